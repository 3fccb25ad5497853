"""Model registry: a folder's config.json names its architecture, which decides the class that reads the rest of it.

    model = load_model("path/to/folder", dtype=torch.bfloat16)

``register`` adds an architecture: a function (config dict, name -> tensor) -> module.
"""

import os
from types import SimpleNamespace

import torch

from .checkpoint import read_config, read_safetensors

_BUILDERS = {}


def register(*names):
    def add(build):
        for name in names:
            _BUILDERS[name] = build
        return build

    return add


def architectures():
    return sorted(_BUILDERS)


def architecture_of(config):
    """Registered name for a parsed config.json; KeyError names what is there if nothing fits."""
    asked = [config.get("architecture"), *(config.get("architectures") or []), config.get("model_type")]
    for name in asked:
        if name in _BUILDERS:
            return name
    raise KeyError(f"no registered architecture among {[a for a in asked if a]}; known: {architectures()}")


@register("Fogilix")
def _fogilix(config, tensors):
    from .fogilix import Fogilix

    return Fogilix.from_checkpoint(config, tensors)


@register("Nufasun")
def _nufasun(config, tensors):
    from .nufasun import Nufasun

    return Nufasun.from_checkpoint(config, tensors)


@register("GPT2Model", "GPT2LMHeadModel", "gpt2")
def _gpt2(config, tensors):
    from .gpt import FusedGPT, convert_huggingface_to_triton

    body = {k.removeprefix("transformer."): v for k, v in tensors.items() if k != "lm_head.weight"}
    state_dict, cfg = convert_huggingface_to_triton(body, SimpleNamespace(**config))
    model = FusedGPT(cfg)
    model.load_state_dict(state_dict)
    return model


def load_model(folder, dtype=torch.bfloat16, device="cuda"):
    """The model of a folder (config.json, model.safetensors), in `dtype` on `device`, ready to run."""
    config = read_config(folder)
    build = _BUILDERS[architecture_of(config)]
    return build(config, read_safetensors(os.path.join(folder, "model.safetensors"))).to(dtype).to(device).eval()
