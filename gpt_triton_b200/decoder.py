"""What the decoders with RMS norms and an fp32 residual stream share: parameters named after a checkpoint's tensors and the
calls that GenerationSession makes (generation.py).

A subclass has ``embed``, ``head``, ``final_norm``, ``config.vocab`` and ``_operand`` and implements ``_run`` (token ids
through all layers to the rows behind the final norm), ``head_logits`` and ``new_cache``.
"""

import torch

from . import kernels as K
from .generation import GeneratesTokens
from .mixers import PromptContext, StepContext
from .module_base import _EvalOnly


class StreamDecoder(GeneratesTokens, _EvalOnly):
    exact_float32 = True  # float32 models run in true 32-bit
    TENSOR_NAMES = ()  # (name in the checkpoint, name of the parameter) where a dot of the one is not a submodule of the other

    # ---- weights
    @classmethod
    def _parameter_name(cls, tensor):
        """Name in the checkpoint -> name of the parameter."""
        name = tensor
        for theirs, ours in cls.TENSOR_NAMES:
            if name == theirs or name.endswith("." + theirs):
                name = name[:len(name) - len(theirs)] + ours
        return "layers." + name[1:] if name[:1] == "l" and name[1:2].isdigit() else name

    @classmethod
    def tensor_name(cls, parameter):
        """The other way round."""
        name = "l" + parameter.removeprefix("layers.") if parameter.startswith("layers.") else parameter
        for theirs, ours in cls.TENSOR_NAMES:
            if name == ours or name.endswith("." + ours):
                name = name[:len(name) - len(ours)] + theirs
        return name

    @classmethod
    def _load(cls, config, tensors):
        model = cls(config)
        model.load_state_dict({cls._parameter_name(k): v for k, v in tensors.items()})
        return model

    # ---- what GenerationSession drives
    def vocab_size(self):
        return self.config.vocab

    def check_capacity(self, capacity):
        pass  # no position table: any length

    def prompt_pass(self, ids, cache, start, pos=None, want=None, tap=None):
        B, n = ids.shape
        rows = self._run(ids.reshape(-1).contiguous(), PromptContext(B, n, start, cache), "prompt", tap)
        if want is None:
            want = torch.tensor([n - 1], device=ids.device)
        index = (torch.arange(B, device=ids.device)[:, None] * n + want[None, :]).reshape(-1)
        return rows if index.numel() == B * n and n == 1 else K.select_rows(rows, index)

    def decode_pass(self, ids, cache, pos):
        return self._run(ids, StepContext(ids.shape[0], pos, cache), "step")

    def pick(self, rows, temperature, top_k, seed, pos):
        logits = self.head_logits(rows)
        if temperature == 0.0:
            return logits.argmax(dim=-1)
        return K.sample_logits(logits, temperature=temperature, top_k=top_k, seed=seed, step=pos)

    def _head_operand(self):
        return self._operand.derived(("head",), (self.head,), lambda: K.operand_rows(self.head.data)[0])

    # ---- whole sequences
    @torch.no_grad()
    def logits(self, ids):
        """ids (batch, n) -> float32 logits (batch, n, vocab)."""
        B, n = ids.shape
        rows = self._run(ids.reshape(-1).contiguous(), PromptContext(B, n, 0, None), "prompt")
        return self.head_logits(rows).view(B, n, -1)

    forward = logits

    @torch.no_grad()
    def logits_and_next_ids(self, ids):
        logits = self.logits(ids)
        return logits, logits.argmax(dim=-1)

    @torch.no_grad()
    def next_ids(self, ids):
        return self.logits(ids).argmax(dim=-1)
