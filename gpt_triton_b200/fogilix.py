"""Fogilix: a decoder that alternates decayed linear attention and sliding-window latent attention (some layers reading
another layer's latents), with optional dense feed-forwards, RMS norms and a residual stream in 32-bit.

``FogilixConfig.from_dict`` reads the model's config.json; the state dict's names follow its tensors: ``embed``,
``l<i>.norm1``, ``l<i>.mix.<name>``, ``l<i>.norm2``, ``l<i>.mlp.<name>``, ``final.norm``, ``head``.  Precisions: bfloat16
(products on the tensor cores, everything in front of a norm, a softmax or a recurrence in fp32) or float32 throughout.
"""

from dataclasses import dataclass

import torch
from torch import nn

from . import kernels as K
from .decoder import StreamDecoder
from .mixers import DenseFeedForward, LatentAttention, LightningAttention, _weight
from .module_base import _OperandCache


@dataclass(frozen=True)
class LatentSpec:
    heads: int
    dim: int
    vdim: int
    kv_rank: int
    window: int
    scale: float
    kv_from: int | None = None


@dataclass(frozen=True)
class LightningSpec:
    heads: int
    dim: int
    vdim: int
    decay: tuple


@dataclass(frozen=True)
class LayerSpec:
    mixer: LatentSpec | LightningSpec
    ff: int | None  # width of the dense feed-forward; None: the layer has none


@dataclass(frozen=True)
class FogilixConfig:
    vocab: int
    width: int
    eps: float
    logit_scale: float
    layers: tuple

    @classmethod
    def from_dict(cls, d):
        layers = []
        for i, layer in enumerate(d["layers"]):
            m, kind = layer["mixer"], layer["type"]
            if kind == "latent_attention":
                spec = LatentSpec(m["heads"], m["dim"], m["vdim"], m["kv_rank"], m["mask"]["size"], float(m["scale"]), m.get("kv_from"))
                if spec.kv_from is not None:
                    owner = layers[spec.kv_from].mixer if 0 <= spec.kv_from < i else None
                    if not isinstance(owner, LatentSpec) or owner.kv_from is not None or owner.kv_rank != spec.kv_rank:
                        raise ValueError(f"layer {i}: kv_from must name an earlier latent attention layer with latents of its own and the same kv_rank")
            elif kind == "lightning":
                spec = LightningSpec(m["heads"], m["dim"], m["vdim"], tuple(float(x) for x in m["decay"]))
                if len(spec.decay) != spec.heads:
                    raise ValueError(f"layer {i}: one decay per head")
            else:
                raise ValueError(f"layer {i}: unknown mixer {kind!r}")
            mlp = layer.get("mlp")
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            layers.append(LayerSpec(spec, None if mlp is None else mlp["ff"]))
        return cls(d["vocab"], d["width"], float(d["norm"]["eps"]), float(d["logit_scale"]), tuple(layers))


class FogilixLayer(nn.Module):
    def __init__(self, i, spec, config):
        super().__init__()
        m, w = spec.mixer, config.width
        self.norm1 = _weight(w)
        if isinstance(m, LatentSpec):
            self.mix = LatentAttention(i, w, m.heads, m.dim, m.vdim, m.kv_rank, m.window, m.scale, config.eps, shares=m.kv_from)
        else:
            self.mix = LightningAttention(i, w, m.heads, m.dim, m.vdim, m.decay, config.eps)
        self.mlp = None
        if spec.ff is not None:
            self.norm2 = _weight(w)
            self.mlp = DenseFeedForward(w, spec.ff)


class Fogilix(StreamDecoder):
    TENSOR_NAMES = (("final.norm", "final_norm"), ("dkv.norm", "dkv_norm"))

    def __init__(self, config):
        super().__init__()
        self.config = config
        self.embed = _weight(config.vocab, config.width)
        self.layers = nn.ModuleList(FogilixLayer(i, spec, config) for i, spec in enumerate(config.layers))
        for layer in self.layers:
            if isinstance(layer.mix, LatentAttention) and layer.mix.shares is not None:
                owner = self.layers[layer.mix.shares].mix
                owner.reach = max(owner.reach, layer.mix.window)
        self.final_norm = _weight(config.width)
        self.head = _weight(config.vocab, config.width)
        self._operand = _OperandCache()

    @classmethod
    def from_checkpoint(cls, config, tensors):
        """config: the parsed config.json; tensors: name -> tensor of model.safetensors."""
        return cls._load(FogilixConfig.from_dict(config), tensors)

    def _gain(self, param):
        """Norm weights are stored around zero."""
        return self._operand.derived(("gain", id(param)), (param,), lambda: (1.0 + param.data.float()).contiguous())

    def _sublayers(self):
        """(sublayer, weights of the norm behind it) in order."""
        subs, gains = [], []
        for layer in self.layers:
            subs.append(layer.mix)
            gains.append(layer.norm1)
            if layer.mlp is not None:
                subs.append(layer.mlp)
                gains.append(layer.norm2)
        return gains[0] if gains else self.final_norm, list(zip(subs, gains[1:] + [self.final_norm]))

    def new_cache(self, batch, capacity):
        dev, dtype = self.embed.device, self.embed.dtype
        return [layer.mix.new_cache(batch, capacity, dev, dtype) for layer in self.layers]

    def _run(self, ids, ctx, phase, tap=None):
        """ids (rows,) -> NormedRows behind the final norm.  `tap` (for tests) is called with the stream after every layer."""
        self._check_eval()
        eps = self.config.eps
        first, subs = self._sublayers()
        x, rows = K.embedding_rms(ids, self.embed.data, self._gain(first), eps)
        for i, (sub, norm) in enumerate(subs):
            rows = getattr(sub, phase)(x, rows, ctx, self._gain(norm), eps)
            if tap is not None and (i + 1 == len(subs) or not isinstance(subs[i + 1][0], DenseFeedForward)):
                tap(x)
        return rows

    def head_logits(self, rows):
        """Final rows -> float32 logits (rows, vocab)."""
        return K.linear(rows, self._head_operand(), out_scale=self.config.logit_scale, out_dtype=torch.float32)
