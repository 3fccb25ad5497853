"""Nufasun: a decoder that alternates differential sliding-window attention and gated delta-rule layers, with clamped gated
feed-forwards, RMS norms in front of and behind every sublayer, soft-capped logits, and a range of layers that runs several
times with the same weights.

``NufasunConfig.from_dict`` reads the model's config.json; the state dict's names follow its tensors: ``embed``, ``loop.step``,
``l<i>.norm1``, ``l<i>.mix.<name>``, ``l<i>.norm1b``, ``l<i>.norm2``, ``l<i>.mlp.<name>``, ``l<i>.norm2b``, ``final.norm``,
``head``.  Precisions: bfloat16 (products on the tensor cores, everything in front of a norm, a softmax or a recurrence in
fp32) or float32 throughout.
"""

from dataclasses import dataclass

import torch
from torch import nn

from . import kernels as K
from .decoder import StreamDecoder
from .mixers import DifferentialAttention, GatedDeltaRule, GatedFeedForward, _weight
from .module_base import _OperandCache


@dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    window: int
    scale: float
    softcap: float
    rot_base: float
    rot_dims: int
    diff: float


@dataclass(frozen=True)
class DeltaSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int


@dataclass(frozen=True)
class FeedForwardSpec:
    ff: int
    limit: float


@dataclass(frozen=True)
class LayerSpec:
    mixer: AttentionSpec | DeltaSpec
    mlp: FeedForwardSpec | None


@dataclass(frozen=True)
class LoopSpec:
    """Layers start .. stop - 1 run `times` times in a row."""

    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class NufasunConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    logit_softcap: float
    loop: LoopSpec
    layers: tuple

    @classmethod
    def from_dict(cls, d):
        layers = []
        for i, layer in enumerate(d["layers"]):
            m, kind = layer["mixer"], layer["type"]
            if m["heads"] % m["kv_heads"]:
                raise ValueError(f"layer {i}: the heads must be a multiple of the key/value heads")
            if kind == "attention":
                spec = AttentionSpec(m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["mask"]["size"], float(m["scale"]), float(m["softcap"]),
                                     float(m["rot"]["base"]), m["rot"]["dims"], float(m["diff"]))
                if spec.rot_dims % 2 or not 0 <= spec.rot_dims <= spec.dim:
                    raise ValueError(f"layer {i}: rot.dims must be even and at most dim")
                if spec.window < 1 or not spec.softcap > 0:
                    raise ValueError(f"layer {i}: a window of at least one token and a positive softcap")
            elif kind == "delta":
                spec = DeltaSpec(m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"])
                if spec.taps < 1:
                    raise ValueError(f"layer {i}: the convolutions need at least one tap")
            else:
                raise ValueError(f"layer {i}: unknown mixer {kind!r}")
            mlp = layer.get("mlp")
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            layers.append(LayerSpec(spec, None if mlp is None else FeedForwardSpec(mlp["ff"], float(mlp["limit"]))))
        loop = LoopSpec(d["loop"]["start"], d["loop"]["stop"], d["loop"]["times"])
        if not (0 <= loop.start < loop.stop <= len(layers) and loop.times >= 1):
            raise ValueError("loop: start < stop <= the number of layers, and at least one pass")
        return cls(d["vocab"], d["width"], float(d["norm"]["eps"]), float(d["embedding"]["scale"]), float(d["logit_softcap"]), loop, tuple(layers))

    def runs(self):
        """(layer, the pass that starts in front of it or None) in the order in which the layers run."""
        a, b = self.loop.start, self.loop.stop
        looped = [(i, t if i == a else None) for t in range(self.loop.times) for i in range(a, b)]
        return [(i, None) for i in range(a)] + looped + [(i, None) for i in range(b, len(self.layers))]


class NufasunLayer(nn.Module):
    def __init__(self, spec, config):
        super().__init__()
        m, w = spec.mixer, config.width
        self.norm1, self.norm1b = _weight(w), _weight(w)
        if isinstance(m, AttentionSpec):
            self.mix = DifferentialAttention(w, m.heads, m.kv_heads, m.dim, m.vdim, m.window, m.scale, m.softcap, m.rot_base, m.rot_dims, m.diff, config.eps)
        else:
            self.mix = GatedDeltaRule(w, m.heads, m.kv_heads, m.dim, m.vdim, m.taps, config.eps)
        self.mlp = None
        if spec.mlp is not None:
            self.norm2, self.norm2b = _weight(w), _weight(w)
            self.mlp = GatedFeedForward(w, spec.mlp.ff, spec.mlp.limit)

    def sublayers(self):
        """(sublayer, weights of the norm in front, weights of the norm behind)"""
        subs = [(self.mix, self.norm1, self.norm1b)]
        return subs if self.mlp is None else subs + [(self.mlp, self.norm2, self.norm2b)]


class Nufasun(StreamDecoder):
    TENSOR_NAMES = (("final.norm", "final_norm"), ("loop.step", "loop_step"), ("q.norm", "q_norm"), ("k.norm", "k_norm"), ("q.conv", "q_conv"),
                    ("k.conv", "k_conv"), ("v.conv", "v_conv"), ("gate.b", "gate_b"), ("up.b", "up_b"), ("down.b", "down_b"))

    def __init__(self, config):
        super().__init__()
        self.config = config
        self.embed = _weight(config.vocab, config.width)
        self.loop_step = _weight(config.loop.times, config.width)
        self.layers = nn.ModuleList(NufasunLayer(spec, config) for spec in config.layers)
        self.final_norm = _weight(config.width)
        self.head = _weight(config.vocab, config.width)
        self._operand = _OperandCache()

    @classmethod
    def from_checkpoint(cls, config, tensors):
        """config: the parsed config.json; tensors: name -> tensor of model.safetensors."""
        return cls._load(NufasunConfig.from_dict(config), tensors)

    def new_cache(self, batch, capacity):
        """One memory per layer run: every pass of a looped layer has its own."""
        dev, dtype = self.embed.device, self.embed.dtype
        return [self.layers[i].mix.new_cache(batch, capacity, dev, dtype) for i, _ in self.config.runs()]

    def _f32(self, param):
        return self._operand.derived(("f32", id(param)), (param,), lambda: param.data.float().contiguous())

    def _run(self, ids, ctx, phase, tap=None):
        """ids (rows,) -> rows behind the final norm.  `tap` (for tests) is called with the stream after every layer run."""
        self._check_eval()
        c = self.config
        steps = self._f32(self.loop_step)
        embedded = dict(ids=ids, table=self.embed.data, table_scale=c.embedding_scale)
        runs = c.runs()
        subs = [(run, i == 0, sub) for run, (layer, _) in enumerate(runs) for i, sub in enumerate(self.layers[layer].sublayers())]
        x, update = ids.numel(), dict(embedded)  # what the next pass over the stream adds to it
        for run, first, (sub, gain, behind) in subs:
            entered = runs[run][1] if first else None
            if first and run > 0 and tap is not None:
                tap(K.stream_update(x, c.eps, **update)[0])
                update = {}
            if entered is not None:
                update |= {"shift": steps[entered], **(embedded if entered > 0 else {})}
            x, rows = K.stream_update(x, c.eps, **update, gain=self._f32(gain), out_dtype=self.embed.dtype)
            ctx.run = run
            update = dict(y=getattr(sub, phase)(rows, ctx), y_gain=self._f32(behind))
        if tap is not None:
            tap(K.stream_update(x, c.eps, **update)[0])
            update = {}
        return K.stream_update(x, c.eps, **update, gain=self._f32(self.final_norm), out_dtype=self.embed.dtype)[1]

    def head_logits(self, rows):
        """Final rows -> float32 logits (rows, vocab)."""
        return K.linear(rows, self._head_operand(), act="softcap", act_param=self.config.logit_softcap, out_dtype=torch.float32)
