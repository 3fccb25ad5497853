"""Sublayers of decoders with RMS norms and a residual stream in 32-bit: sliding-window latent attention with a sink,
decayed linear ("lightning") attention, and the dense feed-forward.

Every sublayer takes the fp32 stream ``x`` (rows, width), updated in place, and the ``NormedRows`` of its input, and
returns the NormedRows for the sublayer that follows it, whose norm weights it gets as ``next_gain``: the norm itself is
finished inside the products (kernels.linear).  ``PromptContext`` / ``StepContext`` say where the tokens stand.
"""

from dataclasses import dataclass, field

import torch
from torch import nn

from . import kernels as K
from .module_base import _EvalOnly, _OperandCache


@dataclass
class PromptContext:
    """`n` new tokens of each of `batch` sequences, the first at position `start` (known on the host).  `cache` is the
    model's list of per-layer memories, or None when nothing is to be remembered (start must be 0)."""

    batch: int
    n: int
    start: int
    cache: list
    latents: dict = field(default_factory=dict)  # layer -> (batch, hist + n, kv_rank) of this call, for the layers that share them


@dataclass
class StepContext:
    """One new token per sequence at the device-side position pos[0]."""

    batch: int
    pos: torch.Tensor
    cache: list


def _weight(*shape):
    return nn.Parameter(torch.rand(*shape))


class _Sublayer(_EvalOnly):
    def __init__(self):
        super().__init__()
        self._operand = _OperandCache()

    def _stacked(self, *names):
        """(operand, section starts) of this module's weights `names` stacked into one product."""
        params = tuple(getattr(self, n) for n in names)
        return self._operand.derived(("stacked",) + names, params, lambda: K.operand_rows(*(p.data for p in params)))

    def _f32(self, name):
        p = getattr(self, name)
        return self._operand.derived(("f32", name), (p,), lambda: p.data.float().contiguous())


class LatentAttention(_Sublayer):
    """Sliding-window softmax attention whose keys and values are linear in one latent vector per token, without
    positions, with a learned extra term exp(sink) in every head's denominator.  With ``shares`` set the layer has no
    latents of its own: it reads those of layer ``shares`` (same kv_rank) with its own projections and window."""

    def __init__(self, layer, width, heads, dim, vdim, kv_rank, window, scale, eps, shares=None):
        super().__init__()
        self.layer, self.heads, self.dim, self.vdim, self.kv_rank = layer, heads, dim, vdim, kv_rank
        self.window, self.scale, self.eps, self.shares = window, scale, eps, shares
        self.source = layer if shares is None else shares
        self.reach = window  # largest window among the layers that read these latents (set by the model on the owner)
        self.q = _weight(heads * dim, width)
        if shares is None:
            self.dkv = _weight(kv_rank, width)
            self.dkv_norm = _weight(kv_rank)
        self.uk, self.uv = _weight(heads * dim, kv_rank), _weight(heads * vdim, kv_rank)
        self.sink = _weight(heads)
        self.o = _weight(width, heads * vdim)

    def new_cache(self, batch, capacity, device, dtype):
        """Latents of the last tokens: as many as any reader's window sees."""
        if self.shares is not None:
            return None
        return torch.empty((batch, min(self.reach, capacity), self.kv_rank), device=device, dtype=dtype)

    def _project(self, rows):
        """-> (queries, latents before their norm or None)"""
        if self.shares is not None:
            return K.linear(rows, self._stacked("q")[0]), None
        w, starts = self._stacked("q", "dkv")
        out = K.linear(rows, w)
        return out[:, :self.heads * self.dim], out[:, starts[1]:]

    def prompt(self, x, rows, ctx, next_gain, next_eps):
        q, raw = self._project(rows)
        if raw is not None:
            cache = None if ctx.cache is None else ctx.cache[self.layer]
            hist = min(ctx.start, self.reach - 1)
            ctx.latents[self.layer] = K.latent_append(raw, self._f32("dkv_norm"), self.eps, ctx.batch, cache=cache, hist=hist, start=ctx.start)
        c = ctx.latents[self.source].view(-1, self.kv_rank)
        w, starts = self._stacked("uk", "uv")
        kv = K.linear(c, w)
        y = K.window_attention(q, kv[:, :self.heads * self.dim], kv[:, starts[1]:], ctx.batch, self.heads, self.dim, self.vdim, self.window, self.scale,
                               self._f32("sink"))
        return K.linear_residual(y, self._stacked("o")[0], x, next_gain, next_eps)

    def step(self, x, rows, ctx, next_gain, next_eps):
        q, raw = self._project(rows)
        cache = ctx.cache[self.source]
        if raw is not None:
            K.latent_append(raw, self._f32("dkv_norm"), self.eps, ctx.batch, cache=cache, pos=ctx.pos, keep_rows=False)
        y = K.latent_decode(q, self.uk.data, self.uv.data, cache, ctx.pos, self.heads, self.dim, self.vdim, self.window, self.scale, self._f32("sink"))
        return K.linear_residual(y, self._stacked("o")[0], x, next_gain, next_eps)


class LightningAttention(_Sublayer):
    """Linear attention with a fixed decay per head (``decay``, one float each): a (dim, vdim) fp32 state per head, silu on
    queries, keys and values, an RMS norm over all heads together and a sigmoid output gate."""

    def __init__(self, layer, width, heads, dim, vdim, decay, eps):
        super().__init__()
        assert len(decay) == heads
        self.layer, self.heads, self.dim, self.vdim, self.eps = layer, heads, dim, vdim, eps
        self.decay = tuple(float(d) for d in decay)
        self.q, self.k = _weight(heads * dim, width), _weight(heads * dim, width)
        self.v, self.g = _weight(heads * vdim, width), _weight(heads * vdim, width)
        self.norm = _weight(heads * vdim)
        self.o = _weight(width, heads * vdim)

    def new_cache(self, batch, capacity, device, dtype):
        return torch.empty((batch, self.heads, self.dim, self.vdim), device=device, dtype=torch.float32)

    def _decay_on(self, device):
        return self._operand.derived(("decay",), (self.q,), lambda: torch.tensor(self.decay, dtype=torch.float64, device=device))

    def _mix(self, x, rows, batch, state, fresh, next_gain, next_eps):
        w, starts = self._stacked("q", "k", "v", "g")
        qkvg = K.linear(rows, w, act="silu", act_split=starts[3], act_after="sigmoid")
        y = K.decayed_attention(qkvg, starts[1:], self._decay_on(x.device), self._f32("norm"), state, batch, self.heads, self.dim, self.vdim, self.eps,
                                fresh=fresh)
        return K.linear_residual(y, self._stacked("o")[0], x, next_gain, next_eps)

    def prompt(self, x, rows, ctx, next_gain, next_eps):
        state = self.new_cache(ctx.batch, 0, x.device, None) if ctx.cache is None else ctx.cache[self.layer]
        return self._mix(x, rows, ctx.batch, state, ctx.start == 0, next_gain, next_eps)

    def step(self, x, rows, ctx, next_gain, next_eps):
        return self._mix(x, rows, ctx.batch, ctx.cache[self.layer], False, next_gain, next_eps)


class DenseFeedForward(_Sublayer):
    """down(act(up(h))), no biases."""

    def __init__(self, width, ff, act="gelu_tanh"):
        super().__init__()
        self.act = act
        self.up, self.down = _weight(ff, width), _weight(width, ff)

    def prompt(self, x, rows, ctx, next_gain, next_eps):
        y = K.linear(rows, self._stacked("up")[0], act=self.act)
        return K.linear_residual(y, self._stacked("down")[0], x, next_gain, next_eps)

    step = prompt
