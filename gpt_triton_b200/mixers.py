"""Sublayers of decoders with RMS norms and a residual stream in 32-bit.  ``PromptContext`` / ``StepContext`` say where the
tokens stand.

Norm in front only (sliding-window latent attention with a sink, decayed linear ("lightning") attention, the dense
feed-forward): a sublayer takes the fp32 stream ``x`` (rows, width), updated in place, and the ``NormedRows`` of its input,
and returns the NormedRows for the sublayer that follows it, whose norm weights it gets as ``next_gain``: the norm itself is
finished inside the products (kernels.linear).

Norm in front and behind (differential attention, the gated delta rule, the clamped gated feed-forward): a sublayer takes the
normed rows and returns its output; kernels.stream_update does what lies between two of them.  The model counts the layer
runs in ``ctx.run``, which is the place of their memory in ``ctx.cache``: a layer may run several times.
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
    run: int = 0


@dataclass
class StepContext:
    """One new token per sequence at the device-side position pos[0]."""

    batch: int
    pos: torch.Tensor
    cache: list
    run: int = 0


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


class DifferentialAttention(_Sublayer):
    """Sliding-window attention with two softmax maps per head over the same values, the second subtracted with a learned
    weight; grouped key/value heads, per-head RMS norms and rotation of queries and keys, soft-capped scores, the difference
    RMS-normed per head, one sigmoid gate per head."""

    def __init__(self, width, heads, kv_heads, dim, vdim, window, scale, softcap, rot_base, rot_dims, diff, eps):
        super().__init__()
        assert heads % kv_heads == 0 and rot_dims % 2 == 0 and 0 <= rot_dims <= dim
        self.heads, self.kv_heads, self.dim, self.vdim, self.window = heads, kv_heads, dim, vdim, window
        self.scale, self.softcap, self.rot_base, self.rot_dims, self.diff, self.eps = scale, softcap, rot_base, rot_dims, diff, eps
        self.q, self.k, self.v = _weight(heads * 2 * dim, width), _weight(kv_heads * 2 * dim, width), _weight(kv_heads * vdim, width)
        self.q_norm, self.k_norm = _weight(dim), _weight(dim)
        self.lq1, self.lk1, self.lq2, self.lk2 = (_weight(dim) for _ in range(4))
        self.g = _weight(heads, width)
        self.o = _weight(width, heads * vdim)

    def new_cache(self, batch, capacity, device, dtype):
        """Keys and values of the tokens that the window can see."""
        ring = min(self.window, capacity)
        return tuple(torch.empty((batch, self.kv_heads, ring, cols), device=device, dtype=dtype) for cols in (2 * self.dim, self.vdim))

    def _lambda(self):
        def make():
            a, b, c, d = (p.data.float() for p in (self.lq1, self.lk1, self.lq2, self.lk2))
            return ((a * b).sum().exp() - (c * d).sum().exp() + self.diff).reshape(1)

        return self._operand.derived(("lambda",), (self.lq1, self.lk1, self.lq2, self.lk2), make)

    def _frequencies(self):
        return self._operand.derived(("freq",), (self.q,), lambda: K.rotary_frequencies(self.rot_base, self.rot_dims, self.q.device))

    def _mix(self, rows, ctx, prompt):
        w, starts = self._stacked("q", "k", "v", "g")
        qkvg = K.linear(rows, w, act=None, act_split=starts[3], act_after="sigmoid")
        cache = None if ctx.cache is None else ctx.cache[ctx.run]
        where = dict(hist=min(ctx.start, self.window - 1), start=ctx.start) if prompt else dict(pos=ctx.pos, keep_rows=False)
        k, v = K.rotary_append(qkvg, starts[1:3], self._f32("q_norm"), self._f32("k_norm"), self._frequencies(), self.eps, ctx.batch, q_heads=2 * self.heads,
                               kv_heads=self.kv_heads, maps=2, dim=self.dim, vdim=self.vdim, cache=cache,
                               v_dtype=K.pair_attention_v_dtype(self.dim, self.vdim, qkvg.dtype), **where)
        if not prompt:
            k, v = cache
        y = K.pair_attention(qkvg[:, :2 * self.heads * self.dim], k, v, qkvg[:, starts[3]:], self._lambda(), ctx.batch, heads=self.heads,
                             kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, window=self.window, scale=self.scale, softcap=self.softcap, eps=self.eps,
                             out_scale=1.0 - self.diff, pos=None if prompt else ctx.pos)
        return K.linear(y, self._stacked("o")[0])

    def prompt(self, rows, ctx):
        return self._mix(rows, ctx, True)

    def step(self, rows, ctx):
        return self._mix(rows, ctx, False)


class GatedDeltaRule(_Sublayer):
    """Linear attention that writes the difference between a token's value and what the state holds under its key: a (dim,
    vdim) fp32 state per head, one decay and one step size per head and token, short causal convolutions in front, query and
    key heads shared by groups of value heads, the output RMS-normed per head and gated by silu."""

    def __init__(self, width, heads, kv_heads, dim, vdim, taps, eps):
        super().__init__()
        assert heads % kv_heads == 0 and taps >= 1
        self.heads, self.kv_heads, self.dim, self.vdim, self.taps, self.eps = heads, kv_heads, dim, vdim, taps, eps
        self.q, self.k, self.v = _weight(kv_heads * dim, width), _weight(kv_heads * dim, width), _weight(heads * vdim, width)
        self.q_conv, self.k_conv, self.v_conv = _weight(kv_heads * dim, taps), _weight(kv_heads * dim, taps), _weight(heads * vdim, taps)
        self.a, self.b, self.g = _weight(heads, width), _weight(heads, width), _weight(heads * vdim, width)
        self.A_log, self.dt_bias = _weight(heads), _weight(heads)
        self.norm = _weight(vdim)
        self.o = _weight(width, heads * vdim)

    def _conv_cols(self):
        up = lambda n: (n + 7) // 8 * 8
        return 2 * up(self.kv_heads * self.dim) + self.heads * self.vdim

    def new_cache(self, batch, capacity, device, dtype):
        """The state and the last inputs of the convolutions."""
        return (torch.empty((batch, self.heads, self.dim, self.vdim), device=device, dtype=torch.float32),
                torch.empty((batch, self.taps, self._conv_cols()), device=device, dtype=dtype))

    def _taps(self, starts):
        """(columns, taps) float32 in the column order of the stacked product."""
        def make():
            w = torch.zeros((self._conv_cols(), self.taps), device=self.q.device, dtype=torch.float32)
            for at, p in zip(starts, (self.q_conv, self.k_conv, self.v_conv)):
                w[at:at + p.shape[0]] = p.data.float()
            return w

        return self._operand.derived(("taps",), (self.q_conv, self.k_conv, self.v_conv), make)

    def _mix(self, rows, ctx, **where):
        w, starts = self._stacked("q", "k", "v", "a", "b", "g")
        x = K.linear(rows, w, act=None, act_split=starts[5], act_after="silu")
        if ctx.cache is None:
            state, conv = torch.empty((ctx.batch, self.heads, self.dim, self.vdim), device=x.device, dtype=torch.float32), None
        else:
            state, conv = ctx.cache[ctx.run]
        y = K.gated_delta(x, starts[1:], self._taps(starts), self._f32("A_log"), self._f32("dt_bias"), self._f32("norm"), state, conv, ctx.batch,
                          heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, eps=self.eps, q_scale=self.dim ** -0.5, **where)
        return K.linear(y, self._stacked("o")[0])

    def prompt(self, rows, ctx):
        return self._mix(rows, ctx, start=ctx.start)

    def step(self, rows, ctx):
        return self._mix(rows, ctx, pos=ctx.pos)


class GatedFeedForward(_Sublayer):
    """down(gate * sigmoid(alpha * gate) * (up + 1)) with the gate bounded above and up on both sides by `limit`; biases."""

    def __init__(self, width, ff, limit, alpha=1.702):
        super().__init__()
        self.ff, self.limit, self.alpha = ff, limit, alpha
        self.gate, self.up, self.down = _weight(ff, width), _weight(ff, width), _weight(width, ff)
        self.gate_b, self.up_b, self.down_b = _weight(ff), _weight(ff), _weight(width)

    def prompt(self, rows, ctx):
        w = self._operand.derived(("pairs",), (self.gate, self.up), lambda: K.operand_rows(K.interleave_gated(self.gate.data, self.up.data))[0])
        b = self._operand.derived(("pair biases",), (self.gate_b, self.up_b), lambda: K.interleave_gated(self.gate_b.data, self.up_b.data).float())
        y = K.gated_linear(rows, w, b, self.ff, limit=self.limit, alpha=self.alpha)
        return K.linear(y, self._stacked("down")[0], bias=self._f32("down_b"))

    step = prompt
