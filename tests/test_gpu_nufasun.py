"""GPU tests of the Nufasun model and its mechanisms against the plain oracle (oracle/nufasun_oracle.py).

Inputs are made so that the classic faults show: a key that dominates its query sits just inside or just outside the window,
the second map is far from negligible, scores reach the cap, decays reach from 1e-3 to 1, keys repeat (so that the delta rule
has something to take back), every portion size cuts windows, chunks and convolutions in the middle."""

import json
import os
import subprocess
import sys

import pytest
import torch

from conftest import ROOT
from nufasun_cases import CONFIGS, attention, config, delta, oracle_logits, relative_error, tokens, weights
from oracle import nufasun_oracle as orc

pytestmark = pytest.mark.gpu
DEV = "cuda"
DTYPES = [torch.float32, torch.bfloat16]
MODEL_TOL = {torch.float32: 3e-5, torch.bfloat16: 6e-2}


def _clean():
    from gpt_triton_b200 import kernels as K

    assert K.device_status() == 0


def build(cfg, w, dtype):
    from gpt_triton_b200.nufasun import Nufasun

    return Nufasun.from_checkpoint(cfg, w).to(dtype).to(DEV).eval()


def randn(*shape, seed=0, scale=1.0):
    return torch.randn(shape, generator=torch.Generator().manual_seed(seed)) * scale


def wide(t, to=8):
    """The same matrix on the GPU with a row pitch of a multiple of `to`."""
    return torch.nn.functional.pad(t, (0, -t.shape[1] % to)).to(DEV)[:, :t.shape[1]]


# ------------------------------------------------------------------ the pass between two sublayers
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,W", [(1, 64), (3, 52), (130, 328), (7, 2048), (5, 4104), (2, 9000)])
def test_stream_update(dtype, M, W):
    from gpt_triton_b200 import kernels as K

    x0, y, table = randn(M, W, seed=1, scale=3.0), randn(M, W, seed=2, scale=0.1).to(dtype), randn(40, W, seed=3).to(dtype)
    gy, g, shift = 1 + randn(W, seed=4, scale=0.3), 1 + randn(W, seed=5, scale=0.3), randn(W, seed=6)
    ids = torch.randint(0, 40, (M,), generator=torch.Generator().manual_seed(7))
    d = lambda t: t.double()
    emb = d(table)[ids] * 0.7
    tol = dict(rtol=2e-5, atol=2e-5) if dtype == torch.float32 else dict(rtol=8e-3, atol=1e-3)
    for kw, ref in (({"y": wide(y), "y_gain": gy.to(DEV)}, d(x0) + orc.rms_norm(d(y), d(gy), 1e-3)),
                    ({"y": wide(y), "y_gain": gy.to(DEV), "ids": ids.to(DEV), "table": table.to(DEV), "table_scale": 0.7, "shift": shift.to(DEV)},
                     d(x0) + orc.rms_norm(d(y), d(gy), 1e-3) + emb + d(shift)),
                    ({"shift": shift.to(DEV)}, d(x0) + d(shift))):
        for gain in (g.to(DEV), None):
            x, rows = K.stream_update(x0.to(DEV), 1e-3, **kw, gain=gain, out_dtype=dtype)
            assert torch.allclose(d(x.cpu()), ref, rtol=2e-6, atol=5e-6)
            assert (rows is None) == (gain is None) and (rows is None or (rows.dtype == dtype and torch.allclose(d(rows.cpu()), orc.rms_norm(ref, d(g), 1e-3), **tol)))
    x, rows = K.stream_update(M, 1e-3, ids=ids.to(DEV), table=table.to(DEV), table_scale=0.7, gain=g.to(DEV))
    assert torch.allclose(d(x.cpu()), emb, rtol=1e-6) and torch.allclose(d(rows.cpu()), orc.rms_norm(emb, d(g), 1e-3), **tol)
    x, _ = K.stream_update(M, 1e-3, ids=torch.full((M,), 40, device=DEV), table=table.to(DEV))
    assert x.abs().sum() == 0  # an id that the table does not have


# ------------------------------------------------------------------ products with a bias, gated pairs, a cap
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,K_,F", [(1, 52, 21), (5, 144, 32), (130, 96, 88), (513, 200, 264), (1100, 64, 520), (700, 1024, 1336)])
def test_biased_gated_and_capped_products(dtype, M, K_, F):
    from gpt_triton_b200 import kernels as K

    a = randn(M, K_, seed=1).to(dtype)
    gate, up = (randn(F, K_, seed=s, scale=1.5 * K_ ** -0.5).to(dtype) for s in (2, 3))
    gb, ub = randn(F, seed=4), randn(F, seed=5)
    rows = wide(a)
    z = lambda w, b: a.double() @ w.double().T + b.double()
    tol = 3e-5 if dtype == torch.float32 else 4e-2
    got = K.linear(rows, K.operand_rows(gate.to(DEV))[0], bias=gb.to(DEV))
    assert got.dtype == dtype and (got.double().cpu() - z(gate, gb)).abs().max() < tol
    for limit, alpha in ((0.8, 1.702), (5.0, 0.6)):
        g, u = z(gate, gb).clamp(max=limit), z(up, ub).clamp(-limit, limit)
        ref = g * torch.sigmoid(alpha * g) * (u + 1)
        w = K.operand_rows(K.interleave_gated(gate, up).to(DEV))[0]
        got = K.gated_linear(rows, w, K.interleave_gated(gb, ub).to(DEV), F, limit=limit, alpha=alpha)
        assert got.shape == (M, F) and got.dtype == dtype and ((got.double().cpu() - ref).abs() / (1 + ref.abs())).max() < tol
    got = K.linear(rows, K.operand_rows(gate.to(DEV))[0], act="softcap", act_param=0.9, out_dtype=torch.float32)
    assert (got.double().cpu() - orc.soft_cap(z(gate, torch.zeros(F)), 0.9)).abs().max() < 3e-5
    got = K.linear(rows, K.operand_rows((gate * 100).to(DEV))[0], act="softcap", act_param=2.0, out_dtype=torch.float32)
    assert torch.isfinite(got).all() and got.abs().max() <= 2.0
    _clean()


# ------------------------------------------------------------------ norm, rotation, ring
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("G,maps,dim,vdim,rot,ring", [(2, 2, 24, 40, 16, 7), (1, 2, 64, 128, 64, 12), (3, 1, 9, 5, 0, 4), (2, 2, 130, 16, 130, 3), (1, 2, 16, 16, 2, 1)])
def test_heads_are_normed_turned_and_remembered(dtype, G, maps, dim, vdim, rot, ring):
    """Portions and single tokens around the ring; queries in place; keys and values behind their history."""
    from gpt_triton_b200 import kernels as K

    B, H, total, base, eps, first = 2, 3, 31, 700.0, 1e-3, 0
    up = lambda c: (c + 7) // 8 * 8
    off_k = up(H * dim)
    off_v = off_k + up(G * maps * dim)
    raw = randn(B, total, off_v + G * vdim, seed=1).to(dtype)
    qw, kw = 1 + randn(dim, seed=2, scale=0.3), 1 + randn(dim, seed=3, scale=0.3)
    turn = lambda x, w, heads, b: orc.rotate_interleaved(orc.rms_norm(x[b].double().view(total, heads, dim), w.double(), eps), torch.arange(total), base, rot)
    q_ref = torch.stack([turn(raw[..., :H * dim], qw, H, b) for b in range(B)])
    k_ref = torch.stack([turn(raw[..., off_k:off_k + G * maps * dim], kw, G * maps, b) for b in range(B)]).view(B, total, G, maps * dim)
    v_ref = raw[..., off_v:].double().view(B, total, G, vdim)
    nan = lambda cols: torch.full((B, G, ring, cols), float("nan"), dtype=dtype, device=DEV)
    cache = (nan(maps * dim), nan(vdim))
    freq = K.rotary_frequencies(base, rot, DEV)
    pos = torch.zeros(2, dtype=torch.int32, device=DEV)
    tol = 2e-5 if dtype == torch.float32 else 4e-2
    for n in (3, 2, 1, 9, 1, 1, 6, 7, 1):
        part = wide(raw[:, first:first + n].reshape(B * n, -1)).clone()
        hist = min(first, ring - 1)
        kw_args = dict(q_heads=H, kv_heads=G, maps=maps, dim=dim, vdim=vdim, cache=cache)
        if n == 1:
            pos.fill_(first)
            assert K.rotary_append(part, (off_k, off_v), qw.to(DEV), kw.to(DEV), freq, eps, B, pos=pos, keep_rows=False, **kw_args) == (None, None)
        else:
            vt = torch.float16 if dtype == torch.bfloat16 and n == 6 else None
            k, v = K.rotary_append(part, (off_k, off_v), qw.to(DEV), kw.to(DEV), freq, eps, B, hist=hist, start=first, v_dtype=vt, **kw_args)
            assert v.dtype == (vt or dtype)
            assert (k.double().cpu().view(B, hist + n, G, -1) - k_ref[:, first - hist:first + n]).abs().max() < tol
            assert (v.double().cpu().view(B, hist + n, G, -1) - v_ref[:, first - hist:first + n]).abs().max() < 1e-6
        assert (part[:, :H * dim].double().cpu().view(B, n, H, dim) - q_ref[:, first:first + n]).abs().max() < tol
        first += n
        for p in range(max(0, first - ring), first):
            assert (cache[0][:, :, p % ring].double().cpu() - k_ref[:, p]).abs().max() < tol
            assert torch.equal(cache[1][:, :, p % ring].double().cpu(), v_ref[:, p])
    assert first == total


def test_angles_stay_exact_far_into_a_sequence():
    from gpt_triton_b200 import kernels as K

    dim, n, start = 32, 64, 3_000_000
    q = randn(n, 3 * dim, seed=1)
    one = torch.ones(dim)
    x = torch.cat([q, torch.zeros(n, 8)], dim=1).to(DEV)
    K.rotary_append(x, (dim, 2 * dim), one.to(DEV), one.to(DEV), K.rotary_frequencies(1e4, dim, DEV), 0.0, 1, q_heads=1, kv_heads=1, maps=1, dim=dim, vdim=dim,
                    start=start)
    unit = orc.rms_unit(q[:, :dim].double(), 0.0)[:, None]
    ref = orc.rotate_interleaved(unit, start + torch.arange(n), 1e4, dim)[:, 0]
    assert (x[:, :dim].double().cpu() - ref).abs().max() < 2e-6


# ------------------------------------------------------------------ differential attention
def _pair_case(B, n, hist, H, G, dim, vdim, window, dtype, scale=None):
    """q, k, v where some queries have a dominating key, in one map, at a chosen distance: just inside the window, just
    outside, at distance 0, the very first token, the token before."""
    m = hist + n
    q, k, v = randn(B, n, H, 2, dim, seed=1), randn(B, m, G, 2, dim, seed=2), randn(B, m, G, vdim, seed=3)
    for t in range(n):
        i = hist + t
        j = (i - window + 1, i - window, i, 0, i - 1)[t % 5]
        if 0 <= j <= i:
            h, mp = t % H, (t // 5) % 2
            q[:, t, h, mp] = k[:, j, h // (H // G), mp] * (4.0 if t % 2 else 2.0)
    gate = torch.sigmoid(randn(B, n, H, seed=4))
    return [z.reshape(B * z.shape[1], -1).to(dtype) for z in (q, k, v, gate)]


def _pair_reference(q, k, v, gate, lam, B, H, G, dim, vdim, window, scale, cap, eps, out_scale):
    n, m = q.shape[0] // B, k.shape[0] // B
    out = []
    for b in range(B):
        qb = q[b * n:(b + 1) * n].double().view(n, H, 2, dim)
        kb = k[b * m:(b + 1) * m].double().view(m, G, 2, dim)
        vb = v[b * m:(b + 1) * m].double().view(m, G, vdim)
        gb = gate[b * n:(b + 1) * n].double()
        heads = []
        for h in range(H):
            g = h // (H // G)
            a = []
            for i in range(2):
                s = (qb[:, h, i] @ kb[:, g, i].T) * scale
                s = (orc.soft_cap(s, cap) if cap > 0 else s).masked_fill(~orc.sliding_window_mask(m, window)[m - n:], -torch.inf)
                a.append(torch.softmax(s, dim=-1) @ vb[:, g])
            heads.append(orc.rms_unit(a[0] - lam * a[1], eps) * out_scale * gb[:, h, None])
        out.append(torch.cat(heads, dim=-1))
    return torch.cat(out)


PAIR_CASES = [
    (1, 1, 0, 1, 1, 16, 16, 1), (2, 7, 0, 3, 1, 10, 6, 3), (1, 70, 0, 2, 2, 32, 48, 1), (2, 65, 12, 6, 2, 64, 64, 13), (1, 130, 63, 4, 1, 64, 32, 64),
    (1, 129, 64, 5, 5, 40, 64, 65), (1, 200, 0, 2, 1, 64, 128, 64), (2, 300, 127, 4, 2, 64, 128, 128), (1, 2, 99, 4, 4, 56, 72, 100), (1, 333, 0, 3, 3, 24, 24, 1000),
    (1, 260, 5, 2, 1, 48, 8, 6), (3, 128, 0, 2, 1, 64, 64, 2), (1, 90, 17, 2, 2, 160, 200, 30), (1, 1100, 0, 8, 2, 64, 128, 400), (2, 190, 60, 2, 1, 128, 128, 61),
    (1, 150, 0, 4, 2, 96, 96, 77), (1, 3, 700, 4, 2, 32, 64, 701)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("B,n,hist,H,G,dim,vdim,window", PAIR_CASES)
def test_pair_attention_over_a_prompt(dtype, B, n, hist, H, G, dim, vdim, window):
    from gpt_triton_b200 import kernels as K

    q, k, v, gate = _pair_case(B, n, hist, H, G, dim, vdim, window, dtype)
    vt = v.to(K.pair_attention_v_dtype(dim, vdim, dtype))
    for cap, lam in ((3.0, 0.7), (30.0, -0.4), (0.0, 1.3)):
        args = dict(heads=H, kv_heads=G, dim=dim, vdim=vdim, window=window, scale=1.3 * dim ** -0.5, softcap=cap, eps=1e-2, out_scale=0.6)
        got = K.pair_attention(wide(q), wide(k), wide(vt), gate.to(DEV), torch.tensor([lam], device=DEV), B, **args)
        ref = _pair_reference(q, k, v, gate, lam, B, H, G, dim, vdim, window, args["scale"], cap, 1e-2, 0.6)
        assert (got.double().cpu() - ref).abs().max() < (6e-5 if dtype == torch.float32 else 2.5e-2)
    _clean()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("B,H,G,dim,vdim,ring,window,pos", [
    (1, 3, 1, 10, 6, 5, 5, 3), (2, 6, 2, 32, 32, 40, 40, 39), (2, 6, 2, 32, 32, 40, 40, 40), (1, 16, 1, 16, 24, 100, 64, 99), (3, 16, 4, 64, 128, 300, 300, 1234),
    (20, 4, 4, 64, 96, 130, 65, 64), (1, 1, 1, 8, 8, 1, 1, 50), (70, 2, 1, 24, 40, 9, 2, 77), (2, 5, 5, 160, 200, 12, 12, 30), (1, 2, 2, 8, 8, 700, 700, 0),
    (1, 8, 2, 64, 128, 1500, 1500, 1400), (2, 20, 1, 128, 128, 257, 257, 2000), (150, 8, 2, 64, 128, 70, 70, 500), (1, 33, 3, 48, 64, 80, 77, 79)])
def test_pair_attention_of_one_token(dtype, B, H, G, dim, vdim, ring, window, pos):
    from gpt_triton_b200 import kernels as K

    m = pos + 1
    q, k, v, gate = randn(B, H, 2, dim, seed=1), randn(B, m, G, 2, dim, seed=2), randn(B, m, G, vdim, seed=3), torch.sigmoid(randn(B, H, seed=4))
    # the oldest visible key answers map 0 of the first head, the newest invisible one map 1 of the last
    if m >= window:
        k[:, m - window, 0, 0] = q[:, 0, 0] * 2
    if m > window:
        k[:, m - window - 1, G - 1, 1] = q[:, H - 1, 1] * 3
    q, k, v, gate = (t.to(dtype) for t in (q, k, v, gate))
    k_cache, v_cache = torch.zeros(B, G, ring, 2 * dim, dtype=dtype), torch.zeros(B, G, ring, vdim, dtype=dtype)
    for p in range(max(0, m - ring), m):
        k_cache[:, :, p % ring], v_cache[:, :, p % ring] = k[:, p].reshape(B, G, -1), v[:, p]
    posd = torch.tensor([pos, 0], dtype=torch.int32, device=DEV)
    lo = max(0, m - window)
    for cap, lam in ((2.0, 0.8), (25.0, -0.3), (0.0, 1.5)):
        args = dict(heads=H, kv_heads=G, dim=dim, vdim=vdim, scale=dim ** -0.5, softcap=cap, eps=1e-2, out_scale=0.7)
        got = K.pair_attention(wide(q.reshape(B, -1)), k_cache.to(DEV), v_cache.to(DEV), gate.to(DEV), torch.tensor([lam], device=DEV), B, window=window, pos=posd, **args)
        ref = _pair_reference(q.reshape(B, -1), k[:, lo:].reshape(B * (m - lo), -1), v[:, lo:].reshape(B * (m - lo), -1), gate, lam, B, H, G, dim, vdim, window,
                              dim ** -0.5, cap, 1e-2, 0.7)
        assert (got.double().cpu() - ref).abs().max() < (4e-5 if dtype == torch.float32 else 2.5e-2)
    _clean()


def test_scores_far_beyond_the_cap_stay_finite():
    from gpt_triton_b200 import kernels as K

    for dtype in DTYPES:
        q, k, v, gate = (t.to(DEV) for t in _pair_case(1, 90, 0, 2, 1, 64, 64, 20, dtype))
        args = dict(heads=2, kv_heads=1, dim=64, vdim=64, window=20, scale=3.0, softcap=20.0, eps=1e-2, out_scale=1.0)
        vt = v.to(K.pair_attention_v_dtype(64, 64, dtype))
        got = K.pair_attention(q * 30, k, vt, gate, torch.tensor([0.5], device=DEV), 1, **args)
        ref = _pair_reference((q * 30).cpu(), k.cpu(), v.cpu(), gate.cpu(), 0.5, 1, 2, 1, 64, 64, 20, 3.0, 20.0, 1e-2, 1.0)
        assert torch.isfinite(got).all() and (got.double().cpu() - ref).abs().max() < 3e-2


# ------------------------------------------------------------------ gated delta rule
def _delta_reference(x, offs, conv, a_log, dt_bias, norm_w, H, G, dim, vdim, eps):
    """x (n, .) raw projections of one sequence -> outputs (n, H * vdim), last state."""
    n, (ok, ov, oa, ob, og) = x.shape[0], offs
    x = x.double()
    mix = orc.silu(orc.causal_convolution(x[:, :ov + H * vdim], conv.double()))
    q, k = orc.unit(mix[:, :G * dim].view(n, G, dim)) * dim ** -0.5, orc.unit(mix[:, ok:ok + G * dim].view(n, G, dim))
    q, k = (t.repeat_interleave(H // G, dim=1) for t in (q, k))
    decay = torch.exp(-torch.exp(a_log.double()) * orc.softplus(x[:, oa:oa + H] + dt_bias.double()))
    o, s = orc.gated_delta_rule(q, k, mix[:, ov:].view(n, H, vdim), decay, torch.sigmoid(x[:, ob:ob + H]))
    return (orc.rms_norm(o, norm_w.double(), eps) * x[:, og:og + H * vdim].view(n, H, vdim)).reshape(n, -1), s


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("B,H,G,dim,vdim,taps", [(1, 2, 2, 32, 32, 4), (2, 6, 3, 24, 40, 3), (1, 2, 1, 10, 14, 1), (1, 2, 1, 128, 128, 4), (2, 2, 1, 72, 64, 2),
                                                 (1, 1, 1, 200, 24, 4), (1, 2, 2, 64, 136, 6), (1, 4, 1, 48, 256, 4)])
@pytest.mark.parametrize("portions", [(1, 1, 1, 1, 1, 1), (5, 1, 31), (32, 2, 64), (65, 63, 1, 70), (300, 40, 2, 129)])
def test_gated_delta_over_portions(dtype, B, H, G, dim, vdim, taps, portions):
    """Any cut of the tokens gives the recurrence's outputs and state."""
    from gpt_triton_b200 import kernels as K

    n = sum(portions)
    up = lambda c: (c + 7) // 8 * 8
    ok, ov = up(G * dim), 2 * up(G * dim)
    oa = up(ov + H * vdim)
    ob = oa + up(H)
    og = ob + up(H)
    x = randn(B, n, up(og + H * vdim), seed=1)
    # keys that come again: the same direction for stretches of tokens
    x[:, :, ok:ok + G * dim] = x[:, :, ok:ok + G * dim] * 0.3 + randn(B, (n + 6) // 7, G * dim, seed=2).repeat_interleave(7, dim=1)[:, :n] * 1.5
    x = x.to(dtype)
    conv = randn(ov + H * vdim, taps, seed=3)
    a_log, dt_bias, norm_w = torch.linspace(-4, 1.5, H) if H > 1 else torch.tensor([-3.0]), randn(H, seed=4), 1 + randn(vdim, seed=5, scale=0.3)
    state = torch.full((B, H, dim, vdim), float("nan"), device=DEV)
    memory = torch.full((B, taps, ov + H * vdim), float("nan"), device=DEV, dtype=dtype)
    pos = torch.zeros(2, dtype=torch.int32, device=DEV)
    ref = [_delta_reference(x[b], (ok, ov, oa, ob, og), conv, a_log, dt_bias, norm_w, H, G, dim, vdim, 1e-3) for b in range(B)]
    start, got = 0, []
    for i, part in enumerate(portions):
        rows = x[:, start:start + part].reshape(B * part, -1).contiguous().to(DEV)
        where = dict(start=start)
        if part == 1 and start > 0:
            pos.fill_(start)
            where = dict(pos=pos)
        y = K.gated_delta(rows, (ok, ov, oa, ob, og), conv.to(DEV), a_log.to(DEV), dt_bias.to(DEV), norm_w.to(DEV), state, memory, B, heads=H, kv_heads=G, dim=dim,
                          vdim=vdim, eps=1e-3, q_scale=dim ** -0.5, **where)
        got.append(y.view(B, part, -1).double().cpu())
        start += part
    got = torch.cat(got, dim=1)
    for b in range(B):
        err = (got[b] - ref[b][0]).abs() / (1 + ref[b][0].abs())
        assert err.max() < (1e-4 if dtype == torch.float32 else 6e-2) and err.pow(2).mean().sqrt() < (1e-5 if dtype == torch.float32 else 4e-3)
        top = ref[b][1].abs().max()
        assert (state[b].double().cpu() - ref[b][1]).abs().max() < (2e-5 if dtype == torch.float32 else 1.5e-2) * top
    _clean()


@pytest.mark.parametrize("B,H,G,dim,vdim,taps", [(38, 4, 2, 40, 48, 3), (19, 4, 4, 128, 64, 4), (10, 8, 1, 72, 128, 2), (5, 16, 8, 64, 64, 4)])
def test_gated_delta_over_many_sequences(B, H, G, dim, vdim, taps):
    """Enough (sequence, head) pairs for the wide column blocks of the chunked kernel; a ragged prompt, then the rest of it."""
    from gpt_triton_b200 import kernels as K

    up = lambda c: (c + 7) // 8 * 8
    ok, ov = up(G * dim), 2 * up(G * dim)
    oa = up(ov + H * vdim)
    ob, og = oa + up(H), oa + 2 * up(H)
    lengths = (135, 40)
    n = sum(lengths)
    x = randn(B, n, og + up(H * vdim), seed=1)
    x[:, :, ok:ok + G * dim] += randn(B, (n + 4) // 5, G * dim, seed=2).repeat_interleave(5, dim=1)[:, :n]
    x = x.bfloat16()
    conv = randn(ov + H * vdim, taps, seed=3)
    a_log, dt_bias, norm_w = torch.linspace(-4, 1.0, H), randn(H, seed=4), 1 + randn(vdim, seed=5, scale=0.3)
    state = torch.full((B, H, dim, vdim), float("nan"), device=DEV)
    memory = torch.full((B, taps, ov + H * vdim), float("nan"), device=DEV, dtype=torch.bfloat16)
    got, start = [], 0
    for part in lengths:
        y = K.gated_delta(x[:, start:start + part].reshape(B * part, -1).contiguous().to(DEV), (ok, ov, oa, ob, og), conv.to(DEV), a_log.to(DEV), dt_bias.to(DEV),
                          norm_w.to(DEV), state, memory, B, heads=H, kv_heads=G, dim=dim, vdim=vdim, eps=1e-3, q_scale=dim ** -0.5, start=start)
        got.append(y.view(B, part, -1).double().cpu())
        start += part
    got = torch.cat(got, dim=1)
    for b in range(0, B, 4):
        ref, last = _delta_reference(x[b], (ok, ov, oa, ob, og), conv, a_log, dt_bias, norm_w, H, G, dim, vdim, 1e-3)
        err = (got[b] - ref).abs() / (1 + ref.abs())
        assert err.max() < 6e-2 and err.pow(2).mean().sqrt() < 4e-3
        assert (state[b].double().cpu() - last).abs().max() < 1.5e-2 * last.abs().max()
    _clean()


@pytest.mark.parametrize("H,G,dim,vdim,taps", [(4, 2, 64, 48, 3), (2, 1, 128, 128, 4), (3, 3, 72, 40, 1)])
def test_chunks_and_single_tokens_agree_to_rounding(H, G, dim, vdim, taps):
    """The same bf16 inputs through the chunked kernel and token by token: the states differ by far less than a bf16 rounding."""
    from gpt_triton_b200 import kernels as K

    n = 200
    up = lambda c: (c + 7) // 8 * 8
    ok, ov = up(G * dim), 2 * up(G * dim)
    oa = up(ov + H * vdim)
    ob, og = oa + up(H), oa + 2 * up(H)
    x = randn(n, og + up(H * vdim), seed=1).bfloat16().to(DEV)
    args = [randn(ov + H * vdim, taps, seed=2).to(DEV), torch.linspace(-4, 1, H).to(DEV), torch.zeros(H, device=DEV), torch.ones(vdim, device=DEV)]
    kw = dict(heads=H, kv_heads=G, dim=dim, vdim=vdim, eps=1e-6, q_scale=dim ** -0.5)
    fresh = lambda: (torch.zeros(1, H, dim, vdim, device=DEV), torch.zeros(1, taps, ov + H * vdim, device=DEV, dtype=torch.bfloat16))
    state, memory = fresh()
    whole = K.gated_delta(x, (ok, ov, oa, ob, og), *args, state, memory, 1, start=0, **kw).double()
    state1, memory1 = fresh()
    pos, rows = torch.zeros(2, dtype=torch.int32, device=DEV), []
    for t in range(n):
        pos.fill_(t)
        rows.append(K.gated_delta(x[t:t + 1].contiguous(), (ok, ov, oa, ob, og), *args, state1, memory1, 1, pos=pos, **kw))
    single = torch.cat(rows).double()
    rms = lambda t: t.view(n, H, vdim).pow(2).mean(-1).sqrt()
    assert (rms(whole - single) / rms(single)).max() < 1.5e-2
    assert (state - state1).abs().max() < 5e-5 * state1.abs().max()
    assert all(torch.equal(memory[0, t % taps], memory1[0, t % taps]) for t in range(n - taps + 1, n))
    _clean()


def test_a_state_without_decay_keeps_its_first_token():
    """g = 1 and beta = 1 to rounding: with orthogonal keys the first value is read back after hundreds of tokens."""
    from gpt_triton_b200 import kernels as K

    dim, vdim, n = 64, 64, 320
    for dtype in DTYPES:
        x = torch.zeros(n, 4 * dim + 16)
        ok, ov, oa, ob, og = dim, 2 * dim, 3 * dim, 3 * dim + 8, 3 * dim + 16
        x[:, oa], x[:, ob], x[:, og:] = -60.0, 30.0, 1.0
        x[:, :dim], x[:, ok:ok + dim] = -60.0, -60.0  # silu: 0
        for t in range(n):
            x[t, ok + (0 if t == 0 else 1 + t % (dim - 1))] = 5.0
        x[-1, 0] = 5.0  # the last query asks for the first key
        x[:, ov:ov + vdim] = randn(n, vdim, seed=1) * 2
        x = x.to(dtype)
        conv = torch.ones(3 * dim, 1)
        state = torch.empty(1, 1, dim, vdim, device=DEV)
        y = K.gated_delta(x.to(DEV), (ok, ov, oa, ob, og), conv.to(DEV), torch.tensor([0.0], device=DEV), torch.tensor([0.0], device=DEV), torch.ones(vdim, device=DEV),
                          state, None, 1, heads=1, kv_heads=1, dim=dim, vdim=vdim, eps=1e-6, q_scale=1.0)
        v0 = orc.rms_unit(orc.silu(x[0, ov:ov + vdim].double()), 1e-6)
        assert (y[-1].double().cpu() - v0).abs().max() < (1e-4 if dtype == torch.float32 else 2e-2)


# ------------------------------------------------------------------ the whole model
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_model_matches_the_oracle_layer_by_layer(name, dtype):
    cfg = CONFIGS[name]
    w = weights(cfg)
    model = build(cfg, w, dtype)
    ids = tokens(cfg, 150)
    ref, streams = orc.forward(cfg, w, ids.tolist(), dtype=torch.float64)
    seen = []
    model.prompt_pass(ids[None].to(DEV), None, 0, tap=lambda x: seen.append(x.clone()))
    assert len(seen) == len(streams) == len(orc.layer_runs(cfg))
    for got, want in zip(seen, streams):
        err = (got.double().cpu() - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt()
        assert err < (1e-5 if dtype == torch.float32 else 3e-2)
    got = model.logits(ids[None].to(DEV))[0]
    assert got.dtype == torch.float32 and relative_error(got, ref).max() < MODEL_TOL[dtype]
    _clean()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
@pytest.mark.parametrize("portions", [[1], [150], [2], [3, 1, 1, 7, 64], [40, 33, 2, 1], [100, 1]])
def test_any_cut_of_a_prompt_gives_the_same_logits(name, dtype, portions):
    """Whole, token by token, and in portions of changing size, through one session that is used again afterwards."""
    from gpt_triton_b200.generation import GenerationSession

    cfg = CONFIGS[name]
    w = weights(cfg, seed=2)
    model = build(cfg, w, dtype)
    session = GenerationSession(model, 1, 150)
    for run in range(2):  # the second request finds the memory the first one left
        ids = tokens(cfg, 150 - 31 * run, seed=5 + run)
        ref = oracle_logits(cfg, w, ids)
        got, at, i = [], 0, 0
        while at < len(ids):
            n = min(portions[i % len(portions)], len(ids) - at)
            rows = session.extend(ids[None, at:at + n].to(DEV), torch.arange(n, device=DEV))
            got.append(model.head_logits(rows))
            at, i = at + n, i + 1
        assert relative_error(torch.cat(got), ref).max() < MODEL_TOL[dtype]
        session.reset()
    _clean()


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_long_prompt_with_wide_heads(dtype):
    """Enough rows for the persistent GEMM, heads of 128, many chunks of the delta rule, windows that reach across query
    tiles; whole, and cut once where the second part has a full window of history."""
    from gpt_triton_b200.generation import GenerationSession

    cfg = config(520, 384, [delta(4, 2, 128, 128, 4, ff=640), attention(4, 2, 64, 128, 190, ff=520), attention(2, 1, 56, 112, 257), delta(2, 2, 64, 96, 3, ff=72)],
                 loop=(1, 3, 2))
    w = weights(cfg, seed=12)
    model = build(cfg, w, dtype)
    ids = tokens(cfg, 1300, seed=4)
    ref = oracle_logits(cfg, w, ids)
    got = model.logits(ids[None].to(DEV))[0]
    assert relative_error(got, ref).max() < MODEL_TOL[dtype]
    session = GenerationSession(model, 1, 1300)
    cut = []
    for lo, hi in ((0, 611), (611, 1300)):
        cut.append(model.head_logits(session.extend(ids[None, lo:hi].to(DEV), torch.arange(hi - lo, device=DEV))))
    assert relative_error(torch.cat(cut), ref).max() < MODEL_TOL[dtype]
    _clean()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_passes_windows_and_rings_many_times(dtype):
    from gpt_triton_b200.generation import GenerationSession

    cfg = CONFIGS["mixed"]
    w = weights(cfg, seed=3)
    model = build(cfg, w, dtype)
    ids = tokens(cfg, 420, seed=8)
    ref = oracle_logits(cfg, w, ids)
    session = GenerationSession(model, 1, 420)
    got = [model.head_logits(session.extend(ids[None, :20].to(DEV)))]
    for t in range(20, 420):
        got.append(model.head_logits(session.extend(ids[None, t:t + 1].to(DEV))))
    assert relative_error(torch.cat(got), ref[19:]).max() < MODEL_TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_batch_gives_what_each_sequence_gives_alone(dtype):
    from gpt_triton_b200.generation import GenerationSession

    cfg = CONFIGS["mixed"]
    w = weights(cfg, seed=4)
    model = build(cfg, w, dtype)
    ids = tokens(cfg, 90, seed=9, batch=5)
    together = GenerationSession(model, 5, 90)
    got = []
    for lo, hi in ((0, 37), (37, 80), (80, 81), (81, 90)):
        rows = together.extend(ids[:, lo:hi].to(DEV).contiguous())
        got.append(model.head_logits(rows))
    for b in range(5):
        ref = oracle_logits(cfg, w, ids[b])
        for g, place in zip(got, (36, 79, 80, 89)):
            assert relative_error(g[b:b + 1], ref[place:place + 1]).max() < 1.5 * MODEL_TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_token_outside_every_window_moves_nothing(dtype):
    """Windows of 6 and 3, the second layer run twice: a token reaches 5 + 2 + 2 further, and not one more."""
    cfg = config(120, 64, [attention(2, 1, 16, 16, 6), attention(2, 2, 16, 16, 3)], loop=(1, 2, 2))
    w = weights(cfg, seed=6, gain=2.0)
    model = build(cfg, w, dtype)
    ids = tokens(cfg, 60, seed=2)
    base = model.logits(ids[None].to(DEV))[0]
    other = ids.clone()
    other[20] = (other[20] + 1) % cfg["vocab"]
    moved = model.logits(other[None].to(DEV))[0]
    assert torch.equal(base[30:], moved[30:]) and not torch.equal(base[29], moved[29]) and torch.equal(base[:20], moved[:20])


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_follows_the_oracle(dtype, tmp_path):
    """model.generate: prompt (also in portions), eager decode steps, captured step; every generated id is an argmax, to
    rounding, of the oracle's logits over prompt + generated ids; graph replay and eager steps agree."""
    cfg = CONFIGS["mixed"]
    w = weights(cfg, seed=7)
    model = build(cfg, w, dtype)
    prompt = tokens(cfg, 45, seed=3, batch=3)
    out = model.generate(prompt.to(DEV), 40).cpu()
    for b in range(3):
        ref = oracle_logits(cfg, w, torch.cat([prompt[b], out[b, :-1]]))[44:]
        spread = (ref - ref.mean(-1, keepdim=True)).pow(2).mean().sqrt()
        gap = (ref.max(-1).values - ref.gather(-1, out[b][:, None])[:, 0]).max() / spread
        assert gap < (1e-4 if dtype == torch.float32 else 0.25)
    if dtype == torch.float32:
        assert torch.equal(model.generate(prompt.to(DEV), 40, portion=7).cpu(), out)
        assert torch.equal(model.generate(prompt[:, :30].to(DEV), 10).cpu(), model.generate(prompt[:, :30].to(DEV), 10, use_cuda_graph=False).cpu())
    a = model.generate(prompt.to(DEV), 20, temperature=0.8, top_k=20, seed=1)
    assert torch.equal(a, model.generate(prompt.to(DEV), 20, temperature=0.8, top_k=20, seed=1))
    assert torch.equal(model.generate(prompt.to(DEV), 12, temperature=0.5, top_k=1, seed=2).cpu(), model.generate(prompt.to(DEV), 12).cpu())
    _clean()


def _write_model(folder, cfg, w):
    from gpt_triton_b200.checkpoint import write_safetensors

    (folder / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(folder / "model.safetensors"), w)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_runner_and_command_line(tmp_path, dtype):
    """bin/trace_run on a model folder: portions, interleaved requests, memory given back and used again; and the command
    line's greedy continuation equals model.generate."""
    cfg = CONFIGS["mixed"]
    w = weights(cfg, seed=9)
    folder, out = tmp_path / "m", tmp_path / "o"
    folder.mkdir(), out.mkdir()
    _write_model(folder, cfg, w)
    a, b, c = tokens(cfg, 70, seed=1), tokens(cfg, 40, seed=2), tokens(cfg, 70, seed=3)
    steps = [([("a", 0, 33, [0, 32])], []), ([("b", 0, 40, [39, 5])], ["b"]), ([("a", 33, 35, [])], []), ([("a", 35, 36, [0])], []),
             ([("a", 36, 70, [33, 1])], ["a"]), ([("c", 0, 2, [1]), ], []), ([("c", 2, 70, [67])], ["c"])]
    ids = {"a": a, "b": b, "c": c}
    lines = [json.dumps({"step": i, "entries": [{"id": r, "tokens": ids[r][lo:hi].tolist(), "want": want} for r, lo, hi, want in entries], "end": end})
             for i, (entries, end) in enumerate(steps)]
    res = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out), "--max-tokens", "110"],
                         input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=600)
    assert res.returncode == 0, res.stderr[-2000:]
    assert [s for s in res.stdout.splitlines() if s.startswith("done")] == [f"done {i}" for i in range(len(steps))]
    tol = MODEL_TOL[getattr(torch, dtype)]
    for i, (entries, _) in enumerate(steps):
        path = out / f"{i}.f32"
        wanted = [(r, lo + p) for r, lo, _, want in entries for p in want]
        assert path.exists() == bool(wanted)
        if wanted:
            got = torch.frombuffer(bytearray(path.read_bytes()), dtype=torch.float32).view(len(wanted), cfg["vocab"])
            for row, (r, p) in zip(got, wanted):
                ref = oracle_logits(cfg, w, ids[r])
                assert relative_error(row[None], ref[p:p + 1]).max() < 1.5 * tol
    res = subprocess.run([sys.executable, "-m", "gpt_triton_b200", "generate", "--model", str(folder), "--dtype", dtype, "--new-tokens", "9",
                          "--ids", ",".join(map(str, a.tolist())), "--ids", ",".join(map(str, b.tolist()))], capture_output=True, text=True, timeout=600, cwd=ROOT)
    assert res.returncode == 0, res.stderr[-2000:]
    rows = [[int(t) for t in line.split(",")] for line in res.stdout.splitlines()]
    model = build(cfg, w, getattr(torch, dtype))
    assert rows == [model.generate(t[None].to(DEV), 9)[0].tolist() for t in (a, b)]
