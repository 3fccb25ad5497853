"""GPU tests of the Fogilix model and its mechanisms against the plain oracle (oracle/fogilix_oracle.py).

Inputs are made so that the classic faults show: a key that dominates its query sits just inside or just outside the
window, sinks are large, decays reach from 0.2 to 1, every portion size cuts windows and chunks in the middle."""

import json
import os
import subprocess
import sys

import pytest
import torch

from conftest import ROOT
from fogilix_cases import CONFIGS, config, latent, lightning, oracle_logits, relative_error, tokens, weights
from oracle import fogilix_oracle as orc

pytestmark = pytest.mark.gpu
DEV = "cuda"
DTYPES = [torch.float32, torch.bfloat16]
MODEL_TOL = {torch.float32: 3e-5, torch.bfloat16: 6e-2}


def _clean():
    from gpt_triton_b200 import kernels as K

    assert K.device_status() == 0


def build(cfg, w, dtype):
    from gpt_triton_b200.fogilix import Fogilix

    return Fogilix.from_checkpoint(cfg, w).to(dtype).to(DEV).eval()


def randn(*shape, seed=0, scale=1.0):
    return torch.randn(shape, generator=torch.Generator().manual_seed(seed)) * scale


# ------------------------------------------------------------------ products around a deferred RMS norm
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,K_,N", [(1, 52, 37), (5, 144, 331), (130, 96, 64), (513, 200, 264), (1100, 64, 520), (700, 1024, 1336)])
def test_linear_finishes_the_norm_and_applies_activations_by_column(dtype, M, K_, N):
    from gpt_triton_b200 import kernels as K

    table = randn(50, K_, seed=1).to(dtype)
    norm_w = randn(K_, seed=2, scale=0.3)
    ids = torch.randint(0, 50, (M,), generator=torch.Generator().manual_seed(3))
    w = randn(N, K_, seed=4, scale=K_ ** -0.5).to(dtype)
    x, rows = K.embedding_rms(ids.to(DEV), table.to(DEV), (1 + norm_w).to(DEV), 0.02)
    xo = table.double()[ids]
    assert torch.equal(x.cpu(), table.float()[ids])
    z = orc.rms_norm_centred(xo, norm_w.double(), 0.02) @ w.double().T
    op, _ = K.operand_rows(w.to(DEV))
    split = N // 3
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    for act, f in ((None, lambda t: t), ("silu", orc.silu), ("gelu_tanh", orc.gelu_tanh)):
        got = K.linear(rows, op, act=act, act_split=split, act_after="sigmoid")
        ref = torch.cat([f(z[:, :split]), torch.sigmoid(z[:, split:])], dim=1)
        assert got.dtype == dtype and (got.double().cpu() - ref).abs().max() < tol
    got = K.linear(rows, op, out_scale=0.3, out_dtype=torch.float32)
    assert got.dtype == torch.float32 and (got.double().cpu() - 0.3 * z).abs().max() < (2e-5 if dtype == torch.float32 else 1.5e-2)
    plain = K.linear(rows.data, op, out_dtype=torch.float32)  # no norm in front
    assert (plain.double().cpu() - rows.data.double().cpu() @ w.double().T).abs().max() < 5e-5
    _clean()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,K_,N", [(1, 40, 52), (3, 64, 144), (200, 96, 80), (513, 128, 264), (1030, 320, 777)])
def test_linear_residual_keeps_the_stream_in_fp32_and_emits_the_next_norm(dtype, M, K_, N):
    from gpt_triton_b200 import kernels as K

    a = randn(M, K_, seed=1).to(dtype)
    w = randn(N, K_, seed=2, scale=K_ ** -0.5).to(dtype)
    x0 = randn(M, N, seed=3, scale=3.0)
    gain = 1 + randn(N, seed=4, scale=0.3)
    x = x0.to(DEV)
    pad = torch.zeros((M, (K_ + 7) // 8 * 8), dtype=dtype, device=DEV)[:, :K_]
    pad.copy_(a)
    rows = K.linear_residual(pad, K.operand_rows(w.to(DEV))[0], x, gain.to(DEV), 1e-3)
    ref = x0.double() + a.double() @ w.double().T
    assert (x.double().cpu() - ref).abs().max() < 2e-5
    second = randn(24, N, seed=5, scale=N ** -0.5).to(dtype)
    got = K.linear(rows, K.operand_rows(second.to(DEV))[0], out_dtype=torch.float32)
    want = orc.rms_norm_centred(ref, gain.double() - 1, 1e-3) @ second.double().T
    assert (got.double().cpu() - want).abs().max() < (2e-5 if dtype == torch.float32 else 2e-2)
    picked = rows.select(torch.tensor([M - 1, 0], device=DEV))
    assert torch.equal(K.linear(picked, K.operand_rows(second.to(DEV))[0], out_dtype=torch.float32)[0], got[M - 1]) or M > 512
    y = x.clone()
    assert K.linear_residual(pad, K.operand_rows(w.to(DEV))[0], y) is None and (y.double().cpu() - 2 * ref + x0.double()).abs().max() < 5e-5
    _clean()


# ------------------------------------------------------------------ window attention
def _window_case(B, n, hist, heads, dim, vdim, window, dtype, seed=0):
    """q, k, v where some queries have a dominating key at a chosen distance: just inside the window, just outside, at
    distance 0, and the very first token."""
    m = hist + n
    q, k, v = randn(B, n, heads, dim, seed=seed), randn(B, m, heads, dim, seed=seed + 1), randn(B, m, heads, vdim, seed=seed + 2)
    for t in range(n):
        i = hist + t
        j = (i - window + 1, i - window, i, 0, i - 1)[t % 5]
        if 0 <= j <= i:
            h = t % heads
            k[:, j, h] = q[:, t, h] * (4.0 if t % 2 else 2.0)
    return [z.reshape(B * z.shape[1], -1).to(dtype) for z in (q, k, v)]


def _window_reference(q, k, v, B, heads, dim, vdim, window, scale, sink):
    n, m = q.shape[0] // B, k.shape[0] // B
    out = []
    for b in range(B):
        qb = q[b * n:(b + 1) * n].double().view(n, heads, dim).transpose(0, 1)
        kb = k[b * m:(b + 1) * m].double().view(m, heads, dim).transpose(0, 1)
        vb = v[b * m:(b + 1) * m].double().view(m, heads, vdim).transpose(0, 1)
        visible = orc.sliding_window_mask(m, window)[m - n:]
        w = orc.softmax_with_sink(qb @ kb.transpose(1, 2) * scale, visible, sink.double())
        out.append((w @ vb).transpose(0, 1).reshape(n, heads * vdim))
    return torch.cat(out)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("B,n,hist,heads,dim,vdim,window", [
    (1, 1, 0, 1, 16, 16, 1), (2, 7, 0, 3, 10, 6, 3), (1, 70, 0, 2, 32, 48, 1), (2, 65, 12, 3, 64, 64, 13), (1, 130, 63, 2, 64, 32, 64),
    (1, 129, 64, 5, 40, 64, 65), (1, 200, 0, 2, 128, 128, 64), (2, 300, 127, 2, 96, 128, 128), (1, 2, 99, 4, 128, 72, 100), (1, 333, 0, 3, 24, 24, 1000),
    (1, 260, 5, 1, 72, 8, 6), (3, 128, 0, 2, 64, 64, 2),
    (1, 90, 17, 2, 160, 200, 30), (1, 1100, 0, 2, 64, 128, 400)])
def test_window_attention(dtype, B, n, hist, heads, dim, vdim, window):
    from gpt_triton_b200 import kernels as K

    q, k, v = _window_case(B, n, hist, heads, dim, vdim, window, dtype)
    sink = randn(heads, seed=9, scale=3.0)
    scale = 1.7 * dim ** -0.5
    wide = lambda t: torch.nn.functional.pad(t, (0, -t.shape[1] % 8)).to(DEV)[:, :t.shape[1]]  # pitch of a multiple of 8
    got = K.window_attention(wide(q), wide(k), wide(v), B, heads, dim, vdim, window, scale, sink.to(DEV))
    ref = _window_reference(q, k, v, B, heads, dim, vdim, window, scale, sink)
    assert (got.double().cpu() - ref).abs().max() < (4e-5 if dtype == torch.float32 else 2.5e-2)
    no_sink = K.window_attention(wide(q), wide(k), wide(v), B, heads, dim, vdim, window, scale)
    ref = _window_reference(q, k, v, B, heads, dim, vdim, window, scale, torch.full((heads,), -1e4))
    assert (no_sink.double().cpu() - ref).abs().max() < (4e-5 if dtype == torch.float32 else 2.5e-2)
    _clean()


def test_window_attention_survives_extreme_sinks_and_scores():
    from gpt_triton_b200 import kernels as K

    B, n, heads, dim = 1, 80, 2, 64
    q, k, v = (t.to(DEV) for t in _window_case(B, n, 0, heads, dim, dim, 20, torch.bfloat16))
    sink = torch.tensor([300.0, -300.0])
    got = K.window_attention(q * 30, k, v, B, heads, dim, dim, 20, 1.0, sink.to(DEV))
    ref = _window_reference((q * 30).cpu(), k.cpu(), v.cpu(), B, heads, dim, dim, 20, 1.0, sink)
    assert torch.isfinite(got).all() and (got.double().cpu() - ref).abs().max() < 3e-2


# ------------------------------------------------------------------ the latent cache and decoding on it
@pytest.mark.parametrize("dtype", DTYPES)
def test_latents_go_around_the_ring(dtype):
    from gpt_triton_b200 import kernels as K

    B, R, ring, total = 2, 40, 7, 31
    raw, w = randn(B, total, R).to(dtype), 1 + randn(R, seed=2, scale=0.3)
    ref = orc.rms_norm_plain(raw.double(), w.double(), 1e-3)
    cache = torch.full((B, ring, R), float("nan"), dtype=dtype, device=DEV)
    start = 0
    pos = torch.zeros(2, dtype=torch.int32, device=DEV)
    for n in (3, 2, 1, 9, 1, 1, 6, 7, 1):
        part = raw[:, start:start + n].reshape(B * n, R).to(DEV)
        hist = min(start, ring - 1)
        if n == 1:
            pos.fill_(start)
            K.latent_append(part, w.to(DEV), 1e-3, B, cache=cache, pos=pos, keep_rows=False)
        else:
            rows = K.latent_append(part, w.to(DEV), 1e-3, B, cache=cache, hist=hist, start=start)
            assert (rows.double().cpu() - ref[:, start - hist:start + n]).abs().max() < (1e-5 if dtype == torch.float32 else 2e-2)
        start += n
        for p in range(max(0, start - ring), start):
            assert (cache[:, p % ring].double().cpu() - ref[:, p]).abs().max() < (1e-5 if dtype == torch.float32 else 2e-2)
    assert start == total


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("B,heads,dim,vdim,R,ring,window,pos", [
    (1, 3, 10, 6, 21, 5, 5, 3), (2, 6, 32, 32, 128, 40, 40, 39), (2, 6, 32, 32, 128, 40, 40, 40), (1, 17, 16, 24, 72, 100, 64, 99), (3, 16, 64, 64, 512, 300, 300, 1234),
    (20, 4, 128, 96, 264, 130, 65, 64), (1, 1, 8, 8, 200, 1, 1, 50), (70, 2, 24, 40, 136, 9, 2, 77), (2, 5, 16, 16, 640, 12, 12, 30), (1, 2, 8, 8, 64, 700, 700, 0)])
def test_latent_decode(dtype, B, heads, dim, vdim, R, ring, window, pos):
    from gpt_triton_b200 import kernels as K

    q = randn(B, heads, dim, seed=1, scale=2.0).to(dtype)
    uk, uv = randn(heads * dim, R, seed=2, scale=R ** -0.5).to(dtype), randn(heads * vdim, R, seed=3, scale=R ** -0.5).to(dtype)
    n = pos + 1
    c = randn(B, n, R, seed=4).to(dtype)
    # the oldest visible latent and the newest invisible one answer the query of head 0
    for j in (pos - window + 1, pos - window):
        if j >= 0:
            d = torch.einsum("bd,dr->br", q[:, 0].float(), uk.view(heads, dim, R)[0].float())
            c[:, j] = (d / d.pow(2).mean(-1, keepdim=True).sqrt() * 1.5).to(dtype)
    cache = torch.full((B, ring, R), float("nan"), dtype=dtype)
    for p in range(max(0, n - ring), n):
        cache[:, p % ring] = c[:, p]
    sink = randn(heads, seed=5, scale=2.0)
    scale = dim ** -0.5
    posd = torch.tensor([pos, 0], dtype=torch.int32, device=DEV)
    cache = torch.nan_to_num(cache)  # (slots nobody has written: any finite value)
    qd = torch.nn.functional.pad(q.reshape(B, -1), (0, -(heads * dim) % 8)).to(DEV)[:, :heads * dim]
    got = K.latent_decode(qd, uk.to(DEV), uv.to(DEV), cache.to(DEV), posd, heads, dim, vdim, window, scale, sink.to(DEV))
    lo = max(0, n - window)
    k = torch.einsum("bjr,hdr->bhjd", c[:, lo:].double(), uk.double().view(heads, dim, R))
    v = torch.einsum("bjr,hdr->bhjd", c[:, lo:].double(), uv.double().view(heads, vdim, R))
    s = torch.einsum("bhd,bhjd->bhj", q.double(), k) * scale
    top = s.amax(-1, keepdim=True)
    e = torch.exp(s - top)
    w = e / (e.sum(-1, keepdim=True) + torch.exp(sink.double()[None, :, None] - top))
    ref = torch.einsum("bhj,bhjd->bhd", w, v).reshape(B, -1)
    assert (got.double().cpu() - ref).abs().max() < (1e-5 if dtype == torch.float32 else 2.5e-2)
    _clean()


# ------------------------------------------------------------------ decayed linear attention
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("B,heads,dim,vdim,decay", [(1, 2, 32, 32, (0.2, 0.999)), (2, 3, 24, 40, (0.5, 0.9, 1.0)), (1, 2, 10, 14, (0.3, 0.99)), (1, 1, 128, 136, (0.9999,)),
                                                    (2, 2, 72, 64, (0.05, 0.98)), (1, 1, 200, 24, (0.9,)), (1, 1, 320, 40, (0.95,))])
@pytest.mark.parametrize("portions", [(1, 1, 1), (5, 1, 31), (32, 2, 64), (65, 63, 1, 70), (600, 40, 257)])
def test_decayed_attention_over_portions(dtype, B, heads, dim, vdim, decay, portions):
    """Any cut of the tokens gives the recurrence's outputs and state (600 tokens of one sequence run in segments)."""
    from gpt_triton_b200 import kernels as K

    n = sum(portions)
    q, k, v = randn(B, n, heads, dim, seed=1), randn(B, n, heads, dim, seed=2), randn(B, n, heads, vdim, seed=3)
    g, wn = randn(B, n, heads, vdim, seed=4), 1 + randn(heads * vdim, seed=5, scale=0.3)
    q, k, v, g = (t.to(dtype) for t in (q, k, v, g))
    pad = lambda c: (c + 7) // 8 * 8
    o1, o2 = pad(heads * dim), 2 * pad(heads * dim)
    o3 = o2 + pad(heads * vdim)
    buf = torch.zeros((B, n, pad(o3 + heads * vdim)), dtype=dtype)
    for at, t in ((0, q), (o1, k), (o2, v), (o3, g)):
        buf[:, :, at:at + t.shape[2] * t.shape[3]] = t.reshape(B, n, -1)
    state = torch.full((B, heads, dim, vdim), float("nan"), device=DEV)
    lam = torch.tensor(decay, dtype=torch.float64)
    ref_state = [None] * B
    eye = torch.eye(heads * vdim, dtype=dtype, device=DEV)
    op, _ = K.operand_rows(eye)
    start = 0
    for part in portions:
        x = buf[:, start:start + part].reshape(B * part, -1).contiguous().to(DEV)
        rows = K.decayed_attention(x, (o1, o2, o3), lam.to(DEV), wn.to(DEV), state, B, heads, dim, vdim, 1e-2, fresh=start == 0)
        got = K.linear(rows, op, out_dtype=torch.float32).view(B, part, -1)  # the identity product finishes the norm
        for b in range(B):
            sl = slice(start, start + part)
            o, ref_state[b] = orc.decayed_linear_attention(q[b, sl].double(), k[b, sl].double(), v[b, sl].double(), lam, ref_state[b])
            ref = orc.rms_norm_plain(o.reshape(part, -1), wn.double(), 1e-2) * g[b, sl].reshape(part, -1).double()
            assert ((got[b].double().cpu() - ref).abs() / (1 + ref.abs())).max() < (6e-5 if dtype == torch.float32 else 1e-2)
            top = ref_state[b].abs().max()
            assert (state[b].double().cpu() - ref_state[b]).abs().max() < 3e-5 * top
        start += part
    _clean()


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
    assert len(seen) == len(cfg["layers"])
    for got, want in zip(seen, streams):
        err = (got.double().cpu() - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt()
        assert err < (1e-5 if dtype == torch.float32 else 2e-2)
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
    """Enough rows for the persistent GEMM, heads of 128, several segments of the chunked recurrence, windows that reach
    across query tiles; whole, and cut once where the second part has a full window of history."""
    from gpt_triton_b200.generation import GenerationSession

    cfg = config(520, 384, [lightning(2, 128, 128, [0.8, 0.9995], ff=640), latent(3, 128, 96, 136, 190), latent(2, 112, 128, 136, 257, kv_from=1, ff=520)])
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
def test_a_far_token_reaches_the_logits_only_through_the_states(dtype):
    """With nothing but windows a change outside every window must not move the logits at all; inside it must."""
    cfg = config(120, 64, [latent(2, 16, 16, 40, 6), latent(2, 16, 16, 40, 3, kv_from=0)])
    w = weights(cfg, seed=6, gain=2.0)
    model = build(cfg, w, dtype)
    ids = tokens(cfg, 60, seed=2)
    base = model.logits(ids[None].to(DEV))[0]
    other = ids.clone()
    other[20] = (other[20] + 1) % cfg["vocab"]
    moved = model.logits(other[None].to(DEV))[0]
    # layer 0 sees 5 back; layer 1 reads layer 0's LATENTS (functions of the stream in front of layer 0) 2 back
    assert torch.equal(base[26:], moved[26:]) and not torch.equal(base[25], moved[25]) and torch.equal(base[:20], moved[:20])


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
        assert gap < (1e-4 if dtype == torch.float32 else 0.2)
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
