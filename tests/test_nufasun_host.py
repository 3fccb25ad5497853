"""CPU tests of what surrounds the Nufasun model: configuration, registry, checkpoint names, weight layouts, argument checks,
and the oracle's own mechanisms against other formulations of the same equations."""

import ctypes
import json
import math

import pytest
import torch

from nufasun_cases import CONFIGS, attention, config, delta, tokens, weights
from oracle import nufasun_oracle as orc


def rnd(*shape, seed=0):
    return torch.randn(shape, generator=torch.Generator().manual_seed(seed), dtype=torch.float64)


def test_delta_rule_equals_its_triangular_system():
    """With the cumulative decays G: (I + A) U = B (V - diag(G) K S0), A = beta_i (G_i / G_j) k_i.k_j below the diagonal."""
    n, d, dv = 19, 6, 5
    q, k, v = rnd(n, 2, d, seed=1), orc.unit(rnd(n, 2, d, seed=2)), rnd(n, 2, dv, seed=3)
    decay, beta = torch.sigmoid(rnd(n, 2, seed=4) + 1), torch.sigmoid(rnd(n, 2, seed=5))
    s0 = rnd(2, d, dv, seed=6)
    out, last = orc.gated_delta_rule(q, k, v, decay, beta, s0)
    for h in range(2):
        G = torch.cumprod(decay[:, h], 0)
        ratio = G[:, None] / G[None, :]
        low = torch.tril(torch.ones(n, n, dtype=torch.float64))
        A = beta[:, h, None] * ratio * (k[:, h] @ k[:, h].T) * (low - torch.eye(n))
        U = torch.linalg.solve(torch.eye(n, dtype=torch.float64) + A, beta[:, h, None] * (v[:, h] - G[:, None] * (k[:, h] @ s0[h])))
        assert torch.allclose(out[:, h], G[:, None] * (q[:, h] @ s0[h]) + (ratio * (q[:, h] @ k[:, h].T) * low) @ U)
        assert torch.allclose(last[h], G[-1] * s0[h] + ((G[-1] / G)[:, None] * k[:, h]).T @ U)
    first, mid = orc.gated_delta_rule(q[:8], k[:8], v[:8], decay[:8], beta[:8], s0)
    rest, end = orc.gated_delta_rule(q[8:], k[8:], v[8:], decay[8:], beta[8:], mid)
    assert torch.allclose(torch.cat([first, rest]), out) and torch.allclose(end, last)


def test_convolution_window_rotation_and_caps_of_the_oracle():
    x, w = rnd(7, 3), rnd(3, 4, seed=1)
    y = orc.causal_convolution(x, w)
    ref = torch.nn.functional.conv1d(torch.nn.functional.pad(x.T[None], (3, 0)), w[:, None], groups=3)[0].T
    assert torch.allclose(y, ref) and torch.allclose(orc.causal_convolution(x[4:], w, before=x[1:4]), y[4:])
    assert torch.allclose(orc.causal_convolution(x, w[:, 3:]), x * w[:, 3])
    m = orc.sliding_window_mask(6, 3)
    assert m[4].tolist() == [False, False, True, True, True, False]
    # scores depend on the distance only, and only through the turned columns
    q, k = rnd(1, 1, 8, seed=2), rnd(1, 1, 8, seed=3)
    dot = lambda i, j: (orc.rotate_interleaved(q, torch.tensor([i]), 100.0, 6) * orc.rotate_interleaved(k, torch.tensor([j]), 100.0, 6)).sum()
    assert torch.allclose(dot(9, 4), dot(25, 20)) and not torch.allclose(dot(9, 4), dot(9, 5))
    a = 1.0 * 100.0 ** (-2 / 6)
    turned = orc.rotate_interleaved(q, torch.tensor([1]), 100.0, 6)[0, 0]
    assert torch.allclose(turned[2], q[0, 0, 2] * math.cos(a) - q[0, 0, 3] * math.sin(a)) and torch.equal(turned[6:], q[0, 0, 6:])
    assert torch.allclose(orc.soft_cap(torch.tensor([0.01, 1e3]), 5.0), torch.tensor([0.01, 5.0]), atol=1e-5)
    assert torch.allclose(orc.softplus(rnd(9)), torch.nn.functional.softplus(rnd(9)))


def test_layer_runs_of_oracle_and_config_agree():
    from gpt_triton_b200.nufasun import NufasunConfig

    for cfg in CONFIGS.values():
        runs = NufasunConfig.from_dict(cfg).runs()
        mine = orc.layer_runs(cfg)
        assert [i for i, _ in runs] == [i for i, _ in mine]
        assert [t for (i, t) in runs if t is not None] == list(range(cfg["loop"]["times"]))
        assert all(i == cfg["loop"]["start"] for i, t in runs if t is not None)
    cfg = config(9, 8, [delta(1, 1, 8, 8, 1)] * 4, loop=(1, 3, 2))
    assert NufasunConfig.from_dict(cfg).runs() == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]


def test_config_is_read_and_checked():
    from gpt_triton_b200.nufasun import AttentionSpec, DeltaSpec, Nufasun, NufasunConfig

    c = NufasunConfig.from_dict(CONFIGS["mixed"])
    assert c.vocab == 331 and c.eps == 3e-4 and c.logit_softcap == 6.0 and c.embedding_scale == 0.7 and (c.loop.start, c.loop.stop, c.loop.times) == (1, 4, 3)
    assert isinstance(c.layers[0].mixer, DeltaSpec) and isinstance(c.layers[1].mixer, AttentionSpec)
    assert c.layers[1].mixer.rot_dims == 16 and c.layers[1].mlp.limit == 0.7 and c.layers[2].mlp is None and c.layers[3].mixer.taps == 2
    model = Nufasun(c)
    caches = model.new_cache(2, 20)
    assert len(caches) == 11 and caches[1][0].shape == (2, 2, 9, 48) and caches[1][1].shape == (2, 2, 9, 40) and caches[2][0].shape == (2, 1, 20, 64)
    assert caches[0][0].shape == (2, 4, 16, 24) and caches[0][0].dtype == torch.float32 and caches[0][1].shape == (2, 4, 64 + 96)
    assert caches[1][0].data_ptr() != caches[4][0].data_ptr()  # every pass has a memory of its own
    good = [attention(2, 1, 8, 8, 3)]
    for bad in (config(9, 8, [attention(3, 2, 8, 8, 3)]), config(9, 8, [attention(2, 1, 8, 8, 0)]), config(9, 8, [attention(2, 1, 8, 8, 3, rot_dims=10)]),
                config(9, 8, [delta(1, 1, 8, 8, 0)]), config(9, 8, good, loop=(0, 2, 1)), config(9, 8, good, loop=(0, 0, 1)), config(9, 8, good, loop=(0, 1, 0)),
                config(9, 8, [dict(good[0], type="other")]), config(9, 8, [dict(good[0], mlp={"kind": "sparse"})])):
        with pytest.raises(ValueError):
            NufasunConfig.from_dict(bad)


def test_checkpoint_names_and_registry(tmp_path, capsys):
    from gpt_triton_b200.__main__ import main
    from gpt_triton_b200.checkpoint import write_safetensors
    from gpt_triton_b200.registry import architectures, load_model

    cfg = CONFIGS["odd"]
    w = weights(cfg)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(tmp_path / "model.safetensors"), w)
    assert "Nufasun" in architectures()
    model = load_model(str(tmp_path), dtype=torch.bfloat16, device="cpu")
    state = model.state_dict()
    assert torch.equal(state["layers.0.mix.q_norm"], w["l0.mix.q.norm"]) and torch.equal(state["layers.1.mix.norm"], w["l1.mix.norm"])
    assert torch.equal(state["layers.1.mlp.gate_b"], w["l1.mlp.gate.b"]) and torch.equal(state["layers.2.mix.v_conv"], w["l2.mix.v.conv"])
    assert {model.tensor_name(n) for n in state} == set(w) and all(torch.equal(state[model._parameter_name(n)], t) for n, t in w.items())
    assert main(["info", "--model", str(tmp_path)]) == 0 and capsys.readouterr().out.startswith("Nufasun:")
    del w["l0.mix.lq2"]
    write_safetensors(str(tmp_path / "model.safetensors"), w)
    with pytest.raises(RuntimeError):
        load_model(str(tmp_path), device="cpu")


def test_gated_weights_alternate_in_blocks():
    from gpt_triton_b200 import kernels as K

    gate, up = torch.arange(40.0).view(40, 1), 100 + torch.arange(40.0).view(40, 1)
    w = K.interleave_gated(gate, up)
    assert w.shape == (128, 1)
    assert torch.equal(w[:32], gate[:32]) and torch.equal(w[32:64], up[:32]) and torch.equal(w[64:72], gate[32:]) and torch.equal(w[96:104], up[32:])
    assert w[72:96].abs().sum() == 0 and w[104:].abs().sum() == 0
    assert torch.equal(K.interleave_gated(gate[:, 0], up[:, 0]), w[:, 0])


def test_frequencies_carry_two_parts():
    from gpt_triton_b200 import kernels as K

    f = K.rotary_frequencies(1e5, 10, "cpu")
    assert f.shape == (5, 2) and torch.allclose(f.double().sum(1), 1e5 ** (-2 * torch.arange(5, dtype=torch.float64) / 10), rtol=1e-13)
    assert K.rotary_frequencies(10.0, 0, "cpu").shape == (0, 2)


def test_looped_layers_differ_from_layers_run_once():
    cfg = config(50, 24, [attention(2, 1, 8, 8, 5, ff=20), delta(2, 1, 8, 8, 3)], loop=(0, 1, 2))
    w = weights(cfg)
    logits, streams = orc.forward(cfg, w, tokens(cfg, 12).tolist(), dtype=torch.float64)
    once, _ = orc.forward(dict(cfg, loop={"start": 0, "stop": 1, "times": 1}), w, tokens(cfg, 12).tolist(), dtype=torch.float64)
    assert logits.shape == (12, 50) and streams.shape == (3, 12, 24) and torch.isfinite(logits).all() and not torch.allclose(logits, once)
    assert logits.abs().max() < cfg["logit_softcap"]


def test_entry_points_check_their_arguments():
    from gpt_triton_b200 import _lib

    lib, one = _lib.load(), 256
    for name in ("b200_stream_update", "b200_rotary_append", "b200_pair_attention", "b200_delta"):
        assert getattr(lib, name)(None, None) == 1
    p = _lib.StreamArgs()
    p.T, p.W, p.dtype = 0, 8, 2
    assert lib.b200_stream_update(ctypes.byref(p), None) == 0  # no rows: nothing to do
    p.T = 2
    assert lib.b200_stream_update(ctypes.byref(p), None) == 1  # no stream
    p.x = p.y = one
    assert lib.b200_stream_update(ctypes.byref(p), None) == 1  # an output without the weights of its norm
    assert lib.b200_gated_pairs(one, 63, one, 8, 1, 8, 1.0, 1.0, 2, None) == 1  # half a block of columns is missing
    r = _lib.RotaryArgs()
    r.B, r.n, r.q_heads, r.kv_heads, r.maps, r.dim, r.vdim, r.dtype, r.v_rows_dtype = 1, 0, 2, 1, 2, 8, 8, 2, 2
    r.off_k, r.off_v, r.ld = 16, 32, 40
    assert lib.b200_rotary_append(ctypes.byref(r), None) == 0
    r.n, r.rows, r.q_weight, r.k_weight, r.rot_dims, r.freq = 1, one, one, one, 10, one
    assert lib.b200_rotary_append(ctypes.byref(r), None) == 1  # more turned columns than a head has
    r.rot_dims, r.hist, r.ring, r.start, r.k_rows, r.v_rows, r.k_cache, r.v_cache, r.ld_k, r.ld_v = 8, 5, 4, 9, one, one, one, one, 16, 8
    assert lib.b200_rotary_append(ctypes.byref(r), None) == 1  # more history than the ring holds
    a = _lib.PairAttentionArgs()
    a.B, a.n, a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.dtype, a.v_dtype = 1, 1, 4, 2, 8, 8, 3, 2, 2
    a.ld_q, a.ld_out, a.ld_gate, a.q, a.k, a.v, a.gate, a.lambda_, a.out = 64, 32, 4, one, one, one, one, one, one
    a.heads = 3
    assert lib.b200_pair_attention(ctypes.byref(a), None) == 1
    a.heads, a.pos_dev, a.ring = 4, one, 2
    assert lib.b200_pair_attention(ctypes.byref(a), None) == 1  # the window reaches beyond the ring
    a.pos_dev = None
    assert lib.b200_pair_attention(ctypes.byref(a), None) == 1  # a ring without a position
    d = _lib.DeltaArgs()
    d.B, d.n, d.heads, d.kv_heads, d.dim, d.vdim, d.taps, d.dtype = 1, 1, 2, 1, 8, 8, 2, 2
    d.off_k, d.off_v, d.off_a, d.off_b, d.off_g, d.conv_cols, d.ld, d.ld_mixed, d.ld_y = 8, 16, 32, 40, 48, 32, 64, 32, 16
    assert lib.b200_delta(ctypes.byref(d), None) == 1  # a memory that is not there
    d.fresh = 1
    assert lib.b200_delta(ctypes.byref(d), None) == 1
    d.off_v = 15
    assert lib.b200_delta(ctypes.byref(d), None) == 1  # sections overlap
