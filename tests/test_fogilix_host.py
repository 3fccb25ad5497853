"""CPU tests of what surrounds the Fogilix model: configuration, registry, checkpoint files, weight stacking, and the
oracle's own mechanisms against other formulations of the same equations."""

import json

import pytest
import torch

from fogilix_cases import CONFIGS, config, latent, lightning, tokens, weights
from oracle import fogilix_oracle as orc


def test_recurrence_equals_the_decayed_score_form():
    g = torch.Generator().manual_seed(0)
    n, heads, dim, vdim = 23, 3, 5, 7
    q, k = (torch.randn((n, heads, dim), generator=g, dtype=torch.float64) for _ in range(2))
    v = torch.randn((n, heads, vdim), generator=g, dtype=torch.float64)
    decay = torch.tensor([0.3, 0.9, 1.0], dtype=torch.float64)
    out, state = orc.decayed_linear_attention(q, k, v, decay)
    for h in range(heads):
        age = (torch.arange(n)[:, None] - torch.arange(n)[None, :]).double()
        a = torch.where(age >= 0, decay[h] ** age.clamp_min(0), torch.zeros(())) * (q[:, h] @ k[:, h].T)
        assert torch.allclose(out[:, h], a @ v[:, h])
        assert torch.allclose(state[h], ((decay[h] ** (n - 1 - torch.arange(n).double()))[:, None] * k[:, h]).T @ v[:, h])
    first, mid = orc.decayed_linear_attention(q[:9], k[:9], v[:9], decay)
    second, last = orc.decayed_linear_attention(q[9:], k[9:], v[9:], decay, mid)
    assert torch.allclose(torch.cat([first, second]), out) and torch.allclose(last, state)


def test_window_and_sink_of_the_oracle():
    m = orc.sliding_window_mask(6, 3)
    assert m[4].tolist() == [False, False, True, True, True, False] and m[0].tolist() == [True] + [False] * 5
    s = torch.zeros(1, 2, 2)
    w = orc.softmax_with_sink(s, orc.sliding_window_mask(2, 2), torch.zeros(1))
    assert torch.allclose(w[0, 0], torch.tensor([0.5, 0.0])) and torch.allclose(w[0, 1], torch.tensor([1 / 3, 1 / 3]))
    w = orc.softmax_with_sink(s, orc.sliding_window_mask(2, 2), torch.tensor([-1e9]))
    assert torch.allclose(w[0, 1], torch.tensor([0.5, 0.5]))


def test_layers_without_a_feed_forward_and_shared_latents_in_the_oracle():
    """A layer that reads another layer's latents ignores the stream it stands on for its keys and values."""
    cfg = config(50, 24, [latent(2, 8, 4, 12, 5), latent(2, 8, 4, 12, 9, kv_from=0, ff=20)])
    w = weights(cfg)
    assert "l1.mix.dkv" not in w and "l0.norm2" not in w
    logits, streams = orc.forward(cfg, w, tokens(cfg, 12).tolist(), dtype=torch.float64)
    assert logits.shape == (12, 50) and streams.shape == (2, 12, 24) and torch.isfinite(logits).all()


def test_config_is_read_and_checked():
    from gpt_triton_b200.fogilix import Fogilix, FogilixConfig, LatentSpec, LightningSpec
    from gpt_triton_b200.mixers import LatentAttention

    c = FogilixConfig.from_dict(CONFIGS["mixed"])
    assert c.vocab == 331 and c.eps == 3e-4 and c.logit_scale == 0.7 and len(c.layers) == 5
    assert isinstance(c.layers[0].mixer, LatentSpec) and isinstance(c.layers[1].mixer, LightningSpec)
    assert c.layers[2].mixer.kv_from == 0 and c.layers[2].ff is None and c.layers[4].ff == 40
    model = Fogilix(c)
    mixes = [layer.mix for layer in model.layers]
    assert [m.reach for m in mixes if isinstance(m, LatentAttention)][0] == 33  # the largest window that reads layer 0's latents
    caches = model.new_cache(2, 20)
    assert caches[0].shape == (2, 20, 72) and caches[2] is None and caches[1].shape == (2, 3, 16, 48) and caches[1].dtype == torch.float32
    assert model.new_cache(1, 1000)[0].shape == (1, 33, 72)
    for bad in (config(9, 8, [latent(1, 8, 8, 8, 3, kv_from=0)]), config(9, 8, [latent(1, 8, 8, 8, 3), latent(1, 8, 8, 16, 3, kv_from=0)]),
                config(9, 8, [latent(1, 8, 8, 8, 3), latent(1, 8, 8, 8, 3, kv_from=0), latent(1, 8, 8, 8, 3, kv_from=1)]),
                config(9, 8, [lightning(1, 8, 8, [0.5]), latent(1, 8, 8, 8, 3, kv_from=0)]), config(9, 8, [dict(lightning(1, 8, 8, [0.5]), type="other")])):
        with pytest.raises(ValueError):
            FogilixConfig.from_dict(bad)


def test_checkpoint_files_and_registry(tmp_path):
    from gpt_triton_b200.checkpoint import read_config, read_safetensors, write_safetensors
    from gpt_triton_b200.registry import architecture_of, architectures, load_model

    cfg = CONFIGS["odd"]
    w = weights(cfg)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    path = str(tmp_path / "model.safetensors")
    write_safetensors(path, dict(w, table=torch.arange(6, dtype=torch.int32).view(2, 3), empty=torch.empty(0, 4)))
    back = read_safetensors(path)
    assert torch.equal(back["table"], torch.arange(6, dtype=torch.int32).view(2, 3)) and back["empty"].shape == (0, 4)
    assert all(torch.equal(back[k], w[k]) for k in w)
    write_safetensors(path, w)
    assert architecture_of(read_config(str(tmp_path))) == "Fogilix" and {"Fogilix", "gpt2"} <= set(architectures())
    model = load_model(str(tmp_path), dtype=torch.bfloat16, device="cpu")
    state = model.state_dict()
    assert torch.equal(state["layers.1.mix.dkv_norm"], w["l1.mix.dkv.norm"]) and torch.equal(state["final_norm"], w["final.norm"])
    assert sum(p.numel() for p in model.parameters()) == sum(t.numel() for t in w.values())
    with pytest.raises(KeyError):
        architecture_of({"architecture": "nothing like it"})
    (tmp_path / "model.safetensors").write_bytes(open(path, "rb").read()[:-2])
    with pytest.raises(ValueError):
        read_safetensors(path)
    bad = dict(w)
    del bad["l1.mix.sink"]
    write_safetensors(path, bad)
    with pytest.raises(RuntimeError):
        load_model(str(tmp_path), device="cpu")


def test_gpt2_folder_loads_through_the_registry(tmp_path):
    from transformers import GPT2Config, GPT2LMHeadModel

    from gpt_triton_b200.gpt import FusedGPT
    from gpt_triton_b200.registry import load_model

    hf = GPT2LMHeadModel(GPT2Config(vocab_size=96, n_positions=32, n_embd=32, n_layer=2, n_head=2))
    hf.save_pretrained(tmp_path)
    model = load_model(str(tmp_path), dtype=torch.float32, device="cpu")
    assert isinstance(model, FusedGPT) and model.config.n_layer == 2 and not model.exact_float32
    assert torch.equal(model.state_dict()["wte_weight"], hf.state_dict()["transformer.wte.weight"])


def test_stacked_weights_start_at_multiples_of_eight_rows():
    from gpt_triton_b200 import kernels as K

    a, b = torch.randn(5, 12).bfloat16(), torch.randn(9, 12).bfloat16()
    op, starts = K.operand_rows(a, b)
    assert starts == [0, 8] and op.shape == (17, 12) and op.stride(0) == 16
    assert torch.equal(op[:5], a) and torch.equal(op[8:], b) and op[5:8].abs().sum() == 0
    whole = torch.randn(6, 16).bfloat16()
    assert K.operand_rows(whole)[0] is whole  # usable as it is


def test_command_line_info(tmp_path, capsys):
    from gpt_triton_b200.__main__ import main
    from gpt_triton_b200.checkpoint import write_safetensors

    cfg = CONFIGS["odd"]
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(tmp_path / "model.safetensors"), weights(cfg))
    assert main(["info", "--model", str(tmp_path)]) == 0
    assert capsys.readouterr().out.startswith("Fogilix:")


def test_new_entry_points_check_their_arguments():
    import ctypes

    from gpt_triton_b200 import _lib

    lib = _lib.load()
    one = 256
    assert lib.b200_linear(None, None) == 1
    p = _lib.LinearArgs()
    p.M, p.N, p.K, p.lda, p.ldb, p.ld_out, p.op_dtype, p.out_dtype = 0, 8, 8, 8, 8, 8, 2, 2
    assert lib.b200_linear(ctypes.byref(p), None) == 0  # no rows: nothing to do
    p.M = 4
    assert lib.b200_linear(ctypes.byref(p), None) == 1  # no operands
    p.a = p.b = p.out = p.x = one
    assert lib.b200_linear(ctypes.byref(p), None) == 1  # a stream and an output: one of the two
    p.x = None
    p.row_sumsq = one
    assert lib.b200_linear(ctypes.byref(p), None) == 1  # sums of squares without slices
    p.row_sumsq, p.act_lo = None, 9
    assert lib.b200_linear(ctypes.byref(p), None) == 1
    p.act_lo, p.op_dtype, p.lda = 0, 2, 9
    assert lib.b200_linear(ctypes.byref(p), None) == 2  # tensor maps need pitches of a multiple of 8
    assert lib.b200_linear_slice_cols(4, 2) == 64 and lib.b200_linear_slice_cols(513, 2) == 128
    assert lib.b200_embedding_rms(None, None, None, None, None, None, 0, 4, 8, 8, 2, None) == 0
    assert lib.b200_latent_gather(one, one, 1, 2, 8, 9, 8, 9, 2, None) == 1  # more history than the ring holds
    assert lib.b200_latent_append(one, 8, one, 1e-5, None, None, 1, 1, 8, 0, 4, 0, None, 2, None) == 1  # nowhere to go
    assert lib.b200_window_attention(one, 8, one, 8, one, 8, one, 8, 1, 1, 0, 1, 8, 8, 0, 1.0, None, 2, None, None) == 1  # empty window
    assert lib.b200_latent_decode(one, 8, one, one, one, one, 8, 1, 1, 8, 8, 8, 4, 5, 1.0, None, 2, one, one, 0, None) == 1  # window beyond the ring
    assert lib.b200_latent_decode(one, 8, one, one, one, one, 8, 1, 1, 8, 8, 8, 4, 4, 1.0, None, 2, one, None, 0, None) == 5
    assert lib.b200_decayed_attention_slices(1, 3, 16, 40, 2) == 6 and lib.b200_decayed_attention_slices(64, 3, 16, 40, 2) == 3
    assert lib.b200_decayed_attention(one, 32, 8, 16, 20, one, one, one, 1, one, 8, one, 1, 1, 1, 1, 8, 8, 2, None, 0, None, None) == 1  # sections overlap
