"""Small random models for the Nufasun tests: configurations of many shapes and weights that make a fault show."""

import torch

from oracle import nufasun_oracle as orc


def attention(heads, kv_heads, dim, vdim, window, rot_dims=None, base=1e4, scale=None, softcap=15.0, diff=0.4, ff=None, limit=3.0):
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window}, "diff": diff, "softcap": softcap,
                      "scale": scale if scale else dim ** -0.5, "rot": {"base": base, "dims": dim // 2 * 2 if rot_dims is None else rot_dims}},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def delta(heads, kv_heads, dim, vdim, taps, ff=None, limit=3.0):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": taps},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def config(vocab, width, layers, loop=(0, 1, 1), eps=1e-5, embedding_scale=1.0, logit_softcap=12.0):
    return {"architecture": "Nufasun", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}, "embedding": {"scale": embedding_scale},
            "logit_softcap": logit_softcap, "loop": dict(zip(("start", "stop", "times"), loop))}


# Sizes that differ from layer to layer; dim != vdim; windows of 1, 2 and more; one key/value head, as many as heads, and
# between; loops at the start, in the middle and at the end, of one pass and of three; layers without a feed-forward; head
# sizes the tensor-core kernels take and some they do not.
CONFIGS = {
    "mixed": config(331, 144, [delta(4, 2, 16, 24, 4, ff=88), attention(6, 2, 24, 40, 9, rot_dims=16, softcap=8.0, ff=200, limit=0.7),
                               attention(2, 1, 32, 64, 33, base=500.0, diff=0.55), delta(3, 3, 32, 16, 2), attention(4, 4, 16, 16, 70, scale=0.5, ff=40)],
                    loop=(1, 4, 3), eps=3e-4, embedding_scale=0.7, logit_softcap=6.0),
    "odd": config(101, 52, [attention(3, 3, 10, 6, 5, rot_dims=4, softcap=50.0, ff=36), delta(2, 1, 10, 14, 3, ff=21), delta(3, 1, 7, 9, 1),
                            attention(4, 2, 9, 13, 12, diff=0.2)], loop=(0, 2, 2), eps=1e-6, embedding_scale=2.5, logit_softcap=30.0),
    "attention_only": config(200, 96, [attention(16, 2, 8, 8, 1, ff=64), attention(4, 2, 64, 128, 70, rot_dims=64, softcap=2.0, ff=72), attention(2, 2, 128, 96, 2)],
                             loop=(1, 3, 2)),
    "delta_only": config(160, 80, [delta(2, 1, 128, 64, 4, ff=96, limit=0.5), delta(6, 3, 24, 72, 5), delta(2, 2, 64, 128, 4)], loop=(2, 3, 4), logit_softcap=3.0),
}


def weights(cfg, seed=0, gain=0.5):
    """bf16 weights (as a checkpoint holds them); queries and keys are scaled so that single scores stand out, decays reach
    from fast to slow, and lambda is far from zero."""
    g = torch.Generator().manual_seed(seed)
    w = cfg["width"]
    mat = lambda n, k, s=1.0: (torch.randn((n, k), generator=g) * s / k ** 0.5).bfloat16()
    vec = lambda n, s=0.3, at=0.0: (at + torch.randn(n, generator=g) * s).bfloat16()
    out = {"embed": torch.randn((cfg["vocab"], w), generator=g).bfloat16(),
           "loop.step": (torch.randn((cfg["loop"]["times"], w), generator=g) * 0.5).bfloat16()}
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}."
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        out |= {p + "norm1": vec(w, at=1.0), p + "norm1b": vec(w, 0.2, gain), p + "mix.o": mat(w, H * dv)}
        if layer["type"] == "delta":
            taps = m["conv"]
            out |= {p + "mix.q": mat(G * d, w), p + "mix.k": mat(G * d, w), p + "mix.v": mat(H * dv, w), p + "mix.g": mat(H * dv, w), p + "mix.a": mat(H, w),
                    p + "mix.b": mat(H, w, 2.0), p + "mix.A_log": vec(H, 1.5, -1.5), p + "mix.dt_bias": vec(H, 1.0, -1.0), p + "mix.norm": vec(dv, at=1.0)}
            out |= {p + f"mix.{x}.conv": mat(n, taps, 1.5) for x, n in (("q", G * d), ("k", G * d), ("v", H * dv))}
        else:
            out |= {p + "mix.q": mat(2 * H * d, w), p + "mix.k": mat(2 * G * d, w), p + "mix.v": mat(G * dv, w), p + "mix.g": mat(H, w),
                    p + "mix.q.norm": vec(d, at=1.4), p + "mix.k.norm": vec(d, at=1.2)}
            out |= {p + "mix." + x: vec(d, 0.35 / d ** 0.25) for x in ("lq1", "lk1", "lq2", "lk2")}
        if layer["mlp"] is not None:
            F = layer["mlp"]["ff"]
            out |= {p + "norm2": vec(w, at=1.0), p + "norm2b": vec(w, 0.2, gain), p + "mlp.gate": mat(F, w, 1.5), p + "mlp.up": mat(F, w, 1.5),
                    p + "mlp.down": mat(w, F), p + "mlp.gate.b": vec(F), p + "mlp.up.b": vec(F), p + "mlp.down.b": vec(w)}
    out["final.norm"] = vec(w, at=1.0)
    out["head"] = mat(cfg["vocab"], w, 3.0)
    return out


def tokens(cfg, n, seed=1, batch=None):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg["vocab"], (n,) if batch is None else (batch, n), generator=g)


def oracle_logits(cfg, w, ids):
    """(n,) ids -> (n, vocab) in float64."""
    return orc.forward(cfg, w, ids.tolist(), dtype=torch.float64)[0]


def relative_error(got, ref):
    """Per row: rms of the difference over the rms of the reference's deviation from its mean."""
    ref = ref.double()
    spread = (ref - ref.mean(-1, keepdim=True)).pow(2).mean().sqrt()
    return (got.double().cpu() - ref).pow(2).mean(-1).sqrt() / spread
