"""Small random models for the Fogilix tests: configurations of many shapes and weights that make a fault show."""

import torch

from oracle import fogilix_oracle as orc


def latent(heads, dim, vdim, kv_rank, window, scale=None, kv_from=None, ff=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "mask": {"size": window}, "scale": scale if scale else dim ** -0.5}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def lightning(heads, dim, vdim, decay, ff=None):
    assert len(decay) == heads
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(vocab, width, layers, eps=1e-5, logit_scale=1.0):
    return {"architecture": "Fogilix", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}, "logit_scale": logit_scale}


# Sizes that differ from layer to layer; dim != vdim; windows of 1, 2 and more; sharers with larger and smaller windows than
# the layer they read; feed-forwards on either kind of mixer; head sizes the tensor-core kernels take and some they do not.
CONFIGS = {
    "mixed": config(331, 144, [latent(3, 24, 40, 72, 9, ff=88), lightning(3, 16, 48, [0.3, 0.9, 0.9995], ff=200),
                               latent(5, 32, 16, 72, 33, kv_from=0), lightning(1, 72, 24, [0.97]), latent(2, 64, 64, 72, 4, kv_from=0, ff=40)],
                    eps=3e-4, logit_scale=0.7),
    "odd": config(101, 52, [lightning(2, 10, 14, [0.5, 0.99]), latent(3, 10, 6, 21, 5, scale=0.45, ff=36), latent(1, 7, 9, 21, 12, kv_from=1)],
                  eps=1e-6, logit_scale=2.5),
    "attention_only": config(200, 96, [latent(17, 8, 8, 136, 1), latent(4, 80, 104, 136, 70, kv_from=0, ff=64), latent(1, 128, 96, 264, 2)]),
    "linear_only": config(160, 80, [lightning(2, 128, 64, [0.999, 1.0], ff=96), lightning(4, 24, 72, [0.2, 0.8, 0.95, 0.9999])], logit_scale=0.1),
}


def weights(cfg, seed=0, gain=1.0):
    """bf16 weights (as a checkpoint holds them); queries and keys are scaled so that single scores stand out and windows,
    sinks and states matter."""
    g = torch.Generator().manual_seed(seed)
    w = cfg["width"]
    mat = lambda n, k, s=1.0: (torch.randn((n, k), generator=g) * s / k ** 0.5).bfloat16()
    vec = lambda n, s=0.3: (torch.randn(n, generator=g) * s).bfloat16()
    out = {"embed": torch.randn((cfg["vocab"], w), generator=g).bfloat16()}
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}."
        out[p + "norm1"] = vec(w)
        hd, hv = m["heads"] * m["dim"], m["heads"] * m["vdim"]
        if layer["type"] == "lightning":
            out |= {p + "mix.q": mat(hd, w), p + "mix.k": mat(hd, w), p + "mix.v": mat(hv, w), p + "mix.g": mat(hv, w), p + "mix.o": mat(w, hv, gain),
                    p + "mix.norm": (1 + vec(hv)).bfloat16()}
        else:
            out |= {p + "mix.q": mat(hd, w, 2.0), p + "mix.uk": mat(hd, m["kv_rank"], 1.5), p + "mix.uv": mat(hv, m["kv_rank"]),
                    p + "mix.sink": vec(m["heads"], 2.0), p + "mix.o": mat(w, hv, 2 * gain)}
            if "kv_from" not in m:
                out |= {p + "mix.dkv": mat(m["kv_rank"], w), p + "mix.dkv.norm": (1 + vec(m["kv_rank"])).bfloat16()}
        if layer["mlp"] is not None:
            out |= {p + "norm2": vec(w), p + "mlp.up": mat(layer["mlp"]["ff"], w), p + "mlp.down": mat(w, layer["mlp"]["ff"], gain)}
    out["final.norm"] = vec(w)
    out["head"] = mat(cfg["vocab"], w, 2.0)
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
