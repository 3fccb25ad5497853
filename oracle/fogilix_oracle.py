"""Plain float32 (or float64) restatement of the Fogilix decoder, one function per mechanism.

Everything is written token by token or as full matrices from the defining equations; nothing is chunked, cached or
fused, and no code is shared with the product path.  Test infrastructure only.
"""

import math

import torch


def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rms_norm_centred(x, w, eps):
    """RMS norm whose stored weight is the gain minus one."""
    return rms_unit(x, eps) * (1 + w)


def rms_norm_plain(x, w, eps):
    return rms_unit(x, eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z / (1 + torch.exp(-z))


def sliding_window_mask(n, size):
    """visible[i, j]: key j is one of the `size` tokens that end at query i."""
    age = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    return (age >= 0) & (age < size)


def softmax_with_sink(scores, visible, sink):
    """scores (heads, n, n) -> weights over the visible keys; the denominator has one extra term exp(sink[head])."""
    s = scores.masked_fill(~visible, -math.inf)
    top = torch.maximum(s.amax(dim=-1), sink[:, None])
    e = torch.exp(s - top[..., None])
    return e / (e.sum(dim=-1) + torch.exp(sink[:, None] - top))[..., None]


def latent_of(h, w_dkv, norm_w, eps):
    """(n, width) -> (n, kv_rank): the only thing an attention layer has to remember per token."""
    return rms_norm_plain(h @ w_dkv.T, norm_w, eps)


def latent_attention(h, c, p, heads, dim, vdim, scale, size):
    """h (n, width) mixer input, c (n, kv_rank) latents (the layer's own or another layer's); p: q, uk, uv, sink, o."""
    n = h.shape[0]
    q = (h @ p["q"].T).view(n, heads, dim).transpose(0, 1)
    k = (c @ p["uk"].T).view(n, heads, dim).transpose(0, 1)
    v = (c @ p["uv"].T).view(n, heads, vdim).transpose(0, 1)
    w = softmax_with_sink((q @ k.transpose(1, 2)) * scale, sliding_window_mask(n, size), p["sink"])
    return (w @ v).transpose(0, 1).reshape(n, heads * vdim) @ p["o"].T


def decayed_linear_attention(q, k, v, decay, state=None):
    """q, k (n, heads, dim), v (n, heads, vdim), decay (heads,) -> outputs (n, heads, vdim) and the last state
    (heads, dim, vdim): S <- decay S + k v^T, then o = S^T q."""
    n, heads, dim = q.shape
    s = torch.zeros(heads, dim, v.shape[2], dtype=q.dtype) if state is None else state.clone()
    out = torch.empty(n, heads, v.shape[2], dtype=q.dtype)
    for t in range(n):
        s = decay[:, None, None] * s + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (s * q[t][:, :, None]).sum(dim=1)
    return out, s


def lightning(h, p, heads, dim, vdim, decay, eps):
    n = h.shape[0]
    q = silu(h @ p["q"].T).view(n, heads, dim)
    k = silu(h @ p["k"].T).view(n, heads, dim)
    v = silu(h @ p["v"].T).view(n, heads, vdim)
    o, _ = decayed_linear_attention(q, k, v, torch.tensor(decay, dtype=h.dtype))
    y = rms_norm_plain(o.reshape(n, heads * vdim), p["norm"], eps) * torch.sigmoid(h @ p["g"].T)
    return y @ p["o"].T


def dense_mlp(h, up, down):
    return gelu_tanh(h @ up.T) @ down.T


def forward(config, weights, tokens, dtype=torch.float32):
    """config: the parsed config.json; weights: name -> tensor; tokens: list of ids.  Returns (logits (n, vocab),
    residual stream after every layer (layers, n, width))."""
    W = {k: v.to(dtype) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens)]
    latents, streams = {}, []
    for i, layer in enumerate(config["layers"]):
        m, pre = layer["mixer"], f"l{i}."
        p = {k[len(pre) + 4:]: t for k, t in W.items() if k.startswith(pre + "mix.")}
        h = rms_norm_centred(x, W[pre + "norm1"], eps)
        if layer["type"] == "lightning":
            x = x + lightning(h, p, m["heads"], m["dim"], m["vdim"], m["decay"], eps)
        elif layer["type"] == "latent_attention":
            source = m.get("kv_from")
            if source is None:
                latents[i] = latent_of(h, p["dkv"], p["dkv.norm"], eps)
                source = i
            x = x + latent_attention(h, latents[source], p, m["heads"], m["dim"], m["vdim"], m["scale"], m["mask"]["size"])
        else:
            raise ValueError(layer["type"])
        if layer["mlp"] is not None:
            assert layer["mlp"]["kind"] == "dense"
            x = x + dense_mlp(rms_norm_centred(x, W[pre + "norm2"], eps), W[pre + "mlp.up"], W[pre + "mlp.down"])
        streams.append(x)
    return rms_norm_centred(x, W["final.norm"], eps) @ W["head"].T * config["logit_scale"], torch.stack(streams)
