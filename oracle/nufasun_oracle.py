"""Plain restatement of the Nufasun decoder in float32 or float64, one function per mechanism.

Everything is written token by token or as full matrices from the defining equations; nothing is chunked, cached or fused,
and no code is shared with the product path.  Test infrastructure only.
"""

import math

import torch


def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return rms_unit(x, eps) * w


def silu(z):
    return z / (1 + torch.exp(-z))


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def soft_cap(z, cap):
    return cap * torch.tanh(z / cap)


def sliding_window_mask(n, size):
    """visible[i, j]: key j is one of the `size` tokens that end at query i."""
    age = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    return (age >= 0) & (age < size)


def rotate_interleaved(x, positions, base, dims):
    """x (n, heads, d): the neighbours (2i, 2i + 1) of the first `dims` columns turn by position * base^(-2i / dims)."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    angle = positions.double()[:, None] * base ** (-2 * i / dims)
    c, s = torch.cos(angle).to(x.dtype)[:, None, :], torch.sin(angle).to(x.dtype)[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def capped_window_attention(q, k, v, scale, cap, size):
    """One head: q, k (n, d), v (n, dv) -> (n, dv)."""
    s = soft_cap((q @ k.T) * scale, cap).masked_fill(~sliding_window_mask(q.shape[0], size), -math.inf)
    e = torch.exp(s - s.amax(dim=-1, keepdim=True))
    return (e / e.sum(dim=-1, keepdim=True)) @ v


def difference_weight(lq1, lk1, lq2, lk2, diff):
    return torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + diff


def attention(h, p, m, eps):
    """h (n, width); p: the mixer's tensors; m: the mixer's part of config.json."""
    n, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    positions = torch.arange(n)
    q = rms_norm((h @ p["q"].T).view(n, H * 2, d), p["q.norm"], eps)
    k = rms_norm((h @ p["k"].T).view(n, G * 2, d), p["k.norm"], eps)
    v = (h @ p["v"].T).view(n, G, dv)
    q = rotate_interleaved(q, positions, m["rot"]["base"], m["rot"]["dims"]).view(n, H, 2, d)
    k = rotate_interleaved(k, positions, m["rot"]["base"], m["rot"]["dims"]).view(n, G, 2, d)
    lam = difference_weight(p["lq1"], p["lk1"], p["lq2"], p["lk2"], m["diff"])
    gate = sigmoid(h @ p["g"].T)
    out = []
    for head in range(H):
        g = head // (H // G)
        a1, a2 = (capped_window_attention(q[:, head, i], k[:, g, i], v[:, g], m["scale"], m["softcap"], m["mask"]["size"]) for i in range(2))
        out.append(rms_unit(a1 - lam * a2, eps) * (1 - m["diff"]) * gate[:, head, None])
    return torch.cat(out, dim=-1) @ p["o"].T


def causal_convolution(x, w, before=None):
    """x (n, channels), w (channels, taps), the last column multiplying the current row; `before` (taps - 1, channels) are the
    rows in front of x (zeros by default)."""
    taps = w.shape[1]
    if before is None:
        before = torch.zeros(taps - 1, x.shape[1], dtype=x.dtype)
    full = torch.cat([before, x])
    return sum(full[t:t + x.shape[0]] * w[:, t] for t in range(taps))


def unit(x):
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def gated_delta_rule(q, k, v, decay, beta, state=None):
    """q, k (n, heads, d), v (n, heads, dv), decay and beta (n, heads) -> outputs (n, heads, dv), last state (heads, d, dv):
    S <- decay S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q."""
    n, heads, d = q.shape
    s = torch.zeros(heads, d, v.shape[2], dtype=q.dtype) if state is None else state.clone()
    out = torch.empty(n, heads, v.shape[2], dtype=q.dtype)
    for t in range(n):
        s = decay[t][:, None, None] * s
        u = beta[t][:, None] * (v[t] - (s * k[t][:, :, None]).sum(dim=1))
        s = s + k[t][:, :, None] * u[:, None, :]
        out[t] = (s * q[t][:, :, None]).sum(dim=1)
    return out, s


def delta(h, p, m, eps):
    n, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_convolution(h @ p[x].T, p[x + ".conv"])) for x in ("q", "k", "v"))
    q, k = unit(q.view(n, G, d)) * d ** -0.5, unit(k.view(n, G, d))
    q, k = (x.repeat_interleave(H // G, dim=1) for x in (q, k))
    beta = sigmoid(h @ p["b"].T)
    decay = torch.exp(-torch.exp(p["A_log"]) * softplus(h @ p["a"].T + p["dt_bias"]))
    o, _ = gated_delta_rule(q, k, v.view(n, H, dv), decay, beta)
    y = rms_norm(o, p["norm"], eps) * silu(h @ p["g"].T).view(n, H, dv)
    return y.reshape(n, H * dv) @ p["o"].T


def clamped_gated_mlp(h, p, limit):
    g = torch.clamp(h @ p["gate"].T + p["gate.b"], max=limit)
    u = torch.clamp(h @ p["up"].T + p["up.b"], min=-limit, max=limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ p["down"].T + p["down.b"]


def layer_runs(config):
    """(layer, pass) in the order they run; pass is None outside the loop."""
    loop, n = config["loop"], len(config["layers"])
    once = lambda lo, hi: [(i, None) for i in range(lo, hi)]
    return once(0, loop["start"]) + [(i, t) for t in range(loop["times"]) for i in range(loop["start"], loop["stop"])] + once(loop["stop"], n)


def forward(config, weights, tokens, dtype=torch.float32):
    """config: the parsed config.json; weights: name -> tensor; tokens: list of ids.  Returns (logits (n, vocab), residual
    stream after every layer run (runs, n, width))."""
    W = {k: v.to(dtype) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x = start = W["embed"][torch.as_tensor(tokens)] * config["embedding"]["scale"]
    streams = []
    for i, t in layer_runs(config):
        if t is not None and i == config["loop"]["start"]:
            if t > 0:
                x = x + start
            x = x + W["loop.step"][t]
        layer, pre = config["layers"][i], f"l{i}."
        part = lambda name: {k[len(pre) + len(name) + 1:]: w for k, w in W.items() if k.startswith(pre + name + ".")}
        mix = {"attention": attention, "delta": delta}[layer["type"]]
        y = mix(rms_norm(x, W[pre + "norm1"], eps), part("mix"), layer["mixer"], eps)
        x = x + rms_norm(y, W[pre + "norm1b"], eps)
        if layer["mlp"] is not None:
            assert layer["mlp"]["kind"] == "dense"
            y = clamped_gated_mlp(rms_norm(x, W[pre + "norm2"], eps), part("mlp"), layer["mlp"]["limit"])
            x = x + rms_norm(y, W[pre + "norm2b"], eps)
        streams.append(x)
    z = rms_norm(x, W["final.norm"], eps) @ W["head"].T
    return soft_cap(z, config["logit_softcap"]), torch.stack(streams)
