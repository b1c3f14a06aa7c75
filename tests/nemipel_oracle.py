"""Plain restatement of the Nemipel decoder, one function per mechanism, whole sequences only, no cache.

Written from the model's equations for the tests; it shares no code with the package.  Everything runs in the dtype
of the weights handed in (the tests use float64 or float32), token by token where the mechanism is a recurrence.
"""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z / (1 + torch.exp(-z))


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def cap(x, c):
    return x if not c else c * torch.tanh(x / c)


def rotate(x, pos, dims, base):
    """``x`` [T, heads, d]: the pairs (0, 1), (2, 3), ... of the first ``dims`` entries turn by pos * base^(-2i / dims)."""
    y = x.clone()
    for i in range(dims // 2):
        a = pos.to(torch.float64) * base ** (-2.0 * i / dims)
        c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        y[:, :, 2 * i], y[:, :, 2 * i + 1] = u * c - v * s, v * c + u * s
    return y


def softcap_attention(q, k, v, scale, softcap):
    """``q`` [T, H, d], ``k`` [T, G, d], ``v`` [T, G, dv] -> [T, H, dv], causal."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = cap((q[:, h] @ k[:, g].T) * scale, softcap)
        for i in range(T):
            w = torch.exp(s[i, : i + 1] - s[i, : i + 1].max())
            out[i, h] = (w / w.sum()) @ v[: i + 1, g]
    return out


def lightning_scan(q, k, v, decay):
    """S <- decay S + k v^T, o = S^T q per head; ``q, k`` [T, H, d], ``v`` [T, H, dv]."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype)
    dec = torch.as_tensor(decay, dtype=q.dtype)
    out = []
    for t in range(T):
        S = dec[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out)


def short_conv(x, w):
    """Causal per-channel convolution, ``x`` [T, C], ``w`` [C, taps], the last tap meets the current row; then silu."""
    taps = w.shape[1]
    y = torch.zeros_like(x)
    for j in range(taps):
        back = taps - 1 - j
        if back < x.shape[0]:
            y[back:] += w[:, j] * x[: x.shape[0] - back]
    return silu(y)


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def channel_delta_scan(q, k, v, g, beta):
    """``q, k`` [T, Hk, d] (unit rows, q scaled), ``v`` [T, H, dv], ``g`` [T, H, d], ``beta`` [T, H]."""
    T, H, dv = v.shape
    rep = H // q.shape[1]
    S = torch.zeros(H, q.shape[2], dv, dtype=q.dtype)
    out = []
    for t in range(T):
        qt, kt = q[t].repeat_interleave(rep, 0), k[t].repeat_interleave(rep, 0)
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, kt))
        S = S + kt[:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, qt))
    return torch.stack(out)


def softplus(z):
    return torch.where(z > 30, z, torch.log1p(torch.exp(torch.clamp(z, max=30))))


def lightning_mixer(h, W, p, m, eps):
    T = h.shape[0]
    q = silu(h @ W[p + "q"].T).view(T, m["heads"], m["dim"])
    k = silu(h @ W[p + "k"].T).view(T, m["heads"], m["dim"])
    v = silu(h @ W[p + "v"].T).view(T, m["heads"], m["vdim"])
    o = lightning_scan(q, k, v, m["decay"]).reshape(T, -1)
    return (rms(o, eps) * W[p + "norm"] * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def attention_keys(h, W, p, m, eps):
    T = h.shape[0]
    k = (rms(h @ W[p + "k"].T, eps) * W[p + "k.norm"]).view(T, m["kv_heads"], m["dim"])
    k = rotate(k, torch.arange(T), m["rot"]["dims"], m["rot"]["base"])
    return k, (h @ W[p + "v"].T).view(T, m["kv_heads"], m["vdim"])


def attention_mixer(h, W, p, m, eps, kv):
    T = h.shape[0]
    q = (rms(h @ W[p + "q"].T, eps) * W[p + "q.norm"]).view(T, m["heads"], m["dim"])
    q = rotate(q, torch.arange(T), m["rot"]["dims"], m["rot"]["base"])
    a = softcap_attention(q, kv[0], kv[1], m["scale"], m.get("softcap"))
    a = a * sigmoid(h @ W[p + "g"].T)[:, :, None]
    return a.reshape(T, -1) @ W[p + "o"].T


def channel_delta_mixer(h, W, p, m, eps):
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v = (short_conv(h @ W[p + n].T, W[p + n + ".conv"]) for n in ("q", "k", "v"))
    q = unit(q.view(T, m["kv_heads"], d)) * d ** -0.5
    k = unit(k.view(T, m["kv_heads"], d))
    beta = sigmoid(h @ W[p + "b"].T)
    raw = (h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "dt_bias"]
    g = torch.exp(-torch.exp(W[p + "A_log"])[None, :, None] * softplus(raw).view(T, H, d))
    o = channel_delta_scan(q, k, v.view(T, H, dv), g, beta)
    o = rms(o, eps) * W[p + "norm"]
    gate = sigmoid((h @ W[p + "g1"].T) @ W[p + "g2"].T).view(T, H, dv)
    return (o * gate).reshape(T, -1) @ W[p + "o"].T


def feed_forward(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def forward(cfg, W, tokens):
    """Logits [T, vocab] and the residual stream after every layer [layers, T, width] of one whole sequence."""
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = W["embed"][torch.as_tensor(tokens)]
    shared, stream = {}, []
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        if L["type"] == "lightning":
            y = lightning_mixer(x, W, p + "mix.", m, eps)
        elif L["type"] == "channel_delta":
            y = channel_delta_mixer(x, W, p + "mix.", m, eps)
        else:
            src = m.get("kv_from")
            shared[i] = attention_keys(x, W, p + "mix.", m, eps) if src is None else shared[src]
            y = attention_mixer(x, W, p + "mix.", m, eps, shared[i])
        x = rms(alpha * x + y, eps) * W[p + "norm1"]
        if L.get("mlp"):
            x = rms(alpha * x + feed_forward(x, W, p + "mlp."), eps) * W[p + "norm2"]
        stream.append(x)
    z = rms(x, eps) * W["final.norm"]
    return cap(z @ W["head"].T, cfg.get("logit_softcap")), torch.stack(stream)
