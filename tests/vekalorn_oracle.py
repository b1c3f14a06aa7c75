"""Plain restatement of the Vekalorn decoder, one function per mechanism, whole sequences only, no cache.

Written from the model's equations for the tests; it shares no code with the package.  Everything runs in the dtype of the
weights handed in (the tests use float64).
"""
import math

import torch


def rms(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def layer_norm(x, w, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def frequencies(rot):
    """Per pair the angle per position, and the factor on sine and cosine."""
    n, base, s = rot["dims"], rot["base"], rot.get("scaling")
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    if not s:
        return f, 1.0
    turns = lambda t: n * math.log(s["original"] / (2 * math.pi * t)) / (2 * math.log(base))
    lo, hi = max(math.floor(turns(s["fast"])), 0), min(math.ceil(turns(s["slow"])), n - 1)
    out = []
    for i, x in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(x / s["factor"] * r + x * (1 - r))
    return out, 0.1 * math.log(s["factor"]) + 1


def rotate(x, rot):
    """``x`` [T, heads, dims], positions 0 .. T - 1: the pairs (0, 1), (2, 3), ... turn."""
    f, m = frequencies(rot)
    pos, y = torch.arange(x.shape[0], dtype=torch.float64), x.clone()
    for i, fi in enumerate(f):
        c, s = (m * torch.cos(pos * fi)).to(x.dtype)[:, None], (m * torch.sin(pos * fi)).to(x.dtype)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        y[:, :, 2 * i], y[:, :, 2 * i + 1] = u * c - v * s, v * c + u * s
    return y


def visible(i, window):
    """First position that position ``i`` sees (``window`` 0: all)."""
    return max(0, i - window + 1) if window else 0


def attention(q, k, v, scale, window=0):
    """``q, k`` [T, H, d], ``v`` [T, H, dv] -> [T, H, dv]; row ``i`` sees the last ``window`` positions up to its own."""
    T, H, _ = q.shape
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        s = (q[:, h] @ k[:, h].T) * scale
        for i in range(T):
            a = visible(i, window)
            w = torch.exp(s[i, a : i + 1] - s[i, a : i + 1].max())
            out[i, h] = (w / w.sum()) @ v[a : i + 1, h]
    return out


def latent_keys_values(h, W, p, m, eps, rot_dim):
    """Per-head keys [T, H, dim + rot_dim] and values [T, H, vdim] from the latent of every token."""
    T, H, c = h.shape[0], m["heads"], m["kv_rank"]
    z = h @ W[p + "dkv"].T
    lat = rms(z[:, :c], W[p + "dkv.norm"], eps)
    k = (lat @ W[p + "uk"].T).view(T, H, m["dim"])
    v = (lat @ W[p + "uv"].T).view(T, H, m["vdim"])
    if rot_dim:
        k = torch.cat((k, rotate(z[:, None, c:], m["rot"]).expand(T, H, rot_dim)), -1)
    return k, v


def latent_queries(h, W, p, m, eps, rot_dim):
    q = (rms(h @ W[p + "dq"].T, W[p + "dq.norm"], eps) @ W[p + "uq"].T).view(h.shape[0], m["heads"], m["dim"] + rot_dim)
    return torch.cat((q[..., : m["dim"]], rotate(q[..., m["dim"] :], m["rot"])), -1) if rot_dim else q


def windowed_mixer(h, W, p, m, eps):
    k, v = latent_keys_values(h, W, p, m, eps, 0)
    a = attention(latent_queries(h, W, p, m, eps, 0), k, v, m["scale"], m["mask"]["size"])
    return a.reshape(h.shape[0], -1) @ W[p + "o"].T


def rotated_mixer(h, W, p, m, eps):
    r = m["rot_dim"]
    k, v = latent_keys_values(h, W, p, m, eps, r)
    a = attention(latent_queries(h, W, p, m, eps, r), k, v, m["scale"]).reshape(h.shape[0], -1)
    return (a * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def route(z, r):
    """Chosen experts [T, top] (best first) and their weights from router logits ``z`` [T, experts]."""
    e = torch.exp(z - z.max(-1, keepdim=True).values)
    s = e / e.sum(-1, keepdim=True)
    n, g = r["experts"], r["groups"]
    size = n // g["count"]
    ids, wts = [], []
    for row in s.tolist():
        best = [max(row[i * size : (i + 1) * size]) for i in range(g["count"])]
        kept = sorted(range(g["count"]), key=lambda i: -best[i])[: g["keep"]]
        pick = sorted((i for i in range(n) if i // size in kept), key=lambda i: -row[i])[: r["top"]]
        ids.append(pick)
        wts.append([row[i] for i in pick])
    return torch.tensor(ids), torch.tensor(wts, dtype=z.dtype)


def experts(h, W, p, ids, wts):
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(ids[t].tolist(), wts[t]):
            a = torch.clamp(W[f"{p}e{e}.up"] @ h[t], min=0) ** 2
            out[t] += w * (W[f"{p}e{e}.down"] @ a)
    return out


def feed_forward(h, W, p, m):
    return experts(h, W, p, *route(h @ W[p + "router"].T, m["router"]))


MIXERS = {"latent_attention": windowed_mixer, "latent_attention_2": rotated_mixer}


def forward(cfg, W, tokens):
    """Logits [T, vocab] and the residual stream after every layer [layers, T, width] of one whole sequence."""
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens)]
    stream = []
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + layer_norm(MIXERS[L["type"]](x, W, p + "mix.", L["mixer"], eps), W[p + "norm1"], eps)
        if L.get("mlp"):
            x = x + layer_norm(feed_forward(x, W, p + "mlp.", L["mlp"]), W[p + "norm2"], eps)
        stream.append(x)
    return layer_norm(x, W["final.norm"], eps) @ W["head"].T, torch.stack(stream)
