"""Plain restatement of the Zeripel decoder, one function per mechanism, whole sequences only, no cache.

Written from the model's equations for the tests; it shares no code with the package.  Everything runs in the dtype of the
weights handed in (the tests use float64).
"""
import math

import torch


def rms(x, eps):
    """Rows divided by their root mean square."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def embed(tokens, W, e):
    """Scaled table rows plus the row of the pair (token in front, token); the first token has the table's last row."""
    b, out = e["bigram"], []
    for i, t in enumerate(tokens):
        pair = (tokens[i - 1] * b["mul_prev"] + t * b["mul_cur"]) % b["buckets"] if i else b["buckets"]
        out.append(W["embed"][t] * e["scale"] + W["bigram"][pair])
    return torch.stack(out)


def shift(h):
    """Every row's predecessor, zeros in front of the first."""
    return torch.cat((torch.zeros_like(h[:1]), h[:-1]))


def decay(mix, W, p):
    """Factor on the state per token and key channel."""
    return torch.exp(-torch.exp(torch.tanh(mix @ W[p + "w1"].T) @ W[p + "w2"].T + W[p + "w0"]))


def recurrence(r, k, v, w, u):
    """``r, k, w`` [T, H, d], ``v`` [T, H, dv], ``u`` [H, d] -> [T, H, dv]."""
    T, H, d = r.shape
    out = torch.zeros(T, H, v.shape[2], dtype=r.dtype)
    for h in range(H):
        S = torch.zeros(d, v.shape[2], dtype=r.dtype)
        for t in range(T):
            kv = k[t, h][:, None] * v[t, h][None]
            out[t, h] = (S + u[h][:, None] * kv).T @ r[t, h]
            S = w[t, h][:, None] * S + kv
    return out


def wkv_mixer(h, W, p, m, eps, shared):
    T, H, d = h.shape[0], m["heads"], m["dim"]
    back = shift(h)
    mix = {n: h + (back - h) * W[p + "mu." + n] for n in "rkvgw"}
    heads = lambda z: z.view(T, H, d)
    r, k, v = (heads(mix[n] @ W[p + n].T) for n in "rkv")
    o = recurrence(r, k, v, heads(decay(mix["w"], W, p)), W[p + "u"])
    return (rms(o, eps).reshape(T, -1) * W[p + "norm"] * silu(mix["g"] @ W[p + "g"].T)) @ W[p + "o"].T


def softmax_rows(s, sink=None):
    """Weights of one head's scores ``s`` [T, T] over the positions up to the row's own; ``sink``: a further term of the
    denominator."""
    out = torch.zeros_like(s)
    for i in range(s.shape[0]):
        z = s[i, : i + 1] if sink is None else torch.cat((s[i, : i + 1], sink.view(1)))
        e = torch.exp(z - z.max())
        out[i, : i + 1] = (e / e.sum())[: i + 1]
    return out


def temperature(T, q_temp):
    return torch.tensor([1 + q_temp["coef"] * math.log((i + 1) // q_temp["every"] + 1) for i in range(T)], dtype=torch.float64)


def attention_mixer(h, W, p, m, eps, shared):
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q, v = (h @ W[p + "q"].T).view(T, H, d), (h @ W[p + "k"].T).view(T, G, d)
    k, q = rms(v, eps) * W[p + "k.norm"], rms(q, eps) * W[p + "q.norm"]
    if m.get("q_temp"):
        q = q * temperature(T, m["q_temp"]).to(q.dtype)[:, None, None]
    a = [softmax_rows(q[:, i] @ k[:, i // (H // G)].T * m["scale"]) @ v[:, i // (H // G)] for i in range(H)]
    return torch.cat(a, 1) @ W[p + "o"].T


def rotate(x, rot):
    """``x`` [T, .., dims], positions 0 .. T - 1: the pairs (0, 1), (2, 3), ... turn."""
    n, y = rot["dims"], x.clone()
    pos = torch.arange(x.shape[0], dtype=torch.float64)
    for i in range(n // 2):
        a = (pos * rot["base"] ** (-2.0 * i / n)).view(-1, *[1] * (x.dim() - 2))
        c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i], y[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return y


def latent(h, W, p, m, eps):
    """Normed latent [T, kv_rank] and rotated key part [T, rot_dim] of every token."""
    z = h @ W[p + "dkv"].T
    return rms(z[:, : m["kv_rank"]], eps) * W[p + "dkv.norm"], rotate(z[:, m["kv_rank"] :], m["rot"])


def latent_mixer(h, W, p, m, eps, shared):
    T, H, d, r = h.shape[0], m["heads"], m["dim"], m["rot_dim"]
    if m.get("kv_from") is None:
        c, kr = latent(h, W, p, m, eps)
        shared[int(p[1 : p.index(".")])] = c, kr
    else:
        c, kr = shared[m["kv_from"]]
    q = (h @ W[p + "q"].T).view(T, H, d + r)
    qr = rotate(q[..., d:], m["rot"])
    k, v = (c @ W[p + "uk"].T).view(T, H, d), (c @ W[p + "uv"].T).view(T, H, m["vdim"])
    gate = sigmoid(h @ W[p + "g"].T)
    out = []
    for i in range(H):
        s = (q[:, i, :d] @ k[:, i].T + qr[:, i] @ kr.T) * m["scale"]
        out.append(softmax_rows(s, W[p + "sink"][i]) @ v[:, i] * gate[:, i : i + 1])
    return torch.cat(out, 1) @ W[p + "o"].T


def glu(h, W, p, act):
    return (act(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def route(z, correction, r):
    """Chosen experts [T, top] (best first) and their weights from router logits ``z`` [T, experts]."""
    s = sigmoid(z)
    ids = [sorted(range(r["experts"]), key=lambda i: -row[i])[: r["top"]] for row in (s + correction).tolist()]
    ids = torch.tensor(ids)
    w = s.gather(1, ids)
    return ids, w / (w.sum(1, keepdim=True) + 1e-20) * r["scale"]


def feed_forward(h, W, p, m):
    if m["kind"] == "dense":
        return glu(h, W, p, gelu)
    ids, wts = route(h @ W[p + "router"].T, W[p + "correction"], m["router"])
    out = torch.stack([sum(w * glu(h[t], W, f"{p}e{e}.", silu) for e, w in zip(ids[t].tolist(), wts[t])) for t in range(h.shape[0])])
    if m.get("shared"):
        out = out + glu(h, W, p + "shared.", silu) * sigmoid(h @ W[p + "shared.sg"].T)
    return out


MIXERS = {"wkv": wkv_mixer, "attention": attention_mixer, "latent_attention": latent_mixer}


def forward(cfg, W, tokens):
    """Logits [T, vocab] and the residual stream after every layer [layers, T, width] of one whole sequence."""
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x, shared, stream = embed(list(tokens), W, cfg["embedding"]), {}, []
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + mult * MIXERS[L["type"]](rms(x, eps) * W[p + "norm1"], W, p + "mix.", L["mixer"], eps, shared)
        if L.get("mlp"):
            x = x + mult * feed_forward(rms(x, eps) * W[p + "norm2"], W, p + "mlp.", L["mlp"])
        stream.append(x)
    return (rms(x, eps) * W["final.norm"]) @ W["head"].T, torch.stack(stream)
