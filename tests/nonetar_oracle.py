"""Plain restatement of the Nonetar decoder, one function per mechanism, whole sequences only, no cache.

Written from the model's equations for the tests; it shares no code with the package.  Everything runs in the dtype of the
weights handed in (the tests use float64).
"""
import math

import torch


def unit(x, eps):
    """Rows divided by their root mean square."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    """RMS norm whose weight is stored around zero."""
    return unit(x, eps) * (1 + w)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log(1 + torch.exp(-z.abs()))


def gelu(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def positions(T, width):
    """Sines at even and cosines at odd places, both of a pair at the rate of its even place."""
    out = torch.zeros(T, width, dtype=torch.float64)
    for p in range(T):
        for e in range(width):
            a = p * 10000.0 ** (-(e - e % 2) / width)
            out[p, e] = math.cos(a) if e % 2 else math.sin(a)
    return out


def embed(tokens, W):
    E = W["embed"]
    return E[torch.tensor(tokens)] + positions(len(tokens), E.shape[1]).to(E.dtype)


def shift(h, w):
    """Every row moved towards its predecessor (zeros in front of the first)."""
    back = torch.cat((torch.zeros_like(h[:1]), h[:-1]))
    return h + (back - h) * w


def gather(streams, W, hc):
    """Input of a sublayer: ``streams`` [s, T, width]."""
    return sum(W[hc + "in"][s] * streams[s] for s in range(streams.shape[0]))


def scatter(streams, y, W, hc):
    """Every stream from all the old ones (the matrix is indexed from, to) and the sublayer's output."""
    n = streams.shape[0]
    return torch.stack([sum(W[hc + "mix"][s, t] * streams[s] for s in range(n)) + W[hc + "out"][t] * y for t in range(n)])


def slopes(H):
    return [2.0 ** (-8.0 * (h + 1) / H) for h in range(H)]


def scores(q, k, m, temp, slope):
    """Biased scores of one head, ``q`` [T, d], ``k`` [T, d] -> [T, T]."""
    s = q @ k.T * m["scale"] * temp
    s = m["softcap"] * torch.tanh(s / m["softcap"])
    i = torch.arange(s.shape[0], dtype=s.dtype)
    return s - slope * (i[:, None] - i[None, :])


def weights_of(s, size):
    """Softmax of every row over itself and the ``size - 1`` places in front of it."""
    out = torch.zeros_like(s)
    for i in range(s.shape[0]):
        a = max(0, i - size + 1)
        e = torch.exp(s[i, a : i + 1] - s[i, a : i + 1].max())
        out[i, a : i + 1] = e / e.sum()
    return out


def attention(h, W, p, m, eps):
    """Heads in front of the output projection, [T, heads * vdim]."""
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = ((h @ W[p + n].T + W[p + n + ".b"]).view(T, x, y) for n, x, y in (("q", H, d), ("k", G, d), ("v", G, dv)))
    q, k = unit(q, eps) * W[p + "q.norm"], unit(k, eps) * W[p + "k.norm"]
    a = [weights_of(scores(q[:, i], k[:, i // (H // G)], m, W[p + "temp"][i], slopes(H)[i]), m["mask"]["size"]) @ v[:, i // (H // G)] for i in range(H)]
    return torch.cat(a, 1)


def conv(x, w, b):
    """Causal convolution per channel, zeros in front of the start; the last tap is the current row's."""
    T, taps = x.shape[0], w.shape[1]
    pad = torch.cat((torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x))
    return torch.stack([(pad[t : t + taps] * w.T).sum(0) + b for t in range(T)])


def block_gate(u, W, p, n):
    """Sigmoid of the block-diagonal projection."""
    blocks = u.view(u.shape[0], W[p + n].shape[0], -1)
    return sigmoid(torch.einsum("tbi,boi->tbo", blocks, W[p + n]) + W[p + n + ".b"]).flatten(1)


def lru(u, r, i, lam):
    """State of every token: a gated linear recurrence per channel."""
    S, out = torch.zeros_like(u[0]), []
    for t in range(u.shape[0]):
        log_a = -8 * r[t] * softplus(lam)
        S = torch.exp(log_a) * S + torch.sqrt(-torch.expm1(2 * log_a)) * i[t] * u[t]
        out.append(S)
    return torch.stack(out)


def griffin(h, W, p, m):
    """The recurrent block in front of its output projection, [T, width]."""
    y = gelu(h @ W[p + "y"].T + W[p + "y.b"])
    u = conv(h @ W[p + "x"].T + W[p + "x.b"], W[p + "conv"], W[p + "conv.b"])
    return lru(u, block_gate(u, W, p, "ra"), block_gate(u, W, p, "ri"), W[p + "lam"]) * y


def parallel_mixer(h, W, p, m, eps):
    left = attention(h, W, p + "left.", m["left"], eps) @ W[p + "left.o"].T
    right = griffin(h, W, p + "right.", m["right"]) @ W[p + "right.o"].T
    return m["left_scale"] * left + m["right_scale"] * right


def ssd(x, B, C, dt, a_log, D):
    """``x`` [T, H, dv], ``B, C`` [T, G, N], ``dt`` [T, H] -> [T, H, dv]."""
    T, H, dv = x.shape
    per = H // B.shape[1]
    out = torch.zeros_like(x)
    for h in range(H):
        S = torch.zeros(B.shape[2], dv, dtype=x.dtype)
        for t in range(T):
            S = torch.exp(-torch.exp(a_log[h]) * dt[t, h]) * S + dt[t, h] * B[t, h // per][:, None] * x[t, h][None]
            out[t, h] = S.T @ C[t, h // per] + D[h] * x[t, h]
    return out


def mamba2_mixer(h, W, p, m, eps):
    T, H, dv, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * dv
    z, c, dt = (h @ W[p + "in"].T).split((inner, inner + 2 * G * N, H), 1)
    x, B, C = silu(conv(c, W[p + "conv"], W[p + "conv.b"])).split((inner, G * N, G * N), 1)
    y = ssd(x.reshape(T, H, dv), B.reshape(T, G, N), C.reshape(T, G, N), softplus(dt + W[p + "dt_bias"]), W[p + "A_log"], W[p + "D"]).reshape(T, inner)
    y = unit((y * silu(z)).view(T, m["norm_groups"], -1), eps).reshape(T, inner)
    return (y * W[p + "norm"]) @ W[p + "o"].T


def xielu(z, p, q):
    return torch.where(z > 0, softplus(p) * z * z, (0.5 + softplus(q)) * (torch.expm1(torch.clamp(z, max=0)) - z)) + 0.5 * z


def feed_forward(h, W, p):
    return xielu(h @ W[p + "up"].T, *W[p + "act"]) @ W[p + "down"].T


MIXERS = {"parallel": parallel_mixer, "mamba2": mamba2_mixer}


def forward(cfg, W, tokens):
    """Logits [T, vocab] and the sum of the streams after every layer [layers, T, width] of one whole sequence."""
    eps, after = cfg["norm"]["eps"], []
    streams = embed(list(tokens), W)[None].repeat(cfg["streams"], 1, 1)
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = norm(gather(streams, W, p + "hc1."), W[p + "norm1"], eps)
        streams = scatter(streams, MIXERS[L["type"]](shift(h, W[p + "shift"]), W, p + "mix.", L["mixer"], eps), W, p + "hc1.")
        if L.get("mlp"):
            h = norm(gather(streams, W, p + "hc2."), W[p + "norm2"], eps)
            streams = scatter(streams, feed_forward(h, W, p + "mlp."), W, p + "hc2.")
        after.append(streams.sum(0))
    return (norm(streams.sum(0), W["final.norm"], eps) @ W["head"].T) * cfg["logit_scale"], torch.stack(after)
