"""Small Zeripel configurations and random weights for the tests of that line."""
import torch

import zeripel_oracle as O
from nemipel_util import checkpoint, error, replayer, run, tokens  # noqa: F401
from vekalorn_util import close_in_bf16  # noqa: F401

V = 203


def _wkv(heads, dim):
    return "wkv", dict(heads=heads, dim=dim)


def _attn(heads, kv, dim, temp=None, scale=None):
    m = dict(heads=heads, kv_heads=kv, dim=dim, vdim=dim, scale=scale or dim ** -0.5)
    if temp:
        m["q_temp"] = dict(coef=temp[0], every=temp[1])
    return "attention", m


def _latent(heads, kv_rank, dim, rot, vdim, kv_from=None, base=300.0, scale=None):
    m = dict(heads=heads, kv_rank=kv_rank, dim=dim, rot_dim=rot, vdim=vdim, scale=scale or 1.3 * (dim + rot) ** -0.5, rot=dict(dims=rot, base=base))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return "latent_attention", m


def _moe(experts, top, ff, shared, scale=1.5):
    m = dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top, scale=scale))
    if shared:
        m["shared"] = dict(ff=shared)
    return m


def _dense(ff):
    return dict(kind="dense", ff=ff)


def _cfg(width, eps, mult, scale, bigram, layers, vocab=V):
    return dict(architecture="Zeripel", vocab=vocab, width=width, norm=dict(eps=eps), residual_mult=mult, embedding=dict(scale=scale, bigram=dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))),
                layers=[dict(type=t, mixer=m, mlp=mlp) for (t, m), mlp in layers])


CONFIGS = {
    # every size its own value; a cache shared by layers with other heads and value sizes than its owner; a layer without
    # feed-forward; a router of other counts per layer
    "mixed": _cfg(72, 1e-5, 0.8, 2.5, (131, 37, 11), [(_wkv(3, 24), _moe(12, 3, 40, 56)), (_latent(5, 56, 16, 8, 40), _dense(88)), (_attn(6, 2, 40, (0.4, 7)), _moe(5, 2, 24, 16, 0.7)),
                                                      (_latent(2, 56, 24, 8, 16, kv_from=1), None), (_wkv(2, 40), _dense(48))]),
    # the sizes the tensor-core kernels are built for
    "wide": _cfg(128, 1e-6, 0.6, 4.0, (509, 127, 3), [(_latent(16, 512, 128, 64, 128), _dense(256)), (_latent(4, 512, 128, 64, 96, kv_from=0, scale=0.1), _moe(16, 4, 64, 128)), (_wkv(2, 128), _moe(8, 2, 128, 64, 2.5)),
                                                      (_attn(8, 2, 128, (0.2, 64)), _moe(8, 1, 64, 32)), (_wkv(4, 64), None)]),
    # nothing is a multiple of 8; more than eight query heads per key head; a temperature that steps at every position
    "odd": _cfg(50, 1e-3, 1.3, 0.7, (97, 5, 1), [(_attn(18, 1, 18, (0.15, 1)), _dense(30)), (_wkv(3, 7), _moe(6, 2, 9, 13)), (_latent(3, 21, 10, 6, 11), _moe(7, 5, 5, 3, 1.0)), (_latent(7, 21, 5, 6, 3, kv_from=2), _dense(21))]),
    # past the tensor-core instances: latents, rotated parts, key widths of the recurrence, attention heads
    "large": _cfg(96, 1e-6, 0.5, 1.0, (1, 1, 1), [(_latent(2, 640, 40, 80, 136), _moe(32, 6, 32, 48)), (_wkv(1, 136), _dense(64)), (_attn(20, 2, 256), _moe(1, 1, 64, 8)), (_wkv(2, 200), None)]),
    # no cache at all; no recurrent layer at all; a mixture without a shared expert
    "recurrent": _cfg(40, 1e-5, 1.0, 3.0, (64, 13, 29), [(_wkv(1, 16), _dense(32)), (_wkv(5, 8), _moe(4, 2, 16, 0))]),
    "cached": _cfg(48, 1e-5, 0.9, 6.928, (311, 2147483647, 7919), [(_latent(4, 32, 24, 2, 8), None), (_latent(2, 128, 16, 32, 24, base=1e4), _dense(40)), (_latent(6, 32, 8, 2, 32, kv_from=0), _moe(9, 4, 8, 16, 3.0)),
                                                                   (_attn(3, 3, 24, (1.0, 1000)), None), (_latent(1, 128, 16, 32, 16, kv_from=1, base=1e4), _dense(24))]),
}


def weights(cfg, seed=0, dtype=torch.bfloat16):
    """Random weights (rounded to ``dtype``) that give peaked attention with sinks that count, decays from fast to slow,
    decided routers and streams of order 1."""
    g = torch.Generator().manual_seed(seed)
    w, W = cfg["width"], {}

    def mat(rows, cols, gain=1.0):
        return torch.randn(rows, cols, generator=g) * gain * cols ** -0.5

    def vec(n, mean=1.0, spread=0.2):
        return mean + spread * torch.randn(n, generator=g)

    def glu(p, ff):
        W[p + "gate"], W[p + "up"], W[p + "down"] = mat(ff, w, 1.5), mat(ff, w), mat(w, ff, 1.5)

    e = cfg["embedding"]
    W["embed"], W["bigram"] = torch.randn(cfg["vocab"], w, generator=g) / e["scale"], torch.randn(e["bigram"]["buckets"] + 1, w, generator=g) * 0.7
    W["final.norm"], W["head"] = vec(w), mat(cfg["vocab"], w, 2.0)
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}.mix."
        H, d = m["heads"], m["dim"]
        n = H * m.get("vdim", d)
        W[f"l{i}.norm1"], W[p + "o"] = vec(w), mat(w, n)
        if L["type"] == "wkv":
            for x in "rkvgw":
                W[p + "mu." + x] = torch.rand(w, generator=g)
            for x in "rkvg":
                W[p + x] = mat(n, w)
            rank = 8 + 3 * (i % 3)
            W[p + "w1"], W[p + "w2"], W[p + "w0"], W[p + "u"], W[p + "norm"] = mat(rank, w), mat(n, rank, 0.7), torch.linspace(-6.0, 1.5, n)[torch.randperm(n, generator=g)], vec(n, 0.5, 0.5).view(H, d), vec(n)
        elif L["type"] == "attention":
            W[p + "q"], W[p + "k"], W[p + "q.norm"], W[p + "k.norm"] = mat(n, w), mat(m["kv_heads"] * d, w), vec(d, 1.5), vec(d, 1.2)
        else:
            c, r = m["kv_rank"], m["rot_dim"]
            W[p + "q"], W[p + "uk"], W[p + "uv"], W[p + "sink"], W[p + "g"] = mat(H * (d + r), w, 1.3), mat(H * d, c, 1.3), mat(n, c), vec(H, 1.5, 1.0), mat(H, w)
            if m.get("kv_from") is None:
                W[p + "dkv"], W[p + "dkv.norm"] = mat(c + r, w), vec(c, 1.1)
        f, q = L["mlp"], f"l{i}.mlp."
        if f:
            W[f"l{i}.norm2"] = vec(w)
            if f["kind"] == "dense":
                glu(q, f["ff"])
            else:
                W[q + "router"], W[q + "correction"] = mat(f["router"]["experts"], w, 1.5), vec(f["router"]["experts"], 0.0, 0.3)
                for x in range(f["router"]["experts"]):
                    glu(f"{q}e{x}.", f["expert"]["ff"])
                if f.get("shared"):
                    glu(q + "shared.", f["shared"]["ff"])
                    W[q + "shared.sg"] = mat(1, w)
    return {k: v.to(dtype).contiguous() for k, v in W.items()}


def truth(cfg, W, toks):
    return O.forward(cfg, {k: v.double() for k, v in W.items()}, toks)[0]
