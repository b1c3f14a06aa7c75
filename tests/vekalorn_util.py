"""Small Vekalorn configurations and random weights for the tests of that line."""
import torch

import vekalorn_oracle as O
from nemipel_util import checkpoint, error, replayer, run, tokens  # noqa: F401

V = 203


def _local(heads, q_rank, kv_rank, dim, vdim, window, scale=None):
    return "latent_attention", dict(heads=heads, q_rank=q_rank, kv_rank=kv_rank, dim=dim, vdim=vdim, scale=scale or 1.3 * dim ** -0.5, mask=dict(size=window))


def _full(heads, q_rank, kv_rank, dim, rot, vdim, base=300.0, yarn=(4.0, 64, 8.0, 1.0), scale=None):
    r = dict(dims=rot, base=base)
    if yarn:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    return "latent_attention_2", dict(heads=heads, q_rank=q_rank, kv_rank=kv_rank, dim=dim, rot_dim=rot, vdim=vdim, scale=scale or 1.3 * (dim + rot) ** -0.5, rot=r)


def _moe(experts, top, ff, groups=1, keep=1):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top, groups=dict(count=groups, keep=keep)))


def _cfg(width, eps, layers, vocab=V):
    return dict(architecture="Vekalorn", vocab=vocab, width=width, norm=dict(eps=eps), layers=[dict(type=t, mixer=m, mlp=mlp) for (t, m), mlp in layers])


CONFIGS = {
    # every size its own value, windows of several lengths, a layer without feed-forward, two rotations
    "mixed": _cfg(72, 1e-5, [(_local(3, 40, 56, 24, 16, 7), _moe(12, 3, 40, 3, 2)), (_full(5, 24, 32, 16, 8, 40), _moe(8, 2, 24, 4, 2)), (_local(2, 16, 64, 40, 32, 33), None),
                             (_full(1, 32, 48, 8, 24, 8, base=900.0, yarn=(2.5, 40, 5.0, 0.5), scale=0.4), _moe(5, 5, 16))]),
    # the sizes the tensor-core kernels are built for, and a latent between two of their instances
    "wide": _cfg(128, 1e-6, [(_full(16, 128, 512, 128, 64, 128), _moe(16, 4, 64, 4, 3)), (_local(16, 96, 512, 128, 128, 70), _moe(16, 4, 128, 8, 4)), (_local(20, 64, 192, 64, 96, 128), _moe(4, 1, 64, 2, 1))]),
    # nothing is a multiple of 8, one expert per group, a window of one position, no scaling of the rotation
    "odd": _cfg(50, 1e-3, [(_full(3, 13, 21, 10, 6, 11, yarn=None), _moe(6, 2, 9, 6, 3)), (_local(7, 9, 15, 5, 3, 1), _moe(7, 2, 5)), (_local(2, 17, 30, 9, 13, 19), _moe(9, 3, 20, 3, 1))]),
    # latents and rotated parts past the tensor-core instances, a single head, one expert only
    "large": _cfg(96, 1e-6, [(_full(2, 72, 640, 40, 80, 136, yarn=(1.0, 128, 32.0, 1.0)), _moe(32, 6, 32, 8, 2)), (_local(1, 32, 264, 136, 8, 300), _moe(1, 1, 64))]),
    # no rotated layer at all; no feed-forward at all
    "local": _cfg(40, 1e-5, [(_local(4, 24, 32, 16, 24, 16), _moe(10, 2, 8, 5, 2)), (_local(4, 24, 32, 16, 24, 64), _moe(10, 4, 8, 2, 1))]),
    "plain": _cfg(48, 1e-5, [(_full(4, 24, 128, 32, 64, 16, base=1e4), None), (_full(2, 40, 256, 24, 16, 48, base=50.0, yarn=(8.0, 1024, 32.0, 1.0)), None)]),
}


def weights(cfg, seed=0, dtype=torch.bfloat16):
    """Random weights (rounded to ``dtype``) that give peaked attention, decided routers and streams of order 1."""
    g = torch.Generator().manual_seed(seed)
    w, W = cfg["width"], {}

    def mat(rows, cols, gain=1.0):
        return torch.randn(rows, cols, generator=g) * gain * cols ** -0.5

    def vec(n, mean=1.0, spread=0.2):
        return mean + spread * torch.randn(n, generator=g)

    W["embed"], W["final.norm"], W["head"] = torch.randn(cfg["vocab"], w, generator=g), vec(w), mat(cfg["vocab"], w, 2.0)
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}.mix."
        H, d, dv, c, r = m["heads"], m["dim"], m["vdim"], m["kv_rank"], m.get("rot_dim", 0)
        W[f"l{i}.norm1"], W[p + "o"] = vec(w, 0.6), mat(w, H * dv)
        W[p + "dq"], W[p + "dq.norm"], W[p + "uq"] = mat(m["q_rank"], w), vec(m["q_rank"], 1.2), mat(H * (d + r), m["q_rank"], 1.3)
        W[p + "dkv"], W[p + "dkv.norm"], W[p + "uk"], W[p + "uv"] = mat(c + r, w), vec(c, 1.1), mat(H * d, c, 1.3), mat(H * dv, c)
        if r:
            W[p + "g"] = mat(H * dv, w)
        if L["mlp"]:
            e, ff, q = L["mlp"]["router"]["experts"], L["mlp"]["expert"]["ff"], f"l{i}.mlp."
            W[f"l{i}.norm2"], W[q + "router"] = vec(w, 0.6), mat(e, w, 2.0)
            for x in range(e):
                W[f"{q}e{x}.up"], W[f"{q}e{x}.down"] = mat(ff, w), mat(w, ff)
    return {k: v.to(dtype).contiguous() for k, v in W.items()}


def truth(cfg, W, toks):
    return O.forward(cfg, {k: v.double() for k, v in W.items()}, toks)[0]


def close_in_bf16(err):
    """bf16 errors of a sequence's positions.  Where a router's choice is close, rounding may take the other expert, and that
    position's logits (and a little those that attend to it) belong to another network; such choices are a small share."""
    return bool(err.median() < 0.03 and err.quantile(0.8) < 0.1)
