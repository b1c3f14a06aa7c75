"""Small Nonetar configurations and random weights for the tests of that line."""
import torch

import nonetar_oracle as O
from nemipel_util import checkpoint, error, replayer, run, tokens  # noqa: F401

V = 203


def _par(heads, kv, dim, vdim, window, width, blocks, conv, scales=(1.3, 0.7), scale=None, softcap=8.0):
    return "parallel", dict(left=dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, mask=dict(size=window), scale=scale or 1.5 * dim ** -0.5, softcap=softcap),
                            right=dict(width=width, blocks=blocks, conv=conv), left_scale=scales[0], right_scale=scales[1])


def _ssd(heads, vdim, state, groups, norm_groups, conv):
    return "mamba2", dict(heads=heads, vdim=vdim, state=state, groups=groups, norm_groups=norm_groups, conv=conv)


def _cfg(width, eps, streams, logit_scale, layers, vocab=V):
    return dict(architecture="Nonetar", vocab=vocab, width=width, norm=dict(eps=eps), streams=streams, logit_scale=logit_scale,
                layers=[dict(type=t, mixer=m, mlp=dict(kind="dense", ff=ff) if ff else None) for (t, m), ff in layers])


CONFIGS = {
    # every size its own value, per layer; layers without feed-forward in the middle and at the end
    "mixed": _cfg(72, 1e-5, 3, 0.6, [(_par(4, 2, 24, 40, 20, 96, 6, 3), 104), (_ssd(6, 16, 24, 3, 2, 4), None), (_par(6, 3, 16, 8, 33, 40, 5, 2, (0.4, 1.6), softcap=3.0), 56), (_ssd(4, 32, 8, 1, 4, 2), 40),
                                     (_par(2, 1, 32, 24, 17, 64, 1, 4), None)]),
    # the sizes the tensor-core kernels are built for
    "wide": _cfg(128, 1e-6, 4, 1.7, [(_par(4, 2, 128, 128, 150, 256, 2, 4), 256), (_ssd(8, 64, 128, 4, 8, 4), 512), (_par(2, 2, 128, 128, 64, 128, 8, 3, (0.8, 0.8), softcap=30.0), 128), (_ssd(2, 128, 64, 2, 1, 3), None)]),
    # nothing is a multiple of 8; more than eight query heads per key head; one tap; more copies than the register form takes
    "odd": _cfg(51, 1e-3, 5, 1.0, [(_par(18, 1, 18, 11, 7, 63, 3, 1), 30), (_ssd(3, 7, 9, 1, 3, 2), 21), (_par(3, 3, 5, 7, 1, 21, 7, 5, (1.0, 1.0)), None), (_ssd(5, 3, 11, 5, 1, 1), 13)]),
    # past the tensor-core instances: attention heads, state widths, taps; one copy of the stream
    "large": _cfg(96, 1e-6, 1, 0.3, [(_par(20, 2, 256, 200, 90, 272, 2, 9), 64), (_ssd(2, 136, 200, 1, 2, 5), 72), (_ssd(1, 40, 136, 1, 1, 16), None)]),
    # no cache at all; no state-space layer at all
    "recurrent": _cfg(40, 1e-5, 2, 2.0, [(_ssd(2, 16, 16, 2, 2, 4), 32), (_ssd(5, 8, 40, 5, 5, 3), 24)]),
    "cached": _cfg(48, 1e-4, 6, 0.9, [(_par(8, 4, 8, 16, 16, 24, 3, 4), 40), (_par(3, 3, 40, 8, 100, 72, 9, 2, (2.0, 0.2)), 88)]),
}


def weights(cfg, seed=0, dtype=torch.bfloat16):
    """Random weights (rounded to ``dtype``) that give peaked attention with a cap that bites, decays from fast to slow, copies of
    the stream that stay apart, and streams of order 1."""
    g = torch.Generator().manual_seed(seed)
    w, n, W = cfg["width"], cfg["streams"], {}

    def mat(rows, cols, gain=1.0):
        return torch.randn(rows, cols, generator=g) * gain * cols ** -0.5

    def vec(k, mean=0.0, spread=0.2):
        return mean + spread * torch.randn(k, generator=g)

    def spread(k, lo, hi):
        return torch.linspace(lo, hi, k)[torch.randperm(k, generator=g)]

    W["embed"], W["final.norm"], W["head"] = torch.randn(cfg["vocab"], w, generator=g), vec(w), mat(cfg["vocab"], w, 2.0)
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}."
        W[p + "norm1"], W[p + "shift"] = vec(w), torch.rand(w, generator=g) * 0.8
        for q in ("hc1.", "hc2.") if L["mlp"] else ("hc1.",):
            W[p + q + "in"], W[p + q + "out"], W[p + q + "mix"] = vec(n, 1 / n, 0.3), vec(n, 0.8, 0.4), 0.8 * torch.eye(n) + 0.2 * torch.randn(n, n, generator=g) * n ** -0.5
        if L["type"] == "parallel":
            a, r, q, t = m["left"], m["right"], p + "mix.left.", p + "mix.right."
            for x, rows in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
                W[q + x], W[q + x + ".b"] = mat(rows, w), vec(rows, 0, 0.5)
            W[q + "q.norm"], W[q + "k.norm"], W[q + "temp"], W[q + "o"] = vec(a["dim"], 1.6), vec(a["dim"], 1.4), vec(a["heads"], 1.2, 0.4), mat(w, a["heads"] * a["vdim"])
            c, b = r["width"], r["blocks"]
            for x in ("y", "x"):
                W[t + x], W[t + x + ".b"] = mat(c, w), vec(c, 0.2, 0.5)
            for x in ("ra", "ri"):
                W[t + x], W[t + x + ".b"] = torch.randn(b, c // b, c // b, generator=g) * 1.5 * (c // b) ** -0.5, vec(c, 0, 0.5).view(b, -1)
            W[t + "conv"], W[t + "conv.b"], W[t + "lam"], W[t + "o"] = mat(c, r["conv"], 1.2), vec(c), spread(c, -7.0, 0.5), mat(w, c, 1.5)
        else:
            inner = m["heads"] * m["vdim"]
            c = inner + 2 * m["groups"] * m["state"]
            W[p + "mix.in"], W[p + "mix.conv"], W[p + "mix.conv.b"] = mat(inner + c + m["heads"], w), mat(c, m["conv"], 1.5), vec(c, 0.1)
            W[p + "mix.dt_bias"], W[p + "mix.A_log"], W[p + "mix.D"] = vec(m["heads"], -1.0, 0.7), spread(m["heads"], -3.0, 1.5), vec(m["heads"], 1.0, 0.5)
            W[p + "mix.norm"], W[p + "mix.o"] = vec(inner, 1.0), mat(w, inner)
        if L["mlp"]:
            ff = L["mlp"]["ff"]
            W[p + "norm2"], W[p + "mlp.up"], W[p + "mlp.down"], W[p + "mlp.act"] = vec(w), mat(ff, w, 1.3), mat(w, ff), torch.tensor([0.3, -0.9]) + vec(2)
    return {k: v.to(dtype).contiguous() for k, v in W.items()}


def truth(cfg, W, toks):
    return O.forward(cfg, {k: v.double() for k, v in W.items()}, toks)[0]
