"""Small Nemipel configurations, random weights and step schedules for the tests of that line."""
import json
import os

import torch

import nemipel_oracle as O

V = 203


def _attn(heads, kv, dim, vdim, rot, scale=None, softcap=None, kv_from=None, base=100.0):
    m = dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, rot=dict(dims=rot, base=base), scale=scale or dim ** -0.5)
    if softcap is not None:
        m["softcap"] = softcap
    if kv_from is not None:
        m["kv_from"] = kv_from
    return "attention", m


def _light(heads, dim, vdim, decay):
    return "lightning", dict(heads=heads, dim=dim, vdim=vdim, decay=list(decay))


def _delta(heads, kv, dim, vdim, conv):
    return "channel_delta", dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, conv=conv)


def _cfg(width, eps, alpha, cap, layers, vocab=V):
    out = dict(architecture="Nemipel", vocab=vocab, width=width, norm=dict(eps=eps), postln_alpha=alpha,
               layers=[dict(type=t, mixer=m, mlp=dict(kind="dense", ff=ff) if ff else None) for (t, m), ff in layers])
    if cap:
        out["logit_softcap"] = cap
    return out


CONFIGS = {
    # key size != value size, two value heads per query / key head, decay and gate ranks that differ, shared cache with
    # another scale and cap than the layer that owns it
    "mixed": _cfg(72, 1e-5, 1.7, 6.0, [(_attn(6, 2, 24, 40, 10, softcap=5.0), 56), (_delta(6, 3, 24, 16, 3), 44), (_light(3, 40, 24, (0.9, 1.0, 0.25)), 40),
                                       (_attn(6, 2, 24, 40, 10, scale=0.31, softcap=9.0, kv_from=0), 0)]),
    # the sizes the tensor-core kernels are built for; no grouping; a convolution of one tap; recurrent layers first
    "wide": _cfg(64, 1e-6, 1.0, 0.0, [(_delta(2, 2, 128, 128, 1), 0), (_light(2, 128, 128, (0.98, 0.6)), 64), (_attn(4, 4, 128, 128, 128, softcap=20.0), 32), (_attn(4, 4, 128, 128, 128, kv_from=2), 64)]),
    # nothing is a multiple of 8; more than eight query heads per KV head; no caps
    "odd": _cfg(50, 1e-3, 0.5, 0.0, [(_attn(18, 1, 18, 13, 2), 30), (_light(5, 6, 11, (0.5, 0.7, 0.8, 0.9, 0.999)), 0), (_delta(3, 1, 7, 9, 5), 21)]),
    # more than eight heads per group, heads of 256, key width past 128, no rotation
    "large": _cfg(128, 1e-6, 2.5, 12.0, [(_attn(20, 2, 256, 72, 64, softcap=50.0), 96), (_light(2, 144, 40, (0.95, 0.8)), 0), (_delta(4, 2, 136, 48, 4), 72), (_attn(2, 1, 32, 64, 0), 24)]),
    # no cache at all; no recurrent state at all
    "recurrent": _cfg(48, 1e-6, 2.0, 9.0, [(_light(2, 24, 8, (0.9, 0.3)), 0), (_delta(2, 1, 16, 8, 2), 32)]),
    "attention": _cfg(40, 1e-6, 2.0, 9.0, [(_attn(2, 2, 16, 8, 4, softcap=3.0), 0), (_attn(3, 1, 40, 24, 40, softcap=8.0), 32)]),
}


# largest error of a position in bf16 (twice what rounding the activations of the plain path to bf16 gives; a small
# postln_alpha lets the sublayers' rounding through)
BF16_ERROR = {"mixed": 0.12, "wide": 0.08, "odd": 0.36, "large": 0.03, "recurrent": 0.08, "attention": 0.08}


def weights(cfg, seed=0, dtype=torch.bfloat16):
    """Random weights (rounded to ``dtype``) that give peaked attention, decays from fast to slow and streams of order 1."""
    g = torch.Generator().manual_seed(seed)
    w, W = cfg["width"], {}

    def mat(rows, cols, gain=1.0):
        return torch.randn(rows, cols, generator=g) * gain * cols ** -0.5

    def vec(n, mean=1.0, spread=0.2):
        return mean + spread * torch.randn(n, generator=g)

    W["embed"], W["final.norm"], W["head"] = torch.randn(cfg["vocab"], w, generator=g), vec(w), mat(cfg["vocab"], w, 2.0)
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}.mix."
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        W[f"l{i}.norm1"], W[p + "o"] = vec(w), mat(w, H * dv, 2.0)
        if L["type"] == "attention":
            W[p + "q"], W[p + "q.norm"], W[p + "g"] = mat(H * d, w), vec(H * d, 1.6), mat(H, w)
            if m.get("kv_from") is None:
                G = m["kv_heads"]
                W[p + "k"], W[p + "k.norm"], W[p + "v"] = mat(G * d, w), vec(G * d, 1.6), mat(G * dv, w)
        elif L["type"] == "lightning":
            for n, r in (("q", H * d), ("k", H * d), ("v", H * dv), ("g", H * dv)):
                W[p + n] = mat(r, w)
            W[p + "norm"] = vec(H * dv)
        else:
            G, ra, rg = m["kv_heads"], 10, 6
            for n, r in (("q", G * d), ("k", G * d), ("v", H * dv)):
                W[p + n], W[p + n + ".conv"] = mat(r, w), torch.randn(r, m["conv"], generator=g) * 0.7
            W[p + "b"], W[p + "A_log"], W[p + "norm"], W[p + "dt_bias"] = mat(H, w), torch.linspace(-4.0, 1.0, H) if H > 1 else torch.tensor([-2.0]), vec(dv), vec(H * d, -1.0, 1.0)
            W[p + "a1"], W[p + "a2"], W[p + "g1"], W[p + "g2"] = mat(ra, w), mat(H * d, ra), mat(rg, w), mat(H * dv, rg)
        if L["mlp"]:
            ff = L["mlp"]["ff"]
            W[f"l{i}.norm2"], W[f"l{i}.mlp.gate"], W[f"l{i}.mlp.up"], W[f"l{i}.mlp.down"] = vec(w), mat(ff, w), mat(ff, w), mat(w, ff, 2.0)
    return {k: v.to(dtype).contiguous() for k, v in W.items()}


def tokens(n, seed, vocab=V):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def truth(cfg, W, toks):
    return O.forward(cfg, {k: v.double() for k, v in W.items()}, toks)[0]


def checkpoint(path, cfg, W):
    from safetensors.torch import save_file

    os.makedirs(path, exist_ok=True)
    save_file(W, os.path.join(path, "model.safetensors"))
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    return str(path)


def replayer(cfg, W, device, dtype, max_tokens, requests=4, **kw):
    """A trace replayer over an engine with these weights."""
    from pegainfer_b200.config import EngineConfig, from_hf
    from pegainfer_b200.engine.build import build_engine
    from pegainfer_b200.loader.sources import DictSource
    from pegainfer_b200.models import registry
    from pegainfer_b200.replay import Replayer

    mcfg = from_hf(cfg)
    mcfg.max_position = 4096
    model = registry.build(mcfg, source=DictSource(W), device=device, dtype=dtype)
    page = kw.pop("page", 16)
    ecfg = EngineConfig(kv_page_size=page, num_kv_blocks=(max_tokens + page - 1) // page + 1, max_decode_batch=requests, state_slots=requests, no_prefix_cache=True, run_ahead=False, **kw)
    return Replayer(build_engine(ecfg, mcfg, device=device, dtype=dtype, model=model, start=False))


def run(rep, schedule, prompts):
    """``schedule``: steps of ``(request, count)``; a name ``a#1`` is prompt ``a`` once more.  Every position's logits are
    asked for; a request ends with its prompt.  Returns request -> logits [T, vocab]."""
    at, out = {}, {}
    for step in schedule:
        entries, done = [], []
        for r, n in step:
            p, lo = prompts[r.split("#")[0]], at.get(r, 0)
            entries.append((r, p[lo : lo + n], list(range(n))))
            at[r] = lo + n
            if at[r] == len(p):
                done.append(r)
        lg, k = rep.step(entries).cpu(), 0
        for r, toks, _ in entries:
            out.setdefault(r, []).append(lg[k : k + len(toks)])
            k += len(toks)
        for r in done:
            rep.end(r)
    assert not rep.live
    return {r: torch.cat(x) for r, x in out.items()}


def error(got, want):
    """Root mean square over the vocabulary of the difference without its mean, per position, over the logits' spread."""
    d = got.double() - want
    d = d - d.mean(1, keepdim=True)
    return d.pow(2).mean(1).sqrt() / (want - want.mean(1, keepdim=True)).pow(2).mean().sqrt()
