"""Vekalorn line on CPU: the operations and whole models of the CPU path against the plain restatement, steps cut in
different ways, generation with shared prefixes, configuration, checkpoint and command line."""
import json

import pytest
import torch

import vekalorn_oracle as O
import vekalorn_util as U
from pegainfer_b200.config import EngineConfig, from_hf, load_model_config, preset
from pegainfer_b200.engine.build import build_engine
from pegainfer_b200.kv.buffer import MixedKvBuffer
from pegainfer_b200.loader.sources import DictSource
from pegainfer_b200.models import registry
from pegainfer_b200.models.vekalorn import VekalornModel, vekalorn_shapes
from pegainfer_b200.ops import reference as R

PROMPTS = {"a": U.tokens(80, 1), "b": U.tokens(37, 2), "c": U.tokens(1, 3), "d": U.tokens(50, 4)}
SCHEDULES = {
    "whole": [[(r, len(p))] for r, p in PROMPTS.items()],
    "tokens": [[("b", 1)]] * 37,
    "portions": [[("a", n)] for n in (2, 3, 14, 45, 1, 15)] + [[("d", 2)]] * 25,
    "batched": [[("a", 33), ("b", 1), ("d", 2), ("c", 1)], [("b", 1), ("a", 2), ("d", 40)], [("a", 1), ("b", 1), ("d", 1)], [("b", 33), ("a", 44)], [("d", 6), ("b", 1)], [("d", 1), ("c#1", 1), ("b#1", 3)],
                [("b#1", 33), ("a#1", 80)], [("b#1", 1)]],
}


@pytest.mark.parametrize("name", sorted(U.CONFIGS))
def test_models_cut_into_steps(name):
    cfg = U.CONFIGS[name]
    W = U.weights(cfg)
    rep = U.replayer(cfg, W, "cpu", torch.float32, 240)
    want = {r: U.truth(cfg, W, p) for r, p in PROMPTS.items()}
    for sched in SCHEDULES.values():
        for r, got in U.run(rep, sched, PROMPTS).items():
            assert U.error(got, want[r.split("#")[0]]).max() < 5e-5
    assert rep.pool.used() == 0


def test_stream_after_every_layer():
    from pegainfer_b200.kv.request_kv import KvView
    from pegainfer_b200.sched.executor import SeqStep, build_meta

    cfg = U.CONFIGS["mixed"]
    W = U.weights(cfg)
    rep = U.replayer(cfg, W, "cpu", torch.float32, 64)
    toks = U.tokens(20, 9)
    ids, meta = build_meta([SeqStep(rid=0, input_tokens=toks, start_pos=0, view=KvView([3, 1], 20, 16))], 16, "cpu")
    rep.ex.model.forward_hidden(ids, meta, rep.ex.kv, aux_layers=range(4))
    stream = O.forward(cfg, {k: v.double() for k, v in W.items()}, toks)[1]
    for got, want in zip(rep.ex.model.last_aux, stream):
        assert (got.double() - want).abs().max() < 1e-4


@pytest.mark.parametrize("plant", ["window_plus", "window_minus", "pairs", "yarn", "factor", "scale", "gate", "mean", "query_norm", "latent_norm", "shared_key", "group_sum", "square", "ungrouped"])
def test_the_restatement_notices_planted_mistakes(plant, monkeypatch):
    """A mistake planted in the plain restatement shows far above the tolerances of these tests."""
    cfg = json.loads(json.dumps(U.CONFIGS["mixed"]))
    W = {k: v.double() for k, v in U.weights(cfg).items()}
    toks = U.tokens(70, 11)
    good = O.forward(cfg, W, toks)[0]
    rot = [L["mixer"] for L in cfg["layers"] if "rot" in L["mixer"]]
    if plant.startswith("window"):
        monkeypatch.setattr(O, "visible", lambda i, w, d=1 if plant == "window_plus" else -1: max(0, i - w + 1 - d) if w else 0)
    elif plant == "pairs":
        def halves(x, r):
            n = r["dims"]
            idx = [i // 2 if i % 2 == 0 else n // 2 + i // 2 for i in range(n)]
            return turn(x[..., idx], r)[..., [idx.index(i) for i in range(n)]]

        turn = O.rotate
        monkeypatch.setattr(O, "rotate", halves)
    elif plant == "yarn":
        for m in rot:
            del m["rot"]["scaling"]
    elif plant == "factor":
        monkeypatch.setattr(O, "frequencies", lambda r, f=O.frequencies: (f(r)[0], 1.0))
    elif plant == "scale":
        for m in rot:
            m["scale"] *= O.frequencies(m["rot"])[1] ** 2
    elif plant == "gate":
        for k in [k for k in W if k.endswith("mix.g")]:
            W[k] = W[k] * 0
    elif plant == "mean":
        monkeypatch.setattr(O, "layer_norm", lambda x, w, eps: O.rms(x, w, eps))
    elif plant in ("query_norm", "latent_norm"):
        for k in [k for k in W if k.endswith("dq.norm" if plant == "query_norm" else "dkv.norm")]:
            W[k] = torch.ones_like(W[k])
    elif plant == "shared_key":  # normed together with the latent
        def keys(h, W, p, m, eps, r):
            W = dict(W)
            if r:
                z = h @ W[p + "dkv"].T
                W[p + "dkv"] = torch.cat((W[p + "dkv"][: m["kv_rank"]], W[p + "dkv"][m["kv_rank"] :] / (z * z).mean().sqrt()))
            return plain(h, W, p, m, eps, r)

        plain = O.latent_keys_values
        monkeypatch.setattr(O, "latent_keys_values", keys)
    elif plant == "square":
        monkeypatch.setattr(O, "experts", lambda h, W, p, ids, wts: torch.stack([sum(w * (W[f"{p}e{e}.down"] @ torch.clamp(W[f"{p}e{e}.up"] @ h[t], min=0)) for e, w in zip(ids[t].tolist(), wts[t])) for t in range(len(h))]))
    elif plant == "ungrouped":
        for L in cfg["layers"]:
            if L["mlp"]:
                L["mlp"]["router"]["groups"] = dict(count=1, keep=1)
    else:
        def other(z, r):
            ids, w = R.router_topk(z, r["top"], "softmax", None, r["groups"]["count"], r["groups"]["keep"], group_top=2)
            return ids.long(), w.double()

        monkeypatch.setattr(O, "route", other)
    bad = O.forward(cfg, W, toks)[0]
    assert U.error(bad, good).max() > 1e-2


# ---- single operations -----------------------------------------------------------------
def paged(lat, table, page, pages, seed=0):
    """Rows [n, w] of one sequence in the pages of ``table``; everything else holds stale values."""
    cache = torch.randn(pages, page * lat.shape[1], generator=torch.Generator().manual_seed(seed)) * 50
    at = torch.arange(lat.shape[0])
    cache.view(-1, lat.shape[1])[torch.tensor(table)[at // page] * page + at % page] = lat
    return cache


def one_sequence(n, q, table, page):
    return R.AttnMeta(q_indptr=torch.tensor([0, q]), kv_lens=torch.tensor([n]), block_table=torch.tensor([table]), slot_mapping=None, positions=torch.arange(n - q, n), page_size=page, num_seqs=1,
                      num_tokens=q, max_q_len=q, max_kv_len=n, h_q_indptr=[0, q], h_kv_lens=[n])


@pytest.mark.parametrize("window", [0, 1, 15, 16, 17, 33])
def test_a_key_that_stands_out(window):
    """Every visible key scores 0 but one, which takes all the weight: exactly the rows whose window holds it answer its
    value, and the others the mean of what they see."""
    heads, c, dim, vdim, n, page, table = 2, 6, 5, 7, 70, 16, [5, 2, 4, 1, 3]
    g = torch.Generator().manual_seed(1)
    uk_t = torch.zeros(heads, c, dim)
    uk_t[:, 0, 0] = 1.0
    uv = torch.randn(heads, vdim, c, generator=g)
    uv[:, :, 0] = 0
    q = torch.zeros(n, heads * dim)
    q[:, 0::dim] = 1.0
    for j in (0, 1, 15, 16, 31, 32, 47, 48, 69):
        lat = torch.randn(n, c, generator=g)
        lat[:, 0] = 0
        lat[j, 0] = 80.0
        out = R.latent_attention(q, uk_t, uv, None, paged(lat, table, page, 6), one_sequence(n, n, table, page), 0, 1.0, window).view(n, heads, vdim)
        v = torch.einsum("tc,hvc->thv", lat, uv)
        for i in range(n):
            lo = O.visible(i, window)
            want = v[j] if lo <= j <= i else v[lo : i + 1].mean(0)
            assert torch.allclose(out[i], want, atol=1e-4), (window, j, i)


def test_rotation_tables():
    for base, n, s in ((300.0, 16, (4.0, 64, 8.0, 1.0)), (1e4, 64, (32.0, 4096, 32.0, 1.0)), (50.0, 2, (8.0, 100, 2.0, 0.5)), (900.0, 24, (1.0, 40, 5.0, 0.5)), (2.0, 8, (3.0, 1 << 20, 4.0, 2.0)), (77.0, 6, None)):
        rot = dict(dims=n, base=base)
        if s:
            rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), s))
        f, gain = O.frequencies(rot)
        cos, sin = R.pair_rope_tables(3000, n, base, "cpu", s or ())
        a = torch.outer(torch.arange(3000, dtype=torch.float64), torch.tensor(f, dtype=torch.float64))
        assert cos.dtype == torch.float32 and (cos.double() - gain * a.cos()).abs().max() < 1e-6 and (sin.double() - gain * a.sin()).abs().max() < 1e-6


@pytest.mark.parametrize("experts,top,groups,keep", [(12, 3, 3, 2), (8, 2, 8, 3), (5, 5, 1, 1), (16, 4, 4, 1), (1, 1, 1, 1)])
def test_router(experts, top, groups, keep):
    z = torch.randn(60, experts, generator=torch.Generator().manual_seed(5)) * 2
    ids, w = R.router_topk(z, top, "softmax", None, groups, keep, group_top=1)
    want_ids, want_w = O.route(z.double(), dict(experts=experts, top=top, groups=dict(count=groups, keep=keep)))
    assert torch.equal(ids.long(), want_ids) and torch.allclose(w.double(), want_w, atol=1e-6)


def test_norms_and_experts():
    g = torch.Generator().manual_seed(3)
    x, y, w = torch.randn(6, 40, generator=g), torch.randn(6, 40, generator=g) * 0.01 + 3, torch.randn(40, generator=g)
    xs = x.clone()
    h = R.add_layer_norm(y, xs, w, 1e-5, torch.bfloat16)
    want = x.double() + O.layer_norm(y.double(), w.double(), 1e-5)
    assert torch.allclose(xs.double(), want, atol=1e-4) and torch.equal(h, xs.bfloat16())
    assert torch.allclose(R.stream_layer_norm(x, w, 1e-3, torch.float32).double(), O.layer_norm(x.double(), w.double(), 1e-3), atol=1e-5)
    up, down, ids, wts = torch.randn(5, 24, 40, generator=g), torch.randn(5, 40, 24, generator=g), torch.tensor([[0, 3], [4, 1], [2, 0], [3, 1], [1, 2], [4, 0]], dtype=torch.int32), torch.rand(6, 2, generator=g)
    want = O.experts(x.double(), {**{f"e{e}.up": up[e].double() for e in range(5)}, **{f"e{e}.down": down[e].double() for e in range(5)}}, "", ids, wts.double())
    rows, pos = R.expert_rows(x, ids, up, down)
    got = (rows[pos.long()].view(6, 2, 40) * wts[:, :, None]).sum(1)
    assert torch.allclose(got.double(), want, rtol=1e-4, atol=1e-3)
    assert torch.allclose(R.moe_experts(x, ids, wts, up, down, act="relu2").double(), want, rtol=1e-4, atol=1e-3)
    xs = x.clone()
    R.add_layer_norm_rows(rows, pos, wts, xs, w, 1e-5, torch.float32)
    assert torch.allclose(xs.double(), x.double() + O.layer_norm(want, w.double(), 1e-5), atol=1e-4)


# ---- engine ------------------------------------------------------------------------------
def _engine(cfg, W, **kw):
    mcfg = from_hf(cfg)
    mcfg.max_position = 512
    return build_engine(EngineConfig(num_kv_blocks=40, **kw), mcfg, device="cpu", dtype=torch.float32, model=registry.build(mcfg, source=DictSource(W), device="cpu", dtype=torch.float32))


def _generate(eng, prompts, n=10):
    try:
        return [toks for toks, term, _ in eng.generate(prompts, max_tokens=n) if term.kind == "finished"]
    finally:
        eng.shutdown()


def test_greedy_generation_through_the_scheduler():
    cfg = U.CONFIGS["mixed"]
    W = U.weights(cfg)
    prompts = [U.tokens(n, 60 + n) for n in (5, 40, 1, 23)]
    together = _generate(_engine(cfg, W, max_prefill_tokens=16, max_decode_batch=3), prompts)
    assert [len(t) for t in together] == [10] * 4
    assert together == [_generate(_engine(cfg, W, max_prefill_tokens=512), [p])[0] for p in prompts]
    for p, toks in zip(prompts, together):
        assert U.truth(cfg, W, p + toks[:-1])[len(p) - 1 :].argmax(-1).tolist() == toks


def test_shared_prefixes_give_the_same_tokens():
    """Everything a request owns is in its pages, so a prompt that begins like an earlier one starts behind the shared pages."""
    cfg = U.CONFIGS["mixed"]
    W = U.weights(cfg)
    head = U.tokens(48, 70)
    prompts = [head + U.tokens(9, 71), head + U.tokens(20, 72), head[:40] + U.tokens(3, 73)]
    eng = _engine(cfg, W)
    try:
        outs = [eng.generate([p], max_tokens=8)[0][0] for p in prompts]
        assert eng.pool.stats.prefix_hits >= 5  # three whole pages of the second prompt, two of the third
    finally:
        eng.shutdown()
    assert outs == [_generate(_engine(cfg, W, no_prefix_cache=True), [p], 8)[0] for p in prompts]


def test_cache_geometry_follows_the_layers():
    cfg = U.CONFIGS["mixed"]
    m = VekalornModel(from_hf(cfg), device="cpu", dtype=torch.float32, source=DictSource(U.weights(cfg)))
    assert m.kv_geometries == [(1, 56, 0), (1, 40, 0), (1, 64, 0), (1, 72, 0)] and m.supports_prefix_cache
    assert MixedKvBuffer.bytes_per_block(m.kv_geometries, 16, torch.float32) == 16 * 232 * 4 == m.kv_geometry()["bytes_per_block"](16)
    with pytest.raises(ValueError):
        build_engine(EngineConfig(num_kv_blocks=8, kv_offload=True), from_hf(cfg), device="cpu", dtype=torch.float32, model=m)


def test_config_reader():
    from pegainfer_b200.loader.export import to_hf_config

    for raw in U.CONFIGS.values():
        cfg = from_hf(raw)
        assert cfg.family == "vekalorn" and cfg.num_layers == len(raw["layers"]) and cfg.rms_eps == raw["norm"]["eps"]
        assert from_hf(to_hf_config(cfg)) == cfg
        for spec, L in zip(cfg.layer_specs, raw["layers"]):
            assert spec.mixer.window == L["mixer"].get("mask", {}).get("size", 0) and spec.mixer.rot_dims == L["mixer"].get("rot_dim", 0) and (spec.moe is None) == (L["mlp"] is None)
    for path, value in ((("layers", 0, "type"), "other"), (("layers", 0, "mixer", "mask", "size"), 0), (("layers", 1, "mixer", "rot", "dims"), 4), (("layers", 0, "mlp", "kind"), "dense"),
                        (("layers", 0, "mlp", "router", "groups", "count"), 5), (("layers", 0, "mlp", "router", "top"), 9)):
        bad = json.loads(json.dumps(U.CONFIGS["mixed"]))
        at = bad
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(ValueError):
            from_hf(bad)


def test_presets_and_weight_shapes():
    for name in ("tiny-vekalorn", "small-vekalorn", "vekalorn-16b-shape"):
        cfg = preset(name)
        shapes = registry.shapes_for(cfg)
        assert cfg.num_layers == len(cfg.layer_specs) and shapes["head"] == (cfg.vocab_size, cfg.hidden_size) and "l0.mix.g" in shapes and "l1.mix.g" not in shapes
    for raw in U.CONFIGS.values():
        assert vekalorn_shapes(from_hf(raw)) == {k: tuple(v.shape) for k, v in U.weights(raw).items()}


def test_checkpoint_round_trip_and_serve_flags(tmp_path):
    from pegainfer_b200.loader.export import export_checkpoint
    from pegainfer_b200.serve import resolve

    cfg = preset("tiny-vekalorn")
    export_checkpoint(cfg, str(tmp_path / "m"), seed=3)
    assert load_model_config(str(tmp_path / "m")).layer_specs == cfg.layer_specs
    ecfg, mcfg, line, _ = resolve(["--model-path", str(tmp_path / "m"), "--dtype", "float32"])
    assert line.name == "vekalorn" and ecfg.dtype == "float32"
    with pytest.raises(SystemExit):
        resolve(["--preset", "tiny-vekalorn", "--state-slots", "4"])
    outs = []
    for e, m in ((EngineConfig(model_path=str(tmp_path / "m"), num_kv_blocks=32), None), (EngineConfig(preset="tiny-vekalorn", num_kv_blocks=32, seed=3), cfg)):
        outs.append(_generate(build_engine(e, m, device="cpu", dtype=torch.float32), [[5, 9, 11, 200]], 6)[0])
    assert outs[0] == outs[1] and len(outs[0]) == 6


def test_trace_program(tmp_path, capsys, monkeypatch):
    """The replay program on CPU, on a line without state slots: entries in their own order, places wanted, pages used again."""
    import io

    from pegainfer_b200 import replay

    cfg = U.CONFIGS["mixed"]
    W = U.weights(cfg)
    U.checkpoint(tmp_path / "m", cfg, W)
    p, q = U.tokens(60, 21), U.tokens(40, 22)
    steps = [dict(step=0, entries=[dict(id="x", tokens=p[:1], want=[]), dict(id="y", tokens=q[:17], want=[0, 16])], end=[]),
             dict(step=1, entries=[dict(id="x", tokens=p[1:59], want=[50, 3])], end=[]),
             dict(step=2, entries=[dict(id="y", tokens=q[17:18], want=[0]), dict(id="x", tokens=p[59:], want=[0])], end=["x"]),
             dict(step=3, entries=[dict(id="z", tokens=p[:57], want=[56]), dict(id="y", tokens=q[18:], want=[21])], end=["y", "z"])]
    monkeypatch.setattr("sys.stdin", io.StringIO("".join(json.dumps(s) + "\n" for s in steps)))
    assert replay.main(["--model", str(tmp_path / "m"), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "128", "--device", "cpu"]) == 0
    assert [l for l in capsys.readouterr().out.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    tx, ty = U.truth(cfg, W, p), U.truth(cfg, W, q)
    for i, w in enumerate([torch.stack([ty[0], ty[16]]), torch.stack([tx[51], tx[4]]), torch.stack([ty[17], tx[59]]), torch.stack([tx[56], ty[39]])]):
        got = torch.frombuffer(bytearray((tmp_path / f"{i}.f32").read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])
        assert got.shape == w.shape and (got.double() - w).abs().max() < 1e-4
