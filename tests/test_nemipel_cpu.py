"""Nemipel line on CPU: the operations and whole models of the CPU path against the plain restatement, steps cut in
different ways, generation, configuration, checkpoint and command line."""
import json
import os
import subprocess
import sys

import pytest
import torch

import nemipel_oracle as O
import nemipel_util as U
from pegainfer_b200.config import EngineConfig, from_hf, load_model_config, preset
from pegainfer_b200.engine.build import build_engine
from pegainfer_b200.kv.buffer import MixedKvBuffer
from pegainfer_b200.kv.state import LayerStates
from pegainfer_b200.loader.sources import DictSource
from pegainfer_b200.models import registry
from pegainfer_b200.models.nemipel import NemipelModel, nemipel_shapes
from pegainfer_b200.ops import reference as R

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
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
    assert rep.pool.used() == 0 and not rep.ex.model.rec.by_rid


def test_stream_after_every_layer():
    cfg = U.CONFIGS["mixed"]
    W = U.weights(cfg)
    rep = U.replayer(cfg, W, "cpu", torch.float32, 64)
    toks = U.tokens(20, 9)
    from pegainfer_b200.kv.request_kv import KvView
    from pegainfer_b200.sched.executor import SeqStep, build_meta

    seqs = [SeqStep(rid=0, input_tokens=toks, start_pos=0, view=KvView([3, 1], 20, 16))]
    ids, meta = build_meta(seqs, 16, "cpu")
    rep.ex.prepare_meta(seqs, meta)
    rep.ex.model.forward_hidden(ids, meta, rep.ex.kv, aux_layers=range(4))
    stream = O.forward(cfg, {k: v.double() for k, v in W.items()}, toks)[1]
    for got, want in zip(rep.ex.model.last_aux, stream):
        assert (got.double() - want).abs().max() < 1e-4


@pytest.mark.parametrize("plant", ["decay", "sharing", "gate", "alpha", "pairs", "cap", "row_norm", "write_after_read"])
def test_the_restatement_notices_planted_mistakes(plant, monkeypatch):
    """A mistake planted in the plain restatement shows far above the tolerances of these tests."""
    cfg = json.loads(json.dumps(U.CONFIGS["mixed"]))
    W = {k: v.double() for k, v in U.weights(cfg).items()}
    toks = U.tokens(70, 11)
    good = O.forward(cfg, W, toks)[0]
    if plant == "decay":
        cfg["layers"][2]["mixer"]["decay"][0] = 0.88
    elif plant == "sharing":
        monkeypatch.setattr(O, "attention_keys", lambda h, W, p, m, eps, f=O.attention_keys: tuple(x.flip(1) for x in f(h, W, p, m, eps)))
    elif plant == "gate":
        W["l0.mix.g"] = torch.zeros_like(W["l0.mix.g"])
    elif plant == "alpha":
        cfg["postln_alpha"] = 1.6
    elif plant == "pairs":
        def halves(x, pos, dims, base):
            idx = [i // 2 if i % 2 == 0 else dims // 2 + i // 2 for i in range(dims)]
            y = x.clone()
            y[..., :dims] = O_rotate(x[..., :dims][..., idx], pos, dims, base)[..., [idx.index(i) for i in range(dims)]]
            return y

        O_rotate = O.rotate
        monkeypatch.setattr(O, "rotate", halves)
    elif plant == "cap":
        cfg["layers"][0]["mixer"]["softcap"] = 9.0
    elif plant == "row_norm":
        monkeypatch.setattr(O, "attention_keys", lambda h, W, p, m, eps, f=O.attention_keys: (lambda k, v: (k * (1 + 0.1 * torch.arange(k.shape[1]).view(1, -1, 1)), v))(*f(h, W, p, m, eps)))
    else:
        def scan(q, k, v, g, beta):
            return torch.cat([torch.zeros_like(v[:1]), O_scan(q[1:], k[:-1], v[:-1], g[:-1], beta[:-1])])

        O_scan = O.channel_delta_scan
        monkeypatch.setattr(O, "channel_delta_scan", scan)
    bad = O.forward(cfg, W, toks)[0]
    assert U.error(bad, good).max() > 1e-2


def test_a_key_that_stands_out():
    heads, kvh, dim, vdim, n, page = 4, 2, 6, 10, 70, 16
    pages = 6
    for j in (0, 15, 16, 47, 48, 69):
        k, v = torch.zeros(n, kvh, dim), torch.randn(n, kvh, vdim, generator=torch.Generator().manual_seed(j))
        k[j, :, 1] = 60.0
        cache = torch.zeros(pages, page * kvh * (dim + vdim))
        kp, vp = R._pages_kv(cache, kvh, dim, vdim, page)
        table = [5, 2, 4, 1, 3]
        for p in range(n):
            kp[table[p // page], p % page], vp[table[p // page], p % page] = k[p], v[p]
        q = torch.zeros(n, heads, dim)
        q[:, :, 1] = 1.0
        meta = R.AttnMeta(q_indptr=torch.tensor([0, n]), kv_lens=torch.tensor([n]), block_table=torch.tensor([table]), slot_mapping=None, positions=None, page_size=page, num_seqs=1, num_tokens=n, max_q_len=n,
                          max_kv_len=n, h_q_indptr=[0, n], h_kv_lens=[n])
        out = R.capped_attention(q, cache, kvh, vdim, meta, 1.0, 50.0).view(n, heads, vdim)
        rep = v.repeat_interleave(2, 1)
        assert torch.allclose(out[j], rep[j], atol=1e-4) and torch.allclose(out[-1], rep[j], atol=1e-4)
        if j:
            assert torch.allclose(out[j - 1], rep[:j].mean(0), atol=1e-4)
        assert torch.allclose(out, O.softcap_attention(q, k, v, 1.0, 50.0), atol=1e-5)


def test_greedy_generation_through_the_scheduler():
    cfg = U.CONFIGS["mixed"]
    W = U.weights(cfg)
    mcfg = from_hf(cfg)
    mcfg.max_position = 512
    prompts = [U.tokens(n, 60 + n) for n in (5, 40, 1, 23)]

    def gen(ps, **kw):
        eng = build_engine(EngineConfig(num_kv_blocks=40, **kw), mcfg, device="cpu", dtype=torch.float32, model=NemipelModel(mcfg, source=DictSource(W), device="cpu", dtype=torch.float32))
        try:
            return [toks for toks, term, _ in eng.generate(ps, max_tokens=10) if term.kind == "finished"]
        finally:
            eng.shutdown()

    together = gen(prompts, max_prefill_tokens=16, max_decode_batch=3, state_slots=2)  # two slots for four requests
    assert [len(t) for t in together] == [10] * 4
    assert together == [gen([p], max_prefill_tokens=512)[0] for p in prompts]
    for p, toks in zip(prompts, together):
        assert U.truth(cfg, W, p + toks[:-1])[len(p) - 1 :].argmax(-1).tolist() == toks


def test_state_slots_are_cleared_and_bounded():
    st = LayerStates(3, [(2, 4, 3, 0, 0), (1, 2, 2, 5, 3), (1, 2, 2, 4, 1)], torch.float32, "cpu")
    a, b = st.slot_for(10, True), st.slot_for(11, True)
    assert sorted((a, b)) == [1, 2] and st.conv[0] is None and st.conv[1].shape == (3, 5, 2) and st.conv[2].shape == (3, 4, 0)
    with pytest.raises(RuntimeError):
        st.slot_for(12, True)
    for t in st.ssm + [st.conv[1]]:
        t.fill_(5.0)
    st.release(10)
    assert st.slot_for(12, False) == a  # a slot that changes hands starts from zero
    assert all((t[a] == 0).all() and (t[b] == 5.0).all() for t in st.ssm + [st.conv[1]])


def test_cache_geometry_follows_the_layers():
    cfg = from_hf(U.CONFIGS["mixed"])
    m = NemipelModel(cfg, device="cpu", dtype=torch.float32, source=DictSource(U.weights(U.CONFIGS["mixed"])))
    assert m.kv_geometries == [(2, 24, 40)] and [L.part.kv_index for L in m.layers if L.mixer.kind == "attention"] == [0, 0]
    assert MixedKvBuffer.bytes_per_block(m.kv_geometries, 16, torch.float32) == 16 * 2 * 64 * 4 == m.kv_geometry()["bytes_per_block"](16)
    assert m.state_bytes(3) == sum(t.numel() * t.element_size() for t in m.make_state(3).ssm) + sum(c.numel() * c.element_size() for c in m.rec.conv if c is not None)
    assert not m.supports_prefix_cache


def test_config_reader():
    for name, raw in U.CONFIGS.items():
        cfg = from_hf(raw)
        assert cfg.family == "nemipel" and cfg.num_layers == len(raw["layers"]) and cfg.postln_alpha == raw["postln_alpha"] and cfg.rms_eps == raw["norm"]["eps"]
        from pegainfer_b200.loader.export import to_hf_config

        assert from_hf(to_hf_config(cfg)) == cfg
        assert cfg.layer_specs[0].ff == (raw["layers"][0]["mlp"] or {"ff": 0})["ff"]
    bad = json.loads(json.dumps(U.CONFIGS["mixed"]))
    bad["layers"][3]["mixer"]["kv_from"] = 1
    with pytest.raises(ValueError):
        from_hf(bad)
    bad["layers"][3] = dict(type="other", mixer=dict(heads=1, dim=8, vdim=8), mlp=None)
    with pytest.raises(ValueError):
        from_hf(bad)


def test_presets_and_weight_shapes():
    for name in ("tiny-nemipel", "small-nemipel", "nemipel-8b-shape"):
        cfg = preset(name)
        kinds = [l.mixer.kind for l in cfg.layer_specs]
        assert set(kinds) == {"attention", "lightning", "channel_delta"} and cfg.num_layers == len(kinds)
        shapes = registry.shapes_for(cfg)
        assert shapes["head"] == (cfg.vocab_size, cfg.hidden_size) and "l4.mix.k" not in shapes and "l4.mix.q" in shapes
    W = U.weights(U.CONFIGS["mixed"])
    cfg = from_hf(U.CONFIGS["mixed"])
    shapes = nemipel_shapes(cfg)
    assert set(shapes) == set(W) and all(tuple(W[k].shape) == s for k, s in shapes.items() if not k.split(".")[-1] in ("a1", "a2", "g1", "g2"))


def test_checkpoint_round_trip_and_serve_flags(tmp_path):
    from pegainfer_b200.loader.export import export_checkpoint
    from pegainfer_b200.serve import resolve

    cfg = preset("tiny-nemipel")
    export_checkpoint(cfg, str(tmp_path / "m"), seed=3)
    back = load_model_config(str(tmp_path / "m"))
    assert [l.mixer.kind for l in back.layer_specs] == [l.mixer.kind for l in cfg.layer_specs]
    ecfg, mcfg, line, _ = resolve(["--model-path", str(tmp_path / "m"), "--dtype", "float32", "--state-slots", "5"])
    assert line.name == "nemipel" and ecfg.dtype == "float32" and ecfg.state_slots == 5
    with pytest.raises(SystemExit):
        resolve(["--preset", "tiny-qwen3", "--dtype", "float32"])
    outs = []
    for e, m in ((EngineConfig(model_path=str(tmp_path / "m"), num_kv_blocks=32), None), (EngineConfig(preset="tiny-nemipel", num_kv_blocks=32, seed=3), cfg)):
        eng = build_engine(e, m, device="cpu", dtype=torch.float32)
        try:
            outs.append(eng.generate([[5, 9, 11, 200]], max_tokens=6)[0][0])
        finally:
            eng.shutdown()
    assert outs[0] == outs[1] and len(outs[0]) == 6


def test_trace_program(tmp_path):
    """The program itself, on CPU: step files, entries in their own order, requests that pause, places wanted."""
    cfg = U.CONFIGS["mixed"]
    W = U.weights(cfg)
    U.checkpoint(tmp_path / "m", cfg, W)
    (tmp_path / "out").mkdir()
    p, q = U.tokens(30, 21), U.tokens(20, 22)
    steps = [dict(step=0, entries=[dict(id="x", tokens=p[:1], want=[]), dict(id="y", tokens=q[:17], want=[0, 16])], end=[]),
             dict(step=1, entries=[dict(id="x", tokens=p[1:29], want=[27, 3])], end=[]),
             dict(step=2, entries=[dict(id="y", tokens=q[17:18], want=[0]), dict(id="x", tokens=p[29:], want=[0])], end=["x"]),
             dict(step=3, entries=[dict(id="y", tokens=q[18:], want=[1])], end=["y"])]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", "float32", "--out", str(tmp_path / "out"), "--max-tokens", "128", "--device", "cpu"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
    tx, ty = U.truth(cfg, W, p), U.truth(cfg, W, q)
    want = [torch.stack([ty[0], ty[16]]), torch.stack([tx[28], tx[4]]), torch.stack([ty[17], tx[29]]), ty[19:20]]
    for i, w in enumerate(want):
        got = torch.frombuffer(bytearray((tmp_path / "out" / f"{i}.f32").read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])
        assert got.shape == w.shape and (got.double() - w).abs().max() < 1e-4


def test_trace_program_refuses_32_bit_on_lines_without_it(tmp_path):
    from pegainfer_b200.loader.export import export_checkpoint

    export_checkpoint(preset("tiny-qwen3"), str(tmp_path / "m"))
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "64"], input="", capture_output=True,
                       text=True, timeout=300)
    assert r.returncode == 3


def test_kernel_units_name_sources():
    for fam, units in registry.KERNEL_UNITS.items():
        assert fam in registry.BUILDERS and all(os.path.exists(os.path.join(ROOT, "csrc", u + ".cu")) for u in units)
