"""Zeripel line on CPU: the operations and whole models of the CPU path against the plain restatement, steps cut in
different ways, generation, configuration, checkpoint and command line."""
import io
import json

import pytest
import torch

import zeripel_oracle as O
import zeripel_util as U
from pegainfer_b200.config import EngineConfig, from_hf, load_model_config, preset
from pegainfer_b200.engine.build import build_engine
from pegainfer_b200.kv.buffer import MixedKvBuffer
from pegainfer_b200.kv.request_kv import KvView
from pegainfer_b200.loader.sources import DictSource
from pegainfer_b200.models import registry
from pegainfer_b200.models.zeripel import ZeripelModel, zeripel_shapes
from pegainfer_b200.ops import reference as R
from pegainfer_b200.sched.executor import SeqStep, build_meta
from test_vekalorn_cpu import one_sequence, paged

PROMPTS = {"a": U.tokens(80, 1), "b": U.tokens(37, 2), "c": U.tokens(1, 3), "d": U.tokens(50, 4)}
SCHEDULES = {
    "whole": [[(r, len(p))] for r, p in PROMPTS.items()],
    "tokens": [[("b", 1)]] * 37,
    "portions": [[("a", n)] for n in (2, 3, 14, 45, 1, 15)] + [[("d", 2)]] * 25,
    "batched": [[("a", 33), ("b", 1), ("d", 2), ("c", 1)], [("b", 1), ("a", 2), ("d", 40)], [("a", 1), ("b", 1), ("d", 1)], [("b", 33), ("a", 44)], [("d", 6), ("b", 1)], [("d", 1), ("c#1", 1), ("b#1", 3)],
                [("b#1", 33), ("a#1", 80)], [("b#1", 1)]],
}
i32 = lambda x: torch.tensor(x, dtype=torch.int32)


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
    seqs = [SeqStep(rid=0, input_tokens=toks, start_pos=0, view=KvView([3, 1], 20, 16))]
    ids, meta = build_meta(seqs, 16, "cpu")
    rep.ex.prepare_meta(seqs, meta)
    rep.ex.model.forward_hidden(ids, meta, rep.ex.kv, aux_layers=range(5))
    stream = O.forward(cfg, {k: v.double() for k, v in W.items()}, toks)[1]
    assert len(rep.ex.model.last_aux) == 5
    for got, want in zip(rep.ex.model.last_aux, stream):
        assert (got.double() - want).abs().max() < 1e-4


def _plant(plant, cfg, W, monkeypatch):
    each = lambda end, f: W.update({k: f(W[k]) for k in list(W) if k.endswith(end)})
    mixers = [L["mixer"] for L in cfg["layers"]]
    if plant == "pair_order":
        b = cfg["embedding"]["bigram"]
        b["mul_prev"], b["mul_cur"] = b["mul_cur"], b["mul_prev"]
    elif plant == "first_pair":
        W["bigram"] = torch.cat((W["bigram"][:-1], W["bigram"][:1]))
    elif plant == "embedding_scale":
        cfg["embedding"]["scale"] *= 1.1
    elif plant == "residual":
        cfg["residual_mult"] = 1.0
    elif plant == "shift":
        monkeypatch.setattr(O, "shift", lambda h: h)
    elif plant == "shift_start":
        monkeypatch.setattr(O, "shift", lambda h: torch.cat((h[:1], h[:-1])))
    elif plant == "decay_bias":
        each(".w0", lambda x: x * 0 - 2)
    elif plant == "decay_tanh":
        monkeypatch.setattr(O, "decay", lambda mix, W, p: torch.exp(-torch.exp(mix @ W[p + "w1"].T @ W[p + "w2"].T + W[p + "w0"])))
    elif plant == "bonus":
        each(".u", lambda x: torch.ones_like(x))
    elif plant == "read_after_write":
        def after(r, k, v, w, u):
            T, H, d = r.shape
            out = torch.zeros(T, H, v.shape[2], dtype=r.dtype)
            for h in range(H):
                S = torch.zeros(d, v.shape[2], dtype=r.dtype)
                for t in range(T):
                    S = w[t, h][:, None] * S + k[t, h][:, None] * v[t, h][None]
                    out[t, h] = S.T @ r[t, h]
            return out

        monkeypatch.setattr(O, "recurrence", after)
    elif plant == "gate":
        monkeypatch.setattr(O, "silu", O.sigmoid)
    elif plant == "sharing":
        monkeypatch.setattr(O, "latent", lambda h, W, p, m, eps, f=O.latent: tuple(x.flip(-1) for x in f(h, W, p, m, eps)))
    elif plant == "normed_values":
        def mixer(h, W, p, m, eps, shared):
            T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
            q = O.rms((h @ W[p + "q"].T).view(T, H, d), eps) * W[p + "q.norm"] * O.temperature(T, m["q_temp"])[:, None, None]
            k = O.rms((h @ W[p + "k"].T).view(T, G, d), eps) * W[p + "k.norm"]
            return torch.cat([O.softmax_rows(q[:, i] @ k[:, i // (H // G)].T * m["scale"]) @ k[:, i // (H // G)] for i in range(H)], 1) @ W[p + "o"].T

        monkeypatch.setitem(O.MIXERS, "attention", mixer)
    elif plant == "temperature":
        monkeypatch.setattr(O, "temperature", lambda T, q: torch.ones(T, dtype=torch.float64))
    elif plant == "temperature_step":
        monkeypatch.setattr(O, "temperature", lambda T, q, f=O.temperature: torch.cat((torch.ones(1, dtype=torch.float64), f(T - 1, q))))
    elif plant == "sink":
        each(".sink", lambda x: x - 30)
    elif plant == "sink_scaled":
        for i, m in enumerate(mixers):
            if "rot" in m:
                W[f"l{i}.mix.sink"] = W[f"l{i}.mix.sink"] * m["scale"]
    elif plant == "pairs":
        def halves(x, r):
            n = r["dims"]
            idx = [i // 2 if i % 2 == 0 else n // 2 + i // 2 for i in range(n)]
            return turn(x[..., idx], r)[..., [idx.index(i) for i in range(n)]]

        turn = O.rotate
        monkeypatch.setattr(O, "rotate", halves)
    elif plant == "own_cache":  # a layer that shares a cache takes the latent of its own input
        W["l3.mix.dkv"], W["l3.mix.dkv.norm"] = W["l1.mix.dkv"], W["l1.mix.dkv.norm"]
        del mixers[3]["kv_from"]
    elif plant == "head_gate":
        each("mix.g", lambda x: x if x.shape[0] > 5 else x * 0)
    elif plant == "activation":
        monkeypatch.setattr(O, "gelu", O.silu)
    elif plant == "correction":
        each(".correction", lambda x: x * 0)
    elif plant == "corrected_weights":
        def route(z, c, r):
            ids, _ = plain(z, c, r)
            s = (O.sigmoid(z) + c).gather(1, ids)
            return ids, s / s.sum(1, keepdim=True) * r["scale"]

        plain = O.route
        monkeypatch.setattr(O, "route", route)
    elif plant == "route_scale":
        for L in cfg["layers"]:
            if L["mlp"] and L["mlp"]["kind"] == "moe":
                L["mlp"]["router"]["scale"] = 1.0
    else:
        assert plant == "shared_gate"
        each(".sg", lambda x: x * 0)


PLANTS = ["pair_order", "first_pair", "embedding_scale", "residual", "shift", "shift_start", "decay_bias", "decay_tanh", "bonus", "read_after_write", "gate", "sharing", "normed_values", "temperature",
          "temperature_step", "sink", "sink_scaled", "pairs", "own_cache", "head_gate", "activation", "correction", "corrected_weights", "route_scale", "shared_gate"]


@pytest.mark.parametrize("plant", PLANTS)
def test_the_restatement_notices_planted_mistakes(plant, monkeypatch):
    """A mistake planted in the plain restatement shows far above the tolerances of these tests."""
    cfg = json.loads(json.dumps(U.CONFIGS["mixed"]))
    W = {k: v.double() for k, v in U.weights(cfg).items()}
    toks = U.tokens(40, 11)
    good = O.forward(cfg, W, toks)[0]
    _plant(plant, cfg, W, monkeypatch)
    assert U.error(O.forward(cfg, W, toks)[0], good).max() > 1e-2


# ---- single operations -----------------------------------------------------------------
def _steps(lens, slots, start=0):
    """Ragged step of sequences of these lengths in these state slots."""
    ind = [0]
    for n in lens:
        ind.append(ind[-1] + n)
    return R.AttnMeta(q_indptr=i32(ind), kv_lens=i32(lens), block_table=None, slot_mapping=None, positions=None, page_size=16, num_seqs=len(lens), num_tokens=ind[-1], max_q_len=max(lens),
                      max_kv_len=max(lens), h_q_indptr=ind, h_kv_lens=list(lens), state_slots=i32(slots), h_state_slots=list(slots))


def test_pair_embedding_carries_the_last_token():
    g = torch.Generator().manual_seed(0)
    e = dict(scale=3.0, bigram=dict(buckets=7, mul_prev=5, mul_cur=3))
    W = {"embed": torch.randn(20, 10, generator=g), "bigram": torch.randn(8, 10, generator=g)}
    w = torch.randn(10, generator=g)
    a, b = [3, 0, 0, 19, 4, 3], [0, 1, 1]
    carried = torch.zeros(4, dtype=torch.int32)
    xs = {"a": [], "b": []}
    for parts in ([("a", a[:1]), ("b", b[:2])], [("a", a[1:4])], [("b", b[2:]), ("a", a[4:5])], [("a", a[5:])]):
        meta = _steps([len(p) for _, p in parts], [1 if n == "a" else 3 for n, _ in parts])
        x, h = R.embed_pairs_norm(i32(sum((p for _, p in parts), [])), W["embed"], W["bigram"], 3.0, (7, 5, 3), carried, w, 1e-3, meta, torch.float32)
        assert torch.allclose(h, O.rms(x, 1e-3) * w, atol=1e-5)
        for (n, p), rows in zip(parts, x.split([len(p) for _, p in parts])):
            xs[n].append(rows)
    assert torch.allclose(torch.cat(xs["a"]), O.embed(a, W, e), atol=1e-6) and torch.allclose(torch.cat(xs["b"]), O.embed(b, W, e), atol=1e-6)
    assert carried.tolist() == [0, 4, 0, 2]


def test_token_mixes_and_recurrence_carry_their_state():
    g = torch.Generator().manual_seed(1)
    n, H, d, dv, w = 23, 3, 6, 5, 12
    h, mu = torch.randn(n, w, generator=g), torch.rand(5, w, generator=g)
    r, k, v = (torch.randn(n, H, x, generator=g) for x in (d, d, dv))
    f, w0, u = torch.randn(n, H * d, generator=g), torch.linspace(-6, 2, H * d), torch.randn(H, d, generator=g)
    carried, state = torch.full((3, w, 1), 7.0), torch.full((3, H, d, dv), 7.0)
    carried[2], state[2] = 0, 0
    mixes, outs, at = [], [], 0
    for m in (1, 2, 13, 1, 6):
        meta = _steps([m], [2])
        mixes.append(R.token_mix(h[at : at + m], mu, carried, meta))
        outs.append(R.wkv_attention(r[at : at + m], k[at : at + m], v[at : at + m], f[at : at + m], w0, u, state, meta))
        at += m
    back = O.shift(h)
    for i in range(5):
        assert torch.allclose(torch.cat(mixes)[:, i], h + (back - h) * mu[i], atol=1e-6)
    dec = torch.exp(-torch.exp(f.double() + w0)).view(n, H, d)
    want = O.recurrence(r.double(), k.double(), v.double(), dec, u.double())
    assert (torch.cat(outs).double() - want).abs().max() < 1e-4
    assert carried[1].eq(7).all() and state[1].eq(7).all() and torch.equal(carried[2, :, 0], h[-1])


def test_residual_norms_and_gated_norm():
    g = torch.Generator().manual_seed(2)
    rnd = lambda *s: torch.randn(*s, generator=g)
    x, y, w = rnd(6, 40), rnd(6, 40), rnd(40)
    xs = x.clone()
    h = R.residual_norm(y, xs, w, 1e-3, 0.7, torch.bfloat16)
    assert torch.allclose(xs, x + 0.7 * y, atol=1e-6) and torch.equal(h, (O.rms(xs, 1e-3) * w).bfloat16())
    rows, pos, wts, shared, sg = rnd(12, 40), torch.randperm(12, generator=g).int(), torch.rand(6, 2, generator=g), rnd(6, 40), rnd(6, 1)
    want = x + 0.7 * ((rows[pos.long()].view(6, 2, 40) * wts[:, :, None]).sum(1) + shared * O.sigmoid(sg))
    xs = x.clone()
    h = R.residual_norm_rows(rows, pos, wts, shared, sg, xs, w, 1e-3, 0.7, torch.float32)
    assert torch.allclose(xs, want, atol=1e-5) and torch.allclose(h, O.rms(want, 1e-3) * w, atol=1e-5)
    o, gate, wh = rnd(4, 3, 8), rnd(4, 24), rnd(24)
    want = O.rms(o, 1e-5).reshape(4, 24) * wh * O.silu(gate)
    assert torch.allclose(R.gated_row_norm(o, gate, wh, 1e-5, "silu").view(4, 24), want, atol=1e-5)
    assert torch.allclose(R.gated_row_norm(o, gate, wh[:8], 1e-5).view(4, 24), O.rms(o, 1e-5).reshape(4, 24) * wh[:8].repeat(3) * O.sigmoid(gate), atol=1e-5)


def test_feed_forwards():
    g = torch.Generator().manual_seed(3)
    rnd = lambda *s: torch.randn(*s, generator=g)
    x, gate, up = rnd(5, 16), rnd(24, 16), rnd(24, 16)
    for act, f in (("silu", O.silu), ("gelu_tanh", O.gelu)):
        want = f(x @ gate.T) * (x @ up.T)
        assert torch.allclose(R.dense_glu(x, torch.cat((gate, up)), False, act), want, atol=1e-4)
        assert torch.allclose(R.dense_glu(x, torch.stack((gate, up), 1).reshape(48, 16), True, act), want, atol=1e-4)
    w1, w2 = rnd(4, 2 * 8, 16), rnd(4, 16, 8)  # rows alternate gate, up
    ids = i32([[0, 3], [1, 0], [3, 2], [2, 1], [0, 1]])
    rows, pos = R.expert_rows(x, ids, w1, w2, "swiglu")
    for t in range(5):
        for j in range(2):
            e = int(ids[t, j])
            want = O.glu(x[t], {"gate": w1[e, 0::2], "up": w1[e, 1::2], "down": w2[e]}, "", O.silu)
            assert torch.allclose(rows[pos[t * 2 + j]], want, atol=1e-3)
    for experts, top, scale in ((12, 3, 1.5), (5, 5, 1.0), (1, 1, 2.5)):
        z, c = rnd(40, experts) * 2, rnd(experts) * 0.5
        ids, w = R.router_topk(z, top, "sigmoid", c, 1, 1, True, scale)
        want_ids, want_w = O.route(z.double(), c.double(), dict(experts=experts, top=top, scale=scale))
        assert torch.equal(ids.long(), want_ids) and torch.allclose(w.double(), want_w, atol=1e-6)


@pytest.mark.parametrize("coef,every", [(0.3, 1), (0.1, 7), (1.0, 64), (0.5, 100000)])
def test_query_temperature(coef, every):
    t = R.temperature_table(500, coef, every)
    assert t.dtype == torch.float32 and (t.double() - O.temperature(500, dict(coef=coef, every=every))).abs().max() < 1e-6


@pytest.mark.parametrize("sink", [-40.0, 0.0, 3.0, 12.0, 200.0])
def test_a_key_that_stands_out_beside_a_sink(sink):
    """Every visible key scores 0 but one; the weight that the keys lose to the sink shows in every row."""
    heads, c, dim, vdim, n, page, table = 2, 6, 5, 7, 70, 16, [5, 2, 4, 1, 3]
    g = torch.Generator().manual_seed(1)
    uk_t, uv = torch.zeros(heads, c, dim), torch.randn(heads, vdim, c, generator=g)
    uk_t[:, 0, 0] = 1.0
    uv[:, :, 0] = 0
    q = torch.zeros(n, heads * dim)
    q[:, 0::dim] = 1.0
    s = torch.tensor([sink, -50.0])
    gate = torch.randn(n, heads, generator=g)
    for j in (0, 1, 15, 16, 47, 48, 69):
        lat = torch.randn(n, c, generator=g)
        lat[:, 0] = 0
        lat[j, 0] = 8.0
        out = R.latent_attention(q, uk_t, uv, None, paged(lat, table, page, 6), one_sequence(n, n, table, page), 0, 1.0, head_gate=gate, sink=s).view(n, heads, vdim)
        for h in range(heads):
            v = lat @ uv[h].T
            for i in range(n):
                e = torch.exp(torch.tensor([8.0 if x == j else 0.0 for x in range(i + 1)], dtype=torch.float64) - max(sink, 8.0))
                den = e.sum() + torch.exp(s[h].double() - max(sink, 8.0))
                assert torch.allclose(out[i, h].double(), (e / den) @ v[: i + 1].double() * O.sigmoid(gate[i, h].double()), atol=1e-4), (j, i, h)


def test_values_are_keys_before_their_norm():
    H, G, d, n, page, table = 4, 2, 6, 40, 16, [2, 3, 1]
    g = torch.Generator().manual_seed(4)
    q, k, qw, kw = torch.randn(n, H * d, generator=g), torch.randn(n, G * d, generator=g) * 3, torch.rand(d, generator=g), torch.rand(d, generator=g)
    meta = one_sequence(n, n, table, page)
    at = torch.arange(n)
    meta.slot_mapping = torch.tensor(table)[at // page] * page + at % page
    cache = torch.full((4, page * G * 2 * d), 9.0)
    temp = R.temperature_table(n, 0.4, 5)
    qn = R.head_norm_append(q, k, k, qw, kw, temp, meta, cache, H, G, d, d, 1e-4)
    out = R.capped_attention(qn, cache, G, d, meta, 0.5)
    qr, v = O.rms(q.view(n, H, d), 1e-4) * qw * temp[:, None, None], k.view(n, G, d)
    kr = O.rms(v, 1e-4) * kw
    want = torch.cat([O.softmax_rows(qr[:, h] @ kr[:, h // 2].T * 0.5) @ v[:, h // 2] for h in range(H)], 1)
    assert torch.allclose(out, want, atol=1e-5)


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
    prompts = [U.tokens(n, 60 + n) for n in (5, 40, 1, 23, 2)]
    together = _generate(_engine(cfg, W, max_prefill_tokens=16, max_decode_batch=3, state_slots=2), prompts)
    assert [len(t) for t in together] == [10] * 5
    for p, toks in zip(prompts, together):
        assert U.truth(cfg, W, p + toks[:-1])[len(p) - 1 :].argmax(-1).tolist() == toks


def test_cache_and_state_geometry_follow_the_layers():
    cfg = U.CONFIGS["mixed"]
    m = ZeripelModel(from_hf(cfg), device="cpu", dtype=torch.float32, source=DictSource(U.weights(cfg)))
    assert m.kv_geometries == [(1, 64, 0), (2, 40, 40)] and not m.supports_prefix_cache and m.layers[1].part.kv_index == m.layers[3].part.kv_index == 0
    assert MixedKvBuffer.bytes_per_block(m.kv_geometries, 16, torch.float32) == 16 * (64 + 160) * 4 == m.kv_geometry()["bytes_per_block"](16)
    st = m.make_state(3)
    assert [tuple(s.shape) for s in st.ssm] == [(4, 3, 24, 24), (4, 2, 40, 40)] and st.token.shape == (4,) and st.conv[0].shape == (4, 72, 1)
    assert m.state_bytes(3) == sum(x.numel() * x.element_size() for x in st.ssm + st.conv + [st.token])
    a = st.slot_for(7, True)
    st.token[a], st.ssm[0][a], st.conv[1][a] = 5, 1.0, 1.0
    st.release(7)
    assert st.slot_for(8, True) == a and int(st.token[a]) == 0 and not st.ssm[0][a].any() and not st.conv[1][a].any()


def test_config_reader():
    from pegainfer_b200.loader.export import to_hf_config

    for raw in U.CONFIGS.values():
        cfg = from_hf(raw)
        assert cfg.family == "zeripel" and cfg.num_layers == len(raw["layers"]) and cfg.rms_eps == raw["norm"]["eps"] and cfg.residual_mult == raw["residual_mult"]
        assert from_hf(to_hf_config(cfg)) == cfg and cfg.bigram == tuple(raw["embedding"]["bigram"][k] for k in ("buckets", "mul_prev", "mul_cur"))
        for spec, L in zip(cfg.layer_specs, raw["layers"]):
            assert (spec.moe is None and not spec.ff) == (L["mlp"] is None) and spec.mixer.kv_from == L["mixer"].get("kv_from", -1) and spec.mixer.sink == (L["type"] == "latent_attention")
    for path, value in ((("layers", 0, "type"), "other"), (("layers", 1, "mixer", "rot", "dims"), 4), (("layers", 0, "mlp", "kind"), "other"), (("layers", 0, "mlp", "router", "top"), 13),
                        (("layers", 2, "mixer", "vdim"), 24), (("layers", 2, "mixer", "kv_heads"), 4), (("layers", 3, "mixer", "kv_from"), 2), (("layers", 3, "mixer", "kv_from"), 3),
                        (("layers", 3, "mixer", "kv_rank"), 64), (("layers", 3, "mixer", "rot", "base"), 10.0), (("layers", 2, "mixer", "q_temp", "every"), 2.5)):
        bad = json.loads(json.dumps(U.CONFIGS["mixed"]))
        at = bad
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(ValueError):
            from_hf(bad)


def test_presets_and_weight_shapes():
    for name in ("tiny-zeripel", "small-zeripel", "zeripel-16b-shape"):
        cfg = preset(name)
        shapes = registry.shapes_for(cfg)
        assert cfg.num_layers == len(cfg.layer_specs) and shapes["head"] == (cfg.vocab_size, cfg.hidden_size) and "l0.mix.dkv" in shapes and "l1.mix.dkv" not in shapes and "l0.mlp.router" not in shapes
    for raw in U.CONFIGS.values():
        want = {k: tuple(v.shape) for k, v in U.weights(raw).items()}
        low = [k for k in want if k.endswith((".w1", ".w2"))]  # their rank is in the tensors only
        got = zeripel_shapes(from_hf(raw))
        assert {k: v for k, v in got.items() if k not in low} == {k: v for k, v in want.items() if k not in low} and set(low) <= set(got)


def test_checkpoint_round_trip_and_serve_flags(tmp_path):
    from pegainfer_b200.loader.export import export_checkpoint
    from pegainfer_b200.serve import resolve

    cfg = preset("tiny-zeripel")
    export_checkpoint(cfg, str(tmp_path / "m"), seed=3)
    got = load_model_config(str(tmp_path / "m"))
    assert got.bigram == cfg.bigram and [l.mixer.kind for l in got.layer_specs] == [l.mixer.kind for l in cfg.layer_specs] and got.layer_specs[1] == cfg.layer_specs[1]
    ecfg, mcfg, line, _ = resolve(["--model-path", str(tmp_path / "m"), "--dtype", "float32", "--state-slots", "4"])
    assert line.name == "zeripel" and ecfg.dtype == "float32" and ecfg.state_slots == 4
    outs = []
    for e, m in ((EngineConfig(model_path=str(tmp_path / "m"), num_kv_blocks=32), None), (EngineConfig(preset="tiny-zeripel", num_kv_blocks=32, seed=3), cfg)):
        outs.append(_generate(build_engine(e, m, device="cpu", dtype=torch.float32), [[5, 9, 11, 200]], 6)[0])
    assert outs[0] == outs[1] and len(outs[0]) == 6


def test_trace_program(tmp_path, capsys, monkeypatch):
    """The replay program on CPU: entries in their own order, places wanted, pages and slots used again."""
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
    assert replay.main(["--model", str(tmp_path / "m"), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "128", "--max-requests", "2", "--device", "cpu"]) == 0
    assert [l for l in capsys.readouterr().out.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    tx, ty = U.truth(cfg, W, p), U.truth(cfg, W, q)
    for i, w in enumerate([torch.stack([ty[0], ty[16]]), torch.stack([tx[51], tx[4]]), torch.stack([ty[17], tx[59]]), torch.stack([tx[56], ty[39]])]):
        got = torch.frombuffer(bytearray((tmp_path / f"{i}.f32").read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])
        assert got.shape == w.shape and (got.double() - w).abs().max() < 1e-4
