"""Nonetar line on CPU: the operations and whole models of the CPU path against the plain restatement, steps cut in different
ways, generation, configuration, checkpoint and command line."""
import io
import json

import pytest
import torch

import nonetar_oracle as O
import nonetar_util as U
from pegainfer_b200.config import EngineConfig, alibi_slopes, from_hf, load_model_config, preset
from pegainfer_b200.engine.build import build_engine
from pegainfer_b200.kv.buffer import MixedKvBuffer
from pegainfer_b200.kv.request_kv import KvView
from pegainfer_b200.loader.sources import DictSource
from pegainfer_b200.models import registry
from pegainfer_b200.models.nonetar import NonetarModel, nonetar_shapes
from pegainfer_b200.ops import reference as R
from pegainfer_b200.sched.executor import SeqStep, build_meta
from test_vekalorn_cpu import one_sequence
from test_zeripel_cpu import _steps

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


def test_copies_after_every_layer():
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


def _plant(plant, cfg, W, mp):
    each = lambda end, f: W.update({k: f(W[k]) for k in list(W) if k.endswith(end)})
    lefts = [L["mixer"]["left"] for L in cfg["layers"] if L["type"] == "parallel"]

    def change_scores(order):
        def scores(q, k, m, temp, slope):
            s, i = q @ k.T * m["scale"], torch.arange(q.shape[0], dtype=q.dtype)
            bias, cap = slope * (i[:, None] - i[None, :]), lambda z: m["softcap"] * torch.tanh(z / m["softcap"])
            return order(s, temp, bias, cap)

        mp.setattr(O, "scores", scores)

    if plant == "plain_norm_weight":
        mp.setattr(O, "norm", lambda x, w, eps: O.unit(x, eps) * w)
    elif plant == "position_pairs":
        mp.setattr(O, "positions", lambda T, w, f=O.positions: f(T, w)[:, [e ^ 1 for e in range(w)]])
    elif plant == "position_start":
        mp.setattr(O, "positions", lambda T, w, f=O.positions: f(T + 1, w)[1:])
    elif plant == "no_positions":
        mp.setattr(O, "positions", lambda T, w: torch.zeros(T, w, dtype=torch.float64))
    elif plant == "no_shift":
        each(".shift", lambda x: x * 0)
    elif plant == "shift_start":
        mp.setattr(O, "shift", lambda h, w: h + (torch.cat((h[:1], h[:-1])) - h) * w)
    elif plant == "shift_of_shifted":
        def shift(h, w):
            out = []
            for row in h:
                out.append(row + ((out[-1] if out else 0 * row) - row) * w)
            return torch.stack(out)

        mp.setattr(O, "shift", shift)
    elif plant == "mix_transposed":
        each(".mix", lambda x: x.T if x.dim() == 2 else x)
    elif plant == "copies_in_place":
        def scatter(streams, y, W, hc):
            new = list(streams)
            for t in range(len(new)):
                new[t] = sum(W[hc + "mix"][s, t] * new[s] for s in range(len(new))) + W[hc + "out"][t] * y
            return torch.stack(new)

        mp.setattr(O, "scatter", scatter)
    elif plant == "plain_sum":
        each(".hc1.in", lambda x: torch.ones_like(x))
    elif plant == "no_temperature":
        each(".temp", lambda x: torch.ones_like(x))
    elif plant == "temperature_after_cap":
        change_scores(lambda s, temp, bias, cap: cap(s) * temp - bias)
    elif plant == "bias_in_cap":
        change_scores(lambda s, temp, bias, cap: cap(s * temp - bias))
    elif plant == "no_cap":
        change_scores(lambda s, temp, bias, cap: s * temp - bias)
    elif plant == "slope_order":
        mp.setattr(O, "slopes", lambda H: [2.0 ** (-8.0 * h / H) for h in range(H)])
    elif plant in ("window_wide", "window_narrow"):
        for a in lefts:
            a["mask"]["size"] += 1 if plant == "window_wide" else -1
    elif plant == "no_bias":
        each(".q.b", lambda x: x * 0)
    elif plant == "value_bias":
        each(".v.b", lambda x: x * 0)
    elif plant == "offset_head_norm":
        each(".q.norm", lambda x: 1 + x)
    elif plant == "scales":
        for L in cfg["layers"]:
            if L["type"] == "parallel":
                L["mixer"]["left_scale"], L["mixer"]["right_scale"] = L["mixer"]["right_scale"], L["mixer"]["left_scale"]
    elif plant == "taps_reversed":
        each(".conv", lambda x: x.flip(1))
    elif plant == "bias_in_front":
        mp.setattr(O, "conv", lambda x, w, b, f=O.conv: f(x, w, b) + torch.stack([w[:, : max(0, w.shape[1] - 1 - t)].sum(1) * 0.3 for t in range(x.shape[0])]))
    elif plant == "gates_swapped":
        for k in [k for k in W if ".ra" in k]:
            W[k], W[k.replace(".ra", ".ri")] = W[k.replace(".ra", ".ri")], W[k]
    elif plant == "gate_blocks_transposed":
        each(".ra", lambda x: x.transpose(1, 2))
    elif plant in ("no_input_scale", "first_token"):
        def lru(u, r, i, lam):
            S, out = torch.zeros_like(u[0]), []
            for t in range(u.shape[0]):
                a = torch.exp(-8 * r[t] * O.softplus(lam))
                S = a * S + (1 if plant == "no_input_scale" or t == 0 else torch.sqrt(1 - a * a)) * i[t] * u[t]
                out.append(S)
            return torch.stack(out)

        mp.setattr(O, "lru", lru)
    elif plant == "gelu":
        mp.setattr(O, "gelu", O.silu)
    elif plant == "norm_in_front_of_gate":
        def mixer(h, W, p, m, eps):
            T, H, dv, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
            z, c, dt = (h @ W[p + "in"].T).split((H * dv, H * dv + 2 * G * N, H), 1)
            x, B, C = O.silu(O.conv(c, W[p + "conv"], W[p + "conv.b"])).split((H * dv, G * N, G * N), 1)
            y = O.ssd(x.reshape(T, H, dv), B.reshape(T, G, N), C.reshape(T, G, N), O.softplus(dt + W[p + "dt_bias"]), W[p + "A_log"], W[p + "D"]).reshape(T, m["norm_groups"], -1)
            return (O.unit(y, eps).reshape(T, -1) * O.silu(z) * W[p + "norm"]) @ W[p + "o"].T

        mp.setitem(O.MIXERS, "mamba2", mixer)
    elif plant == "norm_groups":
        for L in cfg["layers"]:
            if L["type"] == "mamba2":
                L["mixer"]["norm_groups"] = 1
    elif plant in ("head_groups", "keys_and_queries"):
        def ssd(x, B, C, dt, a_log, D, f=O.ssd):
            if plant == "keys_and_queries":
                return f(x, C, B, dt, a_log, D)
            pick = [h % B.shape[1] for h in range(x.shape[1])]
            return f(x, B[:, pick], C[:, pick], dt, a_log, D)

        mp.setattr(O, "ssd", ssd)
    elif plant == "no_skip":
        each(".D", lambda x: x * 0)
    elif plant == "no_step_size":
        mp.setattr(O, "ssd", lambda x, B, C, dt, a_log, D, f=O.ssd: f(x, B / dt.mean(), C, dt, a_log, D))
    elif plant == "dt_bias":
        each(".dt_bias", lambda x: x * 0)
    elif plant == "activation_order":
        each(".act", lambda x: x.flip(0))
    else:
        assert plant == "logit_scale"
        each("head", lambda x: x.roll(1, 0))


PLANTS = ["plain_norm_weight", "position_pairs", "position_start", "no_positions", "no_shift", "shift_start", "shift_of_shifted", "mix_transposed", "copies_in_place", "plain_sum", "no_temperature",
          "temperature_after_cap", "bias_in_cap", "no_cap", "slope_order", "window_wide", "window_narrow", "no_bias", "value_bias", "offset_head_norm", "scales", "taps_reversed", "bias_in_front", "gates_swapped",
          "gate_blocks_transposed", "no_input_scale", "first_token", "gelu", "norm_in_front_of_gate", "norm_groups", "head_groups", "keys_and_queries", "no_skip", "no_step_size", "dt_bias", "activation_order",
          "logit_scale"]


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
@pytest.mark.parametrize("width", [2, 7, 24])
def test_positions_from_coarse_and_fine_tables(width):
    table, n = torch.zeros(3, width), 1500
    tables = R.position_tables(2000, width)
    assert tables[0].shape == (8, (width + 1) // 2, 2) and tables[1].shape == (256, (width + 1) // 2, 2)
    meta = one_sequence(n, n, [1], 16)
    got = R.embed_positions(torch.zeros(n, dtype=torch.int32), table, tables, meta)
    assert got.dtype == torch.float32 and (got.double() - O.positions(n, width)).abs().max() < 4e-7


@pytest.mark.parametrize("s_in,s_out", [(1, 1), (1, 4), (3, 3), (4, 4), (6, 6)])
def test_copies_and_shift_carry_the_last_row(s_in, s_out):
    g = torch.Generator().manual_seed(1)
    rnd = lambda *s: torch.randn(*s, generator=g)
    n, w = 23, 12
    x, y, mix, out, gather, nw, mu = rnd(n, s_in, w), rnd(n, w), rnd(s_in, s_out), rnd(s_out), rnd(s_out), rnd(w), torch.rand(w, generator=g)
    m = R.StreamMix(mix, out, gather)
    W = {"hc.in": gather, "hc.mix": torch.zeros(max(s_in, s_out), s_out), "hc.out": out}
    W["hc.mix"][:s_in] = mix
    copies = torch.cat((x.transpose(0, 1), torch.zeros(max(0, s_out - s_in), n, w)))
    want = O.scatter(copies, y, W, "hc.")[:s_out] if s_in >= s_out else torch.stack([sum(mix[s, t] * x[:, s] for s in range(s_in)) + out[t] * y for t in range(s_out)])
    h = O.unit(O.gather(want, W, "hc."), 1e-3) * nw
    carried = torch.full((3, 1, 1, w), 7.0)
    carried[2] = 0
    at, news, hs = 0, [], []
    for k in (1, 2, 13, 1, 6):
        a, b = R.streams_norm(x[at : at + k], y[at : at + k], m, nw, 1e-3, torch.float32, shift=mu, carried=carried, meta=_steps([k], [2]))
        news.append(a)
        hs.append(b)
        at += k
    assert torch.allclose(torch.cat(news).transpose(0, 1), want, atol=1e-5) and torch.allclose(torch.cat(hs), O.shift(h, mu), atol=1e-4)
    assert carried[1].eq(7).all() and torch.allclose(carried[2, 0, 0], h[-1], atol=1e-5)
    plain = R.streams_norm(x, y, m, nw, 1e-3, torch.bfloat16, keep=False)
    assert plain[0] is None and torch.allclose(plain[1].float(), h, atol=0.02, rtol=0.02)
    same = R.streams_norm(x, None, m, nw, 1e-3, torch.float32)
    assert same[0] is x


def test_recurrences_carry_their_state():
    g = torch.Generator().manual_seed(2)
    rnd = lambda *s: torch.randn(*s, generator=g)
    n, c, b = 29, 12, 3
    u, y, yb, lam = rnd(n, c), rnd(n, c), rnd(c), torch.linspace(-9, 3, c)
    W = {"ra": rnd(b, 4, 4), "ra.b": rnd(b, 4), "ri": rnd(b, 4, 4), "ri.b": rnd(b, 4)}
    mats, bias = torch.cat((W["ra"], W["ri"]), 1), torch.cat((W["ra.b"], W["ri.b"]), 1)
    H, G, N, dv = 6, 2, 5, 3
    x, B, C, dt = rnd(n, H, dv), rnd(n, G, N), rnd(n, G, N), rnd(n, H)
    dtb, al, D = rnd(H), torch.linspace(-4, 2, H), rnd(H)
    state, S = torch.full((3, 1, 1, c), 7.0), torch.full((3, H, N, dv), 7.0)
    state[1], S[1] = 0, 0
    outs, ys, at = [], [], 0
    for k in (1, 2, 13, 1, 12):
        part, meta = slice(at, at + k), _steps([k], [1])
        gates = R.multi_dense(u[part].view(k, b, 4), mats, torch.float32)
        both = torch.zeros(k, c + 5)
        R.gated_lru(gates, bias, u[part], lam, y[part], yb, state, meta, 0.7, both[:, 5:])
        outs.append(both[:, 5:])
        ys.append(R.ssd_attention(x[part], B[part], C[part], dt[part], dtb, al, D, S, meta))
        at += k
    d = lambda z: z.double()
    Wd = {k: d(v) for k, v in W.items()}
    want = O.lru(d(u), O.block_gate(d(u), Wd, "", "ra"), O.block_gate(d(u), Wd, "", "ri"), d(lam))
    assert (torch.cat(outs).double() - want * O.gelu(d(y) + d(yb)) * 0.7).abs().max() < 1e-5
    assert (torch.cat(ys).double() - O.ssd(d(x), d(B), d(C), O.softplus(d(dt) + d(dtb)), d(al), d(D))).abs().max() < 1e-4
    assert state[2].eq(7).all() and S[0].eq(7).all() and (state[1, 0, 0].double() - want[-1]).abs().max() < 1e-5


@pytest.mark.parametrize("taps", [1, 2, 5])
def test_convolution_with_biases(taps):
    g = torch.Generator().manual_seed(3)
    x, w, b, ib = torch.randn(19, 6, generator=g), torch.randn(6, taps, generator=g), torch.randn(6, generator=g), torch.randn(6, generator=g)
    for act, f in (("silu", O.silu), ("none", lambda z: z)):
        state, outs, at = torch.zeros(2, 6, taps - 1), [], 0
        for k in (1, 1, 2, 11, 4):
            outs.append(R.short_conv(x[at : at + k], w, b, state, _steps([k], [1]), act, ib))
            at += k
        assert torch.allclose(torch.cat(outs), f(O.conv(x + ib, w, b)), atol=1e-5)
        if taps > 1:
            assert torch.allclose(state[1], (x + ib)[-(taps - 1) :].T, atol=1e-6)


def test_gate_in_front_of_the_norm_and_xielu():
    g = torch.Generator().manual_seed(4)
    o, gate, w = torch.randn(4, 3, 8, generator=g), torch.randn(4, 24, generator=g), torch.randn(24, generator=g)
    want = O.unit(o * O.silu(gate).view(4, 3, 8), 1e-4).reshape(4, 24) * w
    assert torch.allclose(R.gated_row_norm(o, gate, w, 1e-4, "silu", gate_first=True).view(4, 24), want, atol=1e-5)
    x, up, act = torch.randn(5, 16, generator=g), torch.randn(24, 16, generator=g), torch.tensor([0.4, -1.1])
    c = torch.nn.functional.softplus(act) + torch.tensor([0.0, 0.5])
    assert torch.allclose(R.dense_xielu(x, up, c), O.xielu(x @ up.T, *act), atol=1e-4)


@pytest.mark.parametrize("window", [1, 15, 16, 17, 33, 0])
@pytest.mark.parametrize("slope", [0.0, 0.05])
def test_a_key_that_stands_out(window, slope):
    """Every visible key scores 0 (less the distance bias) but one, which takes most of the weight in exactly the rows whose
    window holds it."""
    H, G, d, dv, n, page, table = 2, 1, 5, 7, 70, 16, [5, 2, 4, 1, 3]
    g = torch.Generator().manual_seed(1)
    v, meta, at = torch.randn(n, G, dv, generator=g), one_sequence(n, n, table, page), torch.arange(n)
    q = torch.zeros(n, H, d)
    q[..., 0] = 1.0
    sl = torch.tensor([slope, 2 * slope])
    for j in (0, 1, 15, 16, 47, 48, 69):
        k = torch.randn(n, G, d, generator=g)
        k[..., 0] = 0
        k[j, :, 0] = 30.0
        cache = torch.randn(6, page * G * (d + dv), generator=g) * 50
        slot = torch.tensor(table)[at // page] * page + at % page
        kp, vp = R._pages_kv(cache, G, d, dv, page)
        kp[slot // page, slot % page], vp[slot // page, slot % page] = k, v
        out = R.capped_attention(q, cache, G, dv, meta, 1.0, 20.0, window=window, slopes=sl, out_scale=0.5).view(n, H, dv)
        for h in range(H):
            s = O.scores(q[:, h].double(), k[:, 0].double(), dict(scale=1.0, softcap=20.0), 1.0, sl[h].item())
            w = O.weights_of(s, window or n)
            assert (out[:, h].double() - 0.5 * w @ v[:, 0].double()).abs().max() < 1e-5
            assert w[n - 1, j] > 0.9 or (window and n - 1 - j >= window)


def test_biases_and_head_factors_in_front_of_the_cache():
    H, G, d, dv, n, page, table = 4, 2, 6, 3, 40, 16, [2, 3, 1]
    g = torch.Generator().manual_seed(4)
    rnd = lambda *s: torch.randn(*s, generator=g)
    q, k, v, qb, kb, vb, qw, kw, temp = rnd(n, H * d), rnd(n, G * d), rnd(n, G * dv), rnd(H * d), rnd(G * d), rnd(G * dv), rnd(d), rnd(d), rnd(H)
    meta, at = one_sequence(n, n, table, page), torch.arange(n)
    meta.slot_mapping = torch.tensor(table)[at // page] * page + at % page
    cache = torch.full((4, page * G * (d + dv)), 9.0)
    got = R.head_norm_append(q, k, v, temp[:, None] * qw, kw, None, meta, cache, H, G, d, dv, 1e-4, bias=(qb, kb, vb))
    assert torch.allclose(got, O.unit((q + qb).view(n, H, d), 1e-4) * qw * temp[:, None], atol=1e-5)
    kp, vp = R._pages_kv(cache, G, d, dv, page)
    slot = meta.slot_mapping
    assert torch.allclose(kp[slot // page, slot % page], O.unit((k + kb).view(n, G, d), 1e-4) * kw, atol=1e-5) and torch.allclose(vp[slot // page, slot % page], (v + vb).view(n, G, dv))


def test_slopes():
    assert alibi_slopes(8) == tuple(2.0 ** -(h + 1) for h in range(8)) and alibi_slopes(1) == (2.0 ** -8,)
    for H in (3, 5, 20):
        assert alibi_slopes(H) == tuple(O.slopes(H)) and len(set(alibi_slopes(H))) == H


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
    m = NonetarModel(from_hf(cfg), device="cpu", dtype=torch.float32, source=DictSource(U.weights(cfg)))
    assert m.kv_geometries == [(2, 24, 40), (3, 16, 8), (1, 32, 24)] and not m.supports_prefix_cache
    assert MixedKvBuffer.bytes_per_block(m.kv_geometries, 16, torch.float32) == 16 * (128 + 72 + 56) * 4 == m.kv_geometry()["bytes_per_block"](16) and m.kv_geometry()["kv_heads"] == 3
    st = m.make_state(3)
    assert [tuple(s.shape[1:]) for s in st.ssm] == [(1, 1, 96), (1, 1, 72), (6, 24, 16), (1, 1, 72), (1, 1, 40), (1, 1, 72), (4, 8, 32), (1, 1, 72), (1, 1, 64), (1, 1, 72)]
    assert [tuple(c.shape[1:]) if c is not None else None for c in st.conv] == [(96, 2), None, (240, 3), None, (40, 1), None, (144, 1), None, (64, 3), None]
    assert m.state_bytes(3) == sum(x.numel() * x.element_size() for x in (*st.ssm, *st.conv) if x is not None)
    a = st.slot_for(7, True)
    for x in (*st.ssm, *st.conv):
        if x is not None:
            x[a] = 1.0
    st.release(7)
    assert st.slot_for(8, True) == a and not any(x[a].any() for x in (*st.ssm, *st.conv) if x is not None)
    rec = NonetarModel(from_hf(U.CONFIGS["recurrent"]), device="cpu", dtype=torch.float32, source=DictSource(U.weights(U.CONFIGS["recurrent"])))
    assert rec.kv_geometries == [] and rec.kv_geometry()["num_layers"] == 1


def test_config_reader():
    from pegainfer_b200.loader.export import to_hf_config

    for raw in U.CONFIGS.values():
        cfg = from_hf(raw)
        assert cfg.family == "nonetar" and cfg.num_layers == len(raw["layers"]) and cfg.rms_eps == raw["norm"]["eps"] and cfg.streams == raw["streams"] and cfg.logit_scale == raw["logit_scale"]
        assert from_hf(to_hf_config(cfg)) == cfg
        for spec, L in zip(cfg.layer_specs, raw["layers"]):
            assert spec.ff == (L["mlp"]["ff"] if L["mlp"] else 0) and spec.mixer.kind == ("parallel" if L["type"] == "parallel" else "ssd")
            if L["type"] == "parallel":
                a, r = spec.mixer.parts
                assert a.window == L["mixer"]["left"]["mask"]["size"] and a.softcap == L["mixer"]["left"]["softcap"] and r.heads * r.dim == L["mixer"]["right"]["width"]
                assert spec.mixer.part_scales == (L["mixer"]["left_scale"], L["mixer"]["right_scale"])
    bare = json.loads(json.dumps(U.CONFIGS["mixed"]))
    del bare["layers"][0]["mixer"]["left"]["mask"], bare["layers"][0]["mixer"]["left"]["softcap"]
    assert from_hf(bare).layer_specs[0].mixer.parts[0].window == 0 and from_hf(to_hf_config(from_hf(bare))) == from_hf(bare)
    for path, value in ((("layers", 0, "type"), "other"), (("layers", 0, "mlp", "kind"), "other"), (("layers", 0, "mixer", "left", "kv_heads"), 3), (("layers", 0, "mixer", "left", "mask", "size"), 0),
                        (("layers", 0, "mixer", "right", "blocks"), 7), (("layers", 1, "mixer", "groups"), 4), (("layers", 1, "mixer", "norm_groups"), 5)):
        bad = json.loads(json.dumps(U.CONFIGS["mixed"]))
        at = bad
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(ValueError):
            from_hf(bad)


def test_presets_and_weight_shapes():
    for name in ("tiny-nonetar", "small-nonetar", "nonetar-8b-shape"):
        cfg = preset(name)
        shapes = registry.shapes_for(cfg)
        assert cfg.num_layers == len(cfg.layer_specs) and shapes["head"] == (cfg.vocab_size, cfg.hidden_size) and "l0.mix.left.q" in shapes and "l2.mix.in" in shapes
    for raw in U.CONFIGS.values():
        assert nonetar_shapes(from_hf(raw)) == {k: tuple(v.shape) for k, v in U.weights(raw).items()}


def test_checkpoint_round_trip_and_serve_flags(tmp_path):
    from pegainfer_b200.loader.export import export_checkpoint
    from pegainfer_b200.serve import resolve

    cfg = preset("tiny-nonetar")
    export_checkpoint(cfg, str(tmp_path / "m"), seed=3)
    got = load_model_config(str(tmp_path / "m"))
    assert got.streams == cfg.streams and got.layer_specs == cfg.layer_specs and got.logit_scale == cfg.logit_scale
    ecfg, mcfg, line, _ = resolve(["--model-path", str(tmp_path / "m"), "--dtype", "float32", "--state-slots", "4"])
    assert line.name == "nonetar" and ecfg.dtype == "float32" and ecfg.state_slots == 4
    outs = []
    for e, m in ((EngineConfig(model_path=str(tmp_path / "m"), num_kv_blocks=32), None), (EngineConfig(preset="tiny-nonetar", num_kv_blocks=32, seed=3), cfg)):
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
