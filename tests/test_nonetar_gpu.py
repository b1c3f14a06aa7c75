"""Nonetar line on a GPU: every kernel against the plain restatement, and whole models through the engine's executor in
bf16 and f32, cut into steps in different ways."""
import pytest
import torch

import nonetar_oracle as O
import nonetar_util as U
from pegainfer_b200.config import alibi_slopes
from pegainfer_b200.ops.reference import StreamMix, position_tables
from test_nemipel_gpu import DEV, K, TOL, TYPES, close, meta_for, rnd

pytestmark = pytest.mark.gpu


# ---- rows --------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("w", [2, 51, 72, 4096])
def test_embedding_with_positions(dtype, w):
    table = rnd(300, w, dtype=dtype).to(DEV)
    pos = [0, 1, 2, 255, 256, 257, 511, 512, 1023, 4000, 65535]
    meta, _ = meta_for([len(pos)], [len(pos)])
    meta.positions = torch.tensor(pos, dtype=torch.int32, device=DEV)
    ids = torch.tensor([(7 * p) % 300 for p in pos], dtype=torch.int32, device=DEV)
    got = K().embed_positions(ids, table, position_tables(65536, w, DEV), meta)
    rate = 10000.0 ** (-(torch.arange(w, dtype=torch.float64) // 2 * 2) / w)
    ang = torch.tensor(pos, dtype=torch.float64)[:, None] * rate
    want = table.double().cpu()[ids.long().cpu()] + torch.where(torch.arange(w) % 2 == 0, ang.sin(), ang.cos())
    assert got.dtype == torch.float32 and (got.double().cpu() - want).abs().max() < 1e-6 and K().read_status(DEV) == 0


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("s_in,s_out,w", [(1, 1, 8), (1, 4, 72), (2, 2, 51), (3, 3, 4096), (4, 4, 8192), (5, 5, 51), (8, 8, 136), (1, 6, 48), (4, 4, 128)])
def test_copies_between_sublayers(dtype, s_in, s_out, w):
    """Ragged sequences in shuffled slots, cut into steps in different ways; long enough for runs of rows per block."""
    lens = {1: 2600 if w < 200 else 40, 2: 3, 3: 70}
    mix, out, gather, nw, mu = rnd(s_in, s_out, seed=1).to(DEV), rnd(s_out, seed=2).to(DEV), rnd(s_out, seed=3).to(DEV), rnd(w, seed=4).to(DEV), torch.rand(w, generator=torch.Generator().manual_seed(5)).to(DEV)
    m = StreamMix(mix, out, gather)
    x, y = {s: rnd(n, s_in, w, seed=10 + s).to(DEV) for s, n in lens.items()}, {s: rnd(n, w, seed=20 + s, dtype=dtype).to(DEV) for s, n in lens.items()}
    new_want = {s: torch.einsum("sn,tsw->tnw", mix.double(), x[s].double()) + out.double()[None, :, None] * y[s].double()[:, None] for s in lens}
    h_want = {s: O.unit(torch.einsum("n,tnw->tw", gather.double(), new_want[s]), 1e-4) * nw.double() for s in lens}
    for moved in (False, True):
        carried = torch.full((5, 1, 1, w), 3.0, device=DEV)
        carried[1:4] = 0
        at, news, hs = {s: 0 for s in lens}, {s: [] for s in lens}, {s: [] for s in lens}
        for step in ([(1, 1), (2, 2)], [(3, 40), (1, lens[1] - 10), (2, 1)], [(1, 1), (3, 1)], [(3, 29), (1, 8)]):
            cut = lambda d: torch.cat([d[s][at[s] : at[s] + n] for s, n in step])
            counts = [n for _, n in step]
            meta, _ = meta_for(counts, counts, slots=[s for s, _ in step])
            wide = torch.zeros(sum(counts), w + 8, dtype=dtype, device=DEV)
            wide[:, :w] = cut(y)
            kw = dict(shift=mu, carried=carried, meta=meta) if moved else {}
            xs = cut(x).contiguous()
            new, h = K().streams_norm(xs, wide[:, :w], m, nw, 1e-4, dtype, **kw)
            assert torch.equal(xs, cut(x))
            none, again = K().streams_norm(xs, wide[:, :w], m, nw, 1e-4, dtype, keep=False)
            assert none is None and (moved or torch.equal(again, h))
            for (s, n), a, b in zip(step, new.split(counts), h.split(counts)):
                news[s].append(a)
                hs[s].append(b)
                at[s] += n
        for s in lens:
            close(torch.cat(news[s]), new_want[s], 1e-5)
            close(torch.cat(hs[s]), O.shift(h_want[s], mu.double()) if moved else h_want[s], TOL[dtype])
            if moved:
                close(carried[s, 0, 0], h_want[s][-1], 1e-4)
        assert carried[0].eq(3).all() and carried[4].eq(3).all()
    first = StreamMix(torch.ones(1, 1, device=DEV), torch.ones(1, device=DEV), torch.full((1,), 1.7, device=DEV))
    same, h = K().streams_norm(x[3][:, :1].contiguous(), None, first, nw, 1e-4, dtype)
    close(h, O.unit(1.7 * x[3][:, 0].double(), 1e-4) * nw.double(), TOL[dtype])


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("t,h,d", [(1, 3, 24), (9, 2, 128), (5, 3, 7), (40, 1, 200), (3, 2, 640), (3, 8, 1024)])
def test_gate_in_front_of_the_norm(dtype, t, h, d):
    x, gate, w = rnd(t, h, d, dtype=dtype).to(DEV), rnd(t, h * d + 8, seed=1, dtype=dtype).to(DEV)[:, : h * d], rnd(h * d, seed=3).to(DEV)
    want = O.unit(x.double() * O.silu(gate.double()).view(t, h, d), 1e-4) * w.double().view(h, d)
    close(K().gated_row_norm(x, gate, w, 1e-4, "silu", gate_first=True), want, TOL[dtype])


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("hq,hkv,d,dv", [(6, 2, 40, 24), (18, 1, 18, 11), (8, 8, 128, 128), (3, 1, 256, 200), (4, 2, 24, 72), (64, 8, 64, 64)])
def test_biases_and_head_factors_in_front_of_the_cache(dtype, hq, hkv, d, dv):
    meta, pages = meta_for([33, 1, 2], [40, 70, 2], 16)
    pad = lambda n: (n + 7) // 8 * 8
    cuts = [pad(hq * d), pad(hkv * d), pad(hkv * dv)]
    z = rnd(36, sum(cuts) + 16, dtype=dtype, gain=3.0).to(DEV)
    q, k, v = (x[:, :n] for x, n in zip(z[:, : sum(cuts)].split(cuts, 1), (hq * d, hkv * d, hkv * dv)))
    qb, kb, vb, qw, kw, temp = (rnd(n, seed=5 + i).to(DEV) for i, n in enumerate((hq * d, hkv * d, hkv * dv, d, d, hq)))
    cache = torch.full((pages, 16 * hkv * (d + dv)), 7.0, dtype=dtype, device=DEV)
    got = K().head_norm_append(q, k, v, (temp[:, None] * qw).contiguous(), kw, None, meta, cache, hq, hkv, d, dv, 1e-3, bias=(qb, kb, vb))
    close(got, O.unit((q.double() + qb.double()).reshape(36, hq, d), 1e-3) * qw.double() * temp.double()[:, None], TOL[dtype])
    slot = meta.slot_mapping.long()
    kp, vp = cache[:, : 16 * hkv * d].reshape(pages * 16, hkv, d), cache[:, 16 * hkv * d :].reshape(pages * 16, hkv, dv)
    close(kp[slot], O.unit((k.double() + kb.double()).reshape(36, hkv, d), 1e-3) * kw.double(), TOL[dtype])
    close(vp[slot], (v.double() + vb.double()).reshape(36, hkv, dv), TOL[dtype])
    assert (cache == 7.0).sum() >= (pages * 16 - 36) * hkv * (d + dv) and K().read_status(DEV) == 0


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 9, 16])
def test_short_convolution(dtype, taps):
    ch = 136
    w, b, ib = rnd(ch, taps, seed=1).to(DEV), rnd(ch, seed=2).to(DEV), rnd(ch, seed=3).to(DEV)
    rows = {s: rnd(n, ch + 8, seed=s, dtype=dtype)[:, :ch] for s, n in ((1, 170), (2, 3), (3, 60))}
    for act, bias, inb in (("none", b, ib), ("silu", b, None), ("none", None, None)):
        state = torch.full((5, ch, taps - 1), 3.0, dtype=dtype, device=DEV)
        state[1:4] = 0
        at, outs = {s: 0 for s in rows}, {s: [] for s in rows}
        for step in ([(1, 1), (2, 2)], [(3, 40), (1, 160), (2, 1)], [(1, 1), (3, 1)], [(3, 19), (1, 8)]):
            counts = [n for _, n in step]
            meta, _ = meta_for(counts, counts, slots=[s for s, _ in step])
            z = torch.zeros(sum(counts), ch + 8, dtype=dtype, device=DEV)
            z[:, :ch] = torch.cat([rows[s][at[s] : at[s] + n] for s, n in step])
            for (s, n), o in zip(step, K().short_conv(z[:, :ch], w, bias, state, meta, act, inb).split(counts)):
                outs[s].append(o)
                at[s] += n
        for s, x in rows.items():
            xd = x.double() + (ib.double().cpu() if inb is not None else 0)
            want = O.conv(xd, w.double().cpu(), b.double().cpu() if bias is not None else torch.zeros(ch, dtype=torch.float64))
            close(torch.cat(outs[s]), O.silu(want) if act == "silu" else want, TOL[dtype])
            if taps > 1:
                k = min(taps - 1, x.shape[0])
                close(state[s, :, taps - 1 - k :], xd[-k:].T, TOL[dtype])
        assert state[0].eq(3).all() and state[4].eq(3).all()


# ---- projections ---------------------------------------------------------------------
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("t,blocks,part", [(1, 3, 32), (33, 3, 21), (64, 16, 256), (700, 8, 64), (5, 1, 136), (2048, 4, 128)])
def test_block_diagonal_gates_in_32_bits(dtype, t, blocks, part):
    x, w = rnd(t, blocks, part, dtype=dtype).to(DEV), rnd(blocks, 2 * part, part, seed=1, dtype=dtype, gain=part ** -0.5).to(DEV)
    got = K().multi_dense(x, w, torch.float32)
    assert got.dtype == torch.float32
    close(got, torch.einsum("tbi,boi->tbo", x.double(), w.double()), 2e-5)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("t,w,ff", [(1, 72, 40), (8, 1024, 2048), (64, 512, 264), (33, 51, 21), (200, 4096, 128), (700, 256, 512), (2048, 1024, 2048)])
def test_xielu_projection(dtype, t, w, ff):
    if dtype == torch.float32 and t > 1000:
        t = 70
    x, up, act = rnd(t, w, dtype=dtype).to(DEV), rnd(ff, w, seed=1, dtype=dtype, gain=1.5 * w ** -0.5).to(DEV), torch.tensor([0.4, -1.1])
    c = (torch.nn.functional.softplus(act) + torch.tensor([0.0, 0.5])).to(DEV)
    close(K().dense_xielu(x, up, c), O.xielu(x.double() @ up.double().T, *act.double().to(DEV)), TOL[dtype] / 3)


# ---- recurrences -----------------------------------------------------------------------
CUTS = ([1] * 210, [2, 8, 7, 1, 15, 17, 20, 64, 4, 72], [128, 5, 3, 74])


def walk(lens, cuts, slots, call):
    """Sequences cut into steps; ``call(rows, step meta)`` -> outputs of those rows.  Returns all outputs."""
    first, at, out = [sum(lens[:b]) for b in range(len(lens))], [0] * len(lens), None
    for i in range(1 if cuts is None else len(cuts)):
        step = list(enumerate(lens)) if cuts is None else [(b, min(cuts[i], n - at[b])) for b, n in enumerate(lens) if at[b] < n]
        if not step:
            break
        idx = torch.cat([torch.arange(first[b] + at[b], first[b] + at[b] + m) for b, m in step]).to(DEV)
        meta, _ = meta_for([m for _, m in step], [m for _, m in step], slots=[slots[b] for b, _ in step])
        o = call(idx, meta)
        out = torch.zeros(sum(lens), *o.shape[1:], dtype=o.dtype, device=DEV) if out is None else out
        out[idx] = o
        for b, m in step:
            at[b] += m
    return out


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("w,blocks", [(40, 5), (96, 3), (21, 7), (256, 2), (1, 1)])
def test_gated_recurrence(dtype, w, blocks):
    lens, slots = [210, 1, 9, 140], [3, 1, 5, 2]
    n = sum(lens)
    g, gb, lam, yb = rnd(n, blocks, 2 * w // blocks, seed=1, gain=2.0).to(DEV), rnd(2 * w, seed=2).to(DEV), torch.linspace(-12, 4, w).to(DEV), rnd(w, seed=3).to(DEV)
    u, z = rnd(n, w, seed=4, dtype=dtype).to(DEV), rnd(n, w + 5, seed=5, dtype=dtype).to(DEV)
    s = O.sigmoid(g.double() + gb.double().view(blocks, -1)).view(n, blocks, 2, -1).cpu()
    want, ends = [], []
    for x, r, i in zip(u.double().cpu().split(lens), s[:, :, 0].reshape(n, w).split(lens), s[:, :, 1].reshape(n, w).split(lens)):
        want.append(O.lru(x, r, i, lam.double().cpu()))
        ends.append(want[-1][-1])
    want = torch.cat(want) * O.gelu(z[:, :w].double().cpu() + yb.double().cpu()) * 0.7
    for cuts in (None, *CUTS):
        state = torch.full((6, 1, 1, w), 5.0, device=DEV)
        state[slots] = 0

        def call(idx, meta):
            both = torch.zeros(len(idx), w + 8, dtype=dtype, device=DEV)
            zz = z[idx]
            K().gated_lru(g[idx], gb, u[idx], lam, zz[:, :w], yb, state, meta, 0.7, both[:, 8:])
            assert not both[:, :8].any()
            return both[:, 8:]

        close(walk(lens, cuts, slots, call), want, TOL[dtype])
        close(state[slots, 0, 0], torch.stack(ends), 1e-4)
        assert state[[0, 4]].eq(5.0).all()


SSD_SHAPES = [(3, 24, 24, 3), (4, 128, 64, 2), (3, 7, 9, 1), (2, 64, 40, 2), (2, 136, 136, 1), (8, 16, 8, 4), (1, 128, 200, 1), (2, 200, 64, 2), (6, 56, 32, 3)]


def ssd_inputs(n, H, N, dv, G, dtype, seed=0):
    """Columns of one convolved row and of a wider projection, as the model has them."""
    c = rnd(n, (H * dv + 2 * G * N + 7) // 8 * 8, seed=seed, dtype=dtype).to(DEV)
    wide = rnd(n, H + 8, seed=seed + 1, dtype=dtype).to(DEV)
    cut = lambda z: (z[:, : H * dv].unflatten(1, (H, dv)), z[:, H * dv : H * dv + G * N].unflatten(1, (G, N)), z[:, H * dv + G * N : H * dv + 2 * G * N].unflatten(1, (G, N)))
    return c, wide[:, :H], cut, rnd(H, seed=seed + 2).to(DEV) - 1, torch.linspace(-5, 2, H).to(DEV), rnd(H, seed=seed + 3).to(DEV)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("H,N,dv,G", SSD_SHAPES)
def test_state_space_duality(dtype, H, N, dv, G):
    lens, slots = [210, 1, 9, 140], [3, 1, 5, 2]
    c, dt, cut, dtb, al, D = ssd_inputs(sum(lens), H, N, dv, G, dtype)
    d = lambda z: z.double().cpu()
    want = torch.cat([O.ssd(*map(d, cut(p)), O.softplus(d(t) + d(dtb)), d(al), d(D)) for p, t in zip(c.split(lens), dt.split(lens))])
    for cuts in (None, *CUTS):
        state = torch.full((6, H, N, dv), 5.0, device=DEV)
        state[slots] = 0
        out = walk(lens, cuts, slots, lambda idx, meta: K().ssd_attention(*cut(c[idx]), dt[idx], dtb, al, D, state, meta))
        close(out, want, TOL[dtype])
        assert state[[0, 4]].eq(5.0).all()


def test_ssd_chunks_and_token_walk_leave_the_same_state():
    """A long sequence over decays from none to immediate, in chunks and token by token; a state that starts non-zero."""
    H, N, dv, G, n = 6, 128, 64, 2, 1300
    c, dt, cut, dtb, _, D = ssd_inputs(n, H, N, dv, G, torch.bfloat16, seed=9)
    al = torch.linspace(-9, 4, H).to(DEV)
    d = lambda z: z.double().cpu()
    want = O.ssd(*map(d, cut(c)), O.softplus(d(dt) + d(dtb)), d(al), d(D))
    meta, _ = meta_for([n], [n], slots=[1])
    states = []
    for chunked in (True, False):
        state = torch.zeros(2, H, N, dv, device=DEV)
        close(K().ssd_attention(*cut(c), dt, dtb, al, D, state, meta, chunked), want, TOL[torch.bfloat16])
        states.append(state.clone())
        again = K().ssd_attention(*cut(c), dt, dtb, al, D, state, meta, chunked)
        states.append((state.clone(), again))
    for a, b in ((states[0], states[2]), (states[1][0], states[3][0])):
        assert ((a - b).abs().amax((1, 2, 3)) / b.abs().amax((1, 2, 3)).clamp(min=1e-3)).max().item() < 1e-3
    close(states[1][1], states[3][1].double(), TOL[torch.bfloat16])


# ---- attention -----------------------------------------------------------------------
def paged_case(dtype, H, G, d, dv, q_lens, kv_lens, page, gain=1.5):
    meta, pages = meta_for(q_lens, kv_lens, page, seed=3)
    cache = torch.full((pages, page * G * (d + dv)), 3.0, dtype=dtype, device=DEV)
    full, _ = meta_for(kv_lens, kv_lens, page, seed=3)
    slot = full.slot_mapping.long()
    k, v, q = rnd(sum(kv_lens), G, d, seed=1, dtype=dtype, gain=gain).to(DEV), rnd(sum(kv_lens), G, dv, seed=2, dtype=dtype).to(DEV), rnd(sum(q_lens), H, d, seed=4, dtype=dtype, gain=gain).to(DEV)
    cut = page * G * d
    cache[:, :cut].view(pages, page, G, d)[slot // page, slot % page] = k
    cache[:, cut:].view(pages, page, G, dv)[slot // page, slot % page] = v
    return meta, cache, q, k, v


def attention_want(q, k, v, H, G, q_lens, kv_lens, m, window, slopes):
    out, qa, ka = [], 0, 0
    for ql, n in zip(q_lens, kv_lens):
        qq, rows = torch.zeros(n, H, q.shape[2], dtype=torch.float64), []
        qq[n - ql :] = q[qa : qa + ql].double().cpu()
        i = torch.arange(n)
        dist = i[:, None] - i[None]
        for h in range(H):
            kk, vv = (z[ka : ka + n, h // (H // G)].double().cpu() for z in (k, v))
            s = O.scores(qq[:, h], kk, m, 1.0, slopes[h]) if m["softcap"] else qq[:, h] @ kk.T * m["scale"] - slopes[h] * dist
            s = s.masked_fill((dist < 0) | (dist >= (window or n)), float("-inf"))
            rows.append((torch.softmax(s, -1) @ vv)[n - ql :])
        out.append(torch.stack(rows, 1))
        qa, ka = qa + ql, ka + n
    return torch.cat(out)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 24, 40), (4, 2, 128, 128), (18, 1, 18, 11), (20, 2, 256, 200), (3, 3, 64, 8), (8, 1, 40, 128)])
def test_windowed_biased_attention(dtype, H, G, d, dv):
    for q_lens, kv_lens, page in (([33, 2, 70], [33, 131, 70], 16), ([1, 1, 1, 1, 1], [1, 16, 17, 200, 65], 32), ([5, 1, 1, 1, 1, 1], [40, 1, 33, 64, 15, 90], 64), ([130, 64], [300, 150], 16)):
        meta, cache, q, k, v = paged_case(dtype, H, G, d, dv, q_lens, kv_lens, page)
        for window, cap, slopes in ((0, 6.0, True), (1, 6.0, True), (16, 0.0, True), (17, 6.0, False), (64, 6.0, True), (63, 0.0, False), (150, 4.0, True)):
            sl = alibi_slopes(H) if slopes else (0.0,) * H
            both = torch.zeros(sum(q_lens), H * dv + 16 - H * dv % 8, dtype=dtype, device=DEV)
            got = K().capped_attention(q, cache, G, dv, meta, d ** -0.5, cap, window=window, slopes=torch.tensor(sl, device=DEV) if slopes else None, out_scale=0.6, out=both[:, : H * dv])
            want = attention_want(q, k, v, H, G, q_lens, kv_lens, dict(scale=d ** -0.5, softcap=cap), window, sl) * 0.6
            close(got.view(-1, H, dv), want, TOL[dtype])
            assert not both[:, H * dv :].any()
    assert K().read_status(DEV) == 0


@pytest.mark.parametrize("window,slopes", [(0, True), (1, True), (64, False), (127, True), (128, True), (129, False), (300, True), (5000, True)])
def test_windowed_prompts_on_the_tcgen05_kernel(window, slopes):
    """Prompt portions beside decoded tokens, edges of the window at every place of a tile."""
    H, G, d = 4, 2, 128
    q_lens, kv_lens = [600, 130, 1, 1], [600, 777, 530, 64]
    meta, cache, q, k, v = paged_case(torch.bfloat16, H, G, d, d, q_lens, kv_lens, 16)
    sl = alibi_slopes(H) if slopes else (0.0,) * H
    for cap in (6.0, 0.0):
        before = K().PREFILL_TC_CALLS["hd128"]
        both = torch.zeros(sum(q_lens), H * d + 64, dtype=torch.bfloat16, device=DEV)
        K().capped_attention(q, cache, G, d, meta, d ** -0.5, cap, window=window, slopes=torch.tensor(sl, device=DEV) if slopes else None, out_scale=1.5, out=both[:, : H * d])
        assert K().PREFILL_TC_CALLS["hd128"] == before + 1
        want = attention_want(q, k, v, H, G, q_lens, kv_lens, dict(scale=d ** -0.5, softcap=cap), window, sl) * 1.5
        close(both[:, : H * d].reshape(-1, H, d), want, TOL[torch.bfloat16])
        assert not both[:, H * d :].any()
    assert K().read_status(DEV) == 0


MARKS = [0, 1, 15, 16, 17, 63, 64, 65, 127, 128, 255, 256, 511, 512, 633, 634, 635, 698, 699]


@pytest.mark.parametrize("dtype,H,G,d", [(torch.bfloat16, 4, 2, 128), (torch.bfloat16, 6, 2, 40), (torch.bfloat16, 18, 1, 18), (torch.float32, 6, 2, 40)])
@pytest.mark.parametrize("window", [65, 188, 0])
def test_one_key_stands_out(dtype, H, G, d, window):
    """Every key scores 0 but one, which takes all the weight of exactly the rows that see it: keys at the first positions, at
    page, tile and window borders and far back, in prompts and in decoding."""
    n, page = 700, 16
    k, v = torch.zeros(len(MARKS) * n, G, d, dtype=dtype), rnd(len(MARKS) * n, G, d, seed=1, dtype=dtype)
    q = torch.zeros(len(MARKS) * n, H, d, dtype=dtype)
    q[..., 0] = 1.0
    for b, j in enumerate(MARKS):
        k[b * n + j, :, 0] = 64.0
    vd = v.double().view(len(MARKS), n, G, d)
    for decode in (False, True):
        q_lens = [1 if decode else n] * len(MARKS)
        meta, cache, *_ = paged_case(dtype, H, G, d, d, q_lens, [n] * len(MARKS), page)
        full, _ = meta_for([n] * len(MARKS), [n] * len(MARKS), page, seed=3)
        slot, cut = full.slot_mapping.long(), page * G * d
        cache[:, :cut].view(-1, page, G, d)[slot // page, slot % page] = k.to(DEV)
        cache[:, cut:].view(-1, page, G, d)[slot // page, slot % page] = v.to(DEV)
        rows = (q.view(len(MARKS), n, H, d)[:, -1] if decode else q).to(DEV).contiguous()
        got = K().capped_attention(rows, cache, G, d, meta, 1.0, 30.0, window=window).view(len(MARKS), -1, H, d)
        for b, j in enumerate(MARKS):
            edge = j + (window or n) - 1  # the last row that sees the key
            for i in [n - 1] if decode else sorted({j - 1, j, j + 1, edge - 1, edge, edge + 1, n - 1} & set(range(n))):
                lo = max(0, i - window + 1) if window else 0
                want = vd[b, j] if lo <= j <= i else vd[b, lo : i + 1].mean(0)
                assert (got[b, -1 if decode else i].double().cpu() - want.repeat_interleave(H // G, 0)).abs().max() < (0.03 if dtype == torch.bfloat16 else 1e-3), (decode, j, i)
    assert K().read_status(DEV) == 0


# ---- whole models ------------------------------------------------------------------------
PROMPTS = {"a": U.tokens(150, 1), "b": U.tokens(61, 2), "c": U.tokens(1, 3), "d": U.tokens(90, 4), "e": U.tokens(34, 5)}
SCHEDULES = {
    "whole": [[(r, len(p))] for r, p in PROMPTS.items()],
    "tokens": [[("b", 1)]] * 61 + [[("e", 2)]] + [[("e", 1)]] * 32,
    "portions": [[("a", n)] for n in (2, 3, 14, 45, 1, 64, 16, 5)] + [[("d", n)] for n in (31, 33, 2, 24)],
    "batched": [[("a", 64), ("b", 1), ("d", 2), ("c", 1)], [("b", 1), ("a", 2), ("d", 40)], [("a", 1), ("b", 1), ("d", 1)], [("b", 57), ("a", 33)], [("d", 45), ("a", 1)], [("d", 1), ("b", 1), ("a", 49)],
                [("d", 1), ("c#1", 1), ("e", 3)], [("b#1", 30), ("e", 31), ("a#1", 100)], [("b#1", 31), ("a#1", 50)]],
}


def _judge(got, want, dtype):
    """In bf16 a row whose copies nearly cancel in front of a norm makes rounding large at its position, whatever computes it."""
    e = U.error(got, want)
    assert e.max() < 1e-4 if dtype == torch.float32 else e.max() < 0.2 and (len(e) == 1 or e.quantile(0.9) < 0.05 and e.median() < 0.02), (e.max().item(), e.median().item())


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("name", sorted(U.CONFIGS))
def test_model_through_the_executor(name, dtype):
    cfg = U.CONFIGS[name]
    W = U.weights(cfg)
    want = {r: U.truth(cfg, W, p) for r, p in PROMPTS.items()}
    rep = U.replayer(cfg, W, DEV, dtype, 384)
    for _ in range(2):  # the second round runs on pages and slots that the first one used
        for sched in SCHEDULES.values():
            for r, got in U.run(rep, sched, PROMPTS).items():
                _judge(got, want[r.split("#")[0]], dtype)
    assert rep.pool.used() == 0 and not rep.ex.model.rec.by_rid and K().read_status(DEV) == 0


@pytest.mark.parametrize("dtype", TYPES)
def test_long_prompts_and_long_decoding(dtype):
    """A prompt whose portions take the tcgen05 attention and the chunk-wise scan, decoded on past its windows."""
    cfg = U.CONFIGS["wide"]
    W = U.weights(cfg, seed=1)
    prompts = {"p": U.tokens(760, 31), "q": U.tokens(260, 32)}
    want = {r: U.truth(cfg, W, p) for r, p in prompts.items()}
    for sched in ([[("p", 760)], [("q", 260)]], [[("p", 600), ("q", 1)]] + [[("p", 1), ("q", 1)]] * 160 + [[("q", 1)]] * 99, [[("p", 530), ("q", 2)], [("q", 1), ("p", 99)], [("p", 2), ("q", 256)], [("p", 129), ("q", 1)]]):
        rep = U.replayer(cfg, W, DEV, dtype, 1088)
        for r, got in U.run(rep, sched, prompts).items():
            _judge(got, want[r], dtype)
    assert K().read_status(DEV) == 0


def test_decode_graph_equals_the_eager_step():
    cfg = U.CONFIGS["mixed"]
    W = U.weights(cfg)
    outs = []
    for graph in (True, False):
        rep = U.replayer(cfg, W, DEV, torch.bfloat16, 384, cuda_graph=graph)
        outs.append(U.run(rep, [[("a", 30), ("b", 20)]] + [[("a", 1), ("b", 1)]] * 41 + [[("a", 1)]] * 79, PROMPTS))
        assert (rep.ex._graphs is not None and rep.ex._graphs.replays > 100) == graph
    for r in "ab":
        assert U.error(outs[0][r], outs[1][r].double()).max() < 0.03  # the KV splits of a graph are fixed at capture


@pytest.mark.parametrize("dtype", TYPES)
def test_greedy_generation_through_the_engine(dtype):
    from pegainfer_b200.config import EngineConfig, from_hf
    from pegainfer_b200.engine.build import build_engine
    from pegainfer_b200.loader.sources import DictSource
    from pegainfer_b200.models import registry

    cfg = U.CONFIGS["mixed"]
    W = U.weights(cfg)
    mcfg = from_hf(cfg)
    mcfg.max_position = 1024
    model = registry.build(mcfg, source=DictSource(W), device=DEV, dtype=dtype)
    eng = build_engine(EngineConfig(num_kv_blocks=64, max_decode_batch=3, max_prefill_tokens=48, state_slots=3), mcfg, device=DEV, dtype=dtype, model=model)
    try:
        prompts = [U.tokens(n, 40 + n) for n in (5, 70, 1, 100, 33)]
        slack = []
        for p, (toks, term, _) in zip(prompts, eng.generate(prompts, max_tokens=20)):
            assert term.kind == "finished" and len(toks) == 20
            lg = U.truth(cfg, W, p + toks[:-1])[len(p) - 1 :]
            slack.append((lg.max(-1).values - lg.gather(1, torch.tensor(toks)[:, None])[:, 0]) / lg.std())  # each token is the best or as good
        slack = torch.cat(slack)
        assert slack.max() < (1e-3 if dtype == torch.float32 else 0.2), slack.max()
    finally:
        eng.shutdown()
