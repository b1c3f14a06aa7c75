"""Nemipel line on a GPU: every kernel against the plain restatement, and whole models through the engine's executor in
bf16 and f32, cut into steps in different ways."""
import pytest
import torch

import nemipel_oracle as O
import nemipel_util as U
from pegainfer_b200.ops.reference import AttnMeta, pair_rope_tables

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
TOL = {torch.float32: 1e-4, torch.bfloat16: 3e-2}
TYPES = [torch.bfloat16, torch.float32]


def K():
    from pegainfer_b200.ops import cuda

    return cuda


def close(got, want, tol, scale=None):
    """Largest difference beyond the rounding of the result itself, over the spread of the values (or ``scale``)."""
    last_bit = 2.0 ** -8 if got.dtype == torch.bfloat16 else 2.0 ** -22
    got, want = got.double().cpu(), want.double().cpu()
    s = scale or want.pow(2).mean().sqrt().item()
    err = ((got - want).abs() - last_bit * want.abs()).max().item() / s
    assert err < tol, err


def rnd(*shape, seed=0, dtype=torch.float32, gain=1.0):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * gain).to(dtype)


def meta_for(q_lens, kv_lens, page=16, slots=None, seed=0):
    """Ragged step over shuffled pages."""
    ind = [0]
    for n in q_lens:
        ind.append(ind[-1] + n)
    need = [(n + page - 1) // page for n in kv_lens]
    perm = (torch.randperm(sum(need), generator=torch.Generator().manual_seed(seed)) + 1).tolist()
    table = torch.zeros(len(q_lens), max(need + [1]), dtype=torch.int32)
    pos, slot = [], []
    for b, n in enumerate(need):
        pages = [perm.pop() for _ in range(n)]
        table[b, :n] = torch.tensor(pages, dtype=torch.int32)
        for p in range(kv_lens[b] - q_lens[b], kv_lens[b]):
            pos.append(p)
            slot.append(pages[p // page] * page + p % page)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)
    slots = slots or list(range(1, len(q_lens) + 1))
    return AttnMeta(q_indptr=i32(ind), kv_lens=i32(kv_lens), block_table=table.to(DEV), slot_mapping=i32(slot), positions=i32(pos), page_size=page, num_seqs=len(q_lens), num_tokens=ind[-1],
                    max_q_len=max(q_lens), max_kv_len=max(kv_lens), decode_only=max(q_lens) <= 1, h_q_indptr=ind, h_kv_lens=list(kv_lens), state_slots=i32(slots), h_state_slots=slots), sum(need) + 1


# ---- rows --------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("t,w", [(1, 8), (5, 50), (3, 4096), (2, 9216), (7, 72)])
def test_stream_rows(dtype, t, w):
    table, ids = rnd(20, w, dtype=dtype).to(DEV), torch.tensor([i * 7 % 20 for i in range(t)], dtype=torch.int32, device=DEV)
    x, h = K().embed_stream(ids, table, dtype)
    assert x.dtype == torch.float32 and h.dtype == dtype and torch.equal(x, table[ids.long()].float()) and torch.equal(h, table[ids.long()])
    wt = rnd(w, seed=2).to(DEV)
    for y in (rnd(t, w, seed=3, dtype=dtype).to(DEV), rnd(t, w, seed=4).to(DEV)):
        want = O.rms(1.7 * x.double() + y.double(), 1e-5) * wt.double()
        xs = x.clone()
        h = K().post_norm(y, xs, wt, 1e-5, 1.7, dtype)
        close(xs, want, 1e-5)
        assert torch.equal(h, xs.to(dtype))
    h = K().stream_norm(x, wt, 1e-3, dtype)
    close(h, O.rms(x.double(), 1e-3) * wt.double(), TOL[dtype])
    assert torch.equal(K().gather_rows(h, ids[:1]), h[ids[:1].long()]) if ids[0] < t else True


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("t,h,d", [(4, 1, 4096), (3, 5, 11), (9, 2, 64), (2, 3, 640), (1, 1, 10000)])
def test_gated_row_norm(dtype, t, h, d):
    x, wide, w = rnd(t, h, d, dtype=dtype).to(DEV), rnd(t, h * d + 24, seed=1, dtype=dtype).to(DEV), rnd(d, seed=2).to(DEV)
    g = wide[:, 8 : 8 + h * d]
    got = K().gated_row_norm(x, g, w, 1e-4)
    close(got, O.rms(x.double(), 1e-4) * w.double() * O.sigmoid(g.double()).view(t, h, d), TOL[dtype])


@pytest.mark.parametrize("t,m,k", [(1, 5, 3), (70, 130, 50), (3, 448, 24), (300, 1100, 264), (64, 7, 18)])
def test_dense_any_size(t, m, k):
    for dtype in TYPES:
        x, w = rnd(t, k + 8, dtype=dtype).to(DEV)[:, :k], rnd(m, k, seed=1, dtype=dtype).to(DEV)
        want = x.double() @ w.double().T
        close(K().dense(x, w, torch.float32), want, 2e-5 if dtype == torch.float32 or m * t < 1 << 17 else 2e-2)
        close(K().dense(x, w), want, TOL[dtype])
    if m % 8 == 0:
        for dtype in TYPES:
            x, w = rnd(t, k, dtype=dtype).to(DEV), rnd(m, k, seed=1, dtype=dtype, gain=0.3).to(DEV)
            z = x.double() @ w.double().T
            want = O.silu(z[:, : m // 2]) * z[:, m // 2 :]
            close(K().dense_glu(x, w), want, 4e-2 if dtype == torch.bfloat16 else 2e-5)
            if dtype == torch.bfloat16:
                il = torch.stack((w[: m // 2], w[m // 2 :]), 1).reshape(m, k).contiguous()
                close(K().dense_glu(x, il, True), want, 4e-2)


def test_softcap_keeps_32_bits():
    x = torch.cat((torch.linspace(-90, 90, 1000), torch.logspace(-6, 1, 500), torch.tensor([0.0]))).view(1, -1).to(DEV)
    want = 15 * torch.tanh(x.double() / 15)
    got = K().softcap_rows(x, 15.0).double()
    assert ((got - want).abs() <= 1e-6 * want.abs() + 1e-12).all()


# ---- attention -----------------------------------------------------------------------
GEOMS = [(6, 2, 24, 40, 10), (4, 4, 128, 128, 128), (18, 1, 18, 13, 2), (20, 2, 256, 72, 64), (6, 3, 96, 96, 32), (9, 1, 64, 64, 0), (16, 2, 128, 128, 32), (4, 1, 16, 128, 16)]


def _filled(meta, pages, heads, kvh, dim, vdim, rot, dtype, kv_lens, seed=0, gain=1.0):
    """Append every sequence's keys and values (one long prompt step per sequence), return cache and the plain tensors."""
    cos, sin = pair_rope_tables(4096, rot, 50.0, DEV)
    cache = rnd(pages, meta.page_size * kvh * (dim + vdim), seed=99, dtype=dtype).to(DEV)  # stale contents
    qw, kw = rnd(heads * dim, seed=5).abs().to(DEV) + 0.5, rnd(kvh * dim, seed=6).abs().to(DEV) + 0.5
    plain = []
    for b, n in enumerate(kv_lens):
        wide = rnd(n, (heads + kvh) * dim + kvh * vdim + 8, seed=seed + 10 + b, dtype=dtype).to(DEV)
        q, k, v = wide[:, : heads * dim], wide[:, heads * dim : (heads + kvh) * dim], wide[:, (heads + kvh) * dim : (heads + kvh) * dim + kvh * vdim]
        m = AttnMeta(q_indptr=None, kv_lens=None, block_table=None, slot_mapping=meta.block_table[b].long().repeat_interleave(meta.page_size)[:n].mul(meta.page_size).add(torch.arange(n, device=DEV) % meta.page_size).int(),
                     positions=torch.arange(n, dtype=torch.int32, device=DEV), page_size=meta.page_size, num_seqs=1, num_tokens=n, max_q_len=n, max_kv_len=n)
        qo = K().row_norm_rope_append(q, k, v, qw, kw, cos, sin, m, cache, heads, kvh, dim, vdim, 1e-5)
        pos = torch.arange(n)
        wq = O.rotate((O.rms(q.double(), 1e-5) * qw.double()).view(n, heads, dim).cpu(), pos, rot, 50.0)
        wk = O.rotate((O.rms(k.double(), 1e-5) * kw.double()).view(n, kvh, dim).cpu(), pos, rot, 50.0)
        close(qo, wq, 2e-2 if dtype == torch.bfloat16 else 2e-5)
        only = K().row_norm_rope_append(q, None, None, qw, None, cos, sin, m, cache, heads, kvh, dim, vdim, 1e-5)  # a layer without keys
        assert torch.equal(only, qo)
        plain.append((qo, wk, v.double().cpu().view(n, kvh, vdim)))
    return cache, plain


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("geom", GEOMS)
def test_attention_shapes(dtype, geom):
    heads, kvh, dim, vdim, rot = geom
    for q_lens, kv_lens, page in (([33, 2, 70], [33, 131, 70], 16), ([1, 1, 1, 1, 1], [1, 16, 17, 200, 65], 32), ([5, 1, 1, 1, 1, 1], [40, 1, 33, 64, 15, 90], 64)):
        meta, pages = meta_for(q_lens, kv_lens, page)
        cache, plain = _filled(meta, pages, heads, kvh, dim, vdim, rot, dtype, kv_lens)
        q = torch.cat([plain[b][0][kv_lens[b] - n :] for b, n in enumerate(q_lens)]).contiguous()
        gate = rnd(q.shape[0], heads + 8, seed=3, dtype=dtype).to(DEV)
        for cap, gt in ((6.0, gate), (0.0, None), (50.0, None)):
            got = K().capped_attention(q, cache, kvh, vdim, meta, 0.4, cap, gt).double().cpu()
            k0 = 0
            for b, n in enumerate(q_lens):
                want = O.softcap_attention(plain[b][0].double().cpu(), plain[b][1].to(dtype).double(), plain[b][2], 0.4, cap)[kv_lens[b] - n :]
                if gt is not None:
                    want = want * O.sigmoid(gt[k0 : k0 + n, :heads].double().cpu())[:, :, None]
                close(got[k0 : k0 + n].view(n, heads, vdim), want, TOL[dtype], scale=1.0)
                k0 += n
    assert K().read_status(DEV) == 0


@pytest.mark.parametrize("dtype,dim,vdim", [(torch.bfloat16, 128, 128), (torch.bfloat16, 64, 32), (torch.bfloat16, 24, 40), (torch.bfloat16, 18, 13), (torch.float32, 24, 40)])
def test_one_key_stands_out(dtype, dim, vdim):
    """Every visible key scores 0 but one, which takes all the weight: the output is that key's value.  Keys at the first
    positions, on both sides of page and tile borders, far back and the query's own; prompts and decoding; a key one past
    the query must not be seen."""
    n, page, kvh, heads = 700, 16, 2, 4
    for decode in (False, True):
        marks = [0, 1, 15, 16, 17, 63, 64, 127, 128, 129, 255, 256, 511, 512, 513, 640, 698, 699]
        q_lens = [1] * len(marks) if decode else [n] * len(marks)
        meta, pages = meta_for(q_lens, [n] * len(marks), page, seed=4)
        v = rnd(len(marks), n, kvh, vdim, seed=1).to(dtype).to(DEV)
        k = torch.zeros(len(marks), n, kvh, dim, dtype=dtype, device=DEV)
        for i, j in enumerate(marks):
            k[i, j, :, 3] = 60.0
        cache = torch.zeros(pages, page * kvh * (dim + vdim), dtype=dtype, device=DEV)
        kp, vp = cache[:, : page * kvh * dim].view(pages, page, kvh, dim), cache[:, page * kvh * dim :].view(pages, page, kvh, vdim)
        for i in range(len(marks)):
            pg = meta.block_table[i].long()
            kp[pg] = torch.nn.functional.pad(k[i], (0, 0, 0, 0, 0, len(pg) * page - n)).view(-1, page, kvh, dim)
            vp[pg] = torch.nn.functional.pad(v[i], (0, 0, 0, 0, 0, len(pg) * page - n)).view(-1, page, kvh, vdim)
        q = torch.zeros(sum(q_lens), heads, dim, dtype=dtype, device=DEV)
        q[:, :, 3] = 1.0
        got = K().capped_attention(q, cache, kvh, vdim, meta, 1.0, 50.0).view(len(marks), -1, heads, vdim)
        for i, j in enumerate(marks):
            rep = v[i].repeat_interleave(heads // kvh, 1)
            assert (got[i, -1] - rep[j]).abs().max() < 0.02
            if not decode:
                assert (got[i, j].float() - rep[j].float()).abs().max() < 0.02  # the row of the key itself
                if j:  # one row earlier: a plain mean of the keys so far
                    close(got[i, j - 1], rep[:j].double().mean(0), 0.02, scale=1.0)
    assert K().read_status(DEV) == 0


def test_long_prompts_take_the_tcgen05_kernel():
    dtype, heads, kvh = torch.bfloat16, 4, 2
    q_lens, kv_lens = [600, 130, 1, 1, 1, 1], [600, 777, 5, 64, 300, 17]
    meta, pages = meta_for(q_lens, kv_lens, 16)
    cache, plain = _filled(meta, pages, heads, kvh, 128, 128, 64, dtype, kv_lens)
    q = torch.cat([plain[b][0][kv_lens[b] - n :] for b, n in enumerate(q_lens)]).contiguous()
    gate = rnd(q.shape[0], heads, seed=3, dtype=dtype).to(DEV)
    for scale, cap in ((0.1, 50.0), (0.1, 4.0), (0.5, 5.0), (0.088, 0.0)):  # far below the cap (polynomial tanh), around it, well above it, none
        before = K().PREFILL_TC_CALLS["hd128"]
        got = K().capped_attention(q, cache, kvh, 128, meta, scale, cap, gate).double().cpu()
        assert K().PREFILL_TC_CALLS["hd128"] == before + 1
        k0 = 0
        for b, n in enumerate(q_lens):
            qd = plain[b][0].double().cpu()
            kk, vv = plain[b][1].to(dtype).double().repeat_interleave(2, 1), plain[b][2].repeat_interleave(2, 1)
            s = O.cap(torch.einsum("qhd,khd->hqk", qd[kv_lens[b] - n :], kk) * scale, cap)
            s = s.masked_fill(torch.arange(kv_lens[b])[None, None] > torch.arange(kv_lens[b] - n, kv_lens[b])[None, :, None], float("-inf"))
            want = torch.einsum("hqk,khd->qhd", torch.softmax(s, -1), vv) * O.sigmoid(gate[k0 : k0 + n].double().cpu())[:, :, None]
            close(got[k0 : k0 + n].view(n, heads, 128), want, 3e-2, scale=1.0)
            k0 += n
    assert K().read_status(DEV) == 0


# ---- recurrences -----------------------------------------------------------------------
def _cuts(n, sizes):
    out, i = [], 0
    while n:
        c = min(sizes[i % len(sizes)], n)
        out.append(c)
        n -= c
        i += 1
    return out


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("h,dk,dv", [(3, 40, 24), (2, 128, 128), (5, 6, 11), (2, 144, 40), (4, 64, 64), (2, 16, 200), (1, 256, 8), (2, 72, 136)])
def test_lightning(dtype, h, dk, dv):
    decay = torch.tensor([0.999, 0.5, 1.0, 0.9, 0.25][:h])
    lens = [300, 64, 33, 1, 65]
    for sizes in ([1000], [2, 31, 64, 1, 130, 3], [7]):
        rows = [rnd(n, 2 * h * dk + h * dv, seed=b, dtype=dtype).to(DEV) for b, n in enumerate(lens)]
        state = torch.zeros(8, h, dk, dv, device=DEV)
        state[6] = 7.0
        cuts, got, at = [_cuts(n, sizes) for n in lens], [[] for _ in lens], [0] * len(lens)
        while any(cuts):
            live = [b for b in range(len(lens)) if cuts[b]]
            n = [cuts[b].pop(0) for b in live]
            meta, _ = meta_for(n, n, slots=[b + 1 for b in live])
            x = torch.cat([rows[b][at[b] : at[b] + c] for b, c in zip(live, n)])
            t = x.shape[0]
            o = K().decay_attention(x[:, : h * dk].view(t, h, dk), x[:, h * dk : 2 * h * dk].view(t, h, dk), x[:, 2 * h * dk :].view(t, h, dv), decay.to(DEV), state, meta)
            k0 = 0
            for b, c in zip(live, n):
                got[b].append(o[k0 : k0 + c])
                at[b] += c
                k0 += c
        for b, n in enumerate(lens):
            z = O.silu(rows[b].double().cpu()).to(dtype).double()
            want = O.lightning_scan(z[:, : h * dk].view(n, h, dk), z[:, h * dk : 2 * h * dk].view(n, h, dk), z[:, 2 * h * dk :].view(n, h, dv), decay.double())
            close(torch.cat(got[b]), want, 2e-2 if dtype == torch.bfloat16 else 1e-4)
        assert (state[6] == 7.0).all() and (state[0] == 0).all() and (state[7] == 0).all()


def test_lightning_chunks_keep_the_state_in_32_bits():
    """A slowly decaying head over a long prompt: chunk-wise and token-wise kernels end in the same f32 state."""
    h, d, n = 2, 128, 1500
    x = rnd(n, 3 * h * d, dtype=torch.bfloat16).to(DEV)
    part = [x[:, i * h * d : (i + 1) * h * d].view(n, h, d) for i in range(3)]
    states = []
    for chunked in (True, False):
        st = torch.zeros(2, h, d, d, device=DEV)
        meta, _ = meta_for([n], [n], slots=[1])
        K().decay_attention(*part, torch.tensor([0.9995, 0.97], device=DEV), st, meta, chunked=chunked)
        states.append(st[1].double())
    close(states[0], states[1], 3e-4)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 7, 16])
def test_conv(dtype, taps):
    ch, lens = 150, [100, 5, 1, 33]
    w = rnd(ch, taps, seed=9).to(DEV)
    for sizes in ([1000], [2], [1], [3, 40, 1]):
        rows = [rnd(n, ch + 10, seed=b, dtype=dtype).to(DEV)[:, :ch] for b, n in enumerate(lens)]
        state = torch.zeros(6, ch, taps - 1, dtype=dtype, device=DEV)
        cuts, got, at = [_cuts(n, sizes) for n in lens], [[] for _ in lens], [0] * len(lens)
        while any(cuts):
            live = [b for b in range(len(lens)) if cuts[b]]
            n = [cuts[b].pop(0) for b in live]
            meta, _ = meta_for(n, n, slots=[b + 1 for b in live])
            wide = torch.cat([torch.nn.functional.pad(rows[b][at[b] : at[b] + c], (0, 6)) for b, c in zip(live, n)])
            o, k0 = K().conv_silu(wide[:, :ch], w, state, meta), 0
            for b, c in zip(live, n):
                got[b].append(o[k0 : k0 + c])
                at[b] += c
                k0 += c
        for b in range(len(lens)):
            close(torch.cat(got[b]), O.short_conv(rows[b].double().cpu(), w.double().cpu()), TOL[dtype])


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("h,hk,dk,dv", [(6, 3, 24, 16), (2, 2, 128, 128), (3, 1, 7, 9), (4, 2, 136, 48), (2, 1, 64, 130), (2, 2, 32, 64)])
def test_channel_delta(dtype, h, hk, dk, dv):
    lens = [90, 17, 1, 40]
    a_log, dt = torch.linspace(-5, 1.5, h), rnd(h * dk, seed=8)
    for sizes in ([1000], [2], [1], [5, 8, 9, 64]):
        rows = [rnd(n, 2 * hk * dk + h * dv, seed=b, dtype=dtype).to(DEV) for b, n in enumerate(lens)]
        f = [rnd(n, h * dk, seed=20 + b, gain=3.0).to(DEV) for b, n in enumerate(lens)]
        bt = [rnd(n, h, seed=30 + b, dtype=dtype).to(DEV) for b, n in enumerate(lens)]
        state = torch.zeros(6, h, dk, dv, device=DEV)
        cuts, got, at = [_cuts(n, sizes) for n in lens], [[] for _ in lens], [0] * len(lens)
        while any(cuts):
            live = [b for b in range(len(lens)) if cuts[b]]
            n = [cuts[b].pop(0) for b in live]
            meta, _ = meta_for(n, n, slots=[b + 1 for b in live])
            cat = lambda xs: torch.cat([xs[b][at[b] : at[b] + c] for b, c in zip(live, n)])
            x, t = cat(rows), sum(n)
            o = K().channel_delta(x[:, : hk * dk].view(t, hk, dk), x[:, hk * dk : 2 * hk * dk].view(t, hk, dk), x[:, 2 * hk * dk :].view(t, h, dv), cat(f), cat(bt), a_log.to(DEV), dt.to(DEV), state, meta)
            k0 = 0
            for b, c in zip(live, n):
                got[b].append(o[k0 : k0 + c])
                at[b] += c
                k0 += c
        for b, n in enumerate(lens):
            z = rows[b].double().cpu()
            g = torch.exp(-torch.exp(a_log.double())[None, :, None] * O.softplus((f[b].double().cpu() + dt.double())).view(n, h, dk))
            want = O.channel_delta_scan(O.unit(z[:, : hk * dk].view(n, hk, dk)) * dk ** -0.5, O.unit(z[:, hk * dk : 2 * hk * dk].view(n, hk, dk)), z[:, 2 * hk * dk :].view(n, h, dv), g, O.sigmoid(bt[b].double().cpu()))
            close(torch.cat(got[b]), want, 3e-2 if dtype == torch.bfloat16 else 1e-4)


# ---- whole models ------------------------------------------------------------------------
PROMPTS = {"a": U.tokens(150, 1), "b": U.tokens(61, 2), "c": U.tokens(1, 3), "d": U.tokens(90, 4), "e": U.tokens(34, 5)}
SCHEDULES = {
    "whole": [[(r, len(p))] for r, p in PROMPTS.items()],
    "tokens": [[("b", 1)]] * 61 + [[("e", 2)]] + [[("e", 1)]] * 32,
    "portions": [[("a", n)] for n in (2, 3, 14, 45, 1, 64, 16, 5)] + [[("d", n)] for n in (31, 33, 2, 24)],
    "batched": [[("a", 64), ("b", 1), ("d", 2), ("c", 1)], [("b", 1), ("a", 2), ("d", 40)], [("a", 1), ("b", 1), ("d", 1)], [("b", 57), ("a", 33)], [("d", 45), ("a", 1)], [("d", 1), ("b", 1), ("a", 49)],
                [("d", 1), ("c#1", 1), ("e", 3)], [("b#1", 30), ("e", 31), ("a#1", 100)], [("b#1", 31), ("a#1", 50)]],
}


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
                e = U.error(got, want[r.split("#")[0]])
                assert e.max() < (2e-4 if dtype == torch.float32 else U.BF16_ERROR[name]), (r, e.max().item(), e.mean().item())
    assert rep.pool.used() == 0 and not rep.ex.model.rec.by_rid and K().read_status(DEV) == 0


def test_decode_graph_equals_the_eager_step():
    cfg = U.CONFIGS["mixed"]
    W = U.weights(cfg)
    outs = []
    for graph in (True, False):
        rep = U.replayer(cfg, W, DEV, torch.bfloat16, 384, cuda_graph=graph)
        outs.append(U.run(rep, [[("a", 30), ("b", 20)]] + [[("a", 1), ("b", 1)]] * 41 + [[("a", 1)]] * 79, PROMPTS))
        assert (rep.ex._graphs is not None and rep.ex._graphs.replays > 100) == graph
    assert all(torch.equal(outs[0][r], outs[1][r]) for r in "ab")


@pytest.mark.parametrize("dtype", TYPES)
def test_greedy_generation_through_the_engine(dtype):
    from pegainfer_b200.config import EngineConfig, from_hf
    from pegainfer_b200.engine.build import build_engine
    from pegainfer_b200.loader.sources import DictSource
    from pegainfer_b200.models.nemipel import NemipelModel

    cfg = U.CONFIGS["mixed"]
    W = U.weights(cfg)
    mcfg = from_hf(cfg)
    mcfg.max_position = 1024
    model = NemipelModel(mcfg, source=DictSource(W), device=DEV, dtype=dtype)
    eng = build_engine(EngineConfig(num_kv_blocks=64, max_decode_batch=3, max_prefill_tokens=48), mcfg, device=DEV, dtype=dtype, model=model)
    try:
        prompts = [U.tokens(n, 40 + n) for n in (5, 70, 33, 1, 100)]
        outs = eng.generate(prompts, max_tokens=20)
        for p, (toks, term, _) in zip(prompts, outs):
            assert term.kind == "finished" and len(toks) == 20
            lg = U.truth(cfg, W, p + toks[:-1])[len(p) - 1 :]
            best = lg.max(-1).values
            slack = (best - lg.gather(1, torch.tensor(toks)[:, None])[:, 0]).max().item()  # each token is the best or as good
            assert slack < (1e-3 if dtype == torch.float32 else 0.5), slack
    finally:
        eng.shutdown()
