"""Zeripel line on a GPU: every kernel against the plain restatement, and whole models through the engine's executor in
bf16 and f32, cut into steps in different ways."""
import pytest
import torch

import zeripel_oracle as O
import zeripel_util as U
from pegainfer_b200.ops.reference import pair_rope_tables, temperature_table
from test_nemipel_gpu import DEV, K, TOL, TYPES, close, meta_for, rnd
from test_vekalorn_gpu import Case

pytestmark = pytest.mark.gpu


# ---- rows --------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("w", [8, 50, 72, 4096, 9216])
def test_pair_embedding(dtype, w):
    e = dict(scale=2.5, bigram=dict(buckets=91, mul_prev=2147483647, mul_cur=7919))
    table, pairs, wt = rnd(300, w, dtype=dtype).to(DEV), rnd(92, w, seed=1, dtype=dtype).to(DEV), rnd(w, seed=2).to(DEV)
    W = {"embed": table.double().cpu(), "bigram": pairs.double().cpu()}
    seqs = {1: U.tokens(40, 1, 300), 2: U.tokens(3, 2, 300), 3: U.tokens(19, 3, 300)}
    carried, at, rows = torch.zeros(5, dtype=torch.int32, device=DEV), {s: 0 for s in seqs}, {s: [] for s in seqs}
    for step in ([(1, 1), (2, 2)], [(3, 7), (1, 30), (2, 1)], [(1, 1), (3, 1)], [(3, 11), (1, 8)]):
        lens = [n for _, n in step]
        meta, _ = meta_for(lens, lens, slots=[s for s, _ in step])
        ids = torch.tensor(sum((seqs[s][at[s] : at[s] + n] for s, n in step), []), dtype=torch.int32, device=DEV)
        x, h = K().embed_pairs_norm(ids, table, pairs, 2.5, (91, 2147483647, 7919), carried, wt, 1e-4, meta, dtype)
        close(h, O.rms(x.double(), 1e-4) * wt.double(), TOL[dtype])
        for (s, n), r in zip(step, x.split(lens)):
            rows[s].append(r)
            at[s] += n
    for s, toks in seqs.items():
        close(torch.cat(rows[s]), O.embed(toks, W, e), 1e-5)
    assert carried.tolist() == [0, seqs[1][-1] + 1, seqs[2][-1] + 1, seqs[3][-1] + 1, 0] and K().read_status(DEV) == 0


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("t,w", [(1, 8), (5, 50), (3, 4096), (2, 9216), (7, 72)])
def test_residual_norm(dtype, t, w):
    x, wt = rnd(t, w).to(DEV), rnd(w, seed=2).to(DEV)
    for y in (rnd(t, w + 8, seed=3, dtype=dtype).to(DEV)[:, :w], rnd(t, w, seed=4).to(DEV)):
        xs = x.clone()
        h = K().residual_norm(y, xs, wt, 1e-5, 0.6, dtype)
        close(xs, x.double() + 0.6 * y.double(), 1e-5)
        close(h, O.rms(xs.double(), 1e-5) * wt.double(), TOL[dtype])
    k = 3
    rows, pos, wts = rnd(t * k, w, seed=6, dtype=dtype).to(DEV), torch.randperm(t * k, generator=torch.Generator().manual_seed(1)).int().to(DEV), rnd(t, k, seed=7).abs().to(DEV)
    y = (rows.double()[pos.long()].view(t, k, w) * wts.double()[:, :, None]).sum(1)
    z = rnd(t, 9, seed=8).to(DEV)
    for shared in (None, rnd(t, w, seed=9, dtype=dtype).to(DEV), rnd(t, w, seed=9).to(DEV)):
        xs = x.clone()
        h = K().residual_norm_rows(rows, pos, wts, shared, None if shared is None else z[:, 8:], xs, wt, 1e-5, 0.6, dtype)
        want = x.double() + 0.6 * (y + (0 if shared is None else shared.double() * O.sigmoid(z[:, 8:].double())))
        close(xs, want, 1e-5)
        close(h, O.rms(want, 1e-5) * wt.double(), TOL[dtype])


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("n,w", [(5, 8), (5, 50), (1, 36), (8, 72), (5, 2048)])
def test_token_mix(dtype, n, w):
    mu = torch.rand(n, w, generator=torch.Generator().manual_seed(5)).to(DEV)
    carried = torch.full((5, w, 1), 3.0, dtype=dtype, device=DEV)
    carried[1:4] = 0
    rows = {s: rnd(m, w, seed=s, dtype=dtype) for s, m in ((1, 700), (2, 3), (3, 60))}
    at, outs = {s: 0 for s in rows}, {s: [] for s in rows}
    for step in ([(1, 1), (2, 2)], [(3, 40), (1, 690), (2, 1)], [(1, 1), (3, 1)], [(3, 19), (1, 8)]):
        lens = [m for _, m in step]
        meta, _ = meta_for(lens, lens, slots=[s for s, _ in step])
        h = torch.cat([rows[s][at[s] : at[s] + m] for s, m in step]).to(DEV)
        for (s, m), r in zip(step, K().token_mix(h, mu, carried, meta).split(lens)):
            outs[s].append(r)
            at[s] += m
    for s, h in rows.items():
        got, hd = torch.cat(outs[s]), h.double()
        for i in range(n):
            close(got[:, i], hd + (O.shift(hd) - hd) * mu[i].double().cpu(), TOL[dtype])
        assert torch.equal(carried[s, :, 0].cpu(), h[-1])
    assert carried[0].eq(3).all() and carried[4].eq(3).all()


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("t,h,d", [(1, 3, 24), (9, 2, 128), (5, 7, 7), (40, 1, 200), (3, 2, 640)])
def test_gated_row_norm_and_tanh(dtype, t, h, d):
    x, gate = rnd(t, h, d, dtype=dtype).to(DEV), rnd(t, h * d + 8, seed=1, dtype=dtype).to(DEV)[:, : h * d]
    for w in (rnd(d, seed=2).to(DEV), rnd(h * d, seed=3).to(DEV)):
        for act, f in (("silu", O.silu), ("sigmoid", O.sigmoid)):
            want = O.rms(x.double(), 1e-4) * w.double().view(-1 if w.numel() > d else 1, d) * f(gate.double()).view(t, h, d)
            close(K().gated_row_norm(x, gate, w, 1e-4, act), want, TOL[dtype])
    close(K().tanh_rows(x * 3), torch.tanh((x * 3).double()), 1e-5 if dtype == torch.float32 else TOL[dtype])


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("hq,hkv,d,dv", [(6, 2, 40, 40), (18, 1, 18, 18), (8, 8, 128, 128), (3, 1, 256, 256), (4, 2, 24, 72), (64, 8, 64, 64)])
def test_head_norm_append(dtype, hq, hkv, d, dv):
    meta, pages = meta_for([33, 1, 2], [40, 70, 2], 16)
    pad = lambda n: (n + 7) // 8 * 8
    z = rnd(36, pad(hq * d) + pad(hkv * d) + hkv * dv, dtype=dtype, gain=3.0).to(DEV)
    q, k, v = z[:, : hq * d], z[:, pad(hq * d) : pad(hq * d) + hkv * d], z[:, pad(hq * d) + pad(hkv * d) :]
    if dv == d:
        v = k
    qw, kw = rnd(d, seed=5).to(DEV), rnd(d, seed=6).to(DEV)
    for temp in (None, temperature_table(128, 0.3, 9, DEV)):
        cache = torch.full((pages, 16 * hkv * (d + dv)), 7.0, dtype=dtype, device=DEV)
        got = K().head_norm_append(q, k, v, qw, kw, temp, meta, cache, hq, hkv, d, dv, 1e-3)
        f = 1 if temp is None else O.temperature(128, dict(coef=0.3, every=9))[meta.positions.long().cpu()][:, None, None]
        close(got, O.rms(q.double().cpu().reshape(36, hq, d), 1e-3) * qw.double().cpu() * f, TOL[dtype])
        slot = meta.slot_mapping.long()
        kp, vp = cache[:, : 16 * hkv * d].reshape(pages * 16, hkv, d), cache[:, 16 * hkv * d :].reshape(pages * 16, hkv, dv)
        close(kp[slot], O.rms(k.double().reshape(36, hkv, d), 1e-3) * kw.double(), TOL[dtype])
        assert torch.equal(vp[slot], v.reshape(36, hkv, dv)) and (cache == 7.0).sum() >= (pages * 16 - 36) * hkv * (d + dv)
    assert K().read_status(DEV) == 0


# ---- projections and experts ---------------------------------------------------------
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("t,w,m", [(1, 72, 40), (33, 50, 21), (64, 1024, 512), (700, 256, 72), (2048, 1024, 1024)])
def test_multi_dense(dtype, t, w, m):
    if dtype == torch.float32 and t > 1000:
        t = 70
    x, wt = rnd(t, 5, w, dtype=dtype).to(DEV)[:, :4], rnd(4, m, w, seed=1, dtype=dtype, gain=w ** -0.5).to(DEV)
    close(K().multi_dense(x, wt), torch.einsum("tnk,nmk->tnm", x.double(), wt.double()), TOL[dtype])


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("t,w,ff", [(1, 72, 40), (8, 1024, 2048), (64, 512, 264), (33, 50, 24), (700, 256, 512), (2048, 1024, 2048)])
def test_gelu_gated_projection(dtype, t, w, ff):
    if dtype == torch.float32 and t > 1000:
        t = 70
    x, gate, up = rnd(t, w, dtype=dtype).to(DEV), rnd(ff, w, seed=1, dtype=dtype, gain=2 * w ** -0.5).to(DEV), rnd(ff, w, seed=2, dtype=dtype, gain=w ** -0.5).to(DEV)
    inter = dtype == torch.bfloat16
    gu = torch.stack((gate, up), 1).reshape(2 * ff, w).contiguous() if inter else torch.cat((gate, up))
    for act, f in (("gelu_tanh", O.gelu), ("silu", O.silu)):
        got, want = K().dense_glu(x, gu, inter, act).double(), f(x.double() @ gate.double().T) * (x.double() @ up.double().T)
        # in bf16 gate and up are rounded before they meet, and so are the activation and the product
        assert ((got - want).abs() - (2.0 ** -6 if inter else 0) * want.abs()).max() < TOL[dtype] * want.pow(2).mean().sqrt()


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("t,w,ff,experts,top", [(1, 72, 40, 12, 3), (200, 128, 64, 4, 1), (33, 50, 16, 6, 2), (70, 264, 136, 8, 8), (300, 512, 200, 16, 4), (5, 8, 8, 1, 1)])
def test_gated_expert_rows(dtype, t, w, ff, experts, top):
    x = rnd(t, w, dtype=dtype).to(DEV)
    gu, down = rnd(experts, 2 * ff, w, seed=1, dtype=dtype, gain=1.5 * w ** -0.5).to(DEV), rnd(experts, w, ff, seed=2, dtype=dtype, gain=ff ** -0.5).to(DEV)
    ids = rnd(t, experts, seed=3).topk(top, -1).indices.int().to(DEV)
    if experts > 2 and top == 1:
        ids[ids == 2] = 0  # an expert nobody asks for
    rows, pos = K().expert_rows(x, ids, gu, down, "swiglu")
    got, xd = rows[pos.long()].view(t, top, w), x.double().cpu()
    for j in range(top):
        e = ids[:, j].long().cpu()
        g, d = gu.double().cpu()[e], down.double().cpu()[e]
        a = O.silu(torch.einsum("tfw,tw->tf", g[:, 0::2], xd)) * torch.einsum("tfw,tw->tf", g[:, 1::2], xd)
        close(got[:, j], torch.einsum("twf,tf->tw", d, a), TOL[dtype])
    assert K().read_status(DEV) == 0


@pytest.mark.parametrize("experts,top,scale", [(12, 3, 1.5), (5, 5, 1.0), (1, 1, 2.5), (64, 6, 2.5), (300, 20, 0.5)])
def test_router(experts, top, scale):
    z, c = (rnd(90, experts + 1, seed=5) * 2).to(DEV), (rnd(experts, seed=6) * 0.5).to(DEV)
    ids, w = K().router_topk(z[:, :experts], top, "sigmoid", c, 1, 1, True, scale)
    want_ids, want_w = O.route(z[:, :experts].double().cpu(), c.double().cpu(), dict(experts=experts, top=top, scale=scale))
    assert torch.equal(ids.long().cpu(), want_ids) and torch.allclose(w.double().cpu(), want_w, rtol=1e-5, atol=1e-7)


# ---- recurrence ------------------------------------------------------------------------
def wkv_inputs(lens, H, dk, dv, dtype, seed=0, w0=(-6.0, 1.5)):
    """Columns of one fused projection per sequence, raw decays in f32, and the oracle's outputs and final states."""
    n = sum(lens)
    pad = (H * max(dk, dv) + 7) // 8 * 8
    z = rnd(n, 3, pad, seed=seed, dtype=dtype)
    f, u = rnd(n, H * dk, seed=seed + 1), rnd(H, dk, seed=seed + 2)
    base = torch.linspace(*w0, H * dk)[torch.randperm(H * dk, generator=torch.Generator().manual_seed(seed))]
    r, k, v = (z[:, i, : H * d].view(n, H, d) for i, d in enumerate((dk, dk, dv)))
    want, at = [], 0
    for m in lens:
        part = slice(at, at + m)
        dec = torch.exp(-torch.exp(f[part].double() + base.double())).view(m, H, dk)
        want.append(O.recurrence(r[part].double(), k[part].double(), v[part].double(), dec, u.double()))
        at += m
    return (r.to(DEV), k.to(DEV), v.to(DEV)), f.to(DEV), base.to(DEV), u.to(DEV), torch.cat(want)


def fused(rkv, H, dk, dv):
    """The three inputs as columns of one buffer on the device (a common row stride, as the model has it)."""
    n, width = rkv[0].shape[0], (H * max(dk, dv) + 7) // 8 * 8
    z = torch.zeros(n, 3, width, dtype=rkv[0].dtype, device=DEV)
    for i, x in enumerate(rkv):
        z[:, i, : x.shape[1] * x.shape[2]] = x.reshape(n, -1)
    return tuple(z[:, i, : H * d].unflatten(1, (H, d)) for i, d in enumerate((dk, dk, dv)))


WKV_SHAPES = [(3, 24, 24), (2, 128, 128), (1, 7, 9), (2, 64, 40), (1, 136, 136), (5, 8, 8), (1, 128, 200), (1, 200, 64)]


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("H,dk,dv", WKV_SHAPES)
def test_wkv_attention(dtype, H, dk, dv):
    """Ragged sequences in shuffled slots, cut into steps in different ways; other slots stay as they are."""
    lens, slots = [70, 1, 9, 33], [3, 1, 5, 2]
    rkv, f, w0, u, want = wkv_inputs(lens, H, dk, dv, dtype)
    rkv = fused(rkv, H, dk, dv)
    first = [0, 70, 71, 80]
    for cuts in (lens, [1] * 70, [16, 16, 38], [2, 8, 7, 1, 15, 17, 20]):
        state = torch.full((6, H, dk, dv), 5.0, device=DEV)
        state[slots] = 0
        out, at = torch.zeros(sum(lens), H, dv, dtype=dtype, device=DEV), [0] * 4
        for i in range(max(len(cuts), 1)):
            if cuts is lens:
                step = list(enumerate(lens)) if i == 0 else []
            else:
                step = [(b, min(cuts[i], lens[b] - at[b])) for b in range(4) if at[b] < lens[b]]
            if not step:
                break
            idx = torch.cat([torch.arange(first[b] + at[b], first[b] + at[b] + m) for b, m in step]).to(DEV)
            meta, _ = meta_for([m for _, m in step], [m for _, m in step], slots=[slots[b] for b, _ in step])
            part = fused(tuple(x[idx] for x in rkv), H, dk, dv)
            out[idx] = K().wkv_attention(*part, f[idx], w0, u, state, meta)
            for b, m in step:
                at[b] += m
        close(out, want, TOL[dtype])
        assert state[[0, 4]].eq(5.0).all()


@pytest.mark.parametrize("dtype", TYPES)
def test_wkv_blocks_and_token_walk_leave_the_same_state(dtype):
    """A long sequence over decays from none to immediate, in blocks and token by token; a state that starts non-zero."""
    H, dk, dv, n = 2, 128, 128, 1200
    rkv, f, w0, u, want = wkv_inputs([n], H, dk, dv, dtype, seed=9, w0=(-12.0, 6.0))
    rkv = fused(rkv, H, dk, dv)
    meta, _ = meta_for([n], [n], slots=[1])
    states = []
    for blocks in (True, False):
        state = torch.zeros(2, H, dk, dv, device=DEV)
        close(K().wkv_attention(*rkv, f, w0, u, state, meta, blocks), want, TOL[dtype])
        states.append(state.clone())
        again = K().wkv_attention(*rkv, f, w0, u, state, meta, blocks)  # the same tokens once more, behind the first pass
        states.append((state.clone(), again))
    for a, b in ((states[0], states[2]), (states[1][0], states[3][0])):
        assert ((a - b).abs().max() / b.abs().max()).item() < 3e-4
    close(states[1][1], states[3][1].double(), TOL[dtype])


@pytest.mark.parametrize("strength", [-30.0, 3.0, 20.0, 100.0])
def test_wkv_extreme_decays(strength):
    """No decay at all, decays that leave nothing, and inputs whose exponential overflows."""
    H, dk, dv, n = 1, 64, 64, 50
    rkv, f, w0, u, want = wkv_inputs([n], H, dk, dv, torch.bfloat16, seed=3, w0=(strength, strength))
    rkv = fused(rkv, H, dk, dv)
    meta, _ = meta_for([n], [n], slots=[1])
    for blocks in (True, False):
        state = torch.zeros(2, H, dk, dv, device=DEV)
        close(K().wkv_attention(*rkv, f, w0, u, state, meta, blocks), want, TOL[torch.bfloat16])
        assert torch.isfinite(state).all()


# ---- attention -----------------------------------------------------------------------
class SinkCase(Case):
    """Plain rotation, a sink and a gate per head; the queries are columns of a wider row."""

    def __init__(self, geom, dtype, q_lens, kv_lens, page, seed=0, gain=1.0, sinks=None):
        super().__init__(geom, dtype, q_lens, kv_lens, page, seed, gain)
        if self.rot:
            self.cos, self.sin = pair_rope_tables(2048, self.rot, 100.0, DEV)
        self.sink = (rnd(self.heads, seed=7) * 2 + 1 if sinks is None else torch.full((self.heads,), sinks)).to(DEV)
        n, w = self.q.shape
        self.row = torch.zeros(n, (w + 7) // 8 * 8 + 16 + (self.heads + 7) // 8 * 8, dtype=dtype, device=DEV)
        self.row[:, :w] = self.q
        at = self.row.shape[1] - (self.heads + 7) // 8 * 8
        self.row[:, at:] = rnd(n, self.row.shape[1] - at, seed=8, dtype=dtype).to(DEV)
        self.gate = self.row[:, at : at + self.heads]

    def run(self, scale, *_):
        from pegainfer_b200.models.layers import LatentHeads

        w, row = LatentHeads(self.uk, self.uv, self.heads), self.row.clone()
        at = self.row.shape[1] - (self.heads + 7) // 8 * 8
        return K().latent_attention(row[:, : self.q.shape[1]], w.uk_t, w.uv, w.ukv, self.cache, self.meta, self.rot, scale, 0, self.cos, self.sin, head_gate=row[:, at : at + self.heads], sink=self.sink)

    def want(self, b, scale, window):
        h, lat, dim, rot, n = self.heads, self.lat, self.dim, self.rot, self.kv_lens[b]
        r = self.rows[b]
        k = (r[:, :lat] @ self.uk.double().cpu().T).view(n, h, dim)
        v = (r[:, :lat] @ self.uv.double().cpu().T).view(n, h, self.vdim)
        q = self.queries[b].double().view(n, h, dim + rot)
        if rot:
            k = torch.cat((k, r[:, None, lat:].expand(n, h, rot)), -1)
            q = torch.cat((q[..., :dim], O.rotate(q[..., dim:], dict(dims=rot, base=100.0))), -1)
        s = torch.einsum("qhd,khd->hqk", q, k) * scale
        s = s.masked_fill(torch.ones(n, n, dtype=torch.bool).triu(1), float("-inf"))
        s = torch.cat((s, self.sink.double().cpu().view(h, 1, 1).expand(h, n, 1)), -1)
        first = sum(self.q_lens[:b])
        gate = O.sigmoid(self.gate[first : first + self.q_lens[b]].double().cpu())
        out = torch.einsum("hqk,khd->qhd", torch.softmax(s, -1)[..., :n], v)[n - self.q_lens[b] :]
        return (out * gate[:, :, None]).reshape(self.q_lens[b], -1)


# heads, latent, dim, rot, vdim
GEOMS = [(5, 32, 16, 8, 40), (16, 512, 128, 64, 128), (20, 192, 64, 0, 96), (7, 15, 5, 0, 3), (3, 21, 10, 6, 11), (2, 640, 40, 80, 136), (1, 264, 136, 24, 8), (17, 128, 8, 16, 8)]


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("geom", GEOMS)
def test_latent_attention_with_sinks(dtype, geom):
    for q_lens, kv_lens, page in (([33, 2, 70], [33, 131, 70], 16), ([1, 1, 1, 1, 1], [1, 16, 17, 200, 65], 32), ([5, 1, 1, 1, 1, 1], [40, 1, 33, 64, 15, 90], 64)):
        SinkCase(geom, dtype, q_lens, kv_lens, page).check(0.3, 0)
    for sinks in (-30.0, 25.0, 300.0):
        SinkCase(geom, dtype, [20, 1], [50, 40], 16, sinks=sinks).check(0.3, 0)


@pytest.mark.parametrize("geom", [(16, 512, 128, 64, 128), (4, 96, 64, 16, 64), (3, 56, 24, 8, 16), (5, 64, 80, 40, 104), (2, 128, 72, 0, 8)])
def test_long_portions_with_sinks_take_the_expanded_form(geom):
    """Prompt portions beside decoded tokens: the portions run on the tcgen05 kernel, the single rows on the absorbed one."""
    for sinks in (None, 12.0, -30.0):
        case = SinkCase(geom, torch.bfloat16, [600, 130, 2, 1, 1], [600, 777, 40, 530, 64], 16, sinks=sinks)
        before = K().PREFILL_TC_CALLS["latent"]
        case.check(0.15, 0)
        assert K().PREFILL_TC_CALLS["latent"] == before + 1


def test_a_latent_past_the_instances_beside_decoded_tokens():
    SinkCase((2, 640, 40, 24, 64), torch.bfloat16, [600, 1, 1], [600, 530, 3], 16).check(0.2, 0)


def test_split_keys_with_sinks_in_decoding():
    """Few rows over many keys: the keys of a row are split over blocks, and the sink counts once where they are merged."""
    for geom in ((16, 512, 128, 64, 128), (24, 512, 128, 0, 128), (5, 120, 16, 8, 24)):
        for sinks in (None, 8.0):
            SinkCase(geom, torch.bfloat16, [1, 1, 1], [1500, 3, 1024], 16, seed=2, sinks=sinks).check(0.3, 0)


MARKS = [0, 1, 15, 16, 17, 31, 32, 63, 64, 65, 127, 128, 255, 256, 511, 512, 513, 698, 699]


@pytest.mark.parametrize("dtype,H,G,d", [(torch.bfloat16, 4, 2, 128), (torch.bfloat16, 6, 2, 40), (torch.bfloat16, 18, 1, 18), (torch.bfloat16, 20, 1, 256), (torch.float32, 6, 2, 40)])
def test_one_key_stands_out(dtype, H, G, d):
    """Every key scores 0 but one, which takes all the weight of the rows that see it: keys at the first positions, at page
    and tile borders and far back, in prompts and in decoding.  Its value is the key as projected, whose norm is 3, not 1."""
    n, page, coef, every = 700, 16, 0.5, 50
    temp = temperature_table(1024, coef, every, DEV)
    ones = torch.ones(d, device=DEV)
    for decode in (False, True):
        q_lens = [1 if decode else n] * len(MARKS)
        meta, pages = meta_for([n] * len(MARKS), [n] * len(MARKS), page, seed=4)
        cache = torch.full((pages, page * G * 2 * d), 3.0, dtype=dtype, device=DEV)
        k = rnd(len(MARKS) * n, G, d, seed=1, dtype=dtype)
        k[..., 0] = 0
        for b, j in enumerate(MARKS):
            k[b * n + j] = 0
            k[b * n + j, :, 0] = 3.0
        q = torch.zeros(len(MARKS) * n, H, d, dtype=dtype)
        q[..., 0] = 1.0
        k, q = k.to(DEV).flatten(1), q.to(DEV).flatten(1)
        z = torch.cat((q, k), 1)
        qn = K().head_norm_append(z[:, : H * d], z[:, H * d :], z[:, H * d :], ones, ones, temp, meta, cache, H, G, d, d, 1e-6)
        if decode:
            qn = qn.view(len(MARKS), n, H, d)[:, -1].contiguous()
            decode_meta, _ = meta_for(q_lens, [n] * len(MARKS), page, seed=4)
            meta = decode_meta
        got = K().capped_attention(qn, cache, G, d, meta, 40.0 / d).view(len(MARKS), -1, H, d)
        tol = 0.04 if dtype == torch.bfloat16 else 2e-3
        kd = k.double().view(len(MARKS), n, G, d)
        total = kd.cumsum(1)
        for b, j in enumerate(MARKS):
            for i in ([n - 1] if decode else sorted({j - 1, j, j + 1, n - 1} & set(range(n)))):
                want = kd[b, j] if i >= j else total[b, i] / (i + 1)
                w = 1 / (1 + i * torch.exp(-40.0 * O.temperature(i + 1, dict(coef=coef, every=every))[-1]))
                assert w > 0.999 or i < j
                assert (got[b, -1 if decode else i].double() - want.repeat_interleave(H // G, 0)).abs().max() < tol, (decode, j, i)
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


def _judge(errors, dtype):
    e = torch.cat(errors)
    assert e.max() < 2e-4 if dtype == torch.float32 else U.close_in_bf16(e), (e.max().item(), e.median().item(), e.quantile(0.8).item())


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("name", sorted(U.CONFIGS))
def test_model_through_the_executor(name, dtype):
    cfg = U.CONFIGS[name]
    W = U.weights(cfg)
    want = {r: U.truth(cfg, W, p) for r, p in PROMPTS.items()}
    rep = U.replayer(cfg, W, DEV, dtype, 384)
    for _ in range(2):  # the second round runs on pages and slots that the first one used
        for sched in SCHEDULES.values():
            _judge([U.error(got, want[r.split("#")[0]]) for r, got in U.run(rep, sched, PROMPTS).items()], dtype)
    assert rep.pool.used() == 0 and not rep.ex.model.rec.by_rid and K().read_status(DEV) == 0


@pytest.mark.parametrize("dtype", TYPES)
def test_long_prompts_and_long_decoding(dtype):
    """A prompt whose portions take the expanded form and the two-SM GEMM's sizes, decoded on over several temperature steps."""
    cfg = U.CONFIGS["wide"]
    W = U.weights(cfg, seed=1)
    prompts = {"p": U.tokens(760, 31), "q": U.tokens(100, 32)}
    want = {r: U.truth(cfg, W, p) for r, p in prompts.items()}
    for sched in ([[("p", 760)], [("q", 100)]], [[("p", 600), ("q", 1)]] + [[("p", 1), ("q", 1)]] * 99 + [[("p", 1)]] * 61, [[("p", 530), ("q", 2)], [("q", 1), ("p", 99)], [("p", 2), ("q", 96)], [("p", 129), ("q", 1)]]):
        rep = U.replayer(cfg, W, DEV, dtype, 1024)
        _judge([U.error(got, want[r]) for r, got in U.run(rep, sched, prompts).items()], dtype)
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
        assert U.error(outs[0][r], outs[1][r].double()).median() < 0.02  # the KV splits of a graph are fixed at capture


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
            slack.append(lg.max(-1).values - lg.gather(1, torch.tensor(toks)[:, None])[:, 0])  # each token is the best or as good
        slack = torch.cat(slack)
        assert slack.max() < 1e-3 if dtype == torch.float32 else slack.quantile(0.8) < 0.3, (slack.max(), slack.quantile(0.8))
    finally:
        eng.shutdown()
