"""Zeripel decoder: a listed order of layers, each with one of three token mixers and an optional feed-forward.

Stream.  Scaled token rows plus the row of the pair (previous token, token); a sublayer reads the RMS norm of the stream and a
constant times its output is added to it.  The stream stays in f32; each sum also forms the next sublayer's normed input.

Mixers.
* ``wkv``: linear attention over an f32 state ``[heads, dim, dim]`` with a decay per token and key channel (two low-rank
  projections) and a bonus for the current token; every projection reads its own mix of a token's row with the previous one's;
  RMS norm per head, SiLU gate.
* ``attention``: grouped-query attention without positions whose values are the projected keys; per-head query and key norms,
  a query temperature that grows with the position's logarithm.
* ``latent``: queries straight from the stream, keys and values as per-head projections of a cached RMS-normed latent, a
  rotated key part shared by the heads, a sink per head in the softmax and a sigmoid gate per head.  With ``kv_from`` the layer
  has no latent: it reads the cache of an earlier layer through its own up-projections.

Feed-forward: a gated one with tanh-GELU, or a mixture of SiLU experts behind a sigmoid router whose choice a learned
correction shifts, with an expert that runs for every token behind a gate of its own.

Layout.  A layer's projections of the normed stream are one weight; the four large projections of a ``wkv`` layer, whose inputs
differ, are one batched product.  Attention and latent layers with projections of their own have a cache in a
``MixedKvBuffer``; ``wkv`` layers have a state and the previous row in ``LayerStates``, which also keeps each request's
previous token.  Runs on one GPU in bf16 or f32.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from .. import ops
from ..config import ExpertsSpec, MixerSpec, ModelConfig
from ..loader.sources import RandomSource, WeightSource
from ..ops.reference import AttnMeta, pair_rope_tables, temperature_table
from ..parallel.tp import SINGLE, TPContext
from .layers import FusedProjection, HybridLayers, LatentHeads, pad8

MIXES = ("r", "k", "v", "g", "w")  # inputs of a wkv layer's projections, the low-rank decay last


def zeripel_shapes(cfg: ModelConfig) -> dict:
    w = cfg.hidden_size
    s = {"embed": (cfg.vocab_size, w), "final.norm": (w,), "head": (cfg.vocab_size, w)}
    if cfg.bigram:
        s["bigram"] = (cfg.bigram[0] + 1, w)
    for i, L in enumerate(cfg.layer_specs):
        m, p, inner = L.mixer, f"l{i}.mix.", L.mixer.heads * L.mixer.vdim
        s[f"l{i}.norm1"], s[p + "o"] = (w,), (w, inner)
        if m.kind == "wkv":
            for n in MIXES:
                s[p + "mu." + n] = (w,)
            for n in MIXES[:4]:
                s[p + n] = (inner, w)
            s[p + "w1"], s[p + "w2"], s[p + "w0"], s[p + "u"], s[p + "norm"] = (m.decay_rank, w), (inner, m.decay_rank), (inner,), (m.heads, m.dim), (inner,)
        elif m.kind == "attention":
            s[p + "q"], s[p + "k"], s[p + "q.norm"], s[p + "k.norm"] = (m.heads * m.dim, w), (m.kv_heads * m.dim, w), (m.dim,), (m.dim,)
        else:
            s[p + "q"], s[p + "uk"], s[p + "uv"] = (m.heads * (m.dim + m.rot_dims), w), (m.heads * m.dim, m.kv_rank), (inner, m.kv_rank)
            s[p + "sink"], s[p + "g"] = (m.heads,), (m.heads, w)
            if m.kv_from < 0:
                s[p + "dkv"], s[p + "dkv.norm"] = (m.kv_rank + m.rot_dims, w), (m.kv_rank,)
        q, e = f"l{i}.mlp.", L.moe
        glu = lambda name, ff: s.update({name + "gate": (ff, w), name + "up": (ff, w), name + "down": (w, ff)})
        if L.ff or e:
            s[f"l{i}.norm2"] = (w,)
        if e:
            s[q + "router"], s[q + "correction"] = (e.experts, w), (e.experts,)
            for x in range(e.experts):
                glu(f"{q}e{x}.", e.ff)
            if e.shared_ff:
                glu(q + "shared.", e.shared_ff)
                s[q + "shared.sg"] = (1, w)
        elif L.ff:
            glu(q, L.ff)
    return s


def _kind(name: str) -> str:
    return "ones" if "norm" in name.rsplit(".", 1)[-1] else "small" if name.endswith(("sink", "correction", ".u", "w0")) or ".mu." in name else "normal"


def zeripel_source(cfg: ModelConfig, seed: int = 0, dtype=torch.bfloat16) -> RandomSource:
    return RandomSource(zeripel_shapes(cfg), seed=seed, dtype=dtype, kind=_kind)


@dataclass
class WkvPart:
    mu: torch.Tensor  # f32 [5, width], in the order of MIXES
    proj: torch.Tensor  # [4, heads * dim, width]
    w1: torch.Tensor
    w2: torch.Tensor
    w0: torch.Tensor
    u: torch.Tensor
    norm: torch.Tensor
    state_index: int


@dataclass
class AttentionPart:
    proj: FusedProjection  # queries | keys, which are the values too
    q_norm: torch.Tensor
    k_norm: torch.Tensor
    temp: Optional[torch.Tensor]
    kv_index: int


@dataclass
class LatentPart:
    proj: FusedProjection  # queries | latent and shared key part, where the layer has its own | head gate
    kv_norm: Optional[torch.Tensor]
    up: LatentHeads
    sink: torch.Tensor
    cos: torch.Tensor
    sin: torch.Tensor
    kv_index: int


@dataclass
class GatedFF:
    gate_up: torch.Tensor
    down: torch.Tensor


@dataclass
class MoePart:
    spec: ExpertsSpec
    router: torch.Tensor  # [experts (+ 1), width]: the last row is the shared expert's gate
    correction: torch.Tensor
    gate_up: torch.Tensor  # [experts, 2 ff, width], rows (gate_0, up_0, gate_1, ...)
    down: torch.Tensor
    shared: Optional[GatedFF]


@dataclass
class ZeripelLayer:
    mixer: MixerSpec
    part: object
    o: torch.Tensor
    norm1: torch.Tensor
    norm2: Optional[torch.Tensor] = None
    ff: Optional[GatedFF] = None
    act: str = "silu"
    moe: Optional[MoePart] = None


class ZeripelModel(HybridLayers):
    family = "zeripel"
    carries_token = True

    def __init__(self, cfg: ModelConfig, source: Optional[WeightSource] = None, device="cpu", dtype=torch.bfloat16, tp: TPContext = SINGLE, seed: int = 0):
        if tp.world != 1:
            raise ValueError("the Zeripel line runs on one GPU")
        self.cfg, self.device, self.dtype, self.tp = cfg, torch.device(device), dtype, tp
        self.kv_geometries, self.state_geometries = [], []
        self._kv_of, self._tables = {}, {}  # layer -> index of the cache it reads
        # fused epilogue layout of the gated feed-forwards (gate_0, up_0, gate_1, ...): bf16 kernels only
        self.interleaved = self.device.type == "cuda" and dtype == torch.bfloat16
        src = source or zeripel_source(cfg, seed=seed, dtype=dtype)
        self.embed = src.get("embed", self.device, dtype)
        self.pairs = src.get("bigram", self.device, dtype) if cfg.bigram else None
        self.head = src.get("head", self.device, dtype)
        self.final_norm = src.get("final.norm", self.device, torch.float32)
        self.layers = [self._load_layer(src, i) for i in range(cfg.num_layers)]

    # -- loading -----------------------------------------------------------------------
    def _table(self, *key):
        """Position tables, one per set of constants: (dims, base) rotation, (coef, every, "temp") query temperature."""
        if key not in self._tables:
            n = self.cfg.max_position
            self._tables[key] = temperature_table(n, key[0], key[1], self.device) if key[-1] == "temp" else pair_rope_tables(n, key[0], key[1], self.device)
        return self._tables[key]

    def _own_cache(self, i: int, geometry: tuple) -> int:
        self._kv_of[i] = len(self.kv_geometries)
        self.kv_geometries.append(geometry)
        return self._kv_of[i]

    def _mixer(self, src: WeightSource, i: int):
        m, p, dev, dt, f32 = self.cfg.layer_specs[i].mixer, f"l{i}.mix.", self.device, self.dtype, torch.float32
        mat = lambda *names: {n: src.get(p + n, dev, dt) for n in names}
        vec = lambda n: src.get(p + n, dev, f32)
        if m.kind == "wkv":
            part = WkvPart(torch.stack([vec("mu." + n) for n in MIXES]), torch.stack(list(mat(*MIXES[:4]).values())), src.get(p + "w1", dev, dt), src.get(p + "w2", dev, dt), vec("w0"), vec("u"),
                           vec("norm"), len(self.state_geometries))
            self.state_geometries.append((m.heads, m.dim, m.vdim, self.cfg.hidden_size, 2))
            return part
        if m.kind == "attention":
            temp = self._table(*m.q_temp, "temp") if m.q_temp else None
            return AttentionPart(FusedProjection(mat("q", "k")), vec("q.norm"), vec("k.norm"), temp, self._own_cache(i, (m.kv_heads, m.dim, m.vdim)))
        if m.kind == "latent":
            own = m.kv_from < 0
            # one "head" whose key is the cache row and whose value is part of it
            index = self._own_cache(i, (1, m.kv_rank + m.rot_dims, 0)) if own else self._kv_of[m.kv_from]
            cos, sin = self._table(m.rot_dims, m.rot_base) if m.rot_dims else (None, None)
            return LatentPart(FusedProjection(mat("q", "dkv", "g") if own else mat("q", "g")), vec("dkv.norm") if own else None, LatentHeads(src.get(p + "uk", dev, dt), src.get(p + "uv", dev, dt), m.heads),
                              vec("sink"), cos, sin, index)
        raise ValueError(f"layer {i}: no mixer of kind {m.kind!r}")

    def _glu(self, src: WeightSource, p: str, ff: int, interleaved: bool) -> GatedFF:
        pad = pad8(ff) - ff  # zero rows: their activations are zero
        g, u = (torch.nn.functional.pad(src.get(p + n, self.device, self.dtype), (0, 0, 0, pad)) for n in ("gate", "up"))
        gu = torch.stack((g, u), 1).reshape(-1, g.shape[1]).contiguous() if interleaved else torch.cat((g, u), 0)
        return GatedFF(gu, torch.nn.functional.pad(src.get(p + "down", self.device, self.dtype), (0, pad)).contiguous())

    def _moe(self, src: WeightSource, p: str, e: ExpertsSpec) -> MoePart:
        dev, dt, w, ff = self.device, self.dtype, self.cfg.hidden_size, pad8(e.ff)
        router = src.get(p + "router", dev, dt)
        shared = self._glu(src, p + "shared.", e.shared_ff, self.interleaved) if e.shared_ff else None
        if shared:
            router = torch.cat((router, src.get(p + "shared.sg", dev, dt)), 0).contiguous()
        gate_up, down = torch.empty((e.experts, 2 * ff, w), dtype=dt, device=dev), torch.empty((e.experts, w, ff), dtype=dt, device=dev)
        for x in range(e.experts):
            one = self._glu(src, f"{p}e{x}.", e.ff, True)
            gate_up[x], down[x] = one.gate_up, one.down
        return MoePart(e, router, src.get(p + "correction", dev, torch.float32), gate_up, down, shared)

    def _load_layer(self, src: WeightSource, i: int) -> ZeripelLayer:
        spec, dev, f32 = self.cfg.layer_specs[i], self.device, torch.float32
        L = ZeripelLayer(spec.mixer, self._mixer(src, i), src.get(f"l{i}.mix.o", dev, self.dtype), src.get(f"l{i}.norm1", dev, f32), act=spec.act)
        if spec.moe:
            L.moe = self._moe(src, f"l{i}.mlp.", spec.moe)
        elif spec.ff:
            L.ff = self._glu(src, f"l{i}.mlp.", spec.ff, self.interleaved)
        if spec.moe or spec.ff:
            L.norm2 = src.get(f"l{i}.norm2", dev, f32)
        return L

    # -- mixers ----------------------------------------------------------------------------
    def wkv(self, L: ZeripelLayer, h, meta: AttnMeta):
        m, A, t = L.mixer, L.part, h.shape[0]
        mix = ops.token_mix(h, A.mu, self.rec.conv[A.state_index], meta)
        z = ops.multi_dense(mix[:, :4], A.proj)
        low = ops.tanh_rows(ops.dense(mix[:, 4], A.w1))
        f = self._f32(low, A.w2)
        r, k, v = (z[:, n].view(t, m.heads, m.dim) for n in range(3))
        o = ops.wkv_attention(r, k, v, f, A.w0, A.u, self.rec.ssm[A.state_index], meta)
        return ops.gated_row_norm(o, z[:, 3], A.norm, self.cfg.rms_eps, "silu").view(t, -1)

    def attention(self, L: ZeripelLayer, h, meta: AttnMeta, kv):
        m, A = L.mixer, L.part
        z, cache = A.proj(h), kv.layer(A.kv_index)
        q = ops.head_norm_append(z["q"], z["k"], z["k"], A.q_norm, A.k_norm, A.temp, meta, cache, m.heads, m.kv_heads, m.dim, m.vdim, self.cfg.rms_eps)
        return ops.capped_attention(q, cache, m.kv_heads, m.vdim, meta, m.scale)

    def latent(self, L: ZeripelLayer, h, meta: AttnMeta, kv):
        m, A = L.mixer, L.part
        z, cache = A.proj(h), kv.layer(A.kv_index)
        if A.kv_norm is not None:
            ops.latent_rows(None, z["dkv"], None, A.kv_norm, A.cos, A.sin, meta, cache, m.kv_rank, self.cfg.rms_eps)
        return ops.latent_attention(z["q"], A.up.uk_t, A.up.uv, A.up.ukv, cache, meta, m.rot_dims, m.scale, 0, A.cos, A.sin, head_gate=z["g"], sink=A.sink)

    def mixer(self, L: ZeripelLayer, h, meta: AttnMeta, kv):
        kind = L.mixer.kind
        return self.wkv(L, h, meta) if kind == "wkv" else self.attention(L, h, meta, kv) if kind == "attention" else self.latent(L, h, meta, kv)

    # -- feed-forward ------------------------------------------------------------------------
    @staticmethod
    def _f32(x, w):
        """Projection with an f32 result at every size: `dense` hands back bf16 where the two-SM GEMM serves."""
        return ops.dense(x, w, torch.float32) if x.dtype == torch.float32 or x.shape[1] % 8 else ops.linear(x, w, out_dtype=torch.float32)

    def gated(self, x, F: GatedFF, act: str = "silu"):
        return ops.dense(ops.dense_glu(x, F.gate_up, self.interleaved, act), F.down, torch.float32)

    def experts(self, M: MoePart, h, x, w):
        e, cfg = M.spec, self.cfg
        z = self._f32(h, M.router)
        ids, wts = ops.router_topk(z[:, : e.experts], e.top, e.scoring, M.correction, 1, 1, e.norm, e.scale)
        rows, pos = ops.expert_rows(h, ids, M.gate_up, M.down, e.act)
        shared, gate = (self.gated(h, M.shared), z[:, e.experts :]) if M.shared else (None, None)
        return ops.residual_norm_rows(rows, pos, wts, shared, gate, x, w, cfg.rms_eps, cfg.residual_mult, self.dtype)

    # -- forward -----------------------------------------------------------------------------
    def forward_hidden(self, token_ids, meta: AttnMeta, kv, aux_layers=()):
        cfg, dt = self.cfg, self.dtype
        eps, mult = cfg.rms_eps, cfg.residual_mult
        x, h = ops.embed_pairs_norm(token_ids, self.embed, self.pairs, cfg.embed_scale, cfg.bigram, self.rec.token, self.layers[0].norm1, eps, meta, dt)
        self.last_aux = []
        for i, L in enumerate(self.layers):
            after = self.layers[i + 1].norm1 if i + 1 < len(self.layers) else self.final_norm
            y = ops.dense(self.mixer(L, h, meta, kv), L.o, torch.float32)
            h = ops.residual_norm(y, x, after if L.norm2 is None else L.norm2, eps, mult, dt)
            if L.moe is not None:
                h = self.experts(L.moe, h, x, after)
            elif L.ff is not None:
                h = ops.residual_norm(self.gated(h, L.ff, L.act), x, after, eps, mult, dt)
            if i in aux_layers:
                self.last_aux.append(x.clone())
        return h

    def logits(self, hidden, rows=None):
        if rows is not None:
            hidden = ops.gather_rows(hidden, rows)
        return ops.dense(hidden, self.head, torch.float32)

    def forward(self, token_ids, meta, kv, logits_rows=None):
        return self.logits(self.forward_hidden(token_ids, meta, kv), logits_rows)
