"""Nonetar decoder: a listed order of layers over several copies of the residual stream, each with one of two token mixers and
an optional feed-forward.

Streams.  Token rows plus the sinusoids of their positions start every copy.  A sublayer reads the RMS norm (weight stored about
zero) of a learned sum of the copies; every copy then becomes a learned sum of all the old ones and of the sublayer's output.
The copies stay in f32; one kernel forms the new copies, the next sublayer's input, its norm and, in front of a mixer, the token
shift: a learned step of every channel towards the previous token's normed row, which is part of a request's state.  The last
norm reads the sum of the copies; the factor on the logits is part of its weight.

Mixers.
* ``parallel``: grouped-query attention and a recurrent block side by side.  Attention: biased projections, per-head query and
  key norms, a factor per head on the scores (part of the query norm's weight), soft cap, a bias that grows with the distance,
  sliding window.  Recurrent block: a linear recurrence per channel whose gates are block-diagonal projections of a short
  convolution's output, times a GELU branch.  Each one's factor is applied where its output is rounded; both share one output
  projection over their columns side by side.
* ``ssd``: Mamba-2's state-space duality, one decay per token and head; a gate in front of an RMS norm in parts.

Feed-forward: up projection, xIELU, down projection.

Layout.  A layer's projections of the same rows are one weight.  Attention has a cache in a ``MixedKvBuffer``; recurrent states,
convolution inputs and the carried rows are in ``LayerStates``.  Runs on one GPU in bf16 or f32.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from .. import ops
from ..config import MixerSpec, ModelConfig
from ..loader.sources import RandomSource, WeightSource
from ..ops.reference import AttnMeta, StreamMix, position_tables
from ..parallel.tp import SINGLE, TPContext
from .layers import FusedProjection, HybridLayers, pad8


def nonetar_shapes(cfg: ModelConfig) -> dict:
    w, n = cfg.hidden_size, cfg.streams
    s = {"embed": (cfg.vocab_size, w), "final.norm": (w,), "head": (cfg.vocab_size, w)}
    for i, L in enumerate(cfg.layer_specs):
        p = f"l{i}."
        s[p + "norm1"], s[p + "shift"] = (w,), (w,)
        if L.mixer.kind == "parallel":
            (a, r), q, t = L.mixer.parts, p + "mix.left.", p + "mix.right."
            for x, rows in (("q", a.heads * a.dim), ("k", a.kv_heads * a.dim), ("v", a.kv_heads * a.vdim)):
                s[q + x], s[q + x + ".b"] = (rows, w), (rows,)
            s[q + "q.norm"], s[q + "k.norm"], s[q + "temp"], s[q + "o"] = (a.dim,), (a.dim,), (a.heads,), (w, a.heads * a.vdim)
            c = r.heads * r.dim
            for x in ("y", "x"):
                s[t + x], s[t + x + ".b"] = (c, w), (c,)
            for x in ("ra", "ri"):
                s[t + x], s[t + x + ".b"] = (r.heads, r.dim, r.dim), (r.heads, r.dim)
            s[t + "conv"], s[t + "conv.b"], s[t + "lam"], s[t + "o"] = (c, r.conv), (c,), (c,), (w, c)
        else:
            m, q = L.mixer, p + "mix."
            inner, c = m.heads * m.vdim, m.heads * m.vdim + 2 * m.kv_heads * m.dim
            s[q + "in"], s[q + "conv"], s[q + "conv.b"], s[q + "o"], s[q + "norm"] = (inner + c + m.heads, w), (c, m.conv), (c,), (w, inner), (inner,)
            s[q + "dt_bias"] = s[q + "A_log"] = s[q + "D"] = (m.heads,)
        subs = ["hc1."]
        if L.ff:
            s[p + "norm2"], s[p + "mlp.up"], s[p + "mlp.down"], s[p + "mlp.act"] = (w,), (L.ff, w), (w, L.ff), (2,)
            subs.append("hc2.")
        for x in subs:
            s[p + x + "in"] = s[p + x + "out"] = (n,)
            s[p + x + "mix"] = (n, n)
    return s


def _kind(name: str) -> str:
    last = name.rsplit(".", 1)[-1]
    if name.endswith((".q.norm", ".k.norm", "mix.norm", ".temp", ".D", ".lam")) or ".hc" in name:
        return "const:0.25" if last == "mix" or last == "in" else "ones"
    return "small" if last in ("norm1", "norm2", "norm", "shift", "b", "dt_bias", "A_log", "act") else "normal"


def nonetar_source(cfg: ModelConfig, seed: int = 0, dtype=torch.bfloat16) -> RandomSource:
    return RandomSource(nonetar_shapes(cfg), seed=seed, dtype=dtype, kind=_kind)


@dataclass
class ParallelPart:
    proj: FusedProjection  # queries | keys | values | GELU branch | recurrent branch
    qkv_bias: tuple
    q_norm: torch.Tensor  # [heads, dim], with the factor per head
    k_norm: torch.Tensor
    slopes: torch.Tensor
    y_bias: torch.Tensor
    x_bias: torch.Tensor
    conv_w: torch.Tensor
    conv_b: torch.Tensor
    gates: torch.Tensor  # [blocks, 2 dim, dim]: a block's two gate matrices
    gate_bias: torch.Tensor
    lam: torch.Tensor
    kv_index: int
    state_index: int


@dataclass
class SsdPart:
    proj: FusedProjection  # gate | convolved columns | step sizes
    conv_w: torch.Tensor
    conv_b: torch.Tensor
    dt_bias: torch.Tensor
    a_log: torch.Tensor
    d: torch.Tensor
    norm: torch.Tensor
    state_index: int


@dataclass
class Feed:
    up: torch.Tensor
    down: torch.Tensor
    act: torch.Tensor  # the activation's two constants as it uses them


@dataclass
class NonetarLayer:
    mixer: MixerSpec
    part: object
    o: torch.Tensor
    norm1: torch.Tensor
    shift: torch.Tensor
    row_index: int  # state that carries the previous token's normed row
    norm2: Optional[torch.Tensor] = None
    ff: Optional[Feed] = None


class NonetarModel(HybridLayers):
    family = "nonetar"

    def __init__(self, cfg: ModelConfig, source: Optional[WeightSource] = None, device="cpu", dtype=torch.bfloat16, tp: TPContext = SINGLE, seed: int = 0):
        if tp.world != 1:
            raise ValueError("the Nonetar line runs on one GPU")
        self.cfg, self.device, self.dtype, self.tp = cfg, torch.device(device), dtype, tp
        self.kv_geometries, self.state_geometries = [], []
        src = source or nonetar_source(cfg, seed=seed, dtype=dtype)
        f32 = lambda n: src.get(n, self.device, torch.float32)
        self.embed = src.get("embed", self.device, dtype)
        self.positions = position_tables(cfg.max_position, cfg.hidden_size, self.device)
        self.head = src.get("head", self.device, dtype)
        self.layers = [self._load_layer(src, i) for i in range(cfg.num_layers)]
        # coefficients in front of every sublayer and of the final norm; the first sublayer has one copy, the embedding
        subs = [f"l{i}.{q}." for i, L in enumerate(self.layers) for q in (("hc1", "hc2") if L.ff else ("hc1",))]
        one = torch.ones(1, dtype=torch.float32, device=self.device)
        gathers = [f32(q + "in") for q in subs] + [one.expand(cfg.streams)]
        self.mixes = [StreamMix(one.view(1, 1), one, gathers[0].sum().view(1))]
        for n, q in enumerate(subs):
            mix = f32(q + "mix")
            self.mixes.append(StreamMix(mix if n else mix.sum(0, keepdim=True), f32(q + "out"), gathers[n + 1]))
        self.final_norm = (1 + f32("final.norm")) * cfg.logit_scale

    # -- loading -----------------------------------------------------------------------
    def _state(self, *geometry) -> int:
        self.state_geometries.append(geometry)
        return len(self.state_geometries) - 1

    def _parallel(self, src: WeightSource, p: str, m: MixerSpec):
        (a, r), dev, dt = m.parts, self.device, self.dtype
        q, t = p + "left.", p + "right."
        vec = lambda n: src.get(n, dev, torch.float32)
        mats = {n: src.get(q + n, dev, dt) for n in ("q", "k", "v")}
        mats.update({n: src.get(t + n, dev, dt) for n in ("y", "x")})
        gates = torch.cat((src.get(t + "ra", dev, dt), src.get(t + "ri", dev, dt)), 1).contiguous()
        gate_bias = torch.cat((vec(t + "ra.b"), vec(t + "ri.b")), 1).contiguous()
        c = r.heads * r.dim
        part = ParallelPart(FusedProjection(mats), tuple(vec(q + n + ".b") for n in ("q", "k", "v")), (vec(q + "temp")[:, None] * vec(q + "q.norm")).contiguous(), vec(q + "k.norm"),
                            torch.tensor(a.slopes, dtype=torch.float32, device=dev), vec(t + "y.b"), vec(t + "x.b"), vec(t + "conv"), vec(t + "conv.b"), gates, gate_bias, vec(t + "lam"),
                            len(self.kv_geometries), self._state(1, 1, c, c, r.conv))
        self.kv_geometries.append((a.kv_heads, a.dim, a.vdim))
        o = torch.cat((src.get(q + "o", dev, dt), src.get(t + "o", dev, dt)), 1)
        return part, torch.nn.functional.pad(o, (0, pad8(o.shape[1]) - o.shape[1])).contiguous()

    def _ssd(self, src: WeightSource, p: str, m: MixerSpec):
        dev, dt, inner, cols = self.device, self.dtype, m.heads * m.vdim, m.heads * m.vdim + 2 * m.kv_heads * m.dim
        vec = lambda n: src.get(p + n, dev, torch.float32)
        z, c, d = src.get(p + "in", dev, dt).split((inner, cols, m.heads), 0)
        part = SsdPart(FusedProjection({"z": z, "c": c, "dt": d}), vec("conv"), vec("conv.b"), vec("dt_bias"), vec("A_log"), vec("D"), vec("norm"), self._state(m.heads, m.dim, m.vdim, cols, m.conv))
        return part, src.get(p + "o", dev, dt)

    def _load_layer(self, src: WeightSource, i: int) -> NonetarLayer:
        spec, dev, p = self.cfg.layer_specs[i], self.device, f"l{i}."
        m = spec.mixer
        if m.kind not in ("parallel", "ssd"):
            raise ValueError(f"layer {i}: no mixer of kind {m.kind!r}")
        vec = lambda n: src.get(p + n, dev, torch.float32)
        part, o = (self._parallel if m.kind == "parallel" else self._ssd)(src, p + "mix.", m)
        L = NonetarLayer(m, part, o, 1 + vec("norm1"), vec("shift"), self._state(1, 1, self.cfg.hidden_size, 0, 0))
        if spec.ff:
            pad = pad8(spec.ff) - spec.ff  # zero rows: their activations are zero
            up, down = src.get(p + "mlp.up", dev, self.dtype), src.get(p + "mlp.down", dev, self.dtype)
            L.ff = Feed(torch.nn.functional.pad(up, (0, 0, 0, pad)).contiguous(), torch.nn.functional.pad(down, (0, pad)).contiguous(),
                        torch.nn.functional.softplus(vec("mlp.act")) + torch.tensor([0.0, 0.5], device=dev))
            L.norm2 = 1 + vec("norm2")
        return L

    # -- mixers ----------------------------------------------------------------------------
    def parallel(self, L: NonetarLayer, h, meta: AttnMeta, kv):
        (a, r), A, t = L.mixer.parts, L.part, h.shape[0]
        sa, sr = L.mixer.part_scales
        z, cache = A.proj(h), kv.layer(A.kv_index)
        cut, cols = a.heads * a.vdim, a.heads * a.vdim + r.heads * r.dim
        both = (torch.empty if cols == L.o.shape[1] else torch.zeros)((t, L.o.shape[1]), dtype=h.dtype, device=h.device)
        q = ops.head_norm_append(z["q"], z["k"], z["v"], A.q_norm, A.k_norm, None, meta, cache, a.heads, a.kv_heads, a.dim, a.vdim, self.cfg.rms_eps, bias=A.qkv_bias)
        ops.capped_attention(q, cache, a.kv_heads, a.vdim, meta, a.scale, a.softcap, window=a.window, slopes=A.slopes, out_scale=sa, out=both[:, :cut])
        u = ops.short_conv(z["x"], A.conv_w, A.conv_b, self.rec.conv[A.state_index], meta, act="none", in_bias=A.x_bias)
        gates = ops.multi_dense(u.view(t, r.heads, r.dim), A.gates, torch.float32)
        ops.gated_lru(gates, A.gate_bias, u, A.lam, z["y"], A.y_bias, self.rec.ssm[A.state_index], meta, scale=sr, out=both[:, cut:cols])
        return both

    def ssd(self, L: NonetarLayer, h, meta: AttnMeta):
        m, A, t = L.mixer, L.part, h.shape[0]
        z, inner, gn = A.proj(h), m.heads * m.vdim, m.kv_heads * m.dim
        c = ops.short_conv(z["c"], A.conv_w, A.conv_b, self.rec.conv[A.state_index], meta)
        x, B, C = c[:, :inner].unflatten(1, (m.heads, m.vdim)), c[:, inner : inner + gn].unflatten(1, (m.kv_heads, m.dim)), c[:, inner + gn :].unflatten(1, (m.kv_heads, m.dim))
        y = ops.ssd_attention(x, B, C, z["dt"], A.dt_bias, A.a_log, A.d, self.rec.ssm[A.state_index], meta)
        return ops.gated_row_norm(y.view(t, m.norm_groups, -1), z["z"], A.norm, self.cfg.rms_eps, "silu", gate_first=True).view(t, -1)

    # -- forward -----------------------------------------------------------------------------
    def forward_hidden(self, token_ids, meta: AttnMeta, kv, aux_layers=()):
        eps, dt = self.cfg.rms_eps, self.dtype
        x = ops.embed_positions(token_ids, self.embed, self.positions, meta).unsqueeze(1)
        # every sublayer: the copies take in the output of the one before, and its input comes out of the same kernel
        y, step = None, iter(self.mixes)
        self.last_aux = []
        for i, L in enumerate(self.layers):
            x, h = ops.streams_norm(x, y, next(step), L.norm1, eps, dt, shift=L.shift, carried=self.rec.ssm[L.row_index], meta=meta)
            if i - 1 in aux_layers:
                self.last_aux.append(x.sum(1))
            y = ops.dense(self.parallel(L, h, meta, kv) if L.mixer.kind == "parallel" else self.ssd(L, h, meta), L.o, torch.float32)
            if L.ff is not None:
                x, h = ops.streams_norm(x, y, next(step), L.norm2, eps, dt)
                y = ops.dense(ops.dense_xielu(h, L.ff.up, L.ff.act), L.ff.down, torch.float32)
        last = len(self.layers) - 1 in aux_layers
        x, h = ops.streams_norm(x, y, next(step), self.final_norm, eps, dt, keep=last)
        if last:
            self.last_aux.append(x.sum(1))
        return h

    def logits(self, hidden, rows=None):
        if rows is not None:
            hidden = ops.gather_rows(hidden, rows)
        return ops.dense(hidden, self.head, torch.float32)

    def forward(self, token_ids, meta, kv, logits_rows=None):
        return self.logits(self.forward_hidden(token_ids, meta, kv), logits_rows)
