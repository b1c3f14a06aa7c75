"""Nemipel decoder: a listed order of layers, each with one of three token mixers and an optional SwiGLU feed-forward.

Stream.  Every sublayer reads the residual stream itself and the norm follows the sum,
``x <- rms_norm(alpha * x + sublayer(x)) * w``; the stream stays in f32 and each norm also writes the activation-dtype
copy that the next projection reads.  A layer without feed-forward has only the first half.

Mixers.
* ``attention``: grouped-query attention with RMS norms over the whole query and key projections, rotation of
  neighbouring pairs on the first ``rot_dims`` entries of a head, a scale and a soft cap on the scores, a sigmoid gate per
  head, value size of its own.  With ``kv_from`` the layer has no keys and values: it reads the cache of an earlier layer.
* ``lightning``: linear attention with a fixed decay per head over an f32 state ``[heads, dim, vdim]``; SiLU on q, k and
  v; RMS norm over all heads of a token, sigmoid gate.
* ``channel_delta``: gated delta rule with a decay per head and key channel; short convolutions on q, k and v, unit rows,
  low-rank decay and output-gate projections; RMS norm per head, sigmoid gate.

Layout.  A layer's projections that read the stream are one weight, its parts padded to multiples of 8 rows so that every
part of the output starts on a 16-byte boundary.  Attention layers with projections of their own have a cache in a
``MixedKvBuffer``; recurrent layers have state in ``LayerStates``.  Runs on one GPU in bf16 or f32.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from .. import ops
from ..config import MixerSpec, ModelConfig
from ..loader.sources import RandomSource, WeightSource
from ..ops.reference import AttnMeta, pair_rope_tables
from ..parallel.tp import SINGLE, TPContext
from .layers import FusedProjection, HybridLayers, pad8


def nemipel_shapes(cfg: ModelConfig) -> dict:
    w = cfg.hidden_size
    s = {"embed": (cfg.vocab_size, w), "final.norm": (w,), "head": (cfg.vocab_size, w)}
    for i, L in enumerate(cfg.layer_specs):
        m, p = L.mixer, f"l{i}.mix."
        s[f"l{i}.norm1"] = (w,)
        if m.kind == "attention":
            s[p + "q"], s[p + "q.norm"], s[p + "g"] = (m.heads * m.dim, w), (m.heads * m.dim,), (m.heads, w)
            if m.kv_from < 0:
                s[p + "k"], s[p + "k.norm"], s[p + "v"] = (m.kv_heads * m.dim, w), (m.kv_heads * m.dim,), (m.kv_heads * m.vdim, w)
        elif m.kind == "lightning":
            s[p + "q"] = s[p + "k"] = (m.heads * m.dim, w)
            s[p + "v"] = s[p + "g"] = (m.heads * m.vdim, w)
            s[p + "norm"] = (m.heads * m.vdim,)
        else:
            for n, rows in (("q", m.kv_heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.heads * m.vdim)):
                s[p + n], s[p + n + ".conv"] = (rows, w), (rows, m.conv)
            s[p + "b"], s[p + "A_log"], s[p + "norm"], s[p + "dt_bias"] = (m.heads, w), (m.heads,), (m.vdim,), (m.heads * m.dim,)
            s[p + "a1"], s[p + "a2"] = (m.decay_rank, w), (m.heads * m.dim, m.decay_rank)
            s[p + "g1"], s[p + "g2"] = (m.gate_rank, w), (m.heads * m.vdim, m.gate_rank)
        s[p + "o"] = (w, m.heads * m.vdim)
        if L.ff:
            q = f"l{i}.mlp."
            s[f"l{i}.norm2"], s[q + "gate"], s[q + "up"], s[q + "down"] = (w,), (L.ff, w), (L.ff, w), (w, L.ff)
    return s


def _kind(name: str) -> str:
    if "norm" in name.rsplit(".", 1)[-1]:
        return "ones"
    if name.endswith("A_log") or name.endswith("dt_bias"):
        return "small"
    return "normal"


def nemipel_source(cfg: ModelConfig, seed: int = 0, dtype=torch.bfloat16) -> RandomSource:
    return RandomSource(nemipel_shapes(cfg), seed=seed, dtype=dtype, kind=_kind)


@dataclass
class AttentionPart:
    proj: FusedProjection
    q_norm: torch.Tensor
    k_norm: Optional[torch.Tensor]
    cos: torch.Tensor
    sin: torch.Tensor
    kv_index: int


@dataclass
class LightningPart:
    proj: FusedProjection
    decay: torch.Tensor
    norm: torch.Tensor
    state_index: int


@dataclass
class ChannelDeltaPart:
    proj: FusedProjection
    conv_cols: int  # q | k | v columns of the projection that pass the convolution (with their padding)
    conv_w: torch.Tensor
    a2: torch.Tensor
    g2: torch.Tensor
    a_log: torch.Tensor
    dt_bias: torch.Tensor
    norm: torch.Tensor
    state_index: int


@dataclass
class NemipelLayer:
    mixer: MixerSpec
    part: object
    o: torch.Tensor
    norm1: torch.Tensor
    gate_up: Optional[torch.Tensor] = None
    down: Optional[torch.Tensor] = None
    norm2: Optional[torch.Tensor] = None


class NemipelModel(HybridLayers):
    family = "nemipel"

    def __init__(self, cfg: ModelConfig, source: Optional[WeightSource] = None, device="cpu", dtype=torch.bfloat16, tp: TPContext = SINGLE, seed: int = 0):
        if tp.world != 1:
            raise ValueError("the Nemipel line runs on one GPU")
        self.cfg, self.device, self.dtype, self.tp = cfg, torch.device(device), dtype, tp
        self.kv_geometries, self.state_geometries = [], []
        self._kv_of = {}  # layer -> index of the cache it reads
        self._rope = {}
        # fused epilogue layout of the feed-forward (gate_0, up_0, gate_1, ...): bf16 kernels only
        self.interleaved = self.device.type == "cuda" and dtype == torch.bfloat16
        src = source or nemipel_source(cfg, seed=seed, dtype=dtype)
        self.embed = src.get("embed", self.device, dtype)
        self.head = src.get("head", self.device, dtype)
        self.final_norm = src.get("final.norm", self.device, torch.float32)
        self.layers = [self._load_layer(src, i) for i in range(cfg.num_layers)]

    # -- loading -----------------------------------------------------------------------
    def _rope_tables(self, m: MixerSpec):
        key = (m.rot_dims, m.rot_base)
        if key not in self._rope:
            self._rope[key] = pair_rope_tables(self.cfg.max_position, m.rot_dims, m.rot_base, self.device)
        return self._rope[key]

    def _load_layer(self, src: WeightSource, i: int) -> NemipelLayer:
        spec, dev, dt = self.cfg.layer_specs[i], self.device, self.dtype
        m, p, f32 = spec.mixer, f"l{i}.mix.", torch.float32
        mat = lambda *names: {n: src.get(p + n, dev, dt) for n in names}
        if m.kind == "attention":
            own = m.kv_from < 0
            if own:
                self._kv_of[i] = len(self.kv_geometries)
                self.kv_geometries.append((m.kv_heads, m.dim, m.vdim))
            else:
                self._kv_of[i] = self._kv_of[m.kv_from]
            cos, sin = self._rope_tables(m)
            part = AttentionPart(FusedProjection(mat("q", "k", "v", "g") if own else mat("q", "g")), src.get(p + "q.norm", dev, f32), src.get(p + "k.norm", dev, f32) if own else None, cos, sin, self._kv_of[i])
        elif m.kind == "lightning":
            part = LightningPart(FusedProjection(mat("q", "k", "v", "g")), torch.tensor(m.decay, dtype=f32, device=dev), src.get(p + "norm", dev, f32), len(self.state_geometries))
            self.state_geometries.append((m.heads, m.dim, m.vdim, 0, 0))
        elif m.kind == "channel_delta":
            proj = FusedProjection(mat("q", "k", "v", "b", "a1", "g1"))
            cols = proj.at["b"][0]
            conv = torch.zeros((cols, m.conv), dtype=f32, device=dev)
            for n in ("q", "k", "v"):
                conv[proj.at[n][0] : proj.at[n][1]] = src.get(p + n + ".conv", dev, f32)
            part = ChannelDeltaPart(proj, cols, conv, src.get(p + "a2", dev, dt), src.get(p + "g2", dev, dt), src.get(p + "A_log", dev, f32), src.get(p + "dt_bias", dev, f32),
                                    src.get(p + "norm", dev, f32), len(self.state_geometries))
            self.state_geometries.append((m.heads, m.dim, m.vdim, cols, m.conv))
        else:
            raise ValueError(f"layer {i}: no mixer of kind {m.kind!r}")
        L = NemipelLayer(m, part, src.get(p + "o", dev, dt), src.get(f"l{i}.norm1", dev, f32))
        if spec.ff:
            q = f"l{i}.mlp."
            pad = pad8(spec.ff) - spec.ff  # zero rows: their activations are zero
            g, u = (torch.nn.functional.pad(src.get(q + n, dev, dt), (0, 0, 0, pad)) for n in ("gate", "up"))
            L.gate_up = torch.stack((g, u), 1).reshape(-1, g.shape[1]).contiguous() if self.interleaved else torch.cat((g, u), 0)
            L.down = torch.nn.functional.pad(src.get(q + "down", dev, dt), (0, pad)).contiguous()
            L.norm2 = src.get(f"l{i}.norm2", dev, f32)
        return L

    # -- mixers ----------------------------------------------------------------------------
    def attention(self, L: NemipelLayer, x, meta: AttnMeta, kv):
        m, A = L.mixer, L.part
        z, cache = A.proj(x), kv.layer(A.kv_index)
        q = ops.row_norm_rope_append(z["q"], z.get("k"), z.get("v"), A.q_norm, A.k_norm, A.cos, A.sin, meta, cache, m.heads, m.kv_heads, m.dim, m.vdim, self.cfg.rms_eps)
        return ops.capped_attention(q, cache, m.kv_heads, m.vdim, meta, m.scale, m.softcap, z["g"])

    def lightning(self, L: NemipelLayer, x, meta: AttnMeta):
        m, A, t = L.mixer, L.part, x.shape[0]
        z = A.proj(x)
        q, k, v = z["q"].view(t, m.heads, m.dim), z["k"].view(t, m.heads, m.dim), z["v"].view(t, m.heads, m.vdim)
        o = ops.decay_attention(q, k, v, A.decay, self.rec.ssm[A.state_index], meta)
        return ops.gated_row_norm(o.view(t, 1, -1), z["g"], A.norm, self.cfg.rms_eps).view(t, -1)

    def channel_delta(self, L: NemipelLayer, x, meta: AttnMeta):
        m, A, t = L.mixer, L.part, x.shape[0]
        y = ops.dense(x, A.proj.w)
        z = {n: y[:, a:b] for n, (a, b) in A.proj.at.items()}
        raw = ops.dense(z["a1"], A.a2, torch.float32)
        if raw.dtype != torch.float32:
            raw = raw.float()
        gate = ops.dense(z["g1"], A.g2)
        c = ops.conv_silu(y[:, : A.conv_cols], A.conv_w, self.rec.conv[A.state_index], meta)
        part = lambda n, h, d: c[:, A.proj.at[n][0] : A.proj.at[n][1]].view(t, h, d)
        o = ops.channel_delta(part("q", m.kv_heads, m.dim), part("k", m.kv_heads, m.dim), part("v", m.heads, m.vdim), raw, z["b"], A.a_log, A.dt_bias, self.rec.ssm[A.state_index], meta)
        return ops.gated_row_norm(o, gate, A.norm, self.cfg.rms_eps).view(t, -1)

    # -- forward -----------------------------------------------------------------------------
    def forward_hidden(self, token_ids, meta: AttnMeta, kv, aux_layers=()):
        eps, alpha, dt = self.cfg.rms_eps, self.cfg.postln_alpha, self.dtype
        x, h = ops.embed_stream(token_ids, self.embed, dt)
        self.last_aux = []
        for i, L in enumerate(self.layers):
            kind = L.mixer.kind
            a = self.attention(L, h, meta, kv) if kind == "attention" else self.lightning(L, h, meta) if kind == "lightning" else self.channel_delta(L, h, meta)
            h = ops.post_norm(ops.dense(a, L.o, torch.float32), x, L.norm1, eps, alpha, dt)
            if L.gate_up is not None:
                y = ops.dense(ops.dense_glu(h, L.gate_up, self.interleaved), L.down, torch.float32)
                h = ops.post_norm(y, x, L.norm2, eps, alpha, dt)
            if i in aux_layers:
                self.last_aux.append(x.clone())
        return ops.stream_norm(x, self.final_norm, eps, dt)

    def logits(self, hidden, rows=None):
        if rows is not None:
            hidden = ops.gather_rows(hidden, rows)
        lg = ops.dense(hidden, self.head, torch.float32)
        if self.cfg.final_logit_softcapping > 0:
            lg = ops.softcap_rows(lg.float(), self.cfg.final_logit_softcapping)
        return lg

    def forward(self, token_ids, meta, kv, logits_rows=None):
        return self.logits(self.forward_hidden(token_ids, meta, kv), logits_rows)
