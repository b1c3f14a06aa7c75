"""Vekalorn decoder: a listed order of latent attention layers, each with an optional mixture of experts.

Stream.  A sublayer reads the residual stream itself and its output is normed before the sum,
``x <- x + layer_norm(sublayer(x)) * w`` (mean and variance, no bias); the stream stays in f32 and each norm also writes the
activation-dtype copy that the next projection reads.

Mixers (``MixerSpec`` of kind ``latent``).  Queries go through an RMS-normed latent of ``q_rank`` columns, keys and values are
per-head projections of an RMS-normed latent of ``kv_rank`` columns; the cache holds that latent and, in layers with
``rot_dims``, one rotated key part that all heads share.  Layers either see all positions, with rotated columns (neighbouring
pairs, YaRN frequencies) and a sigmoid gate on every output element, or the last ``window`` positions without any position
signal.

Feed-forward.  Softmax router over all experts in f32, the ``top`` best experts of the ``keep`` best groups, weighted by their
scores as they are; an expert is an up projection, the squared ReLU and a down projection.  The weighted sum of a token's
experts is formed inside the norm that follows it.

Layout.  A layer's projections of the stream (query latent, key / value latent, gate) are one weight; a layer's cache has its
own row width in a ``MixedKvBuffer``.  Everything a request owns lies in its pages, so prefixes can be shared.  Runs on one
GPU in bf16 or f32.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from .. import ops
from ..config import ExpertsSpec, MixerSpec, ModelConfig
from ..kv.buffer import MixedKvBuffer
from ..loader.sources import RandomSource, WeightSource
from ..ops.reference import AttnMeta, pair_rope_tables
from ..parallel.tp import SINGLE, TPContext
from .layers import FusedProjection, LatentHeads, pad8


def vekalorn_shapes(cfg: ModelConfig) -> dict:
    w = cfg.hidden_size
    s = {"embed": (cfg.vocab_size, w), "final.norm": (w,), "head": (cfg.vocab_size, w)}
    for i, L in enumerate(cfg.layer_specs):
        m, p = L.mixer, f"l{i}.mix."
        s[f"l{i}.norm1"] = (w,)
        s[p + "dq"], s[p + "dq.norm"], s[p + "uq"] = (m.q_rank, w), (m.q_rank,), (m.heads * (m.dim + m.rot_dims), m.q_rank)
        s[p + "dkv"], s[p + "dkv.norm"] = (m.kv_rank + m.rot_dims, w), (m.kv_rank,)
        s[p + "uk"], s[p + "uv"] = (m.heads * m.dim, m.kv_rank), (m.heads * m.vdim, m.kv_rank)
        if m.out_gate:
            s[p + "g"] = (m.heads * m.vdim, w)
        s[p + "o"] = (w, m.heads * m.vdim)
        if L.moe:
            q = f"l{i}.mlp."
            s[f"l{i}.norm2"], s[q + "router"] = (w,), (L.moe.experts, w)
            for e in range(L.moe.experts):
                s[f"{q}e{e}.up"], s[f"{q}e{e}.down"] = (L.moe.ff, w), (w, L.moe.ff)
    return s


def _kind(name: str) -> str:
    return "ones" if "norm" in name.rsplit(".", 1)[-1] else "normal"


def vekalorn_source(cfg: ModelConfig, seed: int = 0, dtype=torch.bfloat16) -> RandomSource:
    return RandomSource(vekalorn_shapes(cfg), seed=seed, dtype=dtype, kind=_kind)


@dataclass
class VekalornLayer:
    mixer: MixerSpec
    proj: FusedProjection  # query latent | key / value latent and shared key part | output gate
    q_norm: torch.Tensor
    kv_norm: torch.Tensor
    uq: torch.Tensor
    up: LatentHeads
    o: torch.Tensor
    norm1: torch.Tensor
    cos: Optional[torch.Tensor] = None
    sin: Optional[torch.Tensor] = None
    experts: Optional[ExpertsSpec] = None
    router: Optional[torch.Tensor] = None
    w_up: Optional[torch.Tensor] = None  # [experts, ff, width]
    w_down: Optional[torch.Tensor] = None  # [experts, width, ff]
    norm2: Optional[torch.Tensor] = None


class VekalornModel:
    family = "vekalorn"
    supports_prefix_cache = True
    supports_kv_offload = False  # the layers' cache rows differ in width: no one slab per block

    def __init__(self, cfg: ModelConfig, source: Optional[WeightSource] = None, device="cpu", dtype=torch.bfloat16, tp: TPContext = SINGLE, seed: int = 0):
        if tp.world != 1:
            raise ValueError("the Vekalorn line runs on one GPU")
        self.cfg, self.device, self.dtype, self.tp = cfg, torch.device(device), dtype, tp
        self._rope = {}
        src = source or vekalorn_source(cfg, seed=seed, dtype=dtype)
        self.embed = src.get("embed", self.device, dtype)
        self.head = src.get("head", self.device, dtype)
        self.final_norm = src.get("final.norm", self.device, torch.float32)
        self.layers = [self._load_layer(src, i) for i in range(cfg.num_layers)]
        # one "head" whose key is the cache row and whose value is part of it
        self.kv_geometries = [(1, l.mixer.kv_rank + l.mixer.rot_dims, 0) for l in cfg.layer_specs]

    # -- loading -----------------------------------------------------------------------
    def _rope_tables(self, m: MixerSpec):
        key = (m.rot_dims, m.rot_base, m.yarn)
        if key not in self._rope:
            self._rope[key] = pair_rope_tables(self.cfg.max_position, m.rot_dims, m.rot_base, self.device, m.yarn)
        return self._rope[key]

    def _load_layer(self, src: WeightSource, i: int) -> VekalornLayer:
        spec, dev, dt, f32 = self.cfg.layer_specs[i], self.device, self.dtype, torch.float32
        m, p = spec.mixer, f"l{i}.mix."
        if m.kind != "latent":
            raise ValueError(f"layer {i}: no mixer of kind {m.kind!r}")
        parts = {n: src.get(p + n, dev, dt) for n in (("dq", "dkv", "g") if m.out_gate else ("dq", "dkv"))}
        L = VekalornLayer(m, FusedProjection(parts), src.get(p + "dq.norm", dev, f32), src.get(p + "dkv.norm", dev, f32), src.get(p + "uq", dev, dt),
                          LatentHeads(src.get(p + "uk", dev, dt), src.get(p + "uv", dev, dt), m.heads), src.get(p + "o", dev, dt), src.get(f"l{i}.norm1", dev, f32))
        if m.rot_dims:
            L.cos, L.sin = self._rope_tables(m)
        if spec.moe:
            q, e = f"l{i}.mlp.", spec.moe
            L.experts, L.router, L.norm2 = e, src.get(q + "router", dev, dt), src.get(f"l{i}.norm2", dev, f32)
            w, ff = self.cfg.hidden_size, pad8(e.ff)  # zero rows and columns: their activations are zero
            L.w_up = torch.zeros((e.experts, ff, w), dtype=dt, device=dev)
            L.w_down = torch.zeros((e.experts, w, ff), dtype=dt, device=dev)
            for x in range(e.experts):
                L.w_up[x, : e.ff] = src.get(f"{q}e{x}.up", dev, dt)
                L.w_down[x, :, : e.ff] = src.get(f"{q}e{x}.down", dev, dt)
        return L

    # -- geometry --------------------------------------------------------------------------
    def kv_geometry(self) -> dict:
        g = self.kv_geometries
        return dict(num_layers=len(g), kv_heads=1, head_dim=max(d for _, d, _ in g), split_plan=False, bytes_per_block=lambda page: MixedKvBuffer.bytes_per_block(g, page, self.dtype))

    def make_kv(self, num_pages: int, page_size: int) -> MixedKvBuffer:
        return MixedKvBuffer(self.kv_geometries, num_pages, page_size, self.dtype, self.device)

    # -- sublayers -------------------------------------------------------------------------
    def attention(self, L: VekalornLayer, x, meta: AttnMeta, cache):
        m = L.mixer
        z = L.proj(x)
        cq = ops.latent_rows(z["dq"], z["dkv"], L.q_norm, L.kv_norm, L.cos, L.sin, meta, cache, m.kv_rank, self.cfg.rms_eps)
        return ops.latent_attention(ops.dense(cq, L.uq), L.up.uk_t, L.up.uv, L.up.ukv, cache, meta, m.rot_dims, m.scale, m.window, L.cos, L.sin, z.get("g"))

    def route(self, L: VekalornLayer, x):
        e = L.experts
        # a shape the two-SM GEMM serves would come back in bf16 from `dense`; the router keeps its 32 bits
        logits = ops.dense(x, L.router, torch.float32) if x.dtype == torch.float32 or x.shape[1] % 8 else ops.linear(x, L.router, out_dtype=torch.float32)
        return ops.router_topk(logits, e.top, "softmax", None, e.groups, e.keep, group_top=1)

    # -- forward -----------------------------------------------------------------------------
    def forward_hidden(self, token_ids, meta: AttnMeta, kv, aux_layers=()):
        eps, dt = self.cfg.rms_eps, self.dtype
        x, h = ops.embed_stream(token_ids, self.embed, dt)
        self.last_aux = []
        for i, L in enumerate(self.layers):
            a = self.attention(L, h, meta, kv.layer(i))
            h = ops.add_layer_norm(ops.dense(a, L.o, torch.float32), x, L.norm1, eps, dt)
            if L.experts is not None:
                ids, wts = self.route(L, h)
                rows, pos = ops.expert_rows(h, ids, L.w_up, L.w_down, "relu2")
                h = ops.add_layer_norm_rows(rows, pos, wts, x, L.norm2, eps, dt)
            if i in aux_layers:
                self.last_aux.append(x.clone())
        return ops.stream_layer_norm(x, self.final_norm, eps, dt)

    def logits(self, hidden, rows=None):
        if rows is not None:
            hidden = ops.gather_rows(hidden, rows)
        return ops.dense(hidden, self.head, torch.float32)

    def forward(self, token_ids, meta, kv, logits_rows=None):
        return self.logits(self.forward_hidden(token_ids, meta, kv), logits_rows)
