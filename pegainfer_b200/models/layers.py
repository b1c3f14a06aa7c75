"""Weight layouts shared by the model lines whose layers are listed one by one."""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from ..kv.buffer import MixedKvBuffer
from ..kv.state import LayerStates
from ..sched.executor import HybridExecutor


def pad8(n: int) -> int:
    return (n + 7) // 8 * 8


class FusedProjection:
    """Matrices that read the same rows, stacked with every part padded to a multiple of 8 rows, so that every part of the
    output starts on a 16-byte boundary."""

    def __init__(self, parts: dict):
        self.at, rows, out = {}, 0, []
        for name, w in parts.items():
            self.at[name] = (rows, rows + w.shape[0])
            out.append(w)
            pad = pad8(w.shape[0]) - w.shape[0]
            if pad:
                out.append(torch.zeros((pad, w.shape[1]), dtype=w.dtype, device=w.device))
            rows += w.shape[0] + pad
        self.w = torch.cat(out, 0).contiguous()

    def __call__(self, x):
        y = ops.dense(x, self.w)
        return {n: y[:, a:b] for n, (a, b) in self.at.items()}


class LatentHeads:
    """Per-head up-projections of a cached latent: ``ukv`` [heads * (dim + vdim), latent] keys then values (expanded form),
    ``uv`` [heads, vdim, latent] a view of it, ``uk_t`` [heads, latent, dim] transposed for folding queries into the latent
    (absorbed form)."""

    def __init__(self, uk: torch.Tensor, uv: torch.Tensor, heads: int):
        self.ukv = torch.cat((uk, uv), 0).contiguous()
        self.uv = self.ukv[uk.shape[0] :].view(heads, -1, uk.shape[1])
        self.uk_t = uk.view(heads, -1, uk.shape[1]).transpose(1, 2).contiguous()


class HybridLayers:
    """Cache, state and executor of a model whose layers are listed one by one, some with pages, some with recurrent state:
    ``kv_geometries`` ``(kv_heads, dim, vdim)`` of the layers that own a cache, ``state_geometries`` as in ``LayerStates``."""

    supports_prefix_cache = False  # recurrent state is per request and not cached
    carries_token = False  # the embedding reads the previous token
    rec: Optional[LayerStates] = None

    def kv_geometry(self) -> dict:
        g = self.kv_geometries or [(1, 8, 8)]
        # KV heads of the attention layers times the groups of up to eight query heads that one CTA of the decode kernel takes
        attn = [m for l in self.cfg.layer_specs for m in l.mixer.flat() if m.kind == "attention"]
        return dict(num_layers=len(g), kv_heads=max([m.kv_heads * ((m.heads // m.kv_heads + 7) // 8) for m in attn] or [1]), head_dim=max(max(d, v) for _, d, v in g),
                    bytes_per_block=lambda page: max(1, MixedKvBuffer.bytes_per_block(self.kv_geometries, page, self.dtype)))

    def make_kv(self, num_pages: int, page_size: int) -> MixedKvBuffer:
        return MixedKvBuffer(self.kv_geometries, num_pages, page_size, self.dtype, self.device)

    def state_bytes(self, slots: int) -> int:
        elem = torch.empty((), dtype=self.dtype).element_size()
        return (slots + 1) * (4 * self.carries_token + sum(4 * h * dk * dv + elem * c * max(taps - 1, 0) for h, dk, dv, c, taps in self.state_geometries))

    def make_state(self, num_slots: int) -> LayerStates:
        self.rec = LayerStates(num_slots + 1, self.state_geometries, self.dtype, self.device, token=self.carries_token)
        return self.rec

    @staticmethod
    def make_executor(model, kv, page_size, cuda_graph=False, max_decode_batch=256, max_blocks_per_seq=0, seed=0, state_slots=None):
        return HybridExecutor(model, kv, page_size, state_slots=state_slots or max_decode_batch, cuda_graph=cuda_graph, max_decode_batch=max_decode_batch, max_blocks_per_seq=max_blocks_per_seq, seed=seed)
