"""Weight layouts shared by the model lines whose layers are listed one by one."""
from __future__ import annotations

import torch

from .. import ops


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
