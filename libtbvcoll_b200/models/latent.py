"""Latent attention as the decoders share it: a paged cache of normed latents and rotated key parts, read in two forms.

    few rows    fold W_uk into the query (grouped GEMM) -> rows kernel over the cache -> expand with W_uv (grouped GEMM)
    many rows   gather the visible context -> expand keys and values (GEMM) -> tiled kernel

What makes the queries, and the rotation, norm and cache write before it, is the decoder's own."""
from __future__ import annotations

from typing import Dict, List

import torch

from .. import ops
from ..engine.batch import StepBatch
from .config import LatentSpec


def pad16(n: int) -> int:
    return (n + 15) // 16 * 16


class LatentAttention:
    """Mixin; needs ``w``, ``_flat`` / ``_buf`` (with ``qa`` and ``lat``), ``block_size``, ``dtype``, ``device`` and ``latents`` (the specs of all such layers)."""
    w: Dict[str, torch.Tensor]
    latents: List[LatentSpec]
    _ctx_rows = 0

    @staticmethod
    def latent_row(m: LatentSpec) -> int:
        return ops.latent_row(pad16(m.kv_rank), pad16(m.rot_dim))

    def _context_scratch(self, rows: int) -> None:
        """Dense context buffers of the many-row form, grown on demand (never inside a captured step)."""
        if rows <= self._ctx_rows:
            return
        rows = (rows + 1023) // 1024 * 1024
        for k, cols in (("ctx_c", max(pad16(m.kv_rank) for m in self.latents)), ("ctx_r", max(pad16(m.rot_dim) for m in self.latents)),
                        ("ctx_kv", max(m.heads * (pad16(m.dim) + pad16(m.vdim)) for m in self.latents))):
            self._flat[k] = torch.empty(rows * cols, dtype=self.dtype, device=self.device)
        self._ctx_rows = rows

    def _latent_attend(self, b: StepBatch, p: str, m: LatentSpec, q: torch.Tensor, qa: torch.Tensor, cache: torch.Tensor, out: torch.Tensor, splits: int) -> None:
        """q [T, heads * dim | heads * rot_dim ..]; the rotated parts of the first n_rows_form rows are in qa already."""
        w, T, n = self.w, b.T, b.n_rows_form
        H, D, V, R, rot = m.heads, pad16(m.dim), pad16(m.vdim), pad16(m.kv_rank), pad16(m.rot_dim)
        sink = w.get(p + "sink")
        if n:
            lat = self._buf("lat", n, H, R)
            ops.linear(q[:n], w[p + "wabs"], qa.view(n, -1), groups=H, x_group=D, y_group=self.latent_row(m))
            ops.latent_attention_rows(qa, cache, b.tables, b.seq_of_row, b.ctx, sink, lat, m.kv_rank, m.scale, self.block_size, splits=splits, window=m.window)
            ops.linear(lat.view(n, -1), w[p + "wuv"], out[:n], groups=H, x_group=R, y_group=V)
        if n < T:
            C = b.dense_slots.shape[0]
            c, kr, kv = self._buf("ctx_c", C, R), self._buf("ctx_r", C, rot), self._buf("ctx_kv", C, H * (D + V))
            ops.latent_gather(cache, b.dense_slots, c, kr)
            ops.linear(c, w[p + "wukv"], kv)
            ops.latent_attention_prefill(q, H * D, kv, kr, b.dense_tiles, sink, out, H, D, V, m.scale, m.window)
