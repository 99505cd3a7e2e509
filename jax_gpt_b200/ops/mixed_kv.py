"""Grouped-query attention operands without rotation, on packed batches over paged ``[K | V]`` rows: queries scaled by a factor of their
position, values mixed with another layer's values of the same token, and means of blocks of cache rows (csrc/mixed_kv.cu).

``mixed_kv`` makes the operands and writes rows and means to the cache; ``window_attention.grouped_attention`` takes them from there.
"""
from __future__ import annotations

import math
from typing import Optional, Sequence, Tuple

import torch

from .. import _ext
from .packed import PackedBatch
from .window_attention import pool_layout


def query_factors(coef: float, every: int, n_pos: int, device="cpu") -> torch.Tensor:
    """fp32 [n_pos]: ``1 + coef ln(floor((p + 1) / every) + 1)`` for position p, so that scores grow with the length of the context."""
    return torch.tensor([1.0 + coef * math.log((p + 1) // every + 1) for p in range(n_pos)], dtype=torch.float32).to(device)


def mixed_kv(batch: PackedBatch, y, cols: Sequence[int], H: int, G: int, dk: int, dv: int, cache, layer: int,
             dense: Optional[Tuple[int, int]] = None, q_factor=None, v_first=None, lam: float = 0.0, window: int = 0):
    """y (N, ...) with q (H dk), k (G dk), v (G dv) at columns ``cols``; ``q_factor`` fp32 [n_pos] multiplies the queries; with ``v_first``
    (N, G dv) the values become ``(1 - lam) v + lam v_first``. Writes the cache rows of ``layer`` and, where the cache keeps block means
    for it (``cache.blocks``), the means of the blocks that the step completes. Returns q (N, H, dk) and None, None, or with ``dense`` =
    (width, value width) q, k, v padded with zeros to these widths, k and v with the means that ``window`` lets be seen in front
    (``pool_layout``)."""
    N, P = batch.n_tok, cache.blocks[layer]
    wk, wv = dense or (dk, dv)
    if y.is_cuda:
        lay = pool_layout(batch, window, P) if dense and P else None
        rows = lay.rows if lay else N
        new = lambda r, h, d: torch.empty(r, h, d, device=y.device, dtype=y.dtype)
        q, k, v = new(N, H, wk), new(rows, G, wk) if dense else None, new(rows, G, wv) if dense else None
        units = 0
        if P:
            units = sum(max(n // P, p) for n, p in zip(batch.lens, lay.pads)) if lay else N // P + batch.n_seq
        _ext.ops().mixed_kv(*batch.desc, y, list(cols), q_factor, v_first, lam, dk, dv, cache.pool[layer], cache.block_table,
                            cache.pooled[layer], P, q, k, v, lay.row0 if lay else None, lay.pad if lay else None, units)
        return q, k, v
    q, k, v = (y[:, c:c + n].float() for c, n in zip(cols, (H * dk, G * dk, G * dv)))
    if q_factor is not None:
        q = q * q_factor[batch.positions()][:, None]
    if v_first is not None:
        v = (1.0 - lam) * v + lam * v_first.float()
    new_rows = torch.cat([k, v], -1)
    for c0, n, slot, start in batch.rows():
        pages, offs = cache.slots(slot, start, n)
        cache.pool[layer][pages, offs] = new_rows[c0:c0 + n].to(cache.dtype)
        if P and (start + n) // P > start // P:
            b0, b1 = start // P, (start + n) // P
            pages, offs = cache.slots(slot, b0 * P, (b1 - b0) * P)
            means = cache.pool[layer][pages, offs].float().reshape(b1 - b0, P, -1).mean(1)
            pages, offs = cache.pooled_slots(layer, slot, b0, b1 - b0)
            cache.pooled[layer][pages, offs] = means.to(cache.dtype)
    return q.to(y.dtype).reshape(N, H, dk), None, None
