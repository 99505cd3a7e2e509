"""Grouped-query attention whose values are rotated by their positions (and the output turned back), with interleaved rotary
pairs and key and value widths of their own, on packed batches over paged ``[K | V]`` rows.

``qkv_rotate`` makes attention operands and the cache rows of a projection row (csrc/rotated_kv.cu). ``causal_attention`` picks the
form: whole bf16 prompts on the tcgen05 flash kernel (operands padded with zeros to its next width), bf16 decode steps of matching
widths on the paged decode kernel, every other case on the any-size kernel of csrc/window_attention.cu. ``turn_back_gate`` undoes the
values' rotation at the query's position and applies a gate per head.
"""
from __future__ import annotations

from typing import Optional, Sequence, Tuple

import torch

from .. import _ext
from .packed import PackedBatch
from .rope import rotate_interleaved
from .window_attention import flash_widths, grouped_attention  # noqa: F401

def qkv_rotate(batch: PackedBatch, y, cols: Sequence[int], bias, H: int, G: int, dk: int, dv: int, rope, vrope, cache, layer: int,
               dense: Optional[Tuple[int, int]]):
    """y (N, ...) with q (H dk), k (G dk), v (G dv) at columns ``cols``; ``bias`` fp32 (H dk + G dk + G dv) or None; ``rope`` /
    ``vrope``: (cos, sin) tables of the interleaved pairs of q and k / of v. Writes the cache rows of ``layer``; returns q (N, H, dk)
    and None, None, or with ``dense`` = (width, value width) q, k, v padded to these widths."""
    N = batch.n_tok
    wk, wv = dense or (dk, dv)
    if y.is_cuda:
        new = lambda h, d: torch.empty(N, h, d, device=y.device, dtype=y.dtype)
        q, k, v = new(H, wk), new(G, wk) if dense else None, new(G, wv) if dense else None
        _ext.ops().qkv_rotate(*batch.desc, y, list(cols), bias, rope[0], rope[1], vrope[0], vrope[1], dk, dv, cache.pool[layer],
                              cache.block_table, q, k, v)
        return q, k, v
    sizes = (H * dk, G * dk, G * dv)
    bs = bias.split(sizes) if bias is not None else (0.0, 0.0, 0.0)
    q, k, v = (y[:, c:c + n].float() + b for c, n, b in zip(cols, sizes, bs))
    pos = batch.positions()
    q, k = (rotate_interleaved(t.reshape(N, -1, dk), pos, rope).to(y.dtype) for t in (q, k))
    v = rotate_interleaved(v.reshape(N, G, dv), pos, vrope).to(y.dtype)
    rows = torch.cat([k.reshape(N, -1), v.reshape(N, -1)], -1)
    for c0, n, slot, start in batch.rows():
        pages, offs = cache.slots(slot, start, n)
        cache.pool[layer][pages, offs] = rows[c0:c0 + n].to(cache.dtype)
    return q, None, None


def causal_attention(batch: PackedBatch, q, k, v, cache, layer: int, G: int, dv: int, scale: float) -> torch.Tensor:
    """Output (N, H, >= dv) of the operands of ``qkv_rotate``: dense prompts, or q against the cached rows."""
    return grouped_attention(batch, q, k, v, cache, layer, G, dv, scale)


def turn_back_gate(batch: PackedBatch, o, g, vrope, scale: float, out) -> None:
    """``out[:, h dv + c] = scale * sigmoid(g[:, h]) * o[:, h, c]`` with o turned back by the row's position; o (N, H, >= dv)."""
    N, H, _ = o.shape
    if o.is_cuda:
        _ext.ops().turn_back_gate(*batch.desc, o, g, vrope[0], vrope[1], scale, out)
        return
    dv = out.shape[1] // H
    t = rotate_interleaved(o[..., :dv].float(), batch.positions(), (vrope[0], -vrope[1]))
    out.copy_((t * (scale * torch.sigmoid(g.float()))[:, :, None]).reshape(N, H * dv).to(out.dtype))
