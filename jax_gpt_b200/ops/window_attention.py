"""Grouped-query attention with a sliding window and kept first tokens on packed batches over paged ``[K | V]`` rows:
position i sees j when ``j <= i and (i - j < window or j < keep_first)``.

``qk_prepare`` makes attention operands of a projection row ``[q heads | k heads]`` (bias, half-split rotation, unit RMS norm
per head) and writes the cache rows; the projected keys double as values. ``window_attention`` then picks the form: whole
prompts of head width 64 / 128 / 256 on the tcgen05 flash kernel, decode steps of these widths on the paged decode kernel,
every other case (other widths, fp32, prompts that continue a cache) on the any-size kernel of csrc/window_attention.cu.
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import _ext
from . import attention as A
from .packed import PackedBatch
from .rope import rotate_half_split

TENSOR_WIDTHS = (64, 128, 256)
NO_WINDOW = 1 << 30


def flash_ok(batch: PackedBatch, t: torch.Tensor, D: int) -> bool:
    """Whole prompts that run on the flash kernel."""
    return t.is_cuda and t.dtype == torch.bfloat16 and batch.fresh and not batch.single and D in TENSOR_WIDTHS


def decode_ok(batch: PackedBatch, t: torch.Tensor, H: int, G: int, D: int) -> bool:
    return t.is_cuda and t.dtype == torch.bfloat16 and batch.single and D in TENSOR_WIDTHS and H // G in (1, 2, 4, 8)


def qk_prepare(batch: PackedBatch, y, bias, H: int, G: int, D: int, unit_norm: bool, eps: float, rope, cache, layer: int,
               dense: bool):
    """y (N, (H + G) D). Returns (q (N, H, D), k, v (N, G, D) or None); the cache rows of ``layer`` are written. ``rope``:
    (cos, sin) tables [max_pos, dims / 2] of half-split pairs; ``bias`` fp32 ((H + G) D) or None."""
    N = batch.n_tok
    if y.is_cuda:
        new = lambda h: torch.empty(N, h, D, device=y.device, dtype=y.dtype)
        q, k, v = new(H), new(G) if dense else None, new(G) if dense else None
        _ext.ops().qk_prepare(*batch.desc, y, bias, unit_norm, eps, rope[0], rope[1], cache.pool[layer], cache.block_table, q, k, v)
        return q, k, v
    x = (y.float() + (0.0 if bias is None else bias)).reshape(N, H + G, D)
    r = rotate_half_split(x, batch.positions(), rope)
    if unit_norm:
        r = r * torch.rsqrt(r.square().mean(-1, keepdim=True) + eps)
    q, k, v = r[:, :H].to(y.dtype), r[:, H:].to(y.dtype), x[:, H:].to(y.dtype)
    rows = torch.cat([k.reshape(N, G * D), v.reshape(N, G * D)], -1)
    for c0, n, slot, start in batch.rows():
        pages, offs = cache.slots(slot, start, n)
        cache.pool[layer][pages, offs] = rows[c0:c0 + n].to(cache.dtype)
    return (q, k, v) if dense else (q, None, None)


def key_splits(batch: PackedBatch, H: int, G: int, window: int, keep_first: int) -> int:
    """Key ranges per query of the any-size kernel: decode steps spread their visible keys over the SMs."""
    if not batch.single:
        return 1
    seen = min(batch.max_len, window + keep_first)
    return max(1, min(592 // max(1, batch.n_seq * G * ((H // G + 7) // 8)), (seen + 63) // 64, 32))


def window_attention_any(batch: PackedBatch, q, cache, layer: int, G: int, window: int, keep_first: int, scale: float,
                         n_splits: int = 0, v_dim: int = 0) -> torch.Tensor:
    """q (N, H, D) over the cached rows of each token's own sequence; values of width ``v_dim`` (0: D). Returns (N, H, v_dim)."""
    N, H, D = q.shape
    DV = v_dim or D
    if q.is_cuda:
        S = n_splits or key_splits(batch, H, G, window, keep_first)
        o = torch.empty(N, H, DV, device=q.device, dtype=q.dtype)
        po = torch.empty(N * H * S * DV, device=q.device, dtype=torch.float32) if S > 1 else None
        pm = torch.empty(N * H * S * 2, device=q.device, dtype=torch.float32) if S > 1 else None
        _ext.ops().window_attention(*batch.desc, q, cache.pool[layer], cache.block_table, window, keep_first, scale, S, po, pm, o)
        return o
    out = torch.empty(N, H, DV, dtype=q.dtype)
    for c0, n, slot, start in batch.rows():
        rows = cache.gather(layer, slot, start + n).float()
        k, v = (t.reshape(start + n, G, -1).repeat_interleave(H // G, 1) for t in rows.split([G * D, G * DV], -1))
        i, j = torch.arange(start, start + n)[:, None], torch.arange(start + n)[None, :]
        seen = (j <= i) & ((i - j < window) | (j < keep_first))
        s = torch.einsum("nhd,khd->hnk", q[c0:c0 + n].float(), k) * scale
        p = torch.softmax(s.masked_fill(~seen, float("-inf")), -1)
        out[c0:c0 + n] = torch.einsum("hnk,khd->nhd", p, v).to(q.dtype)
    return out


def flash_prompts(batch: PackedBatch, q, k, v, scale: float, window: int = 0, keep_first: int = 0) -> torch.Tensor:
    """Whole prompts on the flash kernel: dense q (N, H, D), k (N, G, D), v (N, G, DV). Returns (N, H, DV)."""
    o = torch.empty(q.shape[0], q.shape[1], v.shape[2], device=q.device, dtype=q.dtype)
    same = len(set(batch.lens)) == 1
    parts = [(0, batch.n_tok, batch.n_seq)] if same else [(sum(batch.lens[:b]), n, 1) for b, n in enumerate(batch.lens)]
    for c0, n, B in parts:
        as4 = lambda t: t[c0:c0 + n].unflatten(0, (B, n // B))
        A.attn_fwd(as4(q), as4(k), as4(v), True, scale, out=as4(o), window=window, keep_first=keep_first)
    return o


def window_attention(batch: PackedBatch, q, k, v, cache, layer: int, G: int, window: Optional[int], keep_first: int,
                     scale: float) -> torch.Tensor:
    """q (N, H, D) and, for whole prompts on the flash kernel, the dense k, v (N, G, D) of ``qk_prepare``. Returns (N, H D)."""
    N, H, D = q.shape
    window = window or NO_WINDOW
    if k is not None and flash_ok(batch, q, D):
        return flash_prompts(batch, q, k, v, scale, window, keep_first).view(N, H * D)
    if decode_ok(batch, q, H, G, D):
        # the step has advanced the lengths already: len_add 0
        return A.attention_decode_paged(q, cache.pool[layer], cache.block_table, batch.ids, cache.seq_lens, G, 0, scale,
                                        max_len=batch.max_len, window=window, keep_first=keep_first).view(N, H * D)
    return window_attention_any(batch, q, cache, layer, G, window, keep_first, scale).view(N, H * D)
