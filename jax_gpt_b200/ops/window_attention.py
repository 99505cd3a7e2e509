"""Grouped-query attention with a sliding window and kept first tokens on packed batches over paged ``[K | V]`` rows:
position i sees j when ``j <= i and (i - j < window or j < keep_first)``; in place of the first tokens it may see one mean key and value
for every block of tokens wholly before its window (``pool``). Scores may be soft-capped, the softmax may have a sink.

``qk_prepare`` makes attention operands of a projection row ``[q heads | k heads]`` (bias, half-split rotation, unit RMS norm
per head) and writes the cache rows; the projected keys double as values. ``grouped_attention`` picks the form: whole
prompts of matching widths on the tcgen05 flash kernel, decode steps of matching widths on the paged decode kernel,
every other case (other widths, fp32, prompts that continue a cache) on the any-size kernel of csrc/window_attention.cu.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

import torch

from .. import _ext
from . import attention as A
from .packed import PackedBatch
from .rope import rotate_half_split

TENSOR_WIDTHS = (64, 128, 256)
NO_WINDOW = 1 << 30


FLASH_WIDTHS = ((64, 64), (128, 128), (192, 128), (256, 256))     # (query and key, value) widths of the flash kernel


def flash_widths(batch: PackedBatch, dtype, is_cuda: bool, dk: int, dv: int) -> Optional[Tuple[int, int]]:
    """Operand widths of the flash kernel for whole prompts (operands padded with zeros), None where it does not apply."""
    if not is_cuda or dtype != torch.bfloat16 or not batch.fresh or batch.single:
        return None
    return next((w for w in FLASH_WIDTHS if w[0] >= dk and w[1] >= dv), None)


def flash_ok(batch: PackedBatch, t: torch.Tensor, D: int) -> bool:
    """Whole prompts that run on the flash kernel."""
    return t.is_cuda and t.dtype == torch.bfloat16 and batch.fresh and not batch.single and D in TENSOR_WIDTHS


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


def key_splits(batch: PackedBatch, H: int, G: int, window: int, keep_first: int, pool: int = 0) -> int:
    """Key ranges per query of the any-size kernel: decode steps spread their visible keys over the SMs."""
    if not batch.single:
        return 1
    seen = min(batch.max_len, window + keep_first) + (max(0, batch.max_len - window) // pool if pool else 0)
    return max(1, min(592 // max(1, batch.n_seq * G * ((H // G + 7) // 8)), (seen + 63) // 64, 32))


def window_attention_any(batch: PackedBatch, q, cache, layer: int, G: int, window: int, keep_first: int, scale: float,
                         n_splits: int = 0, v_dim: int = 0, softcap: float = 0.0, sink=None, pool: int = 0) -> torch.Tensor:
    """q (N, H, D) over the cached rows of each token's own sequence; values of width ``v_dim`` (0: D). ``softcap`` > 0: scores become
    softcap tanh(score / softcap); ``sink`` (H,) fp32: exp(sink) joins the denominators; ``pool`` > 0 (the cache's block size of this
    layer): block means before the window are seen too. Returns (N, H, v_dim)."""
    N, H, D = q.shape
    DV = v_dim or D
    if q.is_cuda:
        S = n_splits or key_splits(batch, H, G, window, keep_first, pool)
        o = torch.empty(N, H, DV, device=q.device, dtype=q.dtype)
        po = torch.empty(N * H * S * DV, device=q.device, dtype=torch.float32) if S > 1 else None
        pm = torch.empty(N * H * S * 2, device=q.device, dtype=torch.float32) if S > 1 else None
        _ext.ops().window_attention(*batch.desc, q, cache.pool[layer], cache.block_table, window, keep_first, scale, S, po, pm, o,
                                    softcap, sink, cache.pooled[layer] if pool else None, pool)
        return o
    out = torch.empty(N, H, DV, dtype=q.dtype)
    for c0, n, slot, start in batch.rows():
        rows = cache.gather(layer, slot, start + n).float()
        i, j = torch.arange(start, start + n)[:, None], torch.arange(start + n)[None, :]
        seen = (j <= i) & ((i - j < window) | (j < keep_first))
        if pool:
            rows = torch.cat([rows, cache.gather_pooled(layer, slot, (start + n) // pool).float()])
            ends = (torch.arange(len(rows) - start - n)[None, :] + 1) * pool
            seen = torch.cat([seen, ends <= i - window + 1], 1)
        k, v = (t.reshape(len(rows), G, -1).repeat_interleave(H // G, 1) for t in rows.split([G * D, G * DV], -1))
        s = torch.einsum("nhd,khd->hnk", q[c0:c0 + n].float(), k) * scale
        s = softcap * torch.tanh(s / softcap) if softcap > 0 else s
        s = s.masked_fill(~seen, float("-inf"))
        if sink is not None:
            s = torch.cat([s, sink.float()[:, None, None].expand(H, n, 1)], -1)
        p = torch.softmax(s, -1)[..., :len(rows)]
        out[c0:c0 + n] = torch.einsum("hnk,khd->nhd", p, v).to(q.dtype)
    return out


def prompt_parts(batch: PackedBatch):
    """(first row, rows, sequences) of the launches of a flash kernel over whole prompts: one for equal lengths, else one each."""
    if len(set(batch.lens)) == 1:
        return [(0, batch.n_tok, batch.n_seq)]
    return [(sum(batch.lens[:b]), n, 1) for b, n in enumerate(batch.lens)]


@dataclass(frozen=True)
class PoolLayout:
    """Dense keys and values of whole prompts with block means: sequence b has ``pads[b]`` rows of means (a multiple of the key tile),
    then its tokens from row ``row0[b]`` on."""
    pads: Tuple[int, ...]
    rows: int                          # all rows
    row0: torch.Tensor                 # int32 device copies
    pad: torch.Tensor


def pool_layout(batch: PackedBatch, window: int, pool: int) -> PoolLayout:
    def make():
        pads = tuple((max(0, n - window) // pool + 127) // 128 * 128 for n in batch.lens)
        at, firsts = 0, []
        for p, n in zip(pads, batch.lens):
            firsts.append(at + p)
            at += p + n
        dev = torch.tensor([firsts, pads], dtype=torch.int32).to(batch.ids.device)
        return PoolLayout(pads, at, dev[0], dev[1])
    return batch.memo(("pool_layout", window, pool), make)


def flash_prompts(batch: PackedBatch, q, k, v, scale: float, window: int = 0, keep_first: int = 0, softcap: float = 0.0, sink=None,
                  pool: int = 0) -> torch.Tensor:
    """Whole prompts on the flash kernel: dense q (N, H, D), k (N, G, D), v (N, G, DV). Returns (N, H, DV). With ``pool`` k and v hold the
    rows of ``pool_layout`` (block means before a sequence's tokens)."""
    o = torch.empty(q.shape[0], q.shape[1], v.shape[2], device=q.device, dtype=q.dtype)
    lay = pool_layout(batch, window, pool) if pool else None
    k0 = 0
    for i, (c0, n, B) in enumerate(prompt_parts(batch)):
        pads = lay.pads[i] if lay else 0
        rows = n + B * pads
        as4 = lambda t: t[c0:c0 + n].unflatten(0, (B, n // B))
        kv4 = lambda t: t[k0:k0 + rows].unflatten(0, (B, rows // B))
        A.attn_fwd(as4(q), kv4(k), kv4(v), True, scale, out=as4(o), window=window, keep_first=keep_first, softcap=softcap, sink=sink,
                   pool=pool if pads else 0, pool_rows=pads)
        k0 += rows
    return o


def grouped_attention(batch: PackedBatch, q, k, v, cache, layer: int, G: int, dv: int, scale: float, window: int = NO_WINDOW,
                      keep_first: int = 0, softcap: float = 0.0, sink=None, pool: int = 0) -> torch.Tensor:
    """Output (N, H, >= dv) of attention operands: dense k, v of whole prompts on the flash kernel, or q against the cached rows."""
    N, H, D = q.shape
    windowed = window < NO_WINDOW
    if k is not None:
        return flash_prompts(batch, q, k, v, scale, window if windowed else 0, keep_first if windowed else 0, softcap, sink, pool)
    if (q.is_cuda and q.dtype == torch.bfloat16 and batch.single and A.decode_widths_ok(H, G, D, dv) and not (softcap > 0 and pool)):
        # the step has advanced the lengths already: len_add 0
        return A.attention_decode_paged(q, cache.pool[layer], cache.block_table, batch.ids, cache.seq_lens, G, 0, scale,
                                        max_len=batch.max_len, window=window if windowed else 0, keep_first=keep_first, v_dim=dv,
                                        softcap=softcap, sink=sink, pooled=cache.pooled[layer] if pool else None, pool_block=pool)
    return window_attention_any(batch, q, cache, layer, G, window, keep_first, scale, v_dim=dv, softcap=softcap, sink=sink, pool=pool)


def window_attention(batch: PackedBatch, q, k, v, cache, layer: int, G: int, window: Optional[int], keep_first: int,
                     scale: float) -> torch.Tensor:
    """q (N, H, D) and, for whole prompts on the flash kernel, the dense k, v (N, G, D) of ``qk_prepare``. Returns (N, H D)."""
    N, H, D = q.shape
    dense = k is not None and flash_ok(batch, q, D)
    return grouped_attention(batch, q, k if dense else None, v if dense else None, cache, layer, G, D, scale, window or NO_WINDOW,
                             keep_first).view(N, H * D)
