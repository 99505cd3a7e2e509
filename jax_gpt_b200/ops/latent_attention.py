"""Multi-head latent attention on packed batches over paged latent rows ``[RMS-normed latent | rotated key part]``.

``mla_prepare`` normalises the query latent and writes the cache rows; the attention then runs in one of three forms:
decompressed keys and values on the tcgen05 flash kernel (whole prompts of the shape 192 / 128), absorbed weights on the
tcgen05 paged kernel (decode, latent 512 + 64, ops/mla_decode.py), or absorbed weights on the any-size kernel
``latent_attention`` (every other size, fp32, prompts that continue a cache). All take a softmax sink.
"""
from __future__ import annotations

import torch

from .. import _ext
from .packed import PackedBatch
from .rope import rotate_interleaved


def _pages(cache, layer, slot, n):
    return cache.gather(layer, slot, n)


def mla_prepare(batch: PackedBatch, y, q_gamma, kv_gamma, eps, rope, cache, layer: int, want_latent: bool):
    """y (N, q_rank + R + dr) = [query latent | kv latent | rotary key]. Returns (cq (N, q_rank), lat (N, R + dr) or
    None); the rows of ``lat`` are written to the cache's pages. ``rope``: (cos, sin) tables [max_pos, dims / 2]."""
    qr, R = q_gamma.numel(), kv_gamma.numel()
    dr = y.shape[1] - qr - R
    if y.is_cuda:
        cq = torch.empty(batch.n_tok, qr, device=y.device, dtype=y.dtype)
        lat = torch.empty(batch.n_tok, R + dr, device=y.device, dtype=y.dtype) if want_latent else None
        _ext.ops().mla_prepare(*batch.desc, y, q_gamma, kv_gamma, eps, rope[0], rope[1], cache.pool[layer], cache.block_table, cq, lat)
        return cq, lat
    yf = y.float()
    rms = lambda t, g: t * torch.rsqrt(t.square().mean(-1, keepdim=True) + eps) * g
    cq = rms(yf[:, :qr], q_gamma).to(y.dtype)
    lat = torch.cat([rms(yf[:, qr:qr + R], kv_gamma), rotate_interleaved(yf[:, qr + R:], batch.positions(), rope)], -1).to(y.dtype)
    for c0, n, slot, start in batch.rows():
        pages, offs = cache.slots(slot, start, n)
        cache.pool[layer][pages, offs] = lat[c0:c0 + n].to(cache.dtype)
    return cq, lat if want_latent else None


def mla_rope_qk(batch: PackedBatch, q, k_nope, lat, R: int, rope) -> torch.Tensor:
    """Rotates the last dr features of every head of q (N, H, dn + dr) in place; returns k (N, H, dn + dr)."""
    k = torch.empty_like(q)
    _ext.ops().mla_rope_qk(*batch.desc, q, k_nope, lat, R, rope[0], rope[1], k)
    return k


def mla_absorb_q(batch: PackedBatch, q, w_uk, rope, dr: int) -> torch.Tensor:
    """q (N, H, dn + dr), w_uk (H * dn, R) -> (N, H, R + dr): the unrotated part in latent coordinates, then the rotated."""
    N, H, D = q.shape
    R = w_uk.shape[1]
    if q.is_cuda:
        qf = torch.empty(N, H, R + dr, device=q.device, dtype=q.dtype)
        _ext.ops().mla_absorb_q(*batch.desc, q, w_uk, rope[0], rope[1], qf)
        return qf
    ql = torch.einsum("nhd,hdr->nhr", q[..., :D - dr].float(), w_uk.float().reshape(H, D - dr, R))
    return torch.cat([ql, rotate_interleaved(q[..., D - dr:].float(), batch.positions(), rope)], -1).to(q.dtype)


def mla_absorb_out(o_lat, w_uv) -> torch.Tensor:
    """o_lat (N, H, R), w_uv (H * dv, R) -> (N, H * dv)."""
    N, H, R = o_lat.shape
    if o_lat.is_cuda:
        o = torch.empty(N, w_uv.shape[0], device=o_lat.device, dtype=o_lat.dtype)
        _ext.ops().mla_absorb_out(o_lat, w_uv, o)
        return o
    return torch.einsum("nhr,hvr->nhv", o_lat.float(), w_uv.float().reshape(H, -1, R)).reshape(N, -1).to(o_lat.dtype)


def key_splits(batch: PackedBatch, n_heads: int) -> int:
    """Key ranges per query of the any-size kernel: decode steps spread a long cache over the SMs."""
    if not batch.single:
        return 1
    return max(1, min(592 // max(1, batch.n_seq * ((n_heads + 7) // 8)), (batch.max_len + 63) // 64, 32))


def latent_attention(batch: PackedBatch, qf, cache, layer: int, R: int, scale: float, sink=None, n_splits: int = 0):
    """qf (N, H, R + dr) over the cached rows of each token's own sequence up to its own position. Returns (N, H, R)."""
    N, H, W = qf.shape
    if qf.is_cuda:
        S = n_splits or key_splits(batch, H)
        o = torch.empty(N, H, R, device=qf.device, dtype=qf.dtype)
        po = torch.empty(N * H * S * R, device=qf.device, dtype=torch.float32) if S > 1 else None
        pm = torch.empty(N * H * S * 2, device=qf.device, dtype=torch.float32) if S > 1 else None
        _ext.ops().latent_attention(*batch.desc, qf, cache.pool[layer], cache.block_table, sink, scale, S, po, pm, o)
        return o
    out = torch.empty(N, H, R, dtype=qf.dtype)
    for c0, n, slot, start in batch.rows():
        rows = _pages(cache, layer, slot, start + n).float()
        s = torch.einsum("nhw,kw->nhk", qf[c0:c0 + n].float(), rows) * scale
        seen = torch.arange(start + n)[None, :] <= torch.arange(start, start + n)[:, None]
        s = s.masked_fill(~seen[:, None, :], float("-inf"))
        if sink is not None:
            s = torch.cat([s, sink.float()[None, :, None].expand(n, H, 1)], -1)
        p = torch.softmax(s, -1)[..., :start + n]
        out[c0:c0 + n] = torch.einsum("nhk,kr->nhr", p, rows[:, :R]).to(qf.dtype)
    return out
