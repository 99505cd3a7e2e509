"""Multi-head latent attention on packed batches over paged latent rows ``[RMS-normed latent | rotated key part]``.

``mla_prepare`` normalises the latents and writes the cache rows; ``attend`` then runs in one of three forms:
decompressed keys and values on the tcgen05 flash kernel (whole prompts of the shape 192 / 128), absorbed weights on the
tcgen05 paged kernel (decode, latent 512 + 64, ops/mla_decode.py), or absorbed weights on the any-size kernel
``latent_attention`` (every other size, fp32, prompts that continue a cache). All take a softmax sink, a sliding window and an
output gate.
"""
from __future__ import annotations

import torch

from .. import _ext
from . import attention as A
from . import mla_decode
from .gemm import linear_rows
from .packed import PackedBatch
from .rope import rotate_interleaved
from .window_attention import NO_WINDOW, prompt_parts


def _pages(cache, layer, slot, n):
    return cache.gather(layer, slot, n)


def mla_prepare(batch: PackedBatch, y, q_gamma, kv_gamma, eps, rope, cache, layer: int, want_latent: bool):
    """y (N, q_rank + R + dr) = [query latent | kv latent | rotary key]; without ``q_gamma`` there is no query latent. Returns (cq
    (N, q_rank) or None, lat (N, R + dr) or None); the rows of ``lat`` are written to the cache's pages. ``rope``: (cos, sin) tables
    [max_pos, dims / 2]."""
    qr, R = 0 if q_gamma is None else q_gamma.numel(), kv_gamma.numel()
    dr = y.shape[1] - qr - R
    if y.is_cuda:
        cq = torch.empty(batch.n_tok, qr, device=y.device, dtype=y.dtype) if qr else None
        lat = torch.empty(batch.n_tok, R + dr, device=y.device, dtype=y.dtype) if want_latent else None
        _ext.ops().mla_prepare(*batch.desc, y, q_gamma, kv_gamma, eps, rope[0], rope[1], cache.pool[layer], cache.block_table, cq, lat)
        return cq, lat
    yf = y.float()
    rms = lambda t, g: t * torch.rsqrt(t.square().mean(-1, keepdim=True) + eps) * g
    cq = rms(yf[:, :qr], q_gamma).to(y.dtype) if qr else None
    lat = torch.cat([rms(yf[:, qr:qr + R], kv_gamma), rotate_interleaved(yf[:, qr + R:], batch.positions(), rope)], -1).to(y.dtype)
    for c0, n, slot, start in batch.rows():
        pages, offs = cache.slots(slot, start, n)
        cache.pool[layer][pages, offs] = lat[c0:c0 + n].to(cache.dtype)
    return cq, lat if want_latent else None


def mla_rope_qk(batch: PackedBatch, q, k_nope, lat, R: int, rope) -> torch.Tensor:
    """Rotates the last dr features of every head of q (N, H, dn + dr) in place; returns k (N, H, dn + dr)."""
    k = torch.empty(q.shape, device=q.device, dtype=q.dtype)
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


def mla_absorb_out(o_lat, w_uv, gate=None) -> torch.Tensor:
    """o_lat (N, H, R), w_uv (H * dv, R) -> (N, H * dv), times sigmoid(gate) with ``gate`` (N, H * dv)."""
    N, H, R = o_lat.shape
    if o_lat.is_cuda:
        o = torch.empty(N, w_uv.shape[0], device=o_lat.device, dtype=o_lat.dtype)
        _ext.ops().mla_absorb_out(o_lat, w_uv, o, gate)
        return o
    o = torch.einsum("nhr,hvr->nhv", o_lat.float(), w_uv.float().reshape(H, -1, R)).reshape(N, -1)
    return (o if gate is None else o * torch.sigmoid(gate.float())).to(o_lat.dtype)


def sigmoid_gate(o, gate) -> torch.Tensor:
    """``o`` (N, D) times sigmoid(gate), in place on CUDA."""
    if o.is_cuda:
        _ext.ops().sigmoid_gate(o, gate)
        return o
    return (o.float() * torch.sigmoid(gate.float())).to(o.dtype)


def key_splits(batch: PackedBatch, n_heads: int, window: int = NO_WINDOW) -> int:
    """Key ranges per query of the any-size kernel: decode steps spread a long cache over the SMs."""
    if not batch.single:
        return 1
    return max(1, min(592 // max(1, batch.n_seq * ((n_heads + 7) // 8)), (min(batch.max_len, window) + 63) // 64, 32))


def latent_attention(batch: PackedBatch, qf, cache, layer: int, R: int, scale: float, sink=None, n_splits: int = 0, window: int = NO_WINDOW):
    """qf (N, H, R + dr) over the cached rows of each token's own sequence up to its own position, the last ``window`` of them.
    Returns (N, H, R)."""
    N, H, W = qf.shape
    if qf.is_cuda:
        S = n_splits or key_splits(batch, H, window)
        o = torch.empty(N, H, R, device=qf.device, dtype=qf.dtype)
        po = torch.empty(N * H * S * R, device=qf.device, dtype=torch.float32) if S > 1 else None
        pm = torch.empty(N * H * S * 2, device=qf.device, dtype=torch.float32) if S > 1 else None
        _ext.ops().latent_attention(*batch.desc, qf, cache.pool[layer], cache.block_table, sink, scale, S, po, pm, o, window)
        return o
    out = torch.empty(N, H, R, dtype=qf.dtype)
    for c0, n, slot, start in batch.rows():
        rows = _pages(cache, layer, slot, start + n).float()
        s = torch.einsum("nhw,kw->nhk", qf[c0:c0 + n].float(), rows) * scale
        back = torch.arange(start, start + n)[:, None] - torch.arange(start + n)[None, :]
        seen = (back >= 0) & (back < window)
        s = s.masked_fill(~seen[:, None, :], float("-inf"))
        if sink is not None:
            s = torch.cat([s, sink.float()[None, :, None].expand(n, H, 1)], -1)
        p = torch.softmax(s, -1)[..., :start + n]
        out[c0:c0 + n] = torch.einsum("nhk,kr->nhr", p, rows[:, :R]).to(qf.dtype)
    return out


def flash_ok(batch: PackedBatch, h, dn: int, dr: int, dv: int, R: int) -> bool:
    """Whole prompts whose heads have the flash kernel's MLA shape."""
    return (h.is_cuda and h.dtype == torch.bfloat16 and batch.fresh and not batch.single and dn + dr == 192 and dv == 128 and R % 8 == 0
            and dr % 8 == 0)


def paged_kernel_ok(batch: PackedBatch, h, R: int, dr: int, page_size: int) -> bool:
    return h.is_cuda and h.dtype == torch.bfloat16 and batch.single and R == 512 and dr == 64 and page_size == 64


def attend(batch: PackedBatch, q, lat, w_ukv, R: int, dv: int, rope, cache, layer: int, scale: float, sink=None, window: int = NO_WINDOW,
           gate=None) -> torch.Tensor:
    """q (N, H, dn + dr), unrotated; ``lat`` (N, R + dr) of ``mla_prepare`` where ``flash_ok``, else None; ``w_ukv`` (H dn + H dv, R) = [key
    | value up-projection]. Returns (N, H dv), times sigmoid(gate) with ``gate`` (N, H dv). May rotate q in place."""
    N, H, D = q.shape
    dn = (w_ukv.shape[0] - H * dv) // H
    dr = D - dn
    if lat is not None:
        kv = linear_rows(lat[:, :R], w_ukv)                           # (N, H dn | H dv)
        k = mla_rope_qk(batch, q, kv[:, :H * dn], lat, R, rope)
        v = kv[:, H * dn:].unflatten(-1, (H, dv))
        o = torch.empty(N, H, dv, device=q.device, dtype=q.dtype)
        for c0, n, B in prompt_parts(batch):
            as4 = lambda t: t[c0:c0 + n].unflatten(0, (B, n // B))
            A.attn_fwd(as4(q), as4(k), as4(v), True, scale, out=as4(o), sink=sink, window=window if window < NO_WINDOW else 0)
        o = o.view(N, H * dv)
        return o if gate is None else sigmoid_gate(o, gate)
    qf = mla_absorb_q(batch, q, w_ukv[:H * dn], rope, dr)
    if paged_kernel_ok(batch, q, R, dr, cache.page_size):
        o_lat = mla_decode.mla_paged_decode(qf, cache, layer, batch.ids, scale, sink=sink, max_len=batch.max_len,
                                            window=window if window < NO_WINDOW else 0)
    else:
        o_lat = latent_attention(batch, qf, cache, layer, R, scale, sink, window=window)
    return mla_absorb_out(o_lat, w_ukv[H * dn:], gate)
