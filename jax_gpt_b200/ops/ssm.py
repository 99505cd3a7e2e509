"""State-space (Mamba-2) operations on packed batches: causal convolution with carried inputs, the state recurrence
(chunked on tcgen05 or token by token), the fused one-token step and the gated group norm.

Kernels: csrc/ssm_kernels.cu, csrc/ssd_scan_sm100.cu. State per cache slot: ``ring`` [slots, taps, C] fp32 with the raw
convolution input of position p in row ``p % taps``, and ``state`` [slots, H, N, P] fp32. A sequence that starts at
position 0 ignores what its slot held before, so a slot can be handed on without clearing it.
"""
from __future__ import annotations

import torch
import torch.nn.functional as F

from .. import _ext
from .packed import PackedBatch


def ssm_conv(batch: PackedBatch, x, w, bias, ring) -> torch.Tensor:
    """silu(causal depthwise convolution + bias) of x (N, C), w (C, taps) with the current token's tap last."""
    N, (C, taps) = x.shape[0], w.shape
    if x.is_cuda:
        y = torch.empty(N, C, device=x.device, dtype=x.dtype)
        _ext.ops().ssm_conv(*batch.desc, x, w, bias, ring, y)
        return y
    y = torch.empty(N, C, dtype=x.dtype)
    for c0, n, slot, start in batch.rows():
        past = [ring[slot, p % taps] if p >= 0 else torch.zeros(C) for p in range(start - taps + 1, start)]
        seq = torch.cat([torch.stack(past), x[c0:c0 + n].float()]) if past else x[c0:c0 + n].float()
        acc = bias + sum(seq[k:k + n] * w[:, k] for k in range(taps))
        y[c0:c0 + n] = F.silu(acc).to(x.dtype)
        for t in range(max(0, n - taps + 1), n):
            ring[slot, (start + t) % taps] = x[c0 + t].float()
    return y


def chunked_ok(x, state) -> bool:
    """True when the tensor-core form of the recurrence takes these tensors."""
    return x.is_cuda and x.dtype == torch.bfloat16 and state.shape[2] == 128 and state.shape[3] % 64 == 0


def ssd_scan(batch: PackedBatch, xbc, dt_raw, dt_bias, a_log, d_skip, state, groups: int, chunked=None) -> torch.Tensor:
    """xbc (N, H P + 2 G N') = [x | B | C] after the convolution, dt_raw (N, H). Returns y (N, H P) including the skip
    term; ``state`` is advanced. ``chunked``: None picks the tensor-core kernel where it applies."""
    H, Ns, P = state.shape[1:]
    if xbc.is_cuda:
        y = torch.empty(xbc.shape[0], H * P, device=xbc.device, dtype=xbc.dtype)
        use = chunked_ok(xbc, state) if chunked is None else chunked
        _ext.ops().ssd_scan(*batch.desc, xbc, dt_raw, dt_bias, a_log, d_skip, state, y, groups, use)
        return y
    y = torch.empty(xbc.shape[0], H * P, dtype=xbc.dtype)
    rep = H // groups
    for c0, n, slot, start in batch.rows():
        S = state[slot].clone() if start > 0 else torch.zeros(H, Ns, P)
        for t in range(c0, c0 + n):
            x, B, C = xbc[t].float().split([H * P, groups * Ns, groups * Ns])
            x = x.reshape(H, P)
            B, C = (v.reshape(groups, Ns).repeat_interleave(rep, 0) for v in (B, C))
            dt = F.softplus(dt_raw[t].float() + dt_bias)
            S = torch.exp(-torch.exp(a_log) * dt)[:, None, None] * S + (dt[:, None] * B)[:, :, None] * x[:, None, :]
            y[t] = (torch.einsum("hnp,hn->hp", S, C) + d_skip[:, None] * x).reshape(-1).to(xbc.dtype)
        state[slot] = S
    return y


def ssm_decode(batch: PackedBatch, zxd, w, bias, ring, dt_bias, a_log, d_skip, state, groups: int) -> torch.Tensor:
    """One token per sequence: zxd (B, inner + C + H) = [z | x | B | C | dt] -> (S^T C + D x) silu(z), fp32 (B, inner)."""
    H, Ns, P = state.shape[1:]
    inner, C = H * P, w.shape[0]
    if zxd.is_cuda:
        y = torch.empty(zxd.shape[0], inner, device=zxd.device, dtype=torch.float32)
        _ext.ops().ssm_decode(*batch.desc, zxd, w, bias, ring, dt_bias, a_log, d_skip, state, y, groups)
        return y
    xbc = ssm_conv(batch, zxd[:, inner:inner + C], w, bias, ring)
    y = ssd_scan(batch, xbc, zxd[:, inner + C:], dt_bias, a_log, d_skip, state, groups)
    return y.float() * F.silu(zxd[:, :inner].float())


def gated_group_norm(y, z, gamma, parts: int, eps: float, dtype) -> torch.Tensor:
    """RMS norm over ``parts`` equal pieces of ``y silu(z)`` (``z`` None: y is gated already), times ``gamma``."""
    rows, D = y.shape
    if y.is_cuda:
        out = torch.empty(rows, D, device=y.device, dtype=dtype)
        _ext.ops().gated_group_norm(y, z, gamma, parts, eps, out)
        return out
    g = y.float() if z is None else y.float() * F.silu(z.float())
    g = g.reshape(rows, parts, D // parts)
    g = g * torch.rsqrt(g.square().mean(-1, keepdim=True) + eps)
    return (g.reshape(rows, D) * gamma).to(dtype)
