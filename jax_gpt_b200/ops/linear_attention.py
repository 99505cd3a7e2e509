"""Linear attention with a matrix state per head on packed batches: ``S_t = a_t S_(t-1) + b_t k_t v_t^T``, ``o_t = S_t^T q_t``
with a fixed decay per head, a decay per key channel (gated linear attention), or with exponential gates, a running maximum
and a normaliser (mLSTM).

Kernels: csrc/linear_attention.cu (token by token, one-token step, norm and output gate), csrc/ssd_scan_sm100.cu (chunked on
tcgen05), csrc/gla_chunk.cu (chunked, decays per key channel). State per cache slot: ``state`` [slots, H, N, P] fp32; gated layers also carry ``vec`` [slots, H, N + 1] fp32 = the
normaliser and the running maximum, both scaled by exp(-maximum). A sequence that starts at position 0 ignores them.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn.functional as F

from .. import _ext
from .packed import PackedBatch

TOKENS, STEP, CHUNKED = 0, 1, 2


@dataclass
class Gates:
    """Exponential gates of one layer and step: ``raw`` (N, 2 H) fp32 = [input | forget] before ``bias`` (2 H) and the cap."""
    raw: torch.Tensor
    bias: torch.Tensor
    cap: float
    vec: torch.Tensor


@dataclass
class ChannelDecay:
    """Decay per key channel from a low-rank projection: log alpha = log sigmoid(``low`` (N, R) ``w``^T + ``bias``) / ``tau`` with
    ``w`` (H N', R) in the activation dtype and ``bias`` (H N') fp32."""
    low: torch.Tensor
    w: torch.Tensor
    bias: torch.Tensor
    tau: float

    def log_alpha(self) -> torch.Tensor:
        return F.logsigmoid(self.low.float() @ self.w.float().t() + self.bias) / self.tau


@dataclass
class Numerators:
    """What a scan leaves for ``head_norm_gate``: y (N, H P) and, for gated layers, the denominators' parts and the advanced
    normaliser (moved to its slot by ``head_norm_gate``)."""
    y: torch.Tensor
    den: Optional[torch.Tensor] = None
    vec_new: Optional[torch.Tensor] = None
    vec: Optional[torch.Tensor] = None


def chunked_ok(batch: PackedBatch, x: torch.Tensor, N: int, P: int) -> bool:
    """True when the chunked tensor-core form takes a layer of key width N and value width P."""
    return x.is_cuda and x.dtype == torch.bfloat16 and not batch.single and N == 128 and P % 64 == 0


def channels_chunked_ok(batch: PackedBatch, x: torch.Tensor, N: int, P: int, rank: int) -> bool:
    """The same for a decay per key channel (csrc/gla_chunk.cu)."""
    return (x.is_cuda and x.dtype == torch.bfloat16 and not batch.single and N % 16 == 0 and N <= 128 and P % 8 == 0 and rank <= 64
            and x.stride(0) % 8 == 0 and x.data_ptr() % 16 == 0)


def log_gates(raw, bias, cap: float):
    """(log input gate, log forget gate), each (N, H)."""
    i, f = (cap * torch.tanh((raw + bias) / cap)).chunk(2, -1)
    return i, F.logsigmoid(f)


def linear_scan(batch: PackedBatch, qkv, state, *, decay=None, gates: Optional[Gates] = None,
                channels: Optional[ChannelDecay] = None, q_scale: float = 1.0, silu: bool = False,
                kind: Optional[int] = None) -> Numerators:
    """qkv (N, 2 H N' + H P) = [q | k | v]; one of ``decay`` (H), ``gates``, ``channels``; ``silu``: they still need their activation (the chunked form wants it applied).
    ``state`` is advanced. ``kind``: None picks the one-token step, the chunked or the token-by-token form."""
    H, Nk, P = state.shape[1:]
    N = batch.n_tok
    if qkv.is_cuda:
        if kind is None:
            chunked = not silu and (chunked_ok(batch, qkv, Nk, P) if channels is None else
                                    channels_chunked_ok(batch, qkv, Nk, P, channels.w.shape[1]))
            kind = STEP if batch.single else CHUNKED if chunked else TOKENS
        new = lambda *s: torch.empty(*s, device=qkv.device, dtype=torch.float32)
        y = torch.empty(N, H * P, device=qkv.device, dtype=torch.bfloat16) if kind == CHUNKED else new(N, H * P)
        if channels is not None:
            _ext.ops().linear_scan(*batch.desc, qkv, None, None, None, 1.0, None, None, None, state, y, q_scale, silu, kind,
                                   channels.low, channels.w, channels.bias, 1.0 / channels.tau)
            return Numerators(y)
        if gates is None:
            _ext.ops().linear_scan(*batch.desc, qkv, decay, None, None, 1.0, None, None, None, state, y, q_scale, silu, kind)
            return Numerators(y)
        den, vec_new = new(N, H, 4), new(batch.n_seq, H, Nk + 1)
        _ext.ops().linear_scan(*batch.desc, qkv, None, gates.raw, gates.bias, gates.cap, gates.vec, vec_new, den, state, y, q_scale,
                               silu, kind)
        return Numerators(y, den, vec_new, gates.vec)
    x = qkv.float()
    x = F.silu(x).to(qkv.dtype).float() if silu else x
    y = torch.empty(N, H * P)
    den, vec_new = torch.zeros(N, H, 4), torch.empty(batch.n_seq, H, Nk + 1)
    if gates is not None:
        gi, gf = log_gates(gates.raw, gates.bias, gates.cap)
    if channels is not None:
        alpha = torch.exp(channels.log_alpha()).reshape(N, H, Nk, 1)
    for b, (c0, n, slot, start) in enumerate(batch.rows()):
        S = state[slot].clone() if start > 0 else torch.zeros(H, Nk, P)
        nv, m = torch.zeros(H, Nk), torch.zeros(H)
        if gates is not None and start > 0:
            nv, m = gates.vec[slot, :, :Nk].clone(), gates.vec[slot, :, Nk].clone()
        for t in range(c0, c0 + n):
            q, k, v = (p.reshape(H, -1) for p in x[t].split([H * Nk, H * Nk, H * P]))
            a, w = decay, torch.ones(H)
            if channels is not None:
                a = alpha[t]
            if gates is not None:
                mn = torch.maximum(gf[t] + m, gi[t])
                a, w, m = torch.exp(gf[t] + m - mn), torch.exp(gi[t] - mn), mn
                nv = a[:, None] * nv + w[:, None] * k
                den[t, :, 0], den[t, :, 2] = (nv * q).sum(-1) * q_scale, torch.exp(-m)
            S = (a if channels is not None else a[:, None, None]) * S + (w[:, None] * k)[:, :, None] * v[:, None, :]
            y[t] = (torch.einsum("hnp,hn->hp", S, q) * q_scale).reshape(-1)
        state[slot] = S
        vec_new[b, :, :Nk], vec_new[b, :, Nk] = nv, m
    return Numerators(y) if gates is None else Numerators(y, den, vec_new, gates.vec)


def head_norm_gate(batch: PackedBatch, s: Numerators, z, gamma, parts: int, eps: float, dtype, den_eps: float = 1e-6,
                   silu: bool = False) -> torch.Tensor:
    """RMS norm over ``parts`` equal pieces of the scan's output (gated layers: after the division by the denominator), times
    ``gamma`` and sigmoid(z) (``silu``: silu(z)). Gated layers hand the advanced normaliser on to its slot here."""
    N, D = s.y.shape
    if s.y.is_cuda:
        out = torch.empty(N, D, device=s.y.device, dtype=dtype)
        _ext.ops().head_norm_gate(*batch.desc, s.y, z, gamma, parts, eps, s.den, den_eps, s.vec_new, s.vec, out, silu)
        return out
    y = s.y.reshape(N, parts, D // parts)
    if s.den is not None:
        y = y / (torch.maximum((s.den[..., 0] + s.den[..., 1]).abs(), s.den[..., 2]) + den_eps)[..., None]
        for b, slot in enumerate(batch.ids.tolist()):
            s.vec[slot] = s.vec_new[b]
    y = y * torch.rsqrt(y.square().mean(-1, keepdim=True) + eps)
    return (y.reshape(N, D) * gamma * (F.silu(z.float()) if silu else torch.sigmoid(z.float()))).to(dtype)
