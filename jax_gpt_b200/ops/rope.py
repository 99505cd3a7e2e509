"""Fused per-head RMSNorm + partial rotary embedding (kernels of csrc/seq_kernels.cu).

PyTorch references: ``rms_norm`` / ``apply_rotary_emb`` of models/qwen35/primitives.py (the
semantics of jax_gpt/models/qwen35/primitives.py:29-32,79-109).
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import _ext



def rmsnorm_rope_ref(x, norm_w, freqs, rope_dim: int, pos0: int = 0, eps: float = 1e-6, one_plus: bool = True):
    """x (B,T,H,dh); freqs (n_pos, rope_dim/2, 2)."""
    from ..models.qwen35.primitives import apply_rotary_emb
    xf = x.float()
    if norm_w is not None:
        xf = xf * torch.rsqrt((xf * xf).mean(-1, keepdim=True) + eps) * ((1.0 + norm_w.float()) if one_plus else norm_w.float())
    if rope_dim:
        xf = apply_rotary_emb(xf, freqs[pos0:pos0 + x.shape[1]], rope_dim)
    return xf.to(x.dtype)


class _RmsnormRopeFn(torch.autograd.Function):
    """Forward and backward on the fused kernels (per-head RMSNorm with (1 + w) or w gain, partial half-split rotary)."""

    @staticmethod
    def forward(ctx, x, norm_w, freqs, rope_dim, pos0, eps, one_plus):
        B, T, H, dh = x.shape
        xc = x.contiguous().view(B * T, H, dh)
        y = torch.empty_like(xc)
        fr = freqs.contiguous() if freqs is not None else None
        _ext.ops().rmsnorm_rope(xc, norm_w, fr, y, T, rope_dim, pos0, eps, one_plus)
        ctx.save_for_backward(xc, norm_w, fr)
        ctx.meta = (B, T, H, dh, rope_dim, pos0, eps, one_plus)
        return y.view(B, T, H, dh)

    @staticmethod
    def backward(ctx, dy):
        xc, norm_w, fr = ctx.saved_tensors
        B, T, H, dh, rope_dim, pos0, eps, one_plus = ctx.meta
        dyc = dy.contiguous().view(B * T, H, dh)
        dx = torch.empty_like(xc)
        dw = torch.zeros(dh, device=xc.device, dtype=torch.float32) if norm_w is not None else None
        _ext.ops().rmsnorm_rope_bwd(xc, dyc, norm_w, fr, dx, dw, T, rope_dim, pos0, eps, one_plus)
        return dx.view(B, T, H, dh), (dw.to(norm_w.dtype) if dw is not None else None), None, None, None, None, None


def rmsnorm_rope(x, norm_w, freqs, rope_dim: int, pos0: int = 0, eps: float = 1e-6, one_plus: bool = True):
    B, T, H, dh = x.shape
    per = dh // 32 if dh % 32 == 0 else 0
    ok = (x.is_cuda and x.dtype == torch.bfloat16 and per and dh <= 256 and
          (rope_dim == 0 or ((rope_dim // 2) % per == 0)))
    if not ok or (norm_w is not None and norm_w.dtype != torch.bfloat16):
        return rmsnorm_rope_ref(x, norm_w, freqs, rope_dim, pos0, eps, one_plus)
    if torch.is_grad_enabled() and (x.requires_grad or (norm_w is not None and norm_w.requires_grad)):
        return _RmsnormRopeFn.apply(x, norm_w, freqs, rope_dim, pos0, eps, one_plus)
    xc = x.contiguous().view(B * T, H, dh)
    y = torch.empty_like(xc)
    _ext.ops().rmsnorm_rope(xc, norm_w, freqs.contiguous() if freqs is not None else None, y, T, rope_dim, pos0, eps, one_plus)
    return y.view(B, T, H, dh)


# ---- interleaved rotation with optional YaRN scaling ---------------------------------------------------------------
def yarn_frequencies(dims: int, base: float, scaling=None):
    """(frequencies [dims / 2] as Python floats, factor of cos and sin). ``scaling`` is None or a mapping with
    ``factor``, ``original``, ``fast``, ``slow``: pairs that turn more than ``fast`` times over ``original`` positions
    keep their frequency, pairs that turn fewer than ``slow`` times are slowed by ``factor``, a linear ramp in between
    (Peng et al., "YaRN: Efficient Context Window Extension of Large Language Models")."""
    import math
    freqs = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return freqs, 1.0
    factor = float(scaling["factor"])
    edge = lambda turns: dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(edge(scaling["fast"])), 0)
    hi = min(math.ceil(edge(scaling["slow"])), dims - 1)
    width = max(hi - lo, 0.001)
    ramp = [min(max((i - lo) / width, 0.0), 1.0) for i in range(dims // 2)]
    return [f / factor * r + f * (1.0 - r) for f, r in zip(freqs, ramp)], 0.1 * math.log(factor) + 1.0


def banded_frequencies(dims: int, base: float, scaling=None):
    """Frequencies [dims / 2] as Python floats. ``scaling`` is None or a mapping with ``factor``, ``low``, ``high``,
    ``original``: waves shorter than original / high keep their frequency, waves longer than original / low are slowed by
    ``factor``, those between are blended linearly in original / wavelength (the Llama 3.1 rule)."""
    import math
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling:
            turns = scaling["original"] * f / (2.0 * math.pi)       # original / wavelength
            low, high = scaling["low"], scaling["high"]
            keep = 1.0 if turns > high else 0.0 if turns < low else (turns - low) / (high - low) if high > low else 1.0
            f = keep * f + (1.0 - keep) * f / scaling["factor"]
        out.append(f)
    return out


def rope_tables(dims: int, base: float, n_pos: int, scaling=None, device="cpu"):
    """(cos, sin) [n_pos, dims / 2] fp32; angles are taken in fp64 before rounding. The scaling's keys tell its kind: YaRN
    (``fast``, ``slow``; the amplitude is folded in) or wavelength bands (``low``, ``high``)."""
    if scaling and "low" in scaling:
        freqs, amp = banded_frequencies(dims, base, scaling), 1.0
    else:
        freqs, amp = yarn_frequencies(dims, base, scaling)
    ang = torch.arange(n_pos, dtype=torch.float64)[:, None] * torch.tensor(freqs, dtype=torch.float64)[None, :]
    return (ang.cos() * amp).float().to(device).contiguous(), (ang.sin() * amp).float().to(device).contiguous()


def rotate_interleaved(x: torch.Tensor, pos: torch.Tensor, tables) -> torch.Tensor:
    """x (N, ..., d): the first ``dims`` features turn in pairs (2i, 2i + 1) by the angles of position ``pos[n]``."""
    cos, sin = tables
    dims = 2 * cos.shape[1]
    if dims == 0:
        return x
    shape = [x.shape[0]] + [1] * (x.dim() - 2) + [dims // 2]
    c, s = cos[pos.long()].reshape(shape), sin[pos.long()].reshape(shape)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    turned = torch.stack([u * c - v * s, v * c + u * s], dim=-1).flatten(-2)
    return torch.cat([turned, x[..., dims:]], dim=-1)


def pair_order(width: int, dims: int) -> torch.Tensor:
    """Order of ``width`` features that turns half-split pairs (i, i + dims / 2) into interleaved ones (2i, 2i + 1); the features
    from ``dims`` on stay. Query and key weights reordered by it give the same scores."""
    half = dims // 2
    return torch.cat([torch.stack([torch.arange(half), torch.arange(half) + half], 1).flatten(), torch.arange(dims, width)])


def rotate_half_split(x: torch.Tensor, pos: torch.Tensor, tables) -> torch.Tensor:
    """x (N, ..., d): of the first ``dims`` features, i and i + dims / 2 turn together by the angles of position ``pos[n]``."""
    cos, sin = tables
    half = cos.shape[1]
    if half == 0:
        return x
    shape = [x.shape[0]] + [1] * (x.dim() - 2) + [half]
    c, s = cos[pos.long()].reshape(shape), sin[pos.long()].reshape(shape)
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], dim=-1)
