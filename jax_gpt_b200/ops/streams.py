"""Several parallel residual streams on packed rows (hyper-connections; Zhu et al., "Hyper-Connections"), norms over groups of
features, and row-wise polynomial activations. Kernels: csrc/stream_kernels.cu; CPU tensors take the PyTorch restatements.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from .. import _ext


@dataclass
class Connection:
    """How one sublayer meets the streams (fp32): ``w_in`` [S] combines them to its input, ``mix`` [S, S] ([from, to]) and
    ``w_out`` [S] make the new streams of the old ones and its output."""
    w_in: torch.Tensor
    mix: Optional[torch.Tensor]
    w_out: torch.Tensor


def group_norm_ref(x, gamma, groups: int, eps: float):
    p = x.reshape(*x.shape[:-1], groups, -1)
    return (p * torch.rsqrt(p.square().mean(-1, keepdim=True) + eps)).reshape(x.shape) * gamma


def stream_norm(y: torch.Tensor, xs: torch.Tensor, done: Connection, w_in: torch.Tensor, gamma: Optional[torch.Tensor], groups: int,
                eps: float, dtype, bias: Optional[torch.Tensor] = None, want_u: bool = False):
    """What lies between two sublayers: the output ``y`` (N, D) (+ ``bias``) of the sublayer ``done`` enters the fp32 streams
    ``xs`` (N, S, D) in place (``done.mix`` None: they start with it), then ``u = sum_s w_in[s] xs[:, s]``. Returns (RMS norm of
    u over ``groups`` equal pieces times ``gamma`` in ``dtype`` or None without ``gamma``, u in fp32 if ``want_u``)."""
    N, S, D = xs.shape
    if xs.is_cuda:
        h = torch.empty(N, D, device=xs.device, dtype=dtype) if gamma is not None else None
        u = torch.empty(N, D, device=xs.device, dtype=torch.float32) if want_u else None
        _ext.ops().stream_norm(y, xs, bias, done.mix, done.w_out, w_in, gamma, groups, eps, h, u)
        return h, u
    v = y.float() + (0.0 if bias is None else bias)
    old = torch.einsum("st,nsd->ntd", done.mix, xs) if done.mix is not None else 0.0
    xs.copy_(old + done.w_out[:, None] * v[:, None, :])
    u = torch.einsum("s,nsd->nd", w_in, xs)
    return group_norm_ref(u, gamma, groups, eps).to(dtype) if gamma is not None else None, u if want_u else None


def poly_norm(z: torch.Tensor, coef: torch.Tensor, eps: float) -> torch.Tensor:
    """``c0 N(z) + c1 N(z^2) + c2 N(z^3) + c3`` with N(v) = v / sqrt(mean(v^2) + eps) over a row (PolyNorm of Zhuo et al.,
    "Polynomial Composition Activations: Unleashing the Dynamics of Large Language Models"); ``coef`` fp32 (4)."""
    if z.is_cuda:
        out = torch.empty(z.shape, device=z.device, dtype=z.dtype)
        _ext.ops().poly_norm(z, coef, eps, out)
        return out
    f = z.float()
    n = lambda v: v * torch.rsqrt(v.square().mean(-1, keepdim=True) + eps)
    return (coef[0] * n(f) + coef[1] * n(f * f) + coef[2] * n(f * f * f) + coef[3]).to(z.dtype)


def group_norm_rows(x: torch.Tensor, gamma: torch.Tensor, groups: int, eps: float, dtype) -> torch.Tensor:
    """RMS norm of fp32 rows (N, D) over ``groups`` equal pieces, times ``gamma``, in ``dtype``."""
    one = torch.ones(1, dtype=torch.float32, device=x.device)
    return stream_norm(x, torch.empty(x.shape[0], 1, x.shape[1], dtype=torch.float32, device=x.device), Connection(one, None, one), one,
                       gamma, groups, eps, dtype)[0]
