"""Gated expert layers whose experts are already chosen or scored, shared by the table and the router layers.

Few tokens (decode), fp32 and odd widths run on two kernels that stream the chosen experts' rows and add straight into the
fp32 result; larger bf16 batches sort the rows by expert on the device and run the library grouped GEMM (weights stored
(E, out, in)) between gather, activation and combine kernels of csrc/serve_kernels.cu.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .. import _ext

GROUPED_MIN_ROWS = 64        # (token, choice) pairs from which the grouped GEMM pays


@dataclass(frozen=True)
class Glu:
    """g = min(gate, limit), u = clamp(up, -limit, limit): g sigmoid(alpha g) (u + shift)."""
    limit: float = float("inf")
    alpha: float = 1.0
    shift: float = 0.0


SILU_GLU = Glu()


def glu_ref(gate, up, glu: Glu):
    g = gate.float().clamp(max=glu.limit)
    u = up.float().clamp(-glu.limit, glu.limit)
    return g * torch.sigmoid(glu.alpha * g) * (u + glu.shift)


def use_grouped(h, w_down, top: int) -> bool:
    return (h.is_cuda and h.dtype == torch.bfloat16 and h.shape[1] % 8 == 0 and w_down.shape[2] % 8 == 0
            and h.shape[0] * top >= GROUPED_MIN_ROWS)


def grouped_experts(h, idx, top: int, w_gate_up, w_down, glu: Glu, out, out_scale: float = 1.0, w_pair=None) -> torch.Tensor:
    """idx (M * top,) int32 experts; ``w_pair`` (M * top,) fp32 scales the experts' inputs, ``out_scale`` the summed output.
    Adds to ``out`` (M, D) fp32."""
    M, D = h.shape
    E, I = w_gate_up.shape[0], w_down.shape[2]
    ops, dev = _ext.ops(), h.device
    counts = torch.empty(E, device=dev, dtype=torch.int32)
    pos = torch.empty(M * top, device=dev, dtype=torch.int32)
    ops.moe_prepare(idx, counts, pos)
    ends = counts.cumsum(0, dtype=torch.int32)
    xs = torch.empty(M * top, D, device=dev, dtype=h.dtype)
    row_of = torch.empty(M * top, device=dev, dtype=torch.int32)
    w_row = torch.empty(M * top, device=dev, dtype=torch.float32) if w_pair is not None else None
    ops.moe_gather_rows(h, idx, pos, ends, counts, top, xs, row_of, w_pair, w_row)
    gu = torch._grouped_mm(xs, w_gate_up.transpose(1, 2), offs=ends)
    act = torch.empty(M * top, I, device=dev, dtype=h.dtype)
    ops.clamped_glu(gu, glu.limit, glu.alpha, glu.shift, w_row, act)
    ys = torch._grouped_mm(act, w_down.transpose(1, 2), offs=ends)
    ops.moe_combine_rows(ys, row_of, top, out_scale, out)
    return out


def stream_experts(h, top: int, w_gate_up, w_down, glu: Glu, out, *, tokens=None, table=None, logits=None) -> torch.Tensor:
    """Experts by ``table[tokens]`` (mean of the outputs) or by the ``top`` largest of ``logits`` (M, E) fp32 (sigmoid scores
    scale the inputs, outputs are summed). Adds to ``out`` (M, D) fp32."""
    act = torch.empty(h.shape[0] * top, w_down.shape[2], device=h.device, dtype=h.dtype)
    _ext.ops().stream_experts(h, tokens, table, logits, top, w_gate_up, w_down, glu.limit, glu.alpha, glu.shift, act, out)
    return out


def experts_ref(h, idx, w_gate_up, w_down, glu: Glu, out, out_scale: float = 1.0, weights=None) -> torch.Tensor:
    """PyTorch restatement; idx (M, top), weights (M, top) of the experts' inputs."""
    I = w_down.shape[2]
    for j in range(idx.shape[1]):
        gu = torch.einsum("mkd,md->mk", w_gate_up[idx[:, j]].float(), h.float())
        if weights is not None:
            gu = gu * weights[:, j:j + 1]
        act = glu_ref(gu[:, :I], gu[:, I:], glu).to(h.dtype).float()
        out += torch.einsum("mdk,mk->md", w_down[idx[:, j]].float(), act) * out_scale
    return out
