"""Experts chosen by a table over token ids, each with weight 1 / top, and the clamped gated activation

    g = min(gate, limit), u = clamp(up, -limit, limit), g * sigmoid(alpha g) * (u + 1).

Few tokens (decode), fp32 and odd widths run on two kernels that stream the chosen experts' rows and add straight into
the fp32 residual; larger bf16 batches sort the rows by expert on the device and run the grouped GEMM of
ops/grouped_gemm.py (weights stored (E, out, in)) between gather, activation and combine kernels.
"""
from __future__ import annotations

import torch

from .. import _ext

GROUPED_MIN_ROWS = 64        # (token, choice) pairs from which the grouped GEMM pays


def clamped_glu_ref(gate, up, limit: float, alpha: float):
    g = gate.float().clamp(max=limit)
    u = up.float().clamp(-limit, limit)
    return g * torch.sigmoid(alpha * g) * (u + 1.0)


def table_moe(h, tokens, table, w_gate_up, w_down, limit: float, alpha: float, out) -> torch.Tensor:
    """h (M, D); tokens (M,) int32; table (vocab, top) int32; w_gate_up (E, 2 I, D), w_down (E, D, I). Adds the layer's
    output to ``out`` (M, D) fp32."""
    M, D = h.shape
    E, two_i, _ = w_gate_up.shape
    I, top = two_i // 2, table.shape[1]
    if not h.is_cuda:
        idx = table[tokens.long()].long()
        for j in range(top):
            gu = torch.einsum("mkd,md->mk", w_gate_up[idx[:, j]].float(), h.float())
            act = clamped_glu_ref(gu[:, :I], gu[:, I:], limit, alpha).to(h.dtype).float()
            out += torch.einsum("mdk,mk->md", w_down[idx[:, j]].float(), act) / top
        return out
    ops = _ext.ops()
    grouped = h.dtype == torch.bfloat16 and D % 8 == 0 and I % 8 == 0 and M * top >= GROUPED_MIN_ROWS
    if not grouped:
        act = torch.empty(M * top, I, device=h.device, dtype=h.dtype)
        ops.table_experts(h, tokens, table, w_gate_up, w_down, limit, alpha, act, out)
        return out
    idx = table.index_select(0, tokens).reshape(-1)
    counts = torch.empty(E, device=h.device, dtype=torch.int32)
    pos = torch.empty(M * top, device=h.device, dtype=torch.int32)
    ops.moe_prepare(idx, counts, pos)
    ends = counts.cumsum(0, dtype=torch.int32)
    xs = torch.empty(M * top, D, device=h.device, dtype=h.dtype)
    row_of = torch.empty(M * top, device=h.device, dtype=torch.int32)
    ops.moe_gather_rows(h, idx, pos, ends, counts, top, xs, row_of)
    gu = torch._grouped_mm(xs, w_gate_up.transpose(1, 2), offs=ends)
    act = torch.empty(M * top, I, device=h.device, dtype=h.dtype)
    ops.clamped_glu(gu, limit, alpha, act)
    ys = torch._grouped_mm(act, w_down.transpose(1, 2), offs=ends)
    ops.moe_combine_rows(ys, row_of, top, 1.0 / top, out)
    return out
