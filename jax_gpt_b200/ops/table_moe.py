"""Experts chosen by a table over token ids, each with weight 1 / top, and the clamped gated activation

    g = min(gate, limit), u = clamp(up, -limit, limit), g * sigmoid(alpha g) * (u + 1).
"""
from __future__ import annotations

import torch

from .expert_mlp import GROUPED_MIN_ROWS, Glu, experts_ref, glu_ref, grouped_experts, stream_experts, use_grouped  # noqa: F401


def clamped_glu_ref(gate, up, limit: float, alpha: float):
    return glu_ref(gate, up, Glu(limit, alpha, 1.0))


def table_moe(h, tokens, table, w_gate_up, w_down, limit: float, alpha: float, out) -> torch.Tensor:
    """h (M, D); tokens (M,) int32; table (vocab, top) int32; w_gate_up (E, 2 I, D), w_down (E, D, I). Adds the layer's
    output to ``out`` (M, D) fp32."""
    top, glu = table.shape[1], Glu(limit, alpha, 1.0)
    if not h.is_cuda:
        return experts_ref(h, table[tokens.long()].long(), w_gate_up, w_down, glu, out, 1.0 / top)
    if use_grouped(h, w_down, top):
        return grouped_experts(h, table.index_select(0, tokens).reshape(-1), top, w_gate_up, w_down, glu, out, 1.0 / top)
    return stream_experts(h, top, w_gate_up, w_down, glu, out, tokens=tokens, table=table)
