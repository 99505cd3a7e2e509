"""Experts chosen by a sigmoid router: the ``top`` experts of the largest scores, each fed with the token times its score
(scores not renormalised), outputs summed; a shared expert runs for every token."""
from __future__ import annotations

import torch

from .. import _ext
from .expert_mlp import SILU_GLU, experts_ref, grouped_experts, stream_experts, use_grouped
from .gemm import linear_rows, silu_glu_rows


def sigmoid_topk(logits: torch.Tensor, top: int):
    """(ids (M, top) int32, scores (M, top) fp32) of the largest sigmoid scores, in falling order."""
    if logits.is_cuda:
        ids = torch.empty(logits.shape[0], top, device=logits.device, dtype=torch.int32)
        w = torch.empty(logits.shape[0], top, device=logits.device, dtype=torch.float32)
        _ext.ops().sigmoid_topk(logits, ids, w)
        return ids, w
    z, ids = logits.topk(top, dim=-1)
    return ids.int(), torch.sigmoid(z)


def sigmoid_moe(h, router, top: int, w_gate_up, w_down, shared_gate_up, shared_down) -> torch.Tensor:
    """h (M, D); router (E, D); w_gate_up (E, 2 I, D), w_down (E, D, I); shared_gate_up (2 I', D), shared_down (D, I').
    Returns the layer's output (M, D) fp32."""
    logits = linear_rows(h, router, f32_out=True)
    out = linear_rows(silu_glu_rows(h, shared_gate_up), shared_down, f32_out=True)
    if not h.is_cuda:
        ids, w = sigmoid_topk(logits, top)
        return experts_ref(h, ids.long(), w_gate_up, w_down, SILU_GLU, out, weights=w)
    if use_grouped(h, w_down, top):
        ids, w = sigmoid_topk(logits, top)
        return grouped_experts(h, ids.view(-1), top, w_gate_up, w_down, SILU_GLU, out, w_pair=w.view(-1))
    return stream_experts(h, top, w_gate_up, w_down, SILU_GLU, out, logits=logits)
