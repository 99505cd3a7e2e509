"""Real-gated linear recurrent unit (De et al., "Griffin: Mixing Gated Linear Recurrences with Local Attention for Efficient
Language Models") on packed batches: a causal depthwise convolution with carried inputs, block-diagonal gates and a diagonal
recurrence. Kernels: csrc/gated_lru.cu. State per cache slot: ``ring`` [slots, taps, W] fp32 with the convolution input of
position p in row ``p % taps``, ``state`` [slots, W] fp32; a sequence that starts at position 0 ignores both.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch
import torch.nn.functional as F

from .. import _ext
from .gemm import gelu_tanh
from .packed import PackedBatch


@dataclass
class LruWeights:
    """``x_bias``, ``y_bias`` (W), ``conv`` (W, taps), ``conv_bias`` (W), ``gates`` (blocks, 2, W / blocks, W / blocks) =
    [recurrence, input] gate as (out, in) in the activation dtype, ``gates_bias`` (blocks, 2, W / blocks), ``decay`` (W):
    log a = -decay * recurrence gate. fp32 but for the gates."""
    x_bias: torch.Tensor
    y_bias: torch.Tensor
    conv: torch.Tensor
    conv_bias: torch.Tensor
    gates: torch.Tensor
    gates_bias: torch.Tensor
    decay: torch.Tensor


def gated_lru(batch: PackedBatch, x, y, w: LruWeights, ring, state, scale: float, out) -> None:
    """``out = scale * S * gelu(y + y_bias)`` with S_t = a S_(t-1) + sqrt(1 - a^2) i u of the convolved ``x + x_bias`` (N, W);
    ``ring`` and ``state`` are advanced. ``out`` (N, W) may be a column slice."""
    N, W = x.shape
    if x.is_cuda:
        _ext.ops().gated_lru(*batch.desc, x, w.x_bias, w.conv, w.conv_bias, ring, w.gates, w.gates_bias, w.decay, state, y, w.y_bias,
                             scale, out)
        return
    taps = w.conv.shape[1]
    nb = w.gates.shape[0]
    for c0, n, slot, start in batch.rows():
        xin = x[c0:c0 + n].float() + w.x_bias
        past = [ring[slot, p % taps] if p >= 0 else torch.zeros(W) for p in range(start - taps + 1, start)]
        seq = torch.cat([torch.stack(past), xin]) if past else xin
        u = w.conv_bias + sum(seq[k:k + n] * w.conv[:, k] for k in range(taps))
        g = torch.einsum("nbk,bgok->gnbo", u.reshape(n, nb, -1), w.gates.float()) + w.gates_bias.transpose(0, 1)[:, None]
        r, i = torch.sigmoid(g).reshape(2, n, W)
        la = -w.decay * r
        inp = torch.sqrt(-torch.expm1(2 * la)) * i * u
        S = state[slot].clone() if start > 0 else torch.zeros(W)
        gate = gelu_tanh(y[c0:c0 + n].float() + w.y_bias)
        for t in range(n):
            S = torch.exp(la[t]) * S + inp[t]
            out[c0 + t] = (scale * S * gate[t]).to(out.dtype)
        state[slot] = S
        for t in range(max(0, n - taps + 1), n):
            ring[slot, (start + t) % taps] = xin[t]


def lru_decay(lam: torch.Tensor, rate: float = 8.0) -> torch.Tensor:
    """``decay`` of ``LruWeights`` from the stored parameter."""
    return rate * F.softplus(lam.float())
