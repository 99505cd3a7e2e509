"""Packed (ragged) batches: the tokens of one step, one sequence after the other, without padding.

A step brings some new tokens for every sequence of a batch. Row ``n`` of every activation is one token; sequence ``b``
owns rows ``cu[b] .. cu[b+1]-1`` and its first row sits at position ``start[b]``, which the device reads from (and
advances in) the cache's length vector, so a captured step needs no host value. On CUDA the operations are the kernels of
csrc/serve_kernels.cu; CPU tensors take the PyTorch restatements below (tests of the host logic).
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import List, Optional

import torch

from .. import _ext
from .norm import LAYERNORM, RMSNORM, norm_ref


@dataclass
class PackedBatch:
    seq_ids: List[int]                 # cache slots (host)
    lens: List[int]                    # new tokens of every sequence (host)
    fresh: bool                        # every sequence starts at position 0 (host)
    max_len: int                       # bound of any sequence's length after this step (host)
    ids: torch.Tensor = field(repr=False)       # int32 device copies
    cu: torch.Tensor = field(repr=False)
    tok_seq: torch.Tensor = field(repr=False)
    start: torch.Tensor = field(repr=False)     # written by seq_begin
    prev_tok: torch.Tensor = field(repr=False)  # written by seq_begin: the token before each sequence's first row
    made: dict = field(default_factory=dict, repr=False)

    @property
    def n_tok(self) -> int:
        return self.tok_seq.shape[0]

    @property
    def n_seq(self) -> int:
        return len(self.seq_ids)

    @property
    def single(self) -> bool:
        """One token per sequence: the decode form of every layer applies."""
        return self.n_tok == self.n_seq

    @property
    def desc(self):
        return self.ids, self.cu, self.tok_seq, self.start

    @staticmethod
    def make(seq_ids, lens, fresh: bool, max_len: int, device) -> "PackedBatch":
        B, N = len(seq_ids), sum(lens)
        cu = [0]
        for n in lens:
            cu.append(cu[-1] + n)
        tok = [b for b, n in enumerate(lens) for _ in range(n)]
        host = torch.tensor(list(seq_ids) + cu + tok, dtype=torch.int32)
        dev = host.to(device)          # one upload
        z = torch.zeros(2, B, dtype=torch.int32, device=device)
        return PackedBatch(list(seq_ids), list(lens), fresh, max_len, dev[:B].clone(), dev[B:2 * B + 1].clone(),
                           dev[2 * B + 1:2 * B + 1 + N].clone(), z[0].clone(), z[1].clone())

    def memo(self, key, make):
        """What ``make()`` derives from the batch's host description, made once."""
        if key not in self.made:
            self.made[key] = make()
        return self.made[key]

    # ---- host views of the device description (restatements on CPU tensors) ----
    def rows(self):
        """(first row, number of rows, slot, start position) of every sequence."""
        out = []
        for b, s in enumerate(self.ids.tolist()):
            c0, c1 = int(self.cu[b]), int(self.cu[b + 1])
            out.append((c0, c1 - c0, s, int(self.start[b])))
        return out

    def positions(self) -> torch.Tensor:
        t = torch.arange(self.n_tok, device=self.cu.device)
        b = self.tok_seq.long()
        return self.start.long()[b] + t - self.cu.long()[b]


def seq_begin(batch: PackedBatch, tokens: torch.Tensor, lens: torch.Tensor, prev: torch.Tensor) -> None:
    """Start positions and preceding tokens of the batch from the per-slot state, which then counts the step's tokens."""
    if tokens.is_cuda:
        _ext.ops().seq_begin(batch.ids, batch.cu, tokens, lens, prev, batch.start, batch.prev_tok)
        return
    for b, s in enumerate(batch.ids.tolist()):
        n = int(batch.cu[b + 1] - batch.cu[b])
        batch.start[b] = lens[s]
        batch.prev_tok[b] = prev[s]
        lens[s] += n
        prev[s] = tokens[int(batch.cu[b + 1]) - 1]


def embed_bigram(batch: PackedBatch, tokens, embed, bigram=None, mul_prev: int = 0, mul_cur: int = 0) -> torch.Tensor:
    """fp32 rows ``embed[token]``, plus with a ``bigram`` table [buckets + 1, D] the row
    ``(previous * mul_prev + token * mul_cur) mod buckets``, or the last row for the first token of a sequence."""
    if tokens.is_cuda:
        x = torch.empty(batch.n_tok, embed.shape[1], device=embed.device, dtype=torch.float32)
        _ext.ops().embed_bigram(*batch.desc, tokens, batch.prev_tok, embed, bigram, mul_prev, mul_cur, x)
        return x
    x = embed[tokens.long()].float()
    if bigram is not None:
        buckets = bigram.shape[0] - 1
        prev = torch.cat([tokens[:1], tokens[:-1]]).long()
        prev[batch.cu[:-1].long()] = batch.prev_tok.long()
        row = (prev * mul_prev + tokens.long() * mul_cur) % buckets
        row = torch.where(batch.positions() == 0, torch.full_like(row, buckets), row)
        x = x + bigram[row].float()
    return x


def norm_rows(mode: int, x: torch.Tensor, gamma: torch.Tensor, beta: Optional[torch.Tensor], eps: float, dtype) -> torch.Tensor:
    """Layer norm (``ops.norm.LAYERNORM``) or RMS norm of an fp32 residual, fp32 parameters, result in ``dtype``."""
    if x.is_cuda:
        out = torch.empty(x.shape, device=x.device, dtype=dtype)
        _ext.ops().norm_rows(0 if mode == LAYERNORM else 1, x, gamma, beta, out, eps)
        return out
    return norm_ref(mode, x, gamma, beta, eps).to(dtype)


def residual_norm_rows(y: torch.Tensor, gamma_post: torch.Tensor, x: torch.Tensor, gamma_next: Optional[torch.Tensor], eps: float,
                       dtype, add: bool = True) -> Optional[torch.Tensor]:
    """A sublayer's output ``y`` through its post-norm into the fp32 residual, and the next sublayer's normed input, in one
    pass: ``x (+)= rms(y) gamma_post`` in place (``add`` False: assigned), returns ``rms(x) gamma_next`` in ``dtype`` (None
    without ``gamma_next``)."""
    out = torch.empty(x.shape, device=x.device, dtype=dtype) if gamma_next is not None else None
    if x.is_cuda:
        _ext.ops().residual_norm(y, gamma_post, x, add, gamma_next, out, eps)
        return out
    r = norm_ref(RMSNORM, y.float(), gamma_post, None, eps)
    x.copy_(x + r if add else r)
    return norm_ref(RMSNORM, x, gamma_next, None, eps).to(dtype) if out is not None else None
