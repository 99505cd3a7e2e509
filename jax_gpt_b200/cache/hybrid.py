"""Cache of models that mix paged attention layers with recurrent layers: pages for the attention rows, one slot of
fixed-size state per sequence for the recurrent layers, and the last token of every sequence (bigram embeddings).

A sequence owns a slot from ``acquire`` to ``release``; its pages, lengths and recurrent state are addressed by the slot
number. State is never cleared: the kernels ignore a slot's state for a sequence that starts at position 0.
"""
from __future__ import annotations

from typing import Dict, Hashable, List, Optional, Sequence, Tuple

import torch

from .paged import PagedCache


class HybridPagedCache:
    def __init__(self, widths: Sequence[int], state_shapes: Sequence[Tuple[int, ...]], ring_shapes: Sequence[Optional[Tuple[int, ...]]],
                 n_pages: int, page_size: int, max_seqs: int, max_pages_per_seq: int, dtype=torch.bfloat16, device="cpu",
                 vec_shapes: Sequence[Optional[Tuple[int, ...]]] = (), blocks: Sequence[int] = ()):
        """``widths``: row width of every attention layer; ``state_shapes`` / ``ring_shapes`` / ``vec_shapes``: per recurrent
        layer the shape of one sequence's state, of its ring of past inputs (None: none) and of what else it carries (a normaliser and
        a running maximum; None: nothing). All fp32. ``blocks``: per attention layer the size of token blocks whose mean rows are
        kept (0: none)."""
        self.paged = PagedCache(len(widths), list(widths), n_pages, page_size, max_seqs, max_pages_per_seq, dtype, device, blocks=blocks)
        self.states = [torch.zeros(max_seqs, *s, dtype=torch.float32, device=device) for s in state_shapes]
        self.rings = [None if s is None else torch.zeros(max_seqs, *s, dtype=torch.float32, device=device) for s in ring_shapes]
        self.vecs = [None if s is None else torch.zeros(max_seqs, *s, dtype=torch.float32, device=device) for s in vec_shapes]
        self.prev = torch.zeros(max_seqs, dtype=torch.int32, device=device)
        self.max_seqs, self.page_size, self.max_pages = max_seqs, page_size, max_pages_per_seq
        self._slots: Dict[Hashable, int] = {}
        self._free: List[int] = list(range(max_seqs - 1, -1, -1))

    @property
    def device(self):
        return self.paged.device

    @property
    def max_len(self) -> int:
        return self.max_pages * self.page_size

    @property
    def n_free_slots(self) -> int:
        return len(self._free)

    def acquire(self, seq: Hashable) -> int:
        if seq in self._slots:
            raise ValueError(f"sequence {seq!r} already holds a slot")
        if not self._free:
            raise MemoryError(f"all {self.max_seqs} sequence slots are in use")
        self._slots[seq] = self._free.pop()
        return self._slots[seq]

    def slot(self, seq: Hashable) -> int:
        return self._slots[seq]

    def __contains__(self, seq: Hashable) -> bool:
        return seq in self._slots

    def length(self, seq: Hashable) -> int:
        return self.paged.length(self._slots[seq])

    def release(self, seq: Hashable) -> None:
        slot = self._slots.pop(seq)
        self.paged.release(slot)
        self._free.append(slot)
