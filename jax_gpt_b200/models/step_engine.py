"""Step engine of the model families that run on packed batches (batches of sequences through one step function, decode
steps as CUDA-graph replays), and the ``forward`` / ``generate`` entry points built on it.

``step`` takes the next tokens of every sequence (prompts, continuations or single tokens, mixed lengths, packed without
padding) and returns the logits of the wanted rows. ``decode`` is the one-token step: everything it needs is on the
device (slots, positions, block table, last tokens), so the whole token step of a batch size is captured in a CUDA graph
at its second use and replayed afterwards; the first use runs eagerly and loads the kernels. The host only reserves the
page of the next token and uploads the block table when a sequence got one.

A family subclasses ``StepEngine`` and names its functions:

    make_cache(config, n_pages, max_seqs, max_pages_per_seq, dtype, device) -> HybridPagedCache
    make_rope(config, n_pos, device) -> whatever ``run_layers`` wants
    run_layers(params, config, cache, batch, tokens, rope, layers_out) -> fp32 residual rows
    output_logits(params, config, rows) -> fp32 logits
"""
from __future__ import annotations

from typing import Dict, Hashable, List, Optional, Sequence

import torch

from ..cache.hybrid import HybridPagedCache
from ..ops.packed import PackedBatch


class _DecodeSlot:
    """Static buffers and the captured step of one batch size."""

    def __init__(self, B: int, max_len: int, device):
        self.batch = PackedBatch.make([0] * B, [1] * B, False, max_len, device)
        self.tokens = torch.zeros(B, dtype=torch.int32, device=device)
        self.slots: Optional[List[int]] = None       # what batch.ids holds
        self.logits = None
        self.graph = None
        self.warm = False


class StepEngine:
    make_cache = make_rope = run_layers = output_logits = None       # staticmethods of the family

    def __init__(self, params: dict, config, cache: Optional[HybridPagedCache] = None, *, max_tokens: int = 4096,
                 max_seqs: int = 64, use_cuda_graph: bool = True):
        """Without a ``cache`` one is made for ``max_tokens`` live tokens in at most ``max_seqs`` sequences."""
        self.params, self.config = params, config
        self.device, self.dtype = params["embed"].device, params["embed"].dtype
        if cache is None:
            per = (max_tokens + config.page_size - 1) // config.page_size
            cache = self.make_cache(config, per + max_seqs, max_seqs, per + 1, self.dtype, self.device)
        self.cache = cache
        self.rope = self.make_rope(config, cache.max_len, self.device)
        self.use_graph = use_cuda_graph and self.device.type == "cuda"
        self._decode: Dict[int, _DecodeSlot] = {}
        if self.device.type == "cuda" and self.dtype == torch.float32:
            torch.backends.cuda.matmul.allow_tf32 = False      # fp32 means fp32

    # ---- sequences -----------------------------------------------------------------------------------
    def release(self, seq: Hashable) -> None:
        """Gives back the pages and the state slot of a finished sequence."""
        self.cache.release(seq)

    def _slots(self, seqs: Sequence[Hashable]) -> List[int]:
        if len(set(seqs)) != len(seqs):
            raise ValueError("a sequence may appear once per step")
        return [self.cache.slot(s) if s in self.cache else self.cache.acquire(s) for s in seqs]

    # ---- steps ----------------------------------------------------------------------------------------
    @torch.no_grad()
    def step(self, seqs: Sequence[Hashable], tokens: Sequence[Sequence[int]], want: Optional[Sequence[Sequence[int]]] = None,
             layers_out: Optional[list] = None) -> Optional[torch.Tensor]:
        """``tokens[i]``: the next tokens of ``seqs[i]`` (unknown sequences start at position 0). ``want[i]``: places
        among them whose logits are returned, (rows, V) fp32 in order; None: the last place of every sequence."""
        c = self.config
        lens = [len(t) for t in tokens]
        if not lens or min(lens) < 1:
            raise ValueError("every sequence of a step brings at least one token")
        flat = [int(t) for ts in tokens for t in ts]
        if min(flat) < 0 or max(flat) >= c.vocab_size:
            raise ValueError(f"token ids must be in 0 .. {c.vocab_size - 1}")
        want = [[n - 1] for n in lens] if want is None else want
        if any(not 0 <= w < n for ws, n in zip(want, lens) for w in ws):
            raise ValueError("a wanted place lies outside the step's tokens")
        if layers_out is None and max(lens) == 1 and all(s in self.cache for s in seqs):
            logits = self.decode(seqs, flat)
            rows = [b for b, ws in enumerate(want) for _ in ws]
            return logits if rows == list(range(len(seqs))) else (logits[rows] if rows else None)
        known = [s in self.cache for s in seqs]
        slots = self._slots(seqs)
        paged = self.cache.paged
        starts = [paged.length(s) for s in slots]
        try:
            paged.begin_step(slots, lens)
        except (MemoryError, ValueError):                      # does not fit: the new sequences hold nothing afterwards
            for s, k in zip(seqs, known):
                if not k:
                    self.release(s)
            raise
        batch = PackedBatch.make(slots, lens, not any(starts), max(s + n for s, n in zip(starts, lens)), self.device)
        tok = torch.tensor(flat, dtype=torch.int32).to(self.device)
        x = self.run_layers(self.params, c, self.cache, batch, tok, self.rope, layers_out)
        paged.end_step(slots, lens)
        rows, c0 = [], 0
        for n, ws in zip(lens, want):
            rows += [c0 + w for w in ws]
            c0 += n
        if not rows:
            return None
        if len(rows) != x.shape[0] or rows != list(range(len(rows))):
            x = x[torch.tensor(rows, device=self.device)]
        return self.output_logits(self.params, c, x)

    @torch.no_grad()
    def decode(self, seqs: Sequence[Hashable], tokens) -> torch.Tensor:
        """One token for every (known) sequence: ids as a list or an integer tensor. Returns logits (B, V) fp32; with a
        captured step the buffer is the graph's own and the next ``decode`` of this batch size overwrites it."""
        B = len(seqs)
        slots = [self.cache.slot(s) for s in seqs]
        if len(set(slots)) != B:
            raise ValueError("a sequence may appear once per step")
        d = self._decode.get(B)
        if d is None:
            d = self._decode[B] = _DecodeSlot(B, self.cache.max_len, self.device)
        paged = self.cache.paged
        ones = [1] * B
        paged.begin_step(slots, ones)
        if torch.is_tensor(tokens):
            d.tokens.copy_(tokens.reshape(-1))
        else:
            if min(tokens) < 0 or max(tokens) >= self.config.vocab_size:
                raise ValueError(f"token ids must be in 0 .. {self.config.vocab_size - 1}")
            d.tokens.copy_(torch.tensor(list(tokens), dtype=torch.int32))
        if d.slots != slots:
            d.batch.ids.copy_(torch.tensor(slots, dtype=torch.int32))
            d.slots = slots
        if not self.use_graph or not d.warm:
            d.logits = self._token_step(d)
            d.warm = True
        else:
            if d.graph is None:
                torch.cuda.synchronize(self.device)
                d.graph = torch.cuda.CUDAGraph()
                with torch.cuda.graph(d.graph):
                    d.logits = self._token_step(d)
            d.graph.replay()                                   # capture does not execute
        paged.end_step(slots, ones)
        return d.logits

    def _token_step(self, d: _DecodeSlot) -> torch.Tensor:
        x = self.run_layers(self.params, self.config, self.cache, d.batch, d.tokens, self.rope)
        return self.output_logits(self.params, self.config, x)


# ---- entry points of a family -------------------------------------------------------------------------
@torch.no_grad()
def forward_tokens(engine_class, params, tokens, config, cache: Optional[HybridPagedCache] = None, seq_ids: Optional[List] = None):
    """tokens (B, T) -> logits (B, T, V). Sequences named by ``seq_ids`` continue from the cache when it holds them and
    start at position 0 otherwise."""
    B, T = tokens.shape
    seq_ids = list(range(B)) if seq_ids is None else list(seq_ids)
    if cache is None:
        per = (T + config.page_size - 1) // config.page_size
        cache = engine_class.make_cache(config, B * per, B, per, params["embed"].dtype, tokens.device)
    eng = engine_class(params, config, cache, use_cuda_graph=False)
    return eng.step(seq_ids, tokens.tolist(), want=[list(range(T))] * B).reshape(B, T, -1)


@torch.no_grad()
def generate_tokens(engine_class, params, prompt_tokens, config, max_new_tokens: int, temperature: float = 0.0,
                    top_k: Optional[int] = None, key=None, cache: Optional[HybridPagedCache] = None, use_cuda_graph: bool = True):
    """Continuation (B, max_new_tokens), greedy or sampled. ``prompt_tokens``: (B, T) tensor, or a list of token lists of
    different lengths."""
    from .gpt2.model import sample_logits
    prompts = prompt_tokens.tolist() if torch.is_tensor(prompt_tokens) else [list(p) for p in prompt_tokens]
    device = params["embed"].device
    gen = key if isinstance(key, torch.Generator) else torch.Generator().manual_seed(int(key) if key is not None else 0)
    B = len(prompts)
    if cache is None:
        per = [(len(p) + max_new_tokens + config.page_size - 1) // config.page_size for p in prompts]
        cache = engine_class.make_cache(config, sum(per), B, max(per), params["embed"].dtype, device)
    eng = engine_class(params, config, cache, use_cuda_graph=use_cuda_graph)
    ids = [("gen", b) for b in range(B)]
    logits = eng.step(ids, prompts, want=[[len(p) - 1] for p in prompts])
    out = [sample_logits(logits, temperature, top_k, gen)]
    for _ in range(max_new_tokens - 1):
        out.append(sample_logits(eng.decode(ids, out[-1]), temperature, top_k, gen))
    for i in ids:
        eng.release(i)
    return torch.stack(out, dim=1)
