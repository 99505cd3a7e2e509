"""Munazen forward pass on packed batches (one function per layer kind; prefill, continuation and decode are one code path whose
operations pick the form that fits the batch).

    x_1 = .. = x_S = embed[token]                                                   fp32 streams throughout
    y = sublayer(norm(sum_s in[s] x_s));   x_t <- sum_s mix[s, t] x_s + out[t] y    mixer, then feed-forward, per layer run
    logits = head(norm(sum_s x_s))

Everything between two sublayers (bias, streams, next combination, group norm) is one kernel. Parallel layers: one projection for both
branches; attention operands and cache row in one kernel, attention on the tcgen05 flash kernel, the paged decode kernel or the any-size
kernel; the recurrent unit from convolution to gated output on a second stream; both branches write the row that one output projection reads. Gated linear
attention: one projection, the scan, then norm and output gate in one kernel.
"""
from __future__ import annotations

from typing import List, Optional

import torch

from ...cache.hybrid import HybridPagedCache
from ...ops import linear_attention as LIN
from ...ops import rotated_kv as RKV
from ...ops.gated_lru import gated_lru
from ...ops.gemm import linear_rows
from ...ops.packed import PackedBatch, embed_bigram, seq_begin
from ...ops.rope import rope_tables
from ...ops.streams import Connection, group_norm_rows, poly_norm, stream_norm
from ...utils.overlap import beside
from ...utils.profiling import scope
from ..step_engine import forward_tokens, generate_tokens
from .config import GatedLinear, MunazenConfig, Parallel


def make_cache(config: MunazenConfig, n_pages: int, max_seqs: int, max_pages_per_seq: int, dtype=torch.bfloat16,
               device="cpu") -> HybridPagedCache:
    c = config
    mixers = [c.layers[i].mixer for i in c.runs]
    par = [m for m in mixers if isinstance(m, Parallel)]
    return HybridPagedCache([m.left.width for m in par],
                            [(m.right.width,) if isinstance(m, Parallel) else (m.heads, m.dim, m.vdim) for m in mixers],
                            [(m.right.conv, m.right.width) if isinstance(m, Parallel) else None for m in mixers],
                            n_pages, c.page_size, max_seqs, max_pages_per_seq, dtype, device)


def make_rope(config: MunazenConfig, n_pos: int, device="cpu") -> list:
    """Per layer the rotary tables of (queries and keys, values), None for layers without attention; equal ones are shared."""
    made = {}

    def tables(dims, base, scaling):
        key = (dims, base, scaling)
        if key not in made:
            made[key] = rope_tables(dims, base, n_pos, dict(scaling) if scaling else None, device)
        return made[key]
    out = []
    for l in config.layers:
        a = l.mixer.left if isinstance(l.mixer, Parallel) else None
        out.append(None if a is None else (tables(a.rot.dims, a.rot.base, a.rot.scaling), tables(a.vdim, a.rot.base, None)))
    return out


# ---- mixers: normed input (N, D) -> output (N, D) in the activation dtype ----------------------------------------------
def parallel_mixer(h, mp, m: Parallel, batch: PackedBatch, cache: HybridPagedCache, layer: int, run: int, rope):
    """``layer`` counts attention runs, ``run`` all runs. The output projection's bias is left to the streams' kernel."""
    a, W = m.left, m.right.width
    (cq, ck, cv, cx, cy, cg), _ = m.segments()
    y = linear_rows(h, mp["in"])
    both = torch.empty(h.shape[0], a.heads * a.vdim + W, device=h.device, dtype=h.dtype)
    lru_done = beside(h.device, lambda: gated_lru(batch, y[:, cx:cx + W], y[:, cy:cy + W], mp["lru"], cache.rings[run], cache.states[run],
                                                  m.right_scale, both[:, -W:]))
    wide = RKV.flash_widths(batch, h.dtype, h.is_cuda, a.dim, a.vdim)
    q, k, v = RKV.qkv_rotate(batch, y, (cq, ck, cv), mp["qkv_b"], a.heads, a.kv_heads, a.dim, a.vdim, rope[0], rope[1], cache.paged, layer, wide)
    o = RKV.causal_attention(batch, q, k, v, cache.paged, layer, a.kv_heads, a.vdim, a.scale)
    RKV.turn_back_gate(batch, o, y[:, cg:cg + a.heads], rope[1], m.left_scale, both[:, :-W])
    lru_done()
    return linear_rows(both, mp["o"])


def gla_mixer(h, mp, m: GatedLinear, batch: PackedBatch, cache: HybridPagedCache, run: int, eps):
    qkv, inner, rank = 2 * m.heads * m.dim + m.heads * m.vdim, m.heads * m.vdim, mp["a2"].shape[1]
    y = linear_rows(h, mp["in"])
    g0 = (qkv + 7) // 8 * 8
    a0 = g0 + (inner + 7) // 8 * 8
    s = LIN.linear_scan(batch, y[:, :qkv], cache.states[run], channels=LIN.ChannelDecay(y[:, a0:a0 + rank], mp["a2"], mp["a2_b"], m.tau),
                        q_scale=m.dim ** -0.5)
    return linear_rows(LIN.head_norm_gate(batch, s, y[:, g0:g0 + inner], mp["norm"], m.heads, eps, h.dtype, silu=True), mp["o"])


def feed_forward(h, f, eps):
    return linear_rows(poly_norm(linear_rows(h, f["up"]), f["act"], eps), f["down"])


# ------------------------------------------------------------------------------------------------
@torch.no_grad()
def run_layers(params, config: MunazenConfig, cache: HybridPagedCache, batch: PackedBatch, tokens: torch.Tensor, rope,
               layers_out: Optional[list] = None) -> torch.Tensor:
    """One step: tokens (N,) int32, packed. Returns the fp32 sum of the streams (N, D) after the last layer; the cache's device state
    (rows, recurrent state, lengths) includes the step's tokens. The caller reserves pages before and advances the host mirrors after
    (``PagedCache.begin_step`` / ``end_step``). ``layers_out`` collects the sum of the streams after every layer run."""
    c = config
    act, eps, groups = params["embed"].dtype, c.norm_eps, c.norm_groups
    layers, ones = params["layers"], params["ones"]
    subs = []                                       # (run, which sublayer) in the order they run
    for r, i in enumerate(c.runs):
        subs += [(r, i, 1)] + ([(r, i, 2)] if c.layers[i].mlp is not None else [])
    seq_begin(batch, tokens, cache.paged.seq_lens, cache.prev)
    y, done, bias = embed_bigram(batch, tokens, params["embed"]), Connection(ones, None, ones), None
    xs = torch.empty(batch.n_tok, c.streams, c.width, device=y.device, dtype=torch.float32)
    n_attn = 0
    for k in range(len(subs) + 1):
        last = k == len(subs)
        lp, which = (None, 0) if last else (layers[subs[k][1]], subs[k][2])
        h, u = stream_norm(y, xs, done, ones if last else lp[f"hc{which}"].w_in, None if last else lp[f"norm{which}"], groups, eps, act,
                           bias=bias, want_u=last)
        if layers_out is not None and k > 0 and (last or which == 1):
            layers_out.append(xs.sum(1))
        if last:
            return u
        r, i, _ = subs[k]
        m, done, bias = c.layers[i].mixer, lp[f"hc{which}"], None
        if which == 2:
            with scope("ffn"):
                y = feed_forward(h, lp["mlp"], eps)
        elif isinstance(m, Parallel):
            with scope("parallel"):
                y, bias = parallel_mixer(h, lp["mix"], m, batch, cache, n_attn, r, rope[i]), lp["mix"]["o_b"]
            n_attn += 1
        else:
            with scope("gla"):
                y = gla_mixer(h, lp["mix"], m, batch, cache, r, eps)


def output_logits(params, config: MunazenConfig, x: torch.Tensor) -> torch.Tensor:
    """fp32 logits of rows of the streams' sum."""
    with scope("output_head"):
        return linear_rows(group_norm_rows(x, params["final_norm"], config.norm_groups, config.norm_eps, params["embed"].dtype),
                           params["head"], f32_out=True)


def init_params(config: MunazenConfig, key: int = 0, dtype=torch.float32, device="cpu", on_device: bool = False) -> dict:
    """Random parameters (``on_device``: drawn on ``device``)."""
    from .weight_loader import load_from_state_dict, random_state_dict
    return load_from_state_dict(random_state_dict(config, int(key), device=device if on_device else "cpu"), config, dtype, device)


def forward(params, tokens, config: MunazenConfig, cache: Optional[HybridPagedCache] = None, seq_ids: Optional[List] = None,
            is_decode: bool = False):
    """tokens (B, T) -> logits (B, T, V), see ``step_engine.forward_tokens``; ``is_decode`` is accepted for signature parity
    with the other families."""
    from .engine import MunazenEngine
    return forward_tokens(MunazenEngine, params, tokens, config, cache, seq_ids)


def generate(params, prompt_tokens, config: MunazenConfig, max_new_tokens: int, temperature: float = 0.0,
             top_k: Optional[int] = None, key=None, cache: Optional[HybridPagedCache] = None, use_cuda_graph: bool = True):
    """Continuation (B, max_new_tokens), see ``step_engine.generate_tokens``."""
    from .engine import MunazenEngine
    return generate_tokens(MunazenEngine, params, prompt_tokens, config, max_new_tokens, temperature, top_k, key, cache, use_cuda_graph)
