"""Mopalorn forward pass on packed batches (one function per layer kind; prefill, continuation and decode are one code path whose
operations pick the form that fits the batch).

    x = embed[token]                                                 fp32 residual throughout
    x += norm(mixer(norm(x)));   x += norm(feed_forward(norm(x)))    per layer
    logits = scale * embed norm(x)

Every "post-norm, add to the residual, next pre-norm" is one kernel. Latent attention: one projection for queries, latent, rotary key and
gate; cache rows in one kernel, then the windowed tcgen05 flash kernel (whole prompts), the tcgen05 paged kernel (decode) or the any-size
kernel, the gate in what follows it. Grouped attention: one projection; query factor, value mixing, cache row and block means in one
kernel (two for prompts with blocks), then the flash kernel, the paged decode kernel or the any-size kernel. Feed-forward: the activation
is the up projection's epilogue.
"""
from __future__ import annotations

from typing import List, Optional

import torch

from ...cache.hybrid import HybridPagedCache
from ...ops import latent_attention as LA
from ...ops import window_attention as WA
from ...ops.gemm import linear_rows
from ...ops.mixed_kv import mixed_kv, query_factors
from ...ops.norm import RMSNORM
from ...ops.packed import PackedBatch, embed_bigram, norm_rows, residual_norm_rows, seq_begin
from ...ops.rope import rope_tables
from ...utils.profiling import scope
from ..step_engine import forward_tokens, generate_tokens
from .config import GroupedAttention, LatentAttention, MopalornConfig


def make_cache(config: MopalornConfig, n_pages: int, max_seqs: int, max_pages_per_seq: int, dtype=torch.bfloat16,
               device="cpu") -> HybridPagedCache:
    mixers = [l.mixer for l in config.layers]
    return HybridPagedCache([m.width for m in mixers], (), (), n_pages, config.page_size, max_seqs, max_pages_per_seq, dtype, device,
                            blocks=[getattr(m, "pool", 0) for m in mixers])


def make_rope(config: MopalornConfig, n_pos: int, device="cpu") -> list:
    """What a layer needs by position: rotary tables, query factors or nothing; equal ones are shared."""
    made = {}
    make = {LatentAttention: lambda r: rope_tables(r.dims, r.base, n_pos, None, device),
            GroupedAttention: lambda t: query_factors(*t, n_pos, device) if t else None}
    out = []
    for l in config.layers:
        kind, key = type(l.mixer), l.mixer.rot if isinstance(l.mixer, LatentAttention) else l.mixer.q_temp
        if (kind, key) not in made:
            made[kind, key] = make[kind](key)
        out.append(made[kind, key])
    return out


# ---- mixers: normed input (N, D) -> output (N, D) in the activation dtype ----------------------------------------------
def latent_attention_mixer(h, mp, m: LatentAttention, batch: PackedBatch, cache: HybridPagedCache, layer: int, rope, eps):
    (cq, cl, cg), _ = m.segments()
    flash = LA.flash_ok(batch, h, m.dim, m.rot_dim, m.vdim, m.kv_rank)
    y = linear_rows(h, mp["in"])
    _, lat = LA.mla_prepare(batch, y[:, cl:cl + m.width], None, mp["kv_norm"], eps, rope, cache.paged, layer, want_latent=flash)
    q = y[:, cq:cq + m.heads * (m.dim + m.rot_dim)].unflatten(-1, (m.heads, m.dim + m.rot_dim))
    o = LA.attend(batch, q, lat, mp["ukv"], m.kv_rank, m.vdim, rope, cache.paged, layer, m.scale, window=m.window or WA.NO_WINDOW,
                  gate=y[:, cg:cg + m.heads * m.vdim])
    return linear_rows(o, mp["o"])


def grouped_attention_mixer(h, mp, m: GroupedAttention, batch: PackedBatch, cache: HybridPagedCache, layer: int, factors, v_first):
    """Returns (output, the layer's own values (N, G dv) before mixing)."""
    cols, _ = m.segments()
    y = linear_rows(h, mp["in"])
    wide = WA.flash_widths(batch, h.dtype, h.is_cuda, m.dim, m.vdim)
    window = m.window or WA.NO_WINDOW
    q, k, v = mixed_kv(batch, y, cols, m.heads, m.kv_heads, m.dim, m.vdim, cache.paged, layer, wide, factors, v_first, mp["vmix"], window)
    o = WA.grouped_attention(batch, q, k, v, cache.paged, layer, m.kv_heads, m.vdim, m.scale, window, softcap=m.softcap, sink=mp["sink"],
                             pool=m.pool)
    return linear_rows(o[..., :m.vdim].reshape(o.shape[0], m.heads * m.vdim), mp["o"]), y[:, cols[2]:cols[2] + m.kv_heads * m.vdim]


def feed_forward(h, f):
    return linear_rows(linear_rows(h, f["up"], act="xielu", act_args=f["act"]), f["down"])


# ------------------------------------------------------------------------------------------------
@torch.no_grad()
def run_layers(params, config: MopalornConfig, cache: HybridPagedCache, batch: PackedBatch, tokens: torch.Tensor, rope,
               layers_out: Optional[list] = None) -> torch.Tensor:
    """One step: tokens (N,) int32, packed. Returns the fp32 residual (N, D) after the last layer; the cache's device state (rows, block
    means, lengths) includes the step's tokens. The caller reserves pages before and advances the host mirrors after
    (``PagedCache.begin_step`` / ``end_step``). ``layers_out`` collects the residual after every layer."""
    c = config
    act, eps, layers = params["embed"].dtype, c.norm_eps, params["layers"]
    seq_begin(batch, tokens, cache.paged.seq_lens, cache.prev)
    x = embed_bigram(batch, tokens, params["embed"])
    h = norm_rows(RMSNORM, x, layers[0]["norm1"], None, eps, act) if layers else None
    v_first = None
    for i, (layer, lp) in enumerate(zip(c.layers, layers)):
        m = layer.mixer
        if isinstance(m, LatentAttention):
            with scope("latent_attention"):
                y = latent_attention_mixer(h, lp["mix"], m, batch, cache, i, rope[i], eps)
        else:
            with scope("pooled_attention" if m.pool else "full_attention"):
                y, values = grouped_attention_mixer(h, lp["mix"], m, batch, cache, i, rope[i], v_first if m.v_mix else None)
            if i == c.first_values:
                v_first = values
        following = layers[i + 1]["norm1"] if i + 1 < len(layers) else None
        h = residual_norm_rows(y, lp["norm1b"], x, lp["norm2"] if layer.mlp else following, eps, act)
        if layer.mlp is not None:
            with scope("ffn"):
                y = feed_forward(h, lp["mlp"])
            h = residual_norm_rows(y, lp["norm2b"], x, following, eps, act)
        if layers_out is not None:
            layers_out.append(x.clone())
    return x


def output_logits(params, config: MopalornConfig, x: torch.Tensor) -> torch.Tensor:
    """fp32 logits of residual rows; the embeddings are the output matrix, their scale is in the norm's gain."""
    with scope("output_head"):
        return linear_rows(norm_rows(RMSNORM, x, params["final_norm"], None, config.norm_eps, params["embed"].dtype), params["embed"],
                           f32_out=True)


def init_params(config: MopalornConfig, key: int = 0, dtype=torch.float32, device="cpu", on_device: bool = False) -> dict:
    """Random parameters (``on_device``: drawn on ``device``)."""
    from .weight_loader import load_from_state_dict, random_state_dict
    return load_from_state_dict(random_state_dict(config, int(key), device=device if on_device else "cpu"), config, dtype, device)


def forward(params, tokens, config: MopalornConfig, cache: Optional[HybridPagedCache] = None, seq_ids: Optional[List] = None,
            is_decode: bool = False):
    """tokens (B, T) -> logits (B, T, V), see ``step_engine.forward_tokens``; ``is_decode`` is accepted for signature parity
    with the other families."""
    from .engine import MopalornEngine
    return forward_tokens(MopalornEngine, params, tokens, config, cache, seq_ids)


def generate(params, prompt_tokens, config: MopalornConfig, max_new_tokens: int, temperature: float = 0.0,
             top_k: Optional[int] = None, key=None, cache: Optional[HybridPagedCache] = None, use_cuda_graph: bool = True):
    """Continuation (B, max_new_tokens), see ``step_engine.generate_tokens``."""
    from .engine import MopalornEngine
    return generate_tokens(MopalornEngine, params, prompt_tokens, config, max_new_tokens, temperature, top_k, key, cache, use_cuda_graph)
