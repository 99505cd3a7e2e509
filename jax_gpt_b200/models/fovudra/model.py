"""Fovudra forward pass on packed batches (one function per layer kind; prefill, continuation and decode are one code path
whose operations pick the form that fits the batch).

    x = norm(embed[token])                                           fp32 residual throughout
    x += norm(mixer(norm(x)));   x += norm(feed_forward(norm(x)))    per layer
    logits = head(norm(x))

Every "post-norm, add to the residual, next pre-norm" is one kernel. Attention: operands (bias, rotation, unit norm, cache
row) in one kernel, then the tcgen05 flash kernel (whole prompts), the paged decode kernel or the any-size kernel. mLSTM and
lightning attention: one projection, the scan (chunked on tcgen05, token by token, or the one-token step), then norm and
output gate in one kernel. Feed-forward: sigmoid router, experts and the shared expert into one fp32 sum.
"""
from __future__ import annotations

from typing import List, Optional

import torch

from ...cache.hybrid import HybridPagedCache
from ...ops import linear_attention as LIN
from ...ops import window_attention as WA
from ...ops.gemm import linear_rows, linear_rows_f32_tail
from ...ops.norm import RMSNORM
from ...ops.packed import PackedBatch, embed_bigram, norm_rows, residual_norm_rows, seq_begin
from ...ops.rope import rope_tables
from ...ops.sigmoid_moe import sigmoid_moe
from ...utils.profiling import scope
from ..step_engine import forward_tokens, generate_tokens
from .config import DEN_EPS, FovudraConfig, Lightning, MLstm, WindowAttention


def make_cache(config: FovudraConfig, n_pages: int, max_seqs: int, max_pages_per_seq: int, dtype=torch.bfloat16,
               device="cpu") -> HybridPagedCache:
    c = config
    rec = [c.layers[i].mixer for i in c.recurrent_layers]
    return HybridPagedCache([c.layers[i].mixer.width for i in c.attention_layers], [(m.heads, m.dim, m.vdim) for m in rec], (),
                            n_pages, c.page_size, max_seqs, max_pages_per_seq, dtype, device,
                            vec_shapes=[(m.heads, m.dim + 1) if isinstance(m, MLstm) else None for m in rec])


def make_rope(config: FovudraConfig, n_pos: int, device="cpu") -> list:
    """Rotary tables of every attention layer (layers with the same rotation share one pair)."""
    made = {}
    for i in config.attention_layers:
        r = config.layers[i].mixer.rot
        if r not in made:
            made[r] = rope_tables(r.dims, r.base, n_pos, dict(r.scaling) if r.scaling else None, device)
    return [made[config.layers[i].mixer.rot] for i in config.attention_layers]


# ---- mixers: normed input (N, D) -> output (N, D) in the activation dtype ----------------------------------------------
def attention_mixer(h, mp, m: WindowAttention, batch: PackedBatch, cache: HybridPagedCache, layer: int, rope, eps):
    """``layer`` counts attention layers."""
    q, k, v = WA.qk_prepare(batch, linear_rows(h, mp["qk"]), mp["qk_b"], m.heads, m.kv_heads, m.dim, True, eps, rope, cache.paged, layer,
                            dense=WA.flash_ok(batch, h, m.dim))
    o = WA.window_attention(batch, q, k, v, cache.paged, layer, m.kv_heads, m.window, m.keep_first, m.scale)
    return linear_rows(o, mp["o"])


def mlstm_mixer(h, mp, m: MLstm, batch: PackedBatch, cache: HybridPagedCache, layer: int, eps):
    """``layer`` counts recurrent layers."""
    inner = m.heads * m.vdim
    y, raw = linear_rows_f32_tail(h, mp["in"], 2 * m.heads)          # (N, q | k | v | g), fp32 (N, i | f)
    gates = LIN.Gates(raw, mp["gate_b"], m.gate_cap, cache.vecs[layer])
    s = LIN.linear_scan(batch, y[:, :-inner], cache.states[layer], gates=gates, q_scale=m.dim ** -0.5)
    return linear_rows(LIN.head_norm_gate(batch, s, y[:, -inner:], mp["norm"], m.heads, eps, h.dtype, DEN_EPS), mp["o"])


def lightning_mixer(h, mp, m: Lightning, batch: PackedBatch, cache: HybridPagedCache, layer: int, eps):
    """``layer`` counts recurrent layers. The chunked scan takes q, k, v with their SiLU from the projection's epilogue, the
    other forms apply it when they read them."""
    inner = m.heads * m.vdim
    w = mp["in"]
    if LIN.chunked_ok(batch, h, m.dim, m.vdim):
        qkv, g = linear_rows(h, w[:-inner], act="silu"), linear_rows(h, w[-inner:])
        s = LIN.linear_scan(batch, qkv, cache.states[layer], decay=mp["decay"])
    else:
        y = linear_rows(h, w)
        g = y[:, -inner:]
        s = LIN.linear_scan(batch, y[:, :-inner], cache.states[layer], decay=mp["decay"], silu=True)
    return linear_rows(LIN.head_norm_gate(batch, s, g, mp["norm"], 1, eps, h.dtype), mp["o"])


# ------------------------------------------------------------------------------------------------
@torch.no_grad()
def run_layers(params, config: FovudraConfig, cache: HybridPagedCache, batch: PackedBatch, tokens: torch.Tensor, rope,
               layers_out: Optional[list] = None) -> torch.Tensor:
    """One step: tokens (N,) int32, packed. Returns the fp32 residual (N, D) after the last layer; the cache's device state
    (rows, recurrent state, lengths) includes the step's tokens. The caller reserves pages before and advances the host
    mirrors after (``PagedCache.begin_step`` / ``end_step``). ``layers_out`` collects the residual after every layer."""
    c = config
    act, eps = params["embed"].dtype, c.norm_eps
    layers = params["layers"]
    seq_begin(batch, tokens, cache.paged.seq_lens, cache.prev)
    e = embed_bigram(batch, tokens, params["embed"])
    x = torch.empty_like(e)
    h = residual_norm_rows(e, params["embed_norm"], x, layers[0]["norm1"] if layers else None, eps, act, add=False)
    n_attn = n_rec = 0
    for i, (layer, lp) in enumerate(zip(c.layers, layers)):
        m = layer.mixer
        if isinstance(m, WindowAttention):
            with scope("window_attention"):
                y = attention_mixer(h, lp["mix"], m, batch, cache, n_attn, rope[n_attn], eps)
            n_attn += 1
        else:
            with scope("mlstm" if isinstance(m, MLstm) else "lightning"):
                y = (mlstm_mixer if isinstance(m, MLstm) else lightning_mixer)(h, lp["mix"], m, batch, cache, n_rec, eps)
            n_rec += 1
        following = layers[i + 1]["norm1"] if i + 1 < len(layers) else None
        h = residual_norm_rows(y, lp["norm1b"], x, lp["norm2"] if layer.mlp else following, eps, act)
        if layer.mlp is not None:
            with scope("ffn"):
                f = lp["mlp"]
                y = sigmoid_moe(h, f["router"], layer.mlp.top, f["gate_up"], f["down"], f["shared_gate_up"], f["shared_down"])
            h = residual_norm_rows(y, lp["norm2b"], x, following, eps, act)
        if layers_out is not None:
            layers_out.append(x.clone())
    return x


def output_logits(params, config: FovudraConfig, x: torch.Tensor) -> torch.Tensor:
    """fp32 logits of residual rows."""
    with scope("output_head"):
        return linear_rows(norm_rows(RMSNORM, x, params["final_norm"], None, config.norm_eps, params["embed"].dtype), params["head"],
                           f32_out=True)


def init_params(config: FovudraConfig, key: int = 0, dtype=torch.float32, device="cpu", on_device: bool = False) -> dict:
    """Random parameters (``on_device``: drawn on ``device``)."""
    from .weight_loader import load_from_state_dict, random_state_dict
    return load_from_state_dict(random_state_dict(config, int(key), device=device if on_device else "cpu"), config, dtype, device)


def forward(params, tokens, config: FovudraConfig, cache: Optional[HybridPagedCache] = None, seq_ids: Optional[List] = None,
            is_decode: bool = False):
    """tokens (B, T) -> logits (B, T, V), see ``step_engine.forward_tokens``; ``is_decode`` is accepted for signature parity
    with the other families."""
    from .engine import FovudraEngine
    return forward_tokens(FovudraEngine, params, tokens, config, cache, seq_ids)


def generate(params, prompt_tokens, config: FovudraConfig, max_new_tokens: int, temperature: float = 0.0,
             top_k: Optional[int] = None, key=None, cache: Optional[HybridPagedCache] = None, use_cuda_graph: bool = True):
    """Continuation (B, max_new_tokens), see ``step_engine.generate_tokens``."""
    from .engine import FovudraEngine
    return generate_tokens(FovudraEngine, params, prompt_tokens, config, max_new_tokens, temperature, top_k, key, cache, use_cuda_graph)
