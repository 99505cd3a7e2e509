"""Vobunex forward pass on packed batches (one function per layer kind; prefill, continuation and decode are one code
path whose operations pick the form that fits the batch).

    x = embed[token] + bigram[previous, token]                       fp32 residual throughout
    x += mixer(layer_norm(x));   x += feed_forward(layer_norm(x))    per layer
    logits = head(layer_norm(x))

Latent attention: whole prompts with heads of 128 + 64 run decompressed on the tcgen05 flash kernel, decode steps over
the 512 + 64 latent on the tcgen05 paged kernel, every other case on the any-size paged kernel with absorbed weights.
Mamba-2: prefill = convolution, chunked (tcgen05) or token-by-token recurrence, gated norm; decode = one fused kernel
and the gated norm. Projections back into the residual accumulate in fp32 from the GEMM's epilogue.
"""
from __future__ import annotations

from typing import List, Optional

import torch

from ...cache.hybrid import HybridPagedCache
from ...ops import latent_attention as LA
from ...ops import ssm
from ...ops.gemm import linear_rows
from ...ops.norm import LAYERNORM
from ...ops.packed import PackedBatch, embed_bigram, norm_rows, seq_begin
from ...ops.rope import rope_tables
from ...ops.table_moe import table_moe
from ...utils.profiling import scope
from ..step_engine import forward_tokens, generate_tokens
from .config import GLU_ALPHA, DenseMlp, LatentAttention, VobunexConfig


def make_cache(config: VobunexConfig, n_pages: int, max_seqs: int, max_pages_per_seq: int, dtype=torch.bfloat16,
               device="cpu") -> HybridPagedCache:
    c = config
    ssm_mixers = [c.layers[i].mixer for i in c.ssm_layers]
    return HybridPagedCache([c.layers[i].mixer.width for i in c.attention_layers],
                            [(m.heads, m.state, m.vdim) for m in ssm_mixers], [(m.conv, m.conv_dim) for m in ssm_mixers],
                            n_pages, c.page_size, max_seqs, max_pages_per_seq, dtype, device)


def make_rope(config: VobunexConfig, n_pos: int, device="cpu") -> list:
    """Rotary tables of every attention layer (layers with the same rotation share one pair)."""
    made = {}
    out = []
    for i in config.attention_layers:
        r = config.layers[i].mixer.rot
        if r not in made:
            made[r] = rope_tables(r.dims, r.base, n_pos, dict(r.scaling) if r.scaling else None, device)
        out.append(made[r])
    return out


def latent_attention_mixer(h, mp, m: LatentAttention, batch: PackedBatch, cache: HybridPagedCache, layer: int, rope, eps, x):
    """Adds the mixer's output for the normed input ``h`` to the residual ``x``; ``layer`` counts attention layers."""
    flash = LA.flash_ok(batch, h, m.dim, m.rot_dim, m.vdim, m.kv_rank)
    y = linear_rows(h, mp["down"])
    cq, lat = LA.mla_prepare(batch, y, mp["q_norm"], mp["kv_norm"], eps, rope, cache.paged, layer, want_latent=flash)
    q = linear_rows(cq, mp["uq"]).view(h.shape[0], m.heads, m.dim + m.rot_dim)
    o = LA.attend(batch, q, lat, mp["ukv"], m.kv_rank, m.vdim, rope, cache.paged, layer, m.scale, mp["sink"])
    linear_rows(o, mp["o"], out=x, accumulate=True)


def mamba2_mixer(h, mp, m, batch: PackedBatch, cache: HybridPagedCache, layer: int, eps, x):
    """``layer`` counts recurrent layers."""
    ring, state = cache.rings[layer], cache.states[layer]
    zxd = linear_rows(h, mp["in"])                                    # (N, z | x | B | C | dt)
    inner, C = m.inner, m.conv_dim
    if batch.single:
        y = ssm.ssm_decode(batch, zxd, mp["conv"], mp["conv_b"], ring, mp["dt_bias"], mp["A_log"], mp["D"], state, m.groups)
        g = ssm.gated_group_norm(y, None, mp["norm"], m.norm_groups, eps, h.dtype)
    else:
        xbc = ssm.ssm_conv(batch, zxd[:, inner:inner + C], mp["conv"], mp["conv_b"], ring)
        y = ssm.ssd_scan(batch, xbc, zxd[:, inner + C:], mp["dt_bias"], mp["A_log"], mp["D"], state, m.groups)
        g = ssm.gated_group_norm(y, zxd[:, :inner], mp["norm"], m.norm_groups, eps, h.dtype)
    linear_rows(g, mp["o"], out=x, accumulate=True)


def feed_forward(h, fp, f, tokens, x):
    if isinstance(f, DenseMlp):
        linear_rows(linear_rows(h, fp["up"], act="relu2"), fp["down"], out=x, accumulate=True)
    else:
        table_moe(h, tokens, fp["table"], fp["gate_up"], fp["down"], f.limit, GLU_ALPHA, x)


# ------------------------------------------------------------------------------------------------
@torch.no_grad()
def run_layers(params, config: VobunexConfig, cache: HybridPagedCache, batch: PackedBatch, tokens: torch.Tensor, rope,
               layers_out: Optional[list] = None) -> torch.Tensor:
    """One step: tokens (N,) int32, packed. Returns the fp32 residual (N, D) after the last layer; the cache's device
    state (rows, recurrent state, lengths, last tokens) includes the step's tokens. The caller reserves pages before
    and advances the host mirrors after (``PagedCache.begin_step`` / ``end_step``). ``layers_out`` collects the
    residual after every layer."""
    c = config
    act = params["embed"].dtype
    seq_begin(batch, tokens, cache.paged.seq_lens, cache.prev)
    big = c.bigram
    x = embed_bigram(batch, tokens, params["embed"], params["bigram"], big.mul_prev if big else 0, big.mul_cur if big else 0)
    n_attn = n_ssm = 0
    for layer, lp in zip(c.layers, params["layers"]):
        h = norm_rows(LAYERNORM, x, lp["norm1"], lp["norm1_b"], c.norm_eps, act)
        if isinstance(layer.mixer, LatentAttention):
            with scope("latent_attention"):
                latent_attention_mixer(h, lp["mix"], layer.mixer, batch, cache, n_attn, rope[n_attn], c.norm_eps, x)
            n_attn += 1
        else:
            with scope("mamba2"):
                mamba2_mixer(h, lp["mix"], layer.mixer, batch, cache, n_ssm, c.norm_eps, x)
            n_ssm += 1
        if layer.mlp is not None:
            with scope("ffn"):
                h = norm_rows(LAYERNORM, x, lp["norm2"], lp["norm2_b"], c.norm_eps, act)
                feed_forward(h, lp["mlp"], layer.mlp, tokens, x)
        if layers_out is not None:
            layers_out.append(x.clone())
    return x


def output_logits(params, config: VobunexConfig, x: torch.Tensor) -> torch.Tensor:
    """fp32 logits of residual rows."""
    with scope("output_head"):
        return linear_rows(norm_rows(LAYERNORM, x, params["final_norm"], params["final_norm_b"], config.norm_eps,
                                     params["embed"].dtype), params["head"], f32_out=True)


def init_params(config: VobunexConfig, key: int = 0, dtype=torch.float32, device="cpu", on_device: bool = False) -> dict:
    """Random parameters (``on_device``: drawn on ``device``)."""
    from .weight_loader import load_from_state_dict, random_state_dict
    return load_from_state_dict(random_state_dict(config, int(key), device=device if on_device else "cpu"), config, dtype, device)


def forward(params, tokens, config: VobunexConfig, cache: Optional[HybridPagedCache] = None, seq_ids: Optional[List] = None,
            is_decode: bool = False):
    """tokens (B, T) -> logits (B, T, V), see ``step_engine.forward_tokens``; ``is_decode`` is accepted for signature parity
    with the other families."""
    from .engine import VobunexEngine
    return forward_tokens(VobunexEngine, params, tokens, config, cache, seq_ids)


def generate(params, prompt_tokens, config: VobunexConfig, max_new_tokens: int, temperature: float = 0.0,
             top_k: Optional[int] = None, key=None, cache: Optional[HybridPagedCache] = None, use_cuda_graph: bool = True):
    """Continuation (B, max_new_tokens), see ``step_engine.generate_tokens``."""
    from .engine import VobunexEngine
    return generate_tokens(VobunexEngine, params, prompt_tokens, config, max_new_tokens, temperature, top_k, key, cache, use_cuda_graph)
