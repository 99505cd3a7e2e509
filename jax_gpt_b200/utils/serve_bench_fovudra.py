"""Fovudra's part of the serving benchmark (utils/serve_bench.py): kernels of its layers beside the like kernels of Vobunex and
the Qwen3.5 hybrid, and whole models at equal width, depth, expert count and expert width."""
from __future__ import annotations

import torch

BF = torch.bfloat16


def kernel_table(dev, width: int = 2048, seqs: int = 2, seq_len: int = 4096, decode_batches=(1, 8), ctx: int = 4096,
                 experts: int = 64, top: int = 6, ff: int = 1024, shared_ff: int = 128, heads: int = 16, kv_heads: int = 2,
                 window: int = 1024, keep_first: int = 64) -> dict:
    from .. import _ext
    from ..cache.paged import PagedCache
    from ..ops import attention as A
    from ..ops import linear_attention as LIN
    from ..ops import ssm
    from ..ops import window_attention as WA
    from ..ops.gemm import gemm, linear_f32out, linear_rows, linear_rows_f32_tail, silu_glu_rows
    from ..ops.norm import LAYERNORM
    from ..ops.packed import norm_rows, residual_norm_rows
    from ..ops.rope import rope_tables
    from ..ops.router import softmax_topk_router
    from ..ops.sigmoid_moe import sigmoid_moe, sigmoid_topk
    from .serve_bench import _fused_experts, _KernelTimer, _start_batch
    tm = _KernelTimer(dev)
    ops = _ext.ops()
    rn = lambda *s, dtype=BF: torch.randn(*s, device=dev, dtype=torch.float32).to(dtype)
    f32 = torch.float32
    N, D, K = seqs * seq_len, width, 128
    H = width // K
    inner = H * K
    out = {"prefill": {}, "decode": {}, "prefill_shape": f"{seqs} x {seq_len} tokens, width {width}",
           "decode_shape": f"context {ctx}, window {window} + {keep_first}"}

    def put(part, name, mine, other, other_name):
        part[name] = {"fovudra": mine, "other": other, "other_kernel": other_name,
                      "distance_ratio": round(other["frac"] / max(mine["frac"], 1e-9), 2)}   # > 1: further from the roofline
    pre = out["prefill"]
    batch = _start_batch(list(range(seqs)), [seq_len] * seqs, 0, dev, seq_len)

    # ---- prefill: recurrent layers beside the state-space layer of Vobunex ----
    Ps, Hs, G = 64, 2 * D // 64, 8
    ssd_inner, C = Hs * Ps, Hs * Ps + 2 * G * K
    xbc, zxd = rn(N, C), rn(N, ssd_inner + C + Hs)
    al, dtb, Dk = torch.log(torch.rand(Hs, device=dev) * 7 + 0.5), torch.rand(Hs, device=dev) * 3 - 4, rn(Hs, dtype=f32)
    ssd_state = torch.zeros(seqs, Hs, K, Ps, device=dev)
    nc = N / 128.0
    ssd = tm(lambda: ssm.ssd_scan(batch, xbc, zxd[:, ssd_inner + C:], dtb, al, Dk, ssd_state, G), 2.0 * N * (C + ssd_inner + Hs) + 4.0 * ssd_state.numel(),
             nc * Hs * 2.0 * 128 * (128 * K + 3 * 128 * Ps))
    qkv, z = rn(N, 3 * inner) * 0.3, rn(N, inner)
    state, vec = torch.zeros(seqs, H, K, K, device=dev), torch.zeros(seqs, H, K + 1, device=dev)
    raw, gb = rn(N, 2 * H, dtype=f32), torch.cat([torch.zeros(H), torch.full((H,), 4.0)]).to(dev)
    decay = 1.0 - 2.0 ** (-5 - 8 * torch.arange(H, device=dev, dtype=f32) / H)
    gates = LIN.Gates(raw, gb, 15.0, vec)
    # q k^T once per head, M V, Q S, K^T V
    flops = nc * H * 2.0 * 128 * (128 * K + 3 * 128 * K)
    put(pre, "mLSTM scan", tm(lambda: LIN.linear_scan(batch, qkv, state, gates=gates, q_scale=K ** -0.5), 2.0 * N * 4 * inner + 24.0 * N * H + 4.0 * state.numel(), flops),
        ssd, "ssd_scan (64 heads of 64, 8 groups)")
    put(pre, "lightning scan", tm(lambda: LIN.linear_scan(batch, qkv, state, decay=decay), 2.0 * N * 4 * inner + 4.0 * state.numel(), flops),
        ssd, "ssd_scan (64 heads of 64, 8 groups)")
    ys, gs = rn(N, ssd_inner), rn(ssd_inner, dtype=f32)
    gn = tm(lambda: ssm.gated_group_norm(ys, zxd[:, :ssd_inner], gs, G, 1e-5, BF), 6.0 * N * ssd_inner)
    gam = rn(inner, dtype=f32)
    s1 = LIN.linear_scan(batch, qkv, state, gates=gates, q_scale=K ** -0.5)
    s2 = LIN.Numerators(s1.y)
    put(pre, "mLSTM denominator, head norm, gate", tm(lambda: LIN.head_norm_gate(batch, s1, z, gam, H, 1e-5, BF), 6.0 * N * inner + 16.0 * N * H), gn, "gated_group_norm")
    put(pre, "lightning norm, gate", tm(lambda: LIN.head_norm_gate(batch, s2, z, gam, 1, 1e-5, BF), 6.0 * N * inner), gn, "gated_group_norm")
    del xbc, zxd, ys
    x16, x32, g1, g2 = rn(N, D), rn(N, D, dtype=f32), rn(D, dtype=f32), rn(D, dtype=f32)
    ln = tm(lambda: norm_rows(LAYERNORM, x32, g1, g2, 1e-5, BF), 6.0 * N * D)
    put(pre, "post-norm, residual, next norm (bf16 in)", tm(lambda: residual_norm_rows(x16, g1, x32, g2, 1e-5, BF), 12.0 * N * D), ln, "norm_rows (layer norm, fp32 in)")
    y32 = rn(N, D, dtype=f32)
    put(pre, "post-norm, residual, next norm (fp32 in)", tm(lambda: residual_norm_rows(y32, g1, x32, g2, 1e-5, BF), 14.0 * N * D), ln, "norm_rows (layer norm, fp32 in)")
    w_in = rn(4 * inner + 2 * H, D) * D ** -0.5
    gf = lambda n: 2.0 * N * D * n
    plain = tm(lambda: gemm(x16, w_in[:3 * inner]), 0, gf(3 * inner))
    put(pre, "projection with SiLU epilogue", tm(lambda: linear_rows(x16, w_in[:3 * inner], act="silu"), 0, gf(3 * inner)), plain, "the same GEMM without it")
    put(pre, "projection q k v g with fp32 gates", tm(lambda: linear_rows_f32_tail(x16, w_in, 2 * H), 0, gf(4 * inner + 2 * H)), plain, "GEMM of 3/4 the width")

    # ---- prefill: windowed attention beside causal attention ----
    Q, Gk, Dh = heads, kv_heads, 128
    rope = rope_tables(Dh, 5e5, ctx + seq_len, None, dev)
    per = max(seq_len, ctx) // 64 + 2
    nb = max(max(decode_batches), seqs)
    cache = PagedCache(1, [2 * Gk * Dh], nb * per, 64, nb, per, BF, dev)
    for i in range(nb):
        cache.reserve(i, max(seq_len, ctx) + 1)
    cache.pool[0].normal_()
    yqk, bqk = rn(N, (Q + Gk) * Dh), rn((Q + Gk) * Dh, dtype=f32)
    prep = lambda: WA.qk_prepare(batch, yqk, bqk, Q, Gk, Dh, True, 1e-5, rope, cache, 0, dense=True)
    from ..models.qwen35.primitives import precompute_rope_freqs
    from ..ops.rope import rmsnorm_rope
    fr = precompute_rope_freqs(64, seq_len, 1e4, device=dev)
    xq, nw = rn(seqs, seq_len, Q, 256), rn(256)
    put(pre, "bias, rotation, unit norm, cache write", tm(prep, 2.0 * N * Dh * ((Q + Gk) * 2 + 3 * Gk)),
        tm(lambda: rmsnorm_rope(xq, nw, fr, 64), 4.0 * xq.numel()), "rmsnorm_rope (16 heads of 256)")
    q, k, v = prep()
    as4 = lambda t: t.unflatten(0, (seqs, seq_len))
    o = torch.empty_like(as4(q))
    pairs = lambda w, kp: sum(min(i + 1, w + min(kp, max(0, i + 1 - w))) for i in range(seq_len))
    fa = lambda w, kp: seqs * Q * pairs(w, kp) * 4.0 * Dh
    full = tm(lambda: A.attn_fwd(as4(q), as4(k), as4(v), True, 0.09, out=o), 0, fa(seq_len, 0))
    put(pre, "flash attention, window + kept tokens", tm(lambda: A.attn_fwd(as4(q), as4(k), as4(v), True, 0.09, out=o, window=window, keep_first=keep_first), 0, fa(window, keep_first)),
        full, "the same kernel, causal")
    del yqk, xq, o, q, k, v

    # ---- experts ----
    wgu, wdn = rn(experts, 2 * ff, D) * D ** -0.5, rn(experts, D, ff) * ff ** -0.5
    sgu, sdn, wr = rn(2 * shared_ff, D) * D ** -0.5, rn(D, shared_ff) * shared_ff ** -0.5, rn(experts, D) * D ** -0.5
    ep = _fused_experts(dev, D, ff, experts, top)
    epw = {"gate_proj": rn(experts, D, ff) * D ** -0.5, "up_proj": rn(experts, D, ff) * D ** -0.5, "down_proj": rn(experts, ff, D) * ff ** -0.5}
    wrt = wr.t().contiguous()
    moe_flops = 2.0 * N * (top * 3 * D * ff + 3 * D * shared_ff + D * experts)

    def other_moe(xx):
        w, idx = softmax_topk_router(linear_f32out(xx, wrt), top)
        y = ep.forward(xx, w, idx, epw)
        return y + linear_rows(silu_glu_rows(xx, sgu), sdn)
    put(pre, "router, experts, shared expert", tm(lambda: sigmoid_moe(x16, wr, top, wgu, wdn, sgu, sdn), 0, moe_flops), tm(lambda: other_moe(x16), 0, moe_flops),
        "router kernel + ep_moe_forward + the same shared expert")
    logits = linear_rows(x16, wr, f32_out=True)
    put(pre, "top-k of sigmoid scores", tm(lambda: sigmoid_topk(logits, top), 4.0 * N * (experts + 2 * top)), tm(lambda: softmax_topk_router(logits, top), 4.0 * N * (experts + 2 * top)),
        "softmax_topk_router")
    _ext.check_status(dev)

    # ---- decode ----
    for B in decode_batches:
        d = out["decode"][f"batch {B}"] = {}
        bd = _start_batch(list(range(B)), [1] * B, ctx, dev, ctx + 1)
        zs, ring, sst = rn(B, ssd_inner + C + Hs), torch.zeros(B, 4, C, device=dev), torch.zeros(B, Hs, K, Ps, device=dev)
        cw, cb = rn(C, 4, dtype=f32), rn(C, dtype=f32)

        def ssd_step():
            yy = ssm.ssm_decode(bd, zs, cw, cb, ring, dtb, al, Dk, sst, G)
            ssm.gated_group_norm(yy, None, gs, G, 1e-5, BF)
        other = tm(ssd_step, 8.0 * sst.numel() + 4.0 * B * C * 4 + 16.0 * C + 2.0 * zs.numel() + 2.0 * B * ssd_inner)
        st1, v1, qk1 = torch.zeros(B, H, K, K, device=dev), torch.zeros(B, H, K + 1, device=dev), rn(B, 4 * inner) * 0.3
        raw1 = rn(B, 2 * H, dtype=f32)
        g1s = LIN.Gates(raw1, gb, 15.0, v1)

        def step(kind):
            s = LIN.linear_scan(bd, qk1[:, :3 * inner], st1, gates=g1s, q_scale=K ** -0.5) if kind else LIN.linear_scan(bd, qk1[:, :3 * inner], st1, decay=decay, silu=True)
            LIN.head_norm_gate(bd, s, qk1[:, 3 * inner:], gam, H if kind else 1, 1e-5, BF)
        b_step = 8.0 * st1.numel() + 2.0 * B * 5 * inner
        put(d, "mLSTM step + norm", tm(lambda: step(1), b_step + 8.0 * v1.numel()), other, "ssm_decode + gated_group_norm (twice the state)")
        put(d, "lightning step + norm", tm(lambda: step(0), b_step), other, "ssm_decode + gated_group_norm (twice the state)")
        cache.seq_lens.fill_(ctx)
        idt = torch.arange(B, dtype=torch.int32, device=dev)
        qd = rn(B, Q, Dh)
        kb = lambda n: 2.0 * B * n * 2 * Gk * Dh
        dec = lambda w, kp: A.attention_decode_paged(qd, cache.pool[0], cache.block_table, idt, cache.seq_lens, Gk, 0, 0.09, max_len=ctx, window=w, keep_first=kp)
        windowed = tm(lambda: dec(window, keep_first), kb(window + keep_first))
        cache.seq_lens.fill_(window + keep_first)
        put(d, "paged attention, window + kept tokens", windowed, tm(lambda: dec(0, 0), kb(window + keep_first)),
            f"the same kernel, {window + keep_first} cached keys, all seen")
        y1 = rn(B, (Q + Gk) * Dh)
        xq1, n1w = rn(B, 1, Q, 256), rn(256)
        put(d, "bias, rotation, unit norm, cache write", tm(lambda: WA.qk_prepare(bd, y1, bqk, Q, Gk, Dh, True, 1e-5, rope, cache, 0, dense=False), 2.0 * B * Dh * (2 * Q + 3 * Gk)),
            tm(lambda: rmsnorm_rope(xq1, n1w, fr, 64), 4.0 * xq1.numel()), "rmsnorm_rope (16 heads of 256)")
        xb, xr, yb = rn(B, D), rn(B, D, dtype=f32), rn(B, D)
        yg = torch.empty(B, 4 * inner, device=dev, dtype=BF)
        put(d, "projection q k v g with fp32 gates", tm(lambda: linear_rows_f32_tail(xb, w_in, 2 * H), 2.0 * w_in.numel()),
            tm(lambda: gemm(xb, w_in[:4 * inner], out=yg), 2.0 * D * 4 * inner), "tcgen05 GEMM")
        put(d, "post-norm, residual, next norm", tm(lambda: residual_norm_rows(yb, g1, xr, g2, 1e-5, BF), 12.0 * B * D), tm(lambda: norm_rows(LAYERNORM, xr, g1, g2, 1e-5, BF), 6.0 * B * D),
            "norm_rows")
        hit = len(set(sigmoid_topk(linear_rows(xb, wr, f32_out=True), top)[0].reshape(-1).tolist()))
        eb = 2.0 * (hit * 3 * D * ff + 3 * D * shared_ff + experts * D)
        put(d, "router, experts, shared expert", tm(lambda: sigmoid_moe(xb, wr, top, wgu, wdn, sgu, sdn), eb), tm(lambda: other_moe(xb), eb),
            "router kernel + ep_moe_forward + the same shared expert")
    _ext.check_status(dev)
    return out


def model_table(dev, sizes=((2048, 16), (4096, 32)), shapes=((1, 4096), (8, 1024)), steps: int = 24) -> list:
    """Prefill and decode tokens/s of eight layers. ``sizes``: (width, attention heads); ``shapes``: (sequences, prompt)."""
    from ..models.fovudra import FovudraConfig
    from ..models.vobunex import VobunexConfig
    from .serve_bench import _qwen_run, _vobunex_run, model_rows, qwen_like, step_engine_run
    E, top, ff, V = 64, 6, 1024, 65536
    rows = []
    for width, heads in sizes:
        fov = FovudraConfig.serving(width=width, experts=E, top=top, ff=ff, heads=heads, kv_heads=heads // 8, vocab=V)
        vob = VobunexConfig.serving(width=width, n_mamba=6, n_attention=2, experts=E, top=top, ff=ff, heads=heads, vocab=V)
        rows += model_rows(dev, width, shapes, steps, (("fovudra_8_layers", lambda *a: step_engine_run("fovudra", *a), fov),
                                                       ("qwen35_8_layers", _qwen_run, qwen_like(width, heads, E, top, ff, V)),
                                                       ("vobunex_hybrid_8_layers", _vobunex_run, vob)))
    return rows
