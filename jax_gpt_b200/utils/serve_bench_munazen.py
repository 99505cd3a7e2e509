"""Munazen's part of the serving benchmark (utils/serve_bench.py): kernels of its layers beside the like kernels of Fovudra, and whole
models beside Fovudra at equal width, depth and active feed-forward weights."""
from __future__ import annotations

import torch

BF = torch.bfloat16


def kernel_table(dev, width: int = 2048, seqs: int = 2, seq_len: int = 4096, decode_batches=(1, 8), ctx: int = 4096, heads: int = 16,
                 kv_heads: int = 2, ff: int = 8192, streams: int = 2, rank: int = 16) -> dict:
    from .. import _ext
    from ..cache.paged import PagedCache
    from ..ops import attention as A
    from ..ops import linear_attention as LIN
    from ..ops import rotated_kv as RKV
    from ..ops import window_attention as WA
    from ..ops.gated_lru import LruWeights, gated_lru
    from ..ops.gemm import gemm, linear_rows
    from ..ops.packed import residual_norm_rows
    from ..ops.rope import rope_tables
    from ..ops.streams import Connection, poly_norm, stream_norm
    from .serve_bench import _KernelTimer, _start_batch
    tm = _KernelTimer(dev)
    f32 = torch.float32
    rn = lambda *s, dtype=BF: torch.randn(*s, device=dev, dtype=f32).to(dtype)
    N, D, K = seqs * seq_len, width, 128
    H = width // K
    inner, W, nb = H * K, width, width // K
    out = {"prefill": {}, "decode": {}, "prefill_shape": f"{seqs} x {seq_len} tokens, width {width}, {streams} streams", "decode_shape": f"context {ctx}"}

    def put(part, name, mine, other, other_name):
        part[name] = {"munazen": mine, "other": other, "other_kernel": other_name,
                      "distance_ratio": round(other["frac"] / max(mine["frac"], 1e-9), 2)}   # > 1: further from the roofline
    pre = out["prefill"]
    batch = _start_batch(list(range(seqs)), [seq_len] * seqs, 0, dev, seq_len)

    # ---- prefill: both recurrences beside the fixed-decay and the gated scan ----
    y_in = rn(N, 3 * inner + 64) * 0.3
    qkv, low, z = y_in[:, :3 * inner], y_in[:, 3 * inner:3 * inner + rank], rn(N, inner)
    state = torch.zeros(seqs, H, K, K, device=dev)
    decay = 1.0 - 2.0 ** (-5 - 8 * torch.arange(H, device=dev, dtype=f32) / H)
    w2, b2 = rn(inner, rank) * rank ** -0.5, rn(inner, dtype=f32) + 2
    channels = LIN.ChannelDecay(low, w2, b2, 16.0)
    nc = N / 128.0
    flops = nc * H * 2.0 * 128 * (128 * K + 3 * 128 * K)
    scan_bytes = 2.0 * N * 4 * inner + 4.0 * state.numel()
    lightning = tm(lambda: LIN.linear_scan(batch, qkv, state, decay=decay), scan_bytes, flops)
    put(pre, "channel-decay scan", tm(lambda: LIN.linear_scan(batch, qkv, state, channels=channels, q_scale=K ** -0.5), scan_bytes + 2.0 * N * rank, flops),
        lightning, "lightning scan")
    raw, gb = rn(N, 2 * H, dtype=f32), torch.cat([torch.zeros(H), torch.full((H,), 4.0)]).to(dev)
    vec = torch.zeros(seqs, H, K + 1, device=dev)
    gates = LIN.Gates(raw, gb, 15.0, vec)
    mlstm = tm(lambda: LIN.linear_scan(batch, qkv, state, gates=gates, q_scale=K ** -0.5), scan_bytes + 24.0 * N * H, flops)
    put(pre, "channel-decay scan (beside the gated scan)", pre["channel-decay scan"]["munazen"], mlstm, "mLSTM scan")
    gam = rn(inner, dtype=f32)
    s1 = LIN.Numerators(LIN.linear_scan(batch, qkv, state, decay=decay).y)
    put(pre, "head norm, SiLU gate", tm(lambda: LIN.head_norm_gate(batch, s1, z, gam, H, 1e-5, BF, silu=True), 6.0 * N * inner),
        tm(lambda: LIN.head_norm_gate(batch, s1, z, gam, 1, 1e-5, BF), 6.0 * N * inner), "lightning norm, sigmoid gate")
    lw = LruWeights(rn(W, dtype=f32), rn(W, dtype=f32), rn(W, 4, dtype=f32), rn(W, dtype=f32), rn(nb, 2, K, K) * K ** -0.5, rn(nb, 2, K, dtype=f32),
                    torch.rand(W, device=dev) * 0.1)
    xy, both = rn(N, 2 * W), torch.empty(N, 2 * W, device=dev, dtype=BF)
    ring, lst = torch.zeros(seqs, 4, W, device=dev), torch.zeros(seqs, W, device=dev)
    put(pre, "recurrent unit (convolution, gates, scan, output gate)",
        tm(lambda: gated_lru(batch, xy[:, :W], xy[:, W:], lw, ring, lst, 1.0, both[:, W:]), 6.0 * N * W + 2.0 * lw.gates.numel(), 2.0 * N * W * 2 * K),
        lightning, "lightning scan")
    del xy, y_in, qkv, low

    # ---- prefill: streams, activation, projections ----
    x16, g1, g2 = rn(N, D), rn(D, dtype=f32), rn(D, dtype=f32)
    x32, xs = rn(N, D, dtype=f32), rn(N, streams, D, dtype=f32)
    conn = Connection(rn(streams, dtype=f32), torch.eye(streams, device=dev), rn(streams, dtype=f32))
    res = tm(lambda: residual_norm_rows(x16, g1, x32, g2, 1e-5, BF), 12.0 * N * D)
    put(pre, "streams, next combination, group norm", tm(lambda: stream_norm(x16, xs, conn, conn.w_in, g1, 8, 1e-5, BF, bias=g2), (4.0 + 8.0 * streams) * N * D),
        res, "post-norm, residual, next norm")
    zf, coef = rn(N, ff), torch.tensor([0.5, 0.3, 0.2, 0.0], device=dev)
    gu, gh = rn(N, 2 * ff), torch.empty(N, ff, device=dev, dtype=BF)
    put(pre, "polynomial activation", tm(lambda: poly_norm(zf, coef, 1e-5), 4.0 * N * ff),
        tm(lambda: _ext.ops().clamped_glu(gu, float("inf"), 1.0, 0.0, None, gh), 6.0 * N * ff), "gate times up (clamped_glu)")
    del gu, gh
    n_in = (heads + 2 * kv_heads) * K + 2 * W + 16
    w_in, w_o, w_up, w_dn = rn(n_in, D) * D ** -0.5, rn(D, heads * K + W) * 0.02, rn(ff, D) * D ** -0.5, rn(D, ff) * ff ** -0.5
    plain = tm(lambda: gemm(x16, w_in[:3 * D]), 0, 6.0 * N * D * D)
    put(pre, "projection q k v x y g", tm(lambda: linear_rows(x16, w_in), 0, 2.0 * N * D * n_in), plain, "GEMM to 3 x width")
    put(pre, "projection of both branches", tm(lambda: linear_rows(both, w_o), 0, 2.0 * N * D * w_o.shape[1]), plain, "GEMM to 3 x width")
    put(pre, "feed-forward up", tm(lambda: linear_rows(x16, w_up), 0, 2.0 * N * D * ff), plain, "GEMM to 3 x width")
    put(pre, "feed-forward down", tm(lambda: linear_rows(zf, w_dn), 0, 2.0 * N * D * ff), plain, "GEMM to 3 x width")
    del zf, xs, x32

    # ---- prefill: attention ----
    Q, G = heads, kv_heads
    rope, vrope = rope_tables(K, 1e6, ctx + seq_len, None, dev), rope_tables(K, 1e6, ctx + seq_len, None, dev)
    per = max(seq_len, ctx) // 64 + 2
    n_seq = max(max(decode_batches), seqs)
    cache = PagedCache(1, [2 * G * K], n_seq * per, 64, n_seq, per, BF, dev)
    for i in range(n_seq):
        cache.reserve(i, max(seq_len, ctx) + 1)
    cache.pool[0].normal_()
    cols = (0, Q * K, (Q + G) * K)
    yq, bq = rn(N, n_in), rn((Q + 2 * G) * K, dtype=f32)
    rotate = lambda yy, bt, dense: RKV.qkv_rotate(bt, yy, cols, bq, Q, G, K, K, rope, vrope, cache, 0, dense)
    y_qk, b_qk = rn(N, (Q + G) * K), rn((Q + G) * K, dtype=f32)
    put(pre, "bias, rotation of q k v, cache write", tm(lambda: rotate(yq, batch, (K, K)), 2.0 * N * K * ((Q + 2 * G) * 2 + 2 * G)),
        tm(lambda: WA.qk_prepare(batch, y_qk, b_qk, Q, G, K, True, 1e-5, rope, cache, 0, dense=True), 2.0 * N * K * ((Q + G) * 2 + 3 * G)),
        "bias, rotation, unit norm, cache write")
    q, k, v = rotate(yq, batch, (K, K))
    as4 = lambda t: t.unflatten(0, (seqs, seq_len))
    fa = lambda d, dv: seqs * Q * (seq_len * (seq_len + 1) / 2) * 2.0 * (d + dv)
    causal = tm(lambda: A.attn_fwd(as4(q), as4(k), as4(v), True, 0.09), 0, fa(K, K))
    put(pre, "flash attention", tm(lambda: WA.flash_prompts(batch, q, k, v, 0.09), 0, fa(K, K)), causal, "the same kernel")
    put(pre, "flash attention, keys of 64 padded to 128", tm(lambda: WA.flash_prompts(batch, q, k, v, 0.09), 0, fa(64, K)), causal, "the same kernel, keys of 128")
    o = rn(N, Q, K)
    put(pre, "turn back, head gate", tm(lambda: RKV.turn_back_gate(batch, o, yq[:, -16:][:, :Q], vrope, 1.0, both[:, :Q * K]), 4.0 * N * Q * K),
        tm(lambda: LIN.head_norm_gate(batch, s1, z, gam, 1, 1e-5, BF), 6.0 * N * inner), "lightning norm, sigmoid gate")
    del yq, y_qk, q, k, v, o, both, s1, z, x16
    _ext.check_status(dev)

    # ---- decode ----
    for B in decode_batches:
        d = out["decode"][f"batch {B}"] = {}
        bd = _start_batch(list(range(B)), [1] * B, ctx, dev, ctx + 1)
        st1, qk1, z1 = torch.zeros(B, H, K, K, device=dev), rn(B, 3 * inner + 64) * 0.3, rn(B, inner)
        ch1 = LIN.ChannelDecay(qk1[:, 3 * inner:3 * inner + rank], w2, b2, 16.0)

        def step(kind):
            s = LIN.linear_scan(bd, qk1[:, :3 * inner], st1, channels=ch1, q_scale=K ** -0.5) if kind else \
                LIN.linear_scan(bd, qk1[:, :3 * inner], st1, decay=decay, silu=True)
            LIN.head_norm_gate(bd, s, z1, gam, H if kind else 1, 1e-5, BF, silu=bool(kind))
        b_step = 8.0 * st1.numel() + 2.0 * B * 5 * inner
        light = tm(lambda: step(0), b_step)
        put(d, "channel-decay step + norm", tm(lambda: step(1), b_step + 2.0 * w2.numel()), light, "lightning step + norm")
        x1, o1 = rn(B, 2 * W), torch.empty(B, 2 * W, device=dev, dtype=BF)
        ring1, l1 = torch.zeros(B, 4, W, device=dev), torch.zeros(B, W, device=dev)
        put(d, "recurrent unit step", tm(lambda: gated_lru(bd, x1[:, :W], x1[:, W:], lw, ring1, l1, 1.0, o1[:, W:]),
                                         2.0 * lw.gates.numel() + B * W * (6.0 + 8.0 + 16.0) + 4.0 * 9 * W), light, "lightning step + norm")
        cache.seq_lens.fill_(ctx)
        idt = torch.arange(B, dtype=torch.int32, device=dev)
        qd = rn(B, Q, K)
        kb = 2.0 * B * ctx * 2 * G * K
        dec = tm(lambda: A.attention_decode_paged(qd, cache.pool[0], cache.block_table, idt, cache.seq_lens, G, 0, 0.09, max_len=ctx), kb)
        half = PagedCache(1, [G * (64 + K)], n_seq * per, 64, n_seq, per, BF, dev)
        for i in range(n_seq):
            half.reserve(i, ctx + 1)
        half.pool[0].normal_()
        half.seq_lens.fill_(ctx)
        qh = rn(B, Q, 64)
        put(d, "paged attention, keys of 64, values of 128",
            tm(lambda: A.attention_decode_paged(qh, half.pool[0], half.block_table, idt, half.seq_lens, G, 0, 0.09, max_len=ctx, v_dim=K), 0.75 * kb),
            dec, "the same kernel, both 128")
        y1, yk1 = rn(B, n_in), rn(B, (Q + G) * K)
        put(d, "bias, rotation of q k v, cache write", tm(lambda: rotate(y1, bd, None), 2.0 * B * K * (2 * Q + 4 * G)),
            tm(lambda: WA.qk_prepare(bd, yk1, b_qk, Q, G, K, True, 1e-5, rope, cache, 0, dense=False), 2.0 * B * K * (2 * Q + 3 * G)),
            "bias, rotation, unit norm, cache write")
        od = rn(B, Q, K)
        gate1 = tm(lambda: LIN.head_norm_gate(bd, LIN.Numerators(z1), z1, gam, 1, 1e-5, BF), 6.0 * B * inner)
        put(d, "turn back, head gate", tm(lambda: RKV.turn_back_gate(bd, od, y1[:, -16:][:, :Q], vrope, 1.0, o1[:, :Q * K]), 4.0 * B * Q * K), gate1,
            "lightning norm, sigmoid gate")
        xb, yb, xr, xs1 = rn(B, D), rn(B, D), rn(B, D, dtype=f32), rn(B, streams, D, dtype=f32)
        put(d, "streams, next combination, group norm", tm(lambda: stream_norm(yb, xs1, conn, conn.w_in, g1, 8, 1e-5, BF, bias=g2), (4.0 + 8.0 * streams) * B * D),
            tm(lambda: residual_norm_rows(yb, g1, xr, g2, 1e-5, BF), 12.0 * B * D), "post-norm, residual, next norm")
        z1f = rn(B, ff)
        put(d, "polynomial activation", tm(lambda: poly_norm(z1f, coef, 1e-5), 4.0 * B * ff), gate1, "lightning norm, sigmoid gate")
        yo = torch.empty(B, 3 * D, device=dev, dtype=BF)
        lin = tm(lambda: gemm(xb, w_in[:3 * D], out=yo), 6.0 * D * D)
        for name, fn, w in (("projection q k v x y g", lambda: linear_rows(xb, w_in), w_in), ("projection of both branches", lambda: linear_rows(o1, w_o), w_o),
                            ("feed-forward up", lambda: linear_rows(xb, w_up), w_up), ("feed-forward down", lambda: linear_rows(z1f, w_dn), w_dn)):
            put(d, name, tm(fn, 2.0 * w.numel()), lin, "tcgen05 GEMM to 3 x width")
    _ext.check_status(dev)
    return out


def model_table(dev, sizes=((2048, 16), (4096, 32)), shapes=((1, 4096), (8, 1024)), steps: int = 24) -> list:
    """Prefill and decode tokens/s of eight layers. ``sizes``: (width, attention heads); ``shapes``: (sequences, prompt)."""
    from ..models.fovudra import FovudraConfig
    from ..models.munazen import MunazenConfig
    from .serve_bench import model_rows, step_engine_run
    E, top, ff, V = 64, 6, 1024, 65536
    rows = []
    for width, heads in sizes:
        # a dense feed-forward (two matrices) with the weights that a token of the other family meets (six experts of three)
        mun = MunazenConfig.serving(width=width, heads=heads, kv_heads=heads // 8, ff=top * ff * 3 // 2, vocab=V)
        gla = MunazenConfig.serving(width=width, n_parallel=2, n_gla=6, heads=heads, kv_heads=heads // 8, ff=top * ff * 3 // 2, vocab=V)
        fov = FovudraConfig.serving(width=width, experts=E, top=top, ff=ff, heads=heads, kv_heads=heads // 8, vocab=V)
        run = lambda family: (lambda *a: step_engine_run(family, *a))
        rows += model_rows(dev, width, shapes, steps, (("munazen_6_parallel_2_gla", run("munazen"), mun), ("munazen_2_parallel_6_gla", run("munazen"), gla),
                                                       ("fovudra_8_layers", run("fovudra"), fov)))
    return rows
