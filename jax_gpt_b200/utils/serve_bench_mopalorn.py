"""Mopalorn's part of the serving benchmark (utils/serve_bench.py): kernels of its layers beside the like kernels of Vobunex, Fovudra and
Munazen, and whole models beside Munazen and the latent-attention layers of Vobunex at equal width, depth and active feed-forward weights."""
from __future__ import annotations

import torch

BF = torch.bfloat16


def kernel_table(dev, width: int = 2048, seqs: int = 2, seq_len: int = 4096, decode_batches=(1, 8), ctx: int = 4096, heads: int = 16,
                 kv_heads: int = 2, ff: int = 9216, window: int = 1024, pool: int = 16) -> dict:
    from .. import _ext
    from ..cache.paged import PagedCache
    from ..ops import attention as A
    from ..ops import latent_attention as LA
    from ..ops import linear_attention as LIN
    from ..ops import rotated_kv as RKV
    from ..ops import window_attention as WA
    from ..ops.gemm import gemm, linear_rows
    from ..ops.mixed_kv import mixed_kv, query_factors
    from ..ops.mla_decode import mla_paged_decode
    from ..ops.rope import rope_tables
    from .serve_bench import _KernelTimer, _start_batch
    tm = _KernelTimer(dev)
    f32 = torch.float32
    rn = lambda *s, dtype=BF: torch.randn(*s, device=dev, dtype=f32).to(dtype)
    N, D, K = seqs * seq_len, width, 128
    H, G = heads, kv_heads
    out = {"prefill": {}, "decode": {}, "prefill_shape": f"{seqs} x {seq_len} tokens, width {width}, window {window}, blocks of {pool}",
           "decode_shape": f"context {ctx}"}

    def put(part, name, mine, other, other_name):
        part[name] = {"mopalorn": mine, "other": other, "other_kernel": other_name,
                      "distance_ratio": round(other["frac"] / max(mine["frac"], 1e-9), 2)}   # > 1: further from the roofline
    pre = out["prefill"]
    batch = _start_batch(list(range(seqs)), [seq_len] * seqs, 0, dev, seq_len)
    nb = max(max(decode_batches), seqs)
    per = max(seq_len, ctx) // 64 + 2

    def pages(w, blocks=0):
        c = PagedCache(1, [w], nb * per, 64, nb, per, BF, dev, blocks=[blocks])
        for i in range(nb):
            c.reserve(i, max(seq_len, ctx) + 1)
        c.pool[0].normal_()
        if blocks:
            c.pooled[0].normal_()
        return c

    # ---- prefill: latent attention ----
    dn, dr, dv, R, qr = 128, 64, 128, 512, 768
    nq, ng = H * (dn + dr), H * dv
    n_in = nq + R + dr + ng
    rope = rope_tables(dr, 5e4, ctx + seq_len, None, dev)
    lat_pages = pages(R + dr)
    y, yv = rn(N, n_in), rn(N, qr + R + dr)
    kg, qg = rn(R, dtype=f32), rn(qr, dtype=f32)
    kn = rn(N, H * dn)
    q3 = lambda t: t[:, :nq].unflatten(-1, (H, dn + dr))
    qv = rn(N, H, dn + dr)

    def operands(yy, gamma, q, c0):
        _, lat = LA.mla_prepare(batch, yy[:, c0:c0 + (qr if gamma is not None else 0) + R + dr], gamma, kg, 1e-5, rope, lat_pages, 0, True)
        return LA.mla_rope_qk(batch, q, kn, lat, R, rope)
    op_bytes = lambda rank: 2.0 * N * (2 * rank + 3 * (R + dr) + 2 * H * dr + H * dn + H * (dn + dr) + R + dr)
    put(pre, "latent norm, rotation, key assembly, cache write", tm(lambda: operands(y, None, q3(y), nq), op_bytes(0)),
        tm(lambda: operands(yv, qg, qv, 0), op_bytes(qr)), "the same kernels with a query latent")
    k = operands(y, None, q3(y), nq)
    v = rn(N, H, dv)
    as4 = lambda t: t.unflatten(0, (seqs, seq_len))
    o = torch.empty(N, H, dv, device=dev, dtype=BF)
    seen = lambda w, P: sum(min(i + 1, w) + (max(0, i - w + 1) // P if P else 0) for i in range(seq_len))
    fa = lambda w, d, e, P=0: seqs * H * seen(w, P) * 2.0 * (d + e)
    flash = lambda w: A.attn_fwd(as4(q3(y)), as4(k), as4(v), True, 0.07, out=as4(o), window=w)
    causal192 = tm(lambda: flash(0), 0, fa(seq_len, dn + dr, dv))
    put(pre, "flash attention 192 / 128, window", tm(lambda: flash(window), 0, fa(window, dn + dr, dv)), causal192, "the same kernel, causal")
    gate = y[:, nq + R + dr:]
    inner = H * dv
    z, gam = rn(N, inner), rn(inner, dtype=f32)
    norm_gate = tm(lambda: LIN.head_norm_gate(batch, LIN.Numerators(z), z, gam, 1, 1e-5, BF), 6.0 * N * inner)
    put(pre, "output gate", tm(lambda: LA.sigmoid_gate(o.view(N, inner), gate), 6.0 * N * inner), norm_gate, "lightning norm, sigmoid gate")
    del y, yv, qv, kn, k, v, o, z

    # ---- prefill: grouped attention ----
    cols = (0, H * K, (H + G) * K)
    yq, vf = rn(N, (H + 2 * G) * K), rn(N, (H + 2 * G) * K)
    v_first = vf[:, cols[2]:]
    factors = query_factors(0.1, 512, ctx + seq_len, dev)
    plain_pages, block_pages = pages(2 * G * K), pages(2 * G * K, pool)
    rt = rope_tables(K, 1e6, ctx + seq_len, None, dev)
    bias = rn((H + 2 * G) * K, dtype=f32)
    mix = lambda bt, yy, first, c, dense, f: mixed_kv(bt, yy, cols, H, G, K, K, c, 0, dense, f, first, 0.4, window)
    op = 2.0 * N * K * ((H + 2 * G) * 2 + 2 * G)
    rotated = tm(lambda: RKV.qkv_rotate(batch, yq, cols, bias, H, G, K, K, rt, rt, plain_pages, 0, (K, K)), op)
    put(pre, "query factor, value mixing, cache write", tm(lambda: mix(batch, yq, v_first, plain_pages, (K, K), factors), op + 2.0 * N * G * K), rotated,
        "bias, rotation of q k v, cache write")
    put(pre, "value mixing, cache write, block means", tm(lambda: mix(batch, yq, v_first, block_pages, (K, K), None), op + 2.0 * N * G * K * 3), rotated,
        "bias, rotation of q k v, cache write")
    q, k, v = mix(batch, yq, v_first, plain_pages, (K, K), factors)
    causal = tm(lambda: WA.flash_prompts(batch, q, k, v, 0.09), 0, fa(seq_len, K, K))
    put(pre, "flash attention, capped scores", tm(lambda: WA.flash_prompts(batch, q, k, v, 0.09, softcap=50.0), 0, fa(seq_len, K, K)), causal,
        "the same kernel without a cap")
    kept = tm(lambda: WA.flash_prompts(batch, q, k, v, 0.09, window, 64), 0, seqs * H * sum(min(i + 1, window + 64) for i in range(seq_len)) * 4.0 * K)
    sink = rn(H, dtype=f32)
    q, k, v = mix(batch, yq, v_first, block_pages, (K, K), None)
    put(pre, "flash attention, window, block means, sink", tm(lambda: WA.flash_prompts(batch, q, k, v, 0.09, window, sink=sink, pool=pool), 0, fa(window, K, K, pool)),
        kept, "the same kernel, window and 64 kept tokens")
    del yq, vf, v_first, q, k, v

    # ---- prefill: projections ----
    x16 = rn(N, D)
    w_in, w_g, w_up, w_dn, w_o = rn(n_in, D) * D ** -0.5, rn((H + 2 * G) * K, D) * D ** -0.5, rn(ff, D) * D ** -0.5, rn(D, ff) * ff ** -0.5, rn(D, inner) * D ** -0.5
    h = rn(N, ff)
    xielu = dict(act="xielu", act_args=(1.1, 1.2))
    plain = tm(lambda: gemm(x16, w_up), 0, 2.0 * N * D * ff)
    for name, fn, w in (("projection q latent gate", lambda: linear_rows(x16, w_in), w_in), ("projection q k v", lambda: linear_rows(x16, w_g), w_g),
                        ("feed-forward up with its activation", lambda: linear_rows(x16, w_up, **xielu), w_up), ("feed-forward down", lambda: linear_rows(h, w_dn), w_dn),
                        ("output projection", lambda: linear_rows(x16[:, :inner], w_o), w_o)):
        put(pre, name, tm(fn, 0, 2.0 * N * w.numel()), plain, "GEMM to the feed-forward's width")
    del h, x16
    _ext.check_status(dev)

    # ---- decode ----
    w_ukv = rn(H * (dn + dv), R) * R ** -0.5
    for B in decode_batches:
        d = out["decode"][f"batch {B}"] = {}
        bd = _start_batch(list(range(B)), [1] * B, ctx, dev, ctx + 1)
        idt = torch.arange(B, dtype=torch.int32, device=dev)
        y1, yv1, q1 = rn(B, n_in), rn(B, qr + R + dr), rn(B, H, R + dr)
        tm(lambda: LA.mla_prepare(bd, yv1, qg, kg, 1e-5, rope, lat_pages, 0, False))     # not reported: the first timing of a part runs cold
        put(d, "latent norm, rotation, cache write", tm(lambda: LA.mla_prepare(bd, y1[:, nq:nq + R + dr], None, kg, 1e-5, rope, lat_pages, 0, False), 4.0 * B * (R + dr)),
            tm(lambda: LA.mla_prepare(bd, yv1, qg, kg, 1e-5, rope, lat_pages, 0, False), 4.0 * B * (qr + R + dr)), "the same kernel with a query latent")
        put(d, "query absorption", tm(lambda: LA.mla_absorb_q(bd, q3(y1), w_ukv[:H * dn], rope, dr), 2.0 * H * dn * R + 2.0 * B * H * (dn + dr + R + dr)),
            tm(lambda: LA.mla_absorb_q(bd, q3(y1).contiguous(), w_ukv[:H * dn], rope, dr), 2.0 * H * dn * R + 2.0 * B * H * (dn + dr + R + dr)), "the same kernel, dense queries")
        ol = rn(B, H, R)
        put(d, "output absorption and gate", tm(lambda: LA.mla_absorb_out(ol, w_ukv[H * dn:], y1[:, nq + R + dr:]), 2.0 * H * dv * R + 2.0 * B * H * (R + 2 * dv)),
            tm(lambda: LA.mla_absorb_out(ol, w_ukv[H * dn:]), 2.0 * H * dv * R + 2.0 * B * H * (R + dv)), "the same kernel without a gate")
        kb = 2.0 * B * window * (R + dr)
        lat_pages.seq_lens.fill_(ctx)
        mine = tm(lambda: mla_paged_decode(q1, lat_pages, 0, idt, 0.07, max_len=ctx, window=window), kb)
        lat_pages.seq_lens.fill_(window)
        put(d, "paged latent attention, window", mine, tm(lambda: mla_paged_decode(q1, lat_pages, 0, idt, 0.07, max_len=window), kb), f"the same kernel, {window} cached tokens")
        qd = rn(B, H, K)
        dec = lambda c, **kw: A.attention_decode_paged(qd, c.pool[0], c.block_table, idt, c.seq_lens, G, 0, 0.09, max_len=ctx, **kw)
        kb = lambda n: 2.0 * B * n * 2 * G * K
        plain_pages.seq_lens.fill_(ctx)
        block_pages.seq_lens.fill_(ctx)
        put(d, "paged attention, capped scores", tm(lambda: dec(plain_pages, softcap=50.0), kb(ctx)), tm(lambda: dec(plain_pages), kb(ctx)), "the same kernel without a cap")
        n_seen = window + (ctx - window) // pool
        put(d, "paged attention, window, block means, sink", tm(lambda: dec(block_pages, window=window, sink=sink, pooled=block_pages.pooled[0], pool_block=pool), kb(n_seen)),
            tm(lambda: dec(plain_pages, window=window, keep_first=n_seen - window), kb(n_seen)), "the same kernel, window and as many kept tokens")
        yq1, vf1 = rn(B, (H + 2 * G) * K), rn(B, G * K)
        rot1 = tm(lambda: RKV.qkv_rotate(bd, yq1, cols, bias, H, G, K, K, rt, rt, plain_pages, 0, None), 2.0 * B * K * (2 * H + 4 * G))
        put(d, "query factor, value mixing, cache write", tm(lambda: mix(bd, yq1, vf1, plain_pages, None, factors), 2.0 * B * K * (2 * H + 5 * G)), rot1,
            "bias, rotation of q k v, cache write")
        last = _start_batch(list(range(B)), [1] * B, ctx - 1, dev, ctx + 1)     # the step that completes a block
        put(d, "value mixing, cache write, a block's mean", tm(lambda: mix(last, yq1, vf1, block_pages, None, None), 2.0 * B * K * (2 * H + 5 * G + 2 * G * (pool + 1))), rot1,
            "bias, rotation of q k v, cache write")
        xb, hb = rn(B, D), rn(B, ff)
        for name, fn, w, x in (("projection q latent gate", lambda: linear_rows(xb, w_in), w_in, xb), ("projection q k v", lambda: linear_rows(xb, w_g), w_g, xb),
                               ("feed-forward up with its activation", lambda: linear_rows(xb, w_up, **xielu), w_up, xb),
                               ("feed-forward down", lambda: linear_rows(hb, w_dn), w_dn, hb)):
            yo = torch.empty(B, w.shape[0], device=dev, dtype=BF)
            put(d, name, tm(fn, 2.0 * w.numel()), tm(lambda: gemm(x, w, out=yo), 2.0 * w.numel()), "tcgen05 GEMM of the same size, no activation")
    _ext.check_status(dev)
    return out


def model_table(dev, sizes=((2048, 16), (4096, 32)), shapes=((1, 4096), (8, 1024)), steps: int = 24) -> list:
    """Prefill and decode tokens/s of eight layers. ``sizes``: (width, attention heads); ``shapes``: (sequences, prompt)."""
    from ..models.mopalorn import MopalornConfig
    from ..models.munazen import MunazenConfig
    from ..models.vobunex import VobunexConfig
    from .serve_bench import model_rows, step_engine_run
    E, top, ff, V = 64, 6, 1024, 65536
    rows = []
    for width, heads in sizes:
        # a dense feed-forward (two matrices) with the weights that a token meets in six experts of three
        dense = top * ff * 3 // 2
        mop = lambda **kw: MopalornConfig.serving(width=width, heads=heads, kv_heads=heads // 8, ff=dense, vocab=V, **kw)
        run = lambda family: (lambda *a: step_engine_run(family, *a))
        rows += model_rows(dev, width, shapes, steps, (
            ("mopalorn_4_latent_2_full_2_pooled", run("mopalorn"), mop()), ("mopalorn_2_latent_3_full_3_pooled", run("mopalorn"), mop(n_latent=2, n_full=3, n_pooled=3)),
            ("munazen_6_parallel_2_gla", run("munazen"), MunazenConfig.serving(width=width, heads=heads, kv_heads=heads // 8, ff=dense, vocab=V)),
            ("vobunex_latent_8_layers", run("vobunex"), VobunexConfig.serving(width=width, n_mamba=0, n_attention=8, experts=E, top=top, ff=ff, heads=heads, vocab=V))))
    return rows
