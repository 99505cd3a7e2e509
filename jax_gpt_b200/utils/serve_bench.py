"""Serving benchmark of Vobunex, Fovudra, Munazen and Mopalorn beside the closest other families at equal widths (random weights, one GPU).

    python bench.py --serve [--serve-part kernels|models|all] [--serve-family vobunex|fovudra|munazen|mopalorn|all]

``models``: prefill and decode tokens/s of whole models. The hybrid (Mamba-2 + latent attention) stands beside the
Qwen3.5-style hybrid (Gated DeltaNet + gated attention), latent-attention-only layers beside the DeepSeek-V3 layers; same
width, depth, expert count and expert width, each family on its own serving path (decode: CUDA-graph engines, the
others' experts on the fused expert kernel). ``kernels``: device time and roofline fraction of every kernel of a layer
beside the like kernel of the other family. The other families'
tables are made in utils/serve_bench_fovudra.py, utils/serve_bench_munazen.py and utils/serve_bench_mopalorn.py.

Timing: CUDA events. Kernels are timed inside a captured graph that writes a 256 MB buffer (larger than L2) before every
launch; the time of the same graph without the launches is subtracted. The roofline of a kernel is the slower of its
algorithmic bytes at the measured copy bandwidth and its FLOPs at the measured bf16 rate.
"""
from __future__ import annotations

import gc
import os
import statistics

import torch

from . import roofline as R

BF = torch.bfloat16


def _sync_free():
    gc.collect()
    torch.cuda.synchronize()
    torch.cuda.empty_cache()


class _KernelTimer:
    def __init__(self, device, n: int = 10):
        self.flush = torch.empty(64 * 1024 * 1024, dtype=torch.float32, device=device)
        self.n, self.peaks = n, R.load_peaks()

    def _run(self, fn):
        if fn is not None:
            fn()
            fn()
        torch.cuda.synchronize()
        g = torch.cuda.CUDAGraph()
        with torch.cuda.graph(g):
            for _ in range(self.n):
                self.flush.fill_(1.0)
                if fn is not None:
                    fn()
        for _ in range(3):
            g.replay()
        times = []
        for _ in range(5):
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            torch.cuda.synchronize()
            a.record()
            g.replay()
            b.record()
            torch.cuda.synchronize()
            times.append(a.elapsed_time(b) / self.n)
        del g
        return statistics.median(times)

    def __call__(self, fn, bytes_: float = 0.0, flops: float = 0.0) -> dict:
        ms = max(self._run(fn) - self._run(None), 1e-4)
        roof = max(bytes_ / (self.peaks["hbm_gbs"] * 1e6), flops / (self.peaks["bf16_tflops"] * 1e9))
        return {"us": round(ms * 1e3, 2), "roofline_us": round(roof * 1e3, 2), "frac": float(f"{roof / ms:.3g}")}


def _start_batch(seq_ids, lens, start, dev, max_len):
    from ..ops.packed import PackedBatch, seq_begin
    b = PackedBatch.make(seq_ids, lens, start == 0, max_len, dev)
    n = max(seq_ids) + 1
    seq_begin(b, torch.zeros(b.n_tok, dtype=torch.int32, device=dev), torch.full((n,), start, dtype=torch.int32, device=dev),
              torch.zeros(n, dtype=torch.int32, device=dev))
    return b


def _fused_experts(dev, D, I, E, top):
    """The fused expert kernel (world size 1) that serves the other families' routed experts."""
    import torch.distributed as dist
    from ..comm.symm import Communicator
    from ..parallel.expert_parallel import EPMoEInferenceRuntime
    if not dist.is_initialized():
        os.environ.setdefault("MASTER_ADDR", "127.0.0.1")
        os.environ.setdefault("MASTER_PORT", "29537")
        dist.init_process_group("nccl", rank=0, world_size=1, device_id=dev)
    return EPMoEInferenceRuntime(Communicator(device=dev, wait_seconds=30.0), D, I, E, top)


# ------------------------------------------------------------------------------------------------
def kernel_table(dev, width: int = 2048, seqs: int = 2, seq_len: int = 4096, decode_batches=(1, 8), ctx: int = 4096,
                 experts: int = 64, top: int = 6, ff: int = 1024) -> dict:
    from .. import _ext
    from ..cache.paged import PagedCache
    from ..ops import attention as A
    from ..ops import latent_attention as LA
    from ..ops import norm as norm_ops
    from ..ops import ssm
    from ..ops.gemm import gemm, linear_rows
    from ..ops.mla_decode import mla_paged_decode
    from ..ops.norm import LAYERNORM
    from ..ops.packed import norm_rows
    from ..ops.rope import rope_tables
    from ..ops.table_moe import table_moe
    tm = _KernelTimer(dev)
    ops = _ext.ops()
    rn = lambda *s, dtype=BF: torch.randn(*s, device=dev, dtype=torch.float32).to(dtype)
    f32 = torch.float32
    N, D = seqs * seq_len, width
    out = {"prefill": {}, "decode": {}, "prefill_shape": f"{seqs} x {seq_len} tokens, width {width}",
           "decode_shape": f"context {ctx}"}

    def put(part, name, mine, other=None, other_name=None):
        e = {"vobunex": mine}
        if other is not None:
            e["other"] = other
            e["other_kernel"] = other_name
            e["distance_ratio"] = round(other["frac"] / max(mine["frac"], 1e-9), 2)   # > 1: further from the roofline than the other
        out[part][name] = e

    # ---- prefill: state-space layer beside the DeltaNet layer ----
    P, Ns, G = 64, 128, 8
    H = 2 * D // P
    inner, C = H * P, H * P + 2 * G * Ns
    Hqk, Hv = 16, 2 * D // 128
    Cd = 2 * Hqk * 128 + Hv * 128
    batch = _start_batch(list(range(seqs)), [seq_len] * seqs, 0, dev, seq_len)
    zxd = rn(N, inner + C + H)
    cw, cb, ring = rn(C, 4, dtype=f32), rn(C, dtype=f32), torch.zeros(seqs, 4, C, device=dev)
    mixed = rn(seqs, seq_len, Cd)
    wd, yd = rn(Cd, 4), torch.empty(seqs, seq_len, Cd, device=dev, dtype=BF)
    put("prefill", "convolution", tm(lambda: ssm.ssm_conv(batch, zxd[:, inner:inner + C], cw, cb, ring), 4.0 * N * C),
        tm(lambda: ops.gdn_conv_silu(mixed, wd, yd, None), 4.0 * N * Cd), "gdn_conv_silu")
    xbc = rn(N, C)
    al, dtb, Dk = torch.log(torch.rand(H, device=dev) * 7 + 0.5), torch.rand(H, device=dev) * 3 - 4, rn(H, dtype=f32)
    state = torch.zeros(seqs, H, Ns, P, device=dev)
    nc = N / 128.0
    # G per group would do once; the kernel computes it per head, which is what its FLOPs count
    scan = tm(lambda: ssm.ssd_scan(batch, xbc, zxd[:, inner + C:], dtb, al, Dk, state, G), 2.0 * N * (C + inner + H) + 4.0 * state.numel(),
              nc * H * 2.0 * 128 * (128 * Ns + 3 * 128 * P))
    bg, ag = rn(seqs, seq_len, Hv), rn(seqs, seq_len, Hv)
    A_log, dt2 = torch.zeros(Hv, device=dev), torch.ones(Hv, device=dev)
    BH, n64 = seqs * Hv, seq_len // 64
    kq, intra = torch.empty(BH, n64, 128, 128, device=dev, dtype=BF), torch.empty(BH, n64, 64, 64, device=dev, dtype=BF)
    kdec, veff = torch.empty(BH, n64, 64, 128, device=dev, dtype=BF), torch.empty(BH, n64, 64, 128, device=dev, dtype=BF)
    e = torch.empty(BH, n64, device=dev)
    o, s_out = torch.empty(BH, n64, 64, 128, device=dev, dtype=BF), torch.empty(BH, 128, 128, device=dev)

    def gdn():
        ops.gdn_chunk_prep(mixed, bg, ag, A_log, dt2, kq, intra, kdec, veff, e, Hqk, Hv)
        ops.gdn_scan(kq, intra, kdec, veff, e, None, o, s_out, None, None)
    # per chunk: both Gram matrices and the triangular solve of the preparation, the scan's three products
    gdn_flops = BH * n64 * 2.0 * (2 * 64 * 64 * 128 + 64 * 64 * 128 + 128 * 128 * 128 + 64 * 64 * 128 + 64 * 128 * 128)
    put("prefill", "recurrence", scan, tm(gdn, 2.0 * N * (Cd + Hv * 128) + 4.0 * s_out.numel(), gdn_flops), "gdn_chunk_prep + gdn_scan")
    y, gam = rn(N, inner), rn(inner, dtype=f32)
    go, gz, gw = rn(seqs * Hv, seq_len, 128), rn(seqs, seq_len, Hv * 128), torch.ones(128, device=dev)
    gy = torch.empty(seqs, seq_len, Hv * 128, device=dev, dtype=BF)
    put("prefill", "gated norm", tm(lambda: ssm.gated_group_norm(y, zxd[:, :inner], gam, G, 1e-5, BF), 6.0 * N * inner),
        tm(lambda: ops.gdn_gated_norm(go, gz, gw, gy, Hv, 1e-6), 6.0 * N * Hv * 128), "gdn_gated_norm")
    del mixed, yd, kq, intra, kdec, veff, o, gz, go, gy, y
    x32, x16 = rn(N, D, dtype=f32), rn(N, D)
    g1, b1, g16 = rn(D, dtype=f32), rn(D, dtype=f32), rn(D)
    put("prefill", "layer norm (fp32 residual in)", tm(lambda: norm_rows(LAYERNORM, x32, g1, b1, 1e-5, BF), 6.0 * N * D),
        tm(lambda: norm_ops.norm_fwd(norm_ops.RMSNORM, x16, g16, None, 1e-6), 4.0 * N * D), "norm_fwd (bf16 in)")

    # ---- prefill: latent attention beside the DeepSeek-V3 layer ----
    Ha, dn, dr, dv, Rk, qr = 16, 128, 64, 128, 512, 768
    sink = rn(Ha, dtype=f32)
    rope = rope_tables(64, 1e4, ctx + seq_len, None, dev)
    per = (max(seq_len, ctx) + 64) // 64 + 1
    nb = max(max(decode_batches), seqs)
    cache = PagedCache(1, [Rk + dr], nb * per, 64, nb, per, BF, dev)
    for i in range(nb):
        cache.reserve(i, max(seq_len, ctx) + 1)
    cache.pool[0].normal_()
    yq = rn(N, qr + Rk + dr)
    qg, kg = rn(qr, dtype=f32), rn(Rk, dtype=f32)
    q, kv = rn(N, Ha, dn + dr), rn(N, Ha * (dn + dv))
    lat = LA.mla_prepare(batch, yq, qg, kg, 1e-6, rope, cache, 0, True)[1]
    from ..models.deepseek_v3.model import rms_norm, rope_half_split
    from ..models.qwen35.primitives import precompute_rope_freqs
    fr = precompute_rope_freqs(dr, seq_len, 1e4, device=dev)
    g_qr, g_rk = rn(qr), rn(Rk)
    yb, kvb = yq.view(seqs, seq_len, -1), kv.view(seqs, seq_len, Ha, dn + dv)
    qb = q.view(seqs, seq_len, Ha, dn + dr)

    def ds_glue():
        rms_norm(yb[..., :qr].contiguous(), g_qr, 1e-6)
        ckv = rms_norm(yb[..., qr:qr + Rk].contiguous(), g_rk, 1e-6)
        qrp = rope_half_split(qb[..., dn:], fr)
        krp = rope_half_split(yb[..., qr + Rk:].reshape(seqs, seq_len, 1, dr), fr)[:, :, 0]
        torch.cat([kvb[..., :dn], krp[:, :, None, :].expand(seqs, seq_len, Ha, dr)], dim=-1)
        torch.cat([qb[..., :dn], qrp], dim=-1)
        torch.cat([ckv, krp], dim=-1)
    glue_bytes = 2.0 * N * (2 * (qr + Rk + dr) + (Rk + dr) + 2 * Ha * dr + Ha * dn + Ha * (dn + dr))

    def my_glue():
        LA.mla_prepare(batch, yq, qg, kg, 1e-6, rope, cache, 0, True)
        LA.mla_rope_qk(batch, q, kv[:, :Ha * dn], lat, Rk, rope)
    put("prefill", "latent norms, rotation, key assembly, cache write", tm(my_glue, glue_bytes), tm(ds_glue, glue_bytes),
        "norm kernels + torch rotation and concatenation")
    k = LA.mla_rope_qk(batch, q, kv[:, :Ha * dn], lat, Rk, rope)
    as4 = lambda t, d: t.unflatten(0, (seqs, seq_len)).unflatten(-1, (Ha, d))
    ob = torch.empty(N, Ha * dv, device=dev, dtype=BF)
    fa_flops = seqs * Ha * seq_len * seq_len * (dn + dr + dv) * 1.0
    q4, k4, v4, o4 = q.view(seqs, seq_len, Ha, -1), k.view(seqs, seq_len, Ha, -1), as4(kv[:, Ha * dn:], dv), as4(ob, dv)
    put("prefill", "flash attention 192 / 128 with sink", tm(lambda: A.attn_fwd(q4, k4, v4, True, 0.07, out=o4, sink=sink), 0, fa_flops),
        tm(lambda: A.attn_fwd(q4, k4, v4, True, 0.07, out=o4), 0, fa_flops), "the same kernel without a sink")
    del yq, kv, kvb, yb, q, qb, k, lat, ob, q4, k4, v4, o4

    # ---- experts ----
    wgu, wdn = (rn(experts, 2 * ff, D) * D ** -0.5), (rn(experts, D, ff) * ff ** -0.5)
    table = torch.rand(4096, experts, device=dev).argsort(-1)[:, :top].int().contiguous()
    tok = torch.randint(0, 4096, (N,), device=dev, dtype=torch.int32)
    ep = _fused_experts(dev, D, ff, experts, top)
    epw = {"gate_proj": rn(experts, D, ff) * D ** -0.5, "up_proj": rn(experts, D, ff) * D ** -0.5, "down_proj": rn(experts, ff, D) * ff ** -0.5}
    wt = torch.full((N, top), 1.0 / top, device=dev)
    moe_flops = 2.0 * N * top * 3 * D * ff
    idx = table[tok.long()]
    put("prefill", "experts (routing, grouped GEMMs, activation, combine)",
        tm(lambda: table_moe(x16, tok, table, wgu, wdn, 7.0, 1.702, x32), 0, moe_flops),
        tm(lambda: ep.forward(x16, wt, idx, epw), 0, moe_flops), "ep_moe_forward (fused, one rank)")
    _ext.check_status(dev)

    # ---- decode ----
    for B in decode_batches:
        d = {}
        out["decode"][f"batch {B}"] = d
        out_part = out["decode"]
        bd = _start_batch(list(range(B)), [1] * B, ctx, dev, ctx + 1)

        def putd(name, mine, other=None, other_name=None, _d=d):
            put("decode", "_tmp", mine, other, other_name)
            _d[name] = out_part.pop("_tmp")
        z1 = rn(B, inner + C + H)
        ring1, st1 = torch.zeros(B, 4, C, device=dev), torch.zeros(B, H, Ns, P, device=dev)

        def mine_step():
            yy = ssm.ssm_decode(bd, z1, cw, cb, ring1, dtb, al, Dk, st1, G)
            ssm.gated_group_norm(yy, None, gam, G, 1e-5, BF)
        # state in and out, one ring row of every earlier tap, the projection, the result
        b_mine = 8.0 * st1.numel() + 4.0 * B * C * 4 + 16.0 * C + 2.0 * z1.numel() + 2.0 * B * inner
        S2, cst = torch.zeros(B, Hv, 128, 128, device=dev), torch.zeros(B, Cd, 4, device=dev)
        m1, zz = rn(B, Cd), rn(B, Hv * 128)
        bb, aa, dtb16, al16, nw = rn(B, Hv), rn(B, Hv), rn(Hv), rn(Hv), rn(128)
        oo = torch.empty(B, Hv * 128, device=dev, dtype=BF)
        b_gdn = 8.0 * S2.numel() + 8.0 * cst.numel() + 2.0 * (m1.numel() + zz.numel() + oo.numel()) + 2.0 * wd.numel()
        putd("recurrent step (+ norm)", tm(mine_step, b_mine),
             tm(lambda: ops.gdn_decode_step(m1, zz, bb, aa, cst, wd, al16, dtb16, nw, S2, oo, Hqk, Hv, 128, 128, 1e-6), b_gdn), "gdn_decode_step")
        ids = list(range(B))
        cache.seq_lens.fill_(ctx)
        idt = torch.arange(B, dtype=torch.int32, device=dev)
        qf = rn(B, Ha, Rk + dr) * 0.3
        pb = 2.0 * B * ctx * (Rk + dr)
        putd("paged latent attention", tm(lambda: mla_paged_decode(qf, cache, 0, idt, 0.07, sink=sink, max_len=ctx), pb),
             tm(lambda: mla_paged_decode(qf, cache, 0, idt, 0.07, max_len=ctx), pb), "the same kernel without a sink")
        putd("latent attention, any-size kernel", tm(lambda: LA.latent_attention(bd, qf, cache, 0, Rk, 0.07, sink), pb))
        q1, ukv, ol = rn(B, Ha, dn + dr), rn(Ha * (dn + dv), Rk), rn(B, Ha, Rk)

        def mine_abs():
            LA.mla_absorb_q(bd, q1, ukv[:Ha * dn], rope, dr)
            LA.mla_absorb_out(ol, ukv[Ha * dn:])
        wkv = rn(Rk, Ha, dn + dv)

        def ds_abs():
            ql = torch.einsum("bhd,khd->bhk", q1[..., :dn], wkv[..., :dn])
            torch.cat([ql, q1[..., dn:]], dim=-1).contiguous()
            torch.einsum("bhk,khd->bhd", ol, wkv[..., dn:]).reshape(B, Ha * dv)
        ab = 2.0 * (ukv.numel() + q1.numel() + qf.numel() + ol.numel() + B * Ha * dv)
        putd("weight absorption (query and output)", tm(mine_abs, ab), tm(ds_abs, ab), "einsum")
        w_in = rn(inner + C + H, D) * D ** -0.5
        w_pad = w_in[:(w_in.shape[0] // 8) * 8]
        xb = rn(B, D)
        yl, yg = torch.empty(B, w_in.shape[0], device=dev, dtype=BF), torch.empty(B, w_pad.shape[0], device=dev, dtype=BF)
        putd("input projection", tm(lambda: linear_rows(xb, w_in, out=yl), 2.0 * w_in.numel()),
             tm(lambda: gemm(xb, w_pad, out=yg), 2.0 * w_pad.numel()), "tcgen05 GEMM")
        xr = rn(B, D, dtype=f32)
        hit = len(set(table[tok[:B].long()].reshape(-1).tolist()))
        eb = 2.0 * hit * 3 * D * ff
        putd("experts", tm(lambda: table_moe(xb, tok[:B], table, wgu, wdn, 7.0, 1.702, xr), eb),
             tm(lambda: ep.forward(xb, wt[:B], idx[:B], epw), eb), "ep_moe_forward (fused, one rank)")
    _ext.check_status(dev)
    return out


# ------------------------------------------------------------------------------------------------
def _time_calls(fn, warmup, n):
    for _ in range(warmup):
        fn()
    ts = []
    for _ in range(n):
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        ts.append(a.elapsed_time(b))
    return statistics.median(ts)


def step_engine_run(family, cfg, B, T, steps, dev):
    """Prefill (last logits), decode and prefill (all logits) times of a family on the shared step engine."""
    from ..models.registry import FAMILIES
    f = FAMILIES[family]
    params = f.mod().init_params(cfg, 0, BF, dev, on_device=True)
    per = (T + steps + 16 + cfg.page_size - 1) // cfg.page_size
    eng = getattr(f.mod(), f.engine)(params, cfg, f.mod().make_cache(cfg, B * per, B, per, BF, dev))
    tok = torch.randint(0, cfg.vocab_size, (B, T)).tolist()
    ids = list(range(B))

    every = [list(range(T))] * B

    def prefill(want=None):
        for i in ids:
            if i in eng.cache:
                eng.release(i)
        return eng.step(ids, tok, want)
    pre = _time_calls(prefill, 2, 3)
    pre_all = _time_calls(lambda: prefill(every), 1, 3)
    nxt = prefill().argmax(-1)
    state = {"t": nxt}

    def decode():
        state["t"] = eng.decode(ids, state["t"]).argmax(-1)
    dec = _time_calls(decode, 4, steps)
    return pre, dec, pre_all


def _vobunex_run(cfg, B, T, steps, dev):
    return step_engine_run("vobunex", cfg, B, T, steps, dev)


def qwen_like(width, heads, experts, top, ff, vocab, shared_ff=128):
    """The Qwen3.5-style hybrid of eight layers at the given widths."""
    from ..models.qwen35 import Qwen35Config
    return Qwen35Config(d_model=width, vocab_size=vocab, n_layers=8, max_position_embeddings=8192, gqa_n_q_heads=heads,
                        gqa_n_kv_heads=heads // 8, gqa_head_dim=256, delta_n_qk_heads=16, delta_n_v_heads=2 * width // 128,
                        delta_qk_head_dim=128, delta_v_head_dim=128, delta_chunk_size=64, n_routed_experts=experts,
                        n_experts_per_token=top, moe_intermediate_size=ff, shared_expert_intermediate_size=shared_ff)


def _qwen_run(cfg, B, T, steps, dev):
    from ..models.qwen35 import forward, init_cache, init_params
    from ..models.qwen35.decode_engine import Qwen35DecodeEngine
    ep = _fused_experts(dev, cfg.d_model, cfg.moe_intermediate_size, cfg.n_routed_experts, cfg.n_experts_per_token)
    params = init_params(cfg, 0, dtype=BF, device=dev, on_device=True)
    tok = torch.randint(0, cfg.vocab_size, (B, T), device=dev)

    @torch.no_grad()
    def prefill():
        cache = init_cache(cfg, B, T + steps + 16, dtype=BF, device=dev)
        return forward(params, tok, cfg, cache=cache, ep_group=ep)
    pre = _time_calls(prefill, 2, 3)
    lg, cache = prefill()
    state = {"t": lg[:, -1].argmax(-1)}
    del lg
    eng = Qwen35DecodeEngine(params, cfg, cache, ep=ep)

    def decode():
        state["t"] = eng.step(state["t"])
    return pre, _time_calls(decode, 4, steps)


def _deepseek_run(cfg, B, T, steps, dev):
    from ..models.deepseek_v3 import forward, init_params, make_cache
    from ..models.deepseek_v3.decode_engine import DeepSeekV3DecodeEngine
    ep = _fused_experts(dev, cfg.d_model, cfg.moe_intermediate_size, cfg.n_routed_experts, cfg.n_experts_per_token)
    params = init_params(cfg, 0, dtype=BF, device=dev, on_device=True)
    tok = torch.randint(0, cfg.vocab_size, (B, T), device=dev)
    per = (T + steps + 16 + 63) // 64
    ids = list(range(B))

    @torch.no_grad()
    def prefill():
        cache = make_cache(cfg, B * per, B, per, BF, dev)
        return forward(params, tok, cfg, cache, ids, ep=ep), cache
    pre = _time_calls(prefill, 2, 3)
    lg, cache = prefill()
    state = {"t": lg[:, -1].argmax(-1)}
    del lg
    eng = DeepSeekV3DecodeEngine(params, cfg, cache, ids, ep=ep, max_len=T + steps + 16)

    def decode():
        state["t"] = eng.step(state["t"]).clone()
    return pre, _time_calls(decode, 4, steps)


def model_table(dev, sizes=((2048, 16), (4096, 32)), shapes=((1, 4096), (8, 1024)), steps: int = 24) -> list:
    """Prefill and decode tokens/s. ``sizes``: (width, attention heads); ``shapes``: (sequences, prompt length)."""
    from ..models.deepseek_v3 import DeepSeekV3Config
    from ..models.vobunex import VobunexConfig
    E, top, ff, V = 64, 6, 1024, 65536
    rows = []
    for width, heads in sizes:
        hybrid = VobunexConfig.serving(width=width, n_mamba=6, n_attention=2, experts=E, top=top, ff=ff, heads=heads, vocab=V)
        qwen = qwen_like(width, heads, E, top, ff, V)
        latent = VobunexConfig.serving(width=width, n_mamba=0, n_attention=4, experts=E, top=top, ff=ff, heads=heads, vocab=V)
        ds = DeepSeekV3Config(d_model=width, vocab_size=V, n_layers=4, first_k_dense=0, max_position_embeddings=8192, n_heads=heads,
                              q_lora_rank=768, n_routed_experts=E, n_experts_per_token=top, n_group=1, topk_group=1,
                              moe_intermediate_size=ff)
        rows += model_rows(dev, width, shapes, steps, (("vobunex_hybrid_8_layers", _vobunex_run, hybrid), ("qwen35_8_layers", _qwen_run, qwen),
                                                       ("vobunex_latent_4_layers", _vobunex_run, latent), ("deepseek_v3_4_layers", _deepseek_run, ds)))
    return rows


def model_rows(dev, width, shapes, steps, models) -> list:
    """One row per shape; ``models``: (name, run function, configuration)."""
    rows = []
    for B, T in shapes:
        row = {"width": width, "batch": B, "prompt": T}
        for name, fn, cfg in models:
            try:
                pre, dec, *pre_all = fn(cfg, B, T, steps, dev)
                row[name] = {"prefill_ms": round(pre, 3), "prefill_tok_s": round(B * T / pre * 1e3), "decode_ms": round(dec, 4),
                             "decode_tok_s": round(B / dec * 1e3, 1)}
                if pre_all:      # the other families' prefill returns the logits of every position
                    row[name]["prefill_all_logits_ms"] = round(pre_all[0], 3)
            except Exception as e:  # noqa: BLE001 - a family that does not fit leaves the others' numbers
                row[name] = {"error": f"{type(e).__name__}: {str(e)[:200]}"}
            _sync_free()
        rows.append(row)
    return rows


def run(part: str = "all", family: str = "all") -> dict:
    dev = torch.device("cuda", 0)
    torch.cuda.set_device(dev)
    out = {"data": "synthetic token ids, random weights", "dtype": "bf16 (fp32 residual, norms, states)"}
    from . import serve_bench_fovudra as fov
    from . import serve_bench_mopalorn as mop
    from . import serve_bench_munazen as mun
    for name, kernels, models in (("vobunex", kernel_table, model_table), ("fovudra", fov.kernel_table, fov.model_table),
                                  ("munazen", mun.kernel_table, mun.model_table), ("mopalorn", mop.kernel_table, mop.model_table)):
        if family not in (name, "all"):
            continue
        out[name] = {}
        if part in ("kernels", "all"):
            out[name]["kernels"] = kernels(dev)
            _sync_free()
        if part in ("models", "all"):
            out[name]["models"] = models(dev)
    from .. import _ext
    _ext.check_status(dev)
    _sync_free()
    import torch.distributed as dist
    if dist.is_initialized():
        dist.destroy_process_group()
    return out
