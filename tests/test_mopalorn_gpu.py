"""Mopalorn on a B200: kernels, engine (eager and captured steps) and generation against mopalorn_oracle.py; fp32 on the any-size kernels,
bf16 also on the tensor-core kernels (flash attention with a window, block means or capped scores, paged decode of both kinds)."""
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import mopalorn_cases as K  # noqa: E402
import mopalorn_oracle as O  # noqa: E402

pytestmark = pytest.mark.gpu
TOL = 5e-4
DEV = "cuda"


@pytest.fixture(autouse=True)
def _needs_gpu(cuda_device):
    n = torch.get_num_threads()
    torch.set_num_threads(4)                                    # the plain implementation works on tiny tensors
    yield
    torch.set_num_threads(n)


# ---- the whole model in fp32 ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", sorted(K.CONFIGS))
def test_prompts_and_cuts(name):
    K.check_prompts_and_cuts(name, DEV, TOL)


@pytest.mark.parametrize("name", sorted(K.CONFIGS))
def test_layers(name):
    K.check_layers(name, DEV, TOL)


@pytest.mark.parametrize("name", sorted(K.CONFIGS))
def test_batches_slots_and_pages_reused(name):
    K.check_batch_and_reuse(name, DEV, TOL)


def test_mixed_step():
    K.check_mixed_step(DEV, TOL)


def test_greedy_and_sampled_generation():
    K.check_generate(DEV, TOL)


def test_long_decode():
    K.check_long_decode(DEV, TOL)


def test_far_tokens():
    K.check_far_tokens(DEV, TOL)


# ---- attention and its operands alone ------------------------------------------------------------------------------------
def test_one_key_stands_out():
    K.check_one_key_stands_out(DEV, 1e-4)
    K.check_one_key_stands_out(DEV, 1e-4, masks=((0, 0),), softcap=9.0)
    K.check_one_key_stands_out(DEV, 1e-4, masks=((17, 0), (12, 3)), softcap=9.0)


SHAPES = [(4, 2, 64, 64), (4, 1, 64, 128), (3, 1, 40, 72), (2, 1, 128, 128), (2, 2, 136, 120), (8, 1, 128, 256), (2, 1, 200, 256)]


@pytest.mark.parametrize("H,G,d,dv", SHAPES)
def test_one_key_stands_out_on_tensor_cores(H, G, d, dv):
    K.check_one_key_stands_out(DEV, 0.05, torch.bfloat16, H, G, d, dv, n=150, ps=64, masks=((20, 5), (70, 16), (1, 3)))


@pytest.mark.parametrize("H,G,d,dv", SHAPES)
def test_capped_scores_on_tensor_cores(H, G, d, dv):
    K.check_one_key_stands_out(DEV, 0.05, torch.bfloat16, H, G, d, dv, n=150, ps=64, masks=((0, 0),), softcap=12.0)


def test_one_latent_stands_out():
    K.check_one_latent_stands_out(DEV, 1e-4)


@pytest.mark.parametrize("H,dn,dr,dv,R", [(3, 128, 64, 128, 512), (20, 128, 64, 128, 512), (2, 136, 56, 128, 40), (3, 24, 8, 32, 64)])
def test_one_latent_stands_out_on_tensor_cores(H, dn, dr, dv, R):
    """Whole prompts on the windowed flash kernel, decode steps on the windowed paged kernel, portions on the any-size kernel."""
    K.check_one_latent_stands_out(DEV, 0.05, torch.bfloat16, H, dn, dr, dv, R, n=150, ps=64, sizes=(20, 64, 70, 1, 400))


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-6), (torch.bfloat16, 0.02)])
@pytest.mark.parametrize("P,ps", [(4, 8), (5, 8), (8, 8), (19, 8), (1, 8), (16, 64), (24, 16)])
def test_block_means_follow_the_rows(P, ps, dtype, tol):
    K.check_block_means(DEV, dtype, tol, P, ps)
    K.check_block_means(DEV, dtype, tol, P, ps, G=1, d=16, dv=8)


@pytest.mark.parametrize("lens", [[700, 700], [1, 513, 64, 700, 129]])
@pytest.mark.parametrize("size,P", [(30, 2), (128, 1), (100, 16), (257, 7), (1000, 4)])
@pytest.mark.parametrize("d,dv", [(64, 64), (40, 56), (128, 128)])
def test_whole_prompts_with_many_blocks(d, dv, size, P, lens):
    """Several key tiles of block means, tiles that mix seen and unseen ones, unequal prompts in one batch; all positions."""
    from jax_gpt_b200.cache.paged import PagedCache
    from jax_gpt_b200.ops import window_attention as WA
    from jax_gpt_b200.ops.mixed_kv import mixed_kv
    from jax_gpt_b200.ops.packed import PackedBatch, seq_begin
    H, G, n, dt = 2, 1, sum(lens), torch.bfloat16
    g = torch.Generator().manual_seed(size + P)
    per = (max(lens) + 63) // 64
    cache = PagedCache(1, [G * (d + dv)], per * len(lens), 64, len(lens), per, dt, DEV, blocks=[P])
    cache.pool[0].fill_(1e3)
    cache.pooled[0].fill_(1e3)
    for i, k in enumerate(lens):
        cache.reserve(i, k)
    y = torch.randn(n, H * d + G * d + G * dv, generator=g).to(dt)
    y[:, :H * d] *= 2
    sink = torch.randn(H, generator=g)
    b = PackedBatch.make(list(range(len(lens))), lens, True, max(lens), DEV)
    zeros = lambda k: torch.zeros(k, dtype=torch.int32, device=DEV)
    seq_begin(b, zeros(n), zeros(len(lens)), zeros(len(lens)))
    wide = WA.flash_widths(b, dt, True, d, dv)
    q, k, v = mixed_kv(b, y.to(DEV), (0, H * d, H * d + G * d), H, G, d, dv, cache, 0, wide, window=size)
    scale = d ** -0.5
    got = WA.grouped_attention(b, q, k, v, cache, 0, G, dv, scale, size, sink=sink.to(DEV), pool=P)[..., :dv].double().cpu()
    at = 0
    for m in lens:
        qq, kk, vv = (t.double().reshape(m, -1, w) for t, w in zip(y[at:at + m].split([H * d, G * d, G * dv], 1), (d, d, dv)))
        rnd = lambda t: t.to(dt).double()
        kk, vv = (torch.cat([t, rnd(O.block_means(t, P))]).expand(-1, H, -1) for t in (kk, vv))
        seen = torch.cat([O.seen_tokens(m, size), O.seen_blocks(m, P, size)], 1)
        s = torch.einsum("ihd,jhd->hij", qq, kk) * scale
        want = torch.einsum("hij,jhd->ihd", O.weights_of(s, seen, sink.double()[:, None, None]), vv)
        assert float((got[at:at + m] - want).abs().max()) < 0.04, m
        at += m


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-4), (torch.bfloat16, 1.0)])
def test_activation(dtype, tol):
    from jax_gpt_b200.ops.gemm import linear_rows
    K.check_activation(linear_rows, DEV, dtype, tol, ((1, 64, 40), (3, 33, 9), (8, 256, 128), (20, 128, 72), (300, 256, 384), (1000, 512, 1024), (70, 21, 10), (100, 64, 77), (257, 128, 200)))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows,N,gap", [(5, 64, 8), (300, 2048, 0), (7, 13, 3)])
def test_sigmoid_gate(rows, N, gap, dtype):
    from jax_gpt_b200.ops.latent_attention import sigmoid_gate
    o, g = torch.randn(rows, N).to(dtype), (4 * torch.randn(rows, N + gap)).to(dtype)
    want = o.double() * torch.sigmoid(g[:, gap:].double())
    got = sigmoid_gate(o.to(DEV), g.to(DEV)[:, gap:]).double().cpu()
    assert float((got - want).abs().max()) < (2e-6 if dtype == torch.float32 else 2e-2)


# Two sublayer inputs or outputs near zero magnify rounding without bound in these small random models (their norms divide by the root
# mean square), so bf16 runs are judged by the median row.
@pytest.mark.parametrize("name", sorted(K.CONFIGS))
def test_bf16_any_size(name):
    cfg = K.CONFIGS[name]
    w = K.weights(cfg, 1, torch.bfloat16)
    toks = K.tokens(cfg, 45, 2)
    want = O.forward(toks, cfg, w)
    eng = K.engine(cfg, w, DEV, torch.bfloat16)
    spread = want.std(-1).mean()
    for k, cuts in enumerate(([45], [30] + [1] * 15, [20, 25])):
        d = (K.run(eng, f"s{k}", toks, cuts).double().cpu() - want).pow(2).mean(-1).sqrt() / spread
        assert float(d.median()) < 0.1, (name, cuts)
        eng.release(f"s{k}")


# ---- tensor-core shapes in the whole model ---------------------------------------------------------------------------------
TENSOR = K.config([(K.latent(heads=3, dim=128, rot_dim=64, vdim=128, kv_rank=512, size=75, scale=0.07), None),
                   (K.pooled(heads=4, kv_heads=1, dim=64, vdim=128, size=70, pool=16, scale=0.1), K.dense(512)),
                   (K.full(heads=8, kv_heads=1, dim=128, vdim=128, scale=0.08, softcap=9.0, coef=0.3, every=64), None),
                   (K.pooled(heads=3, kv_heads=1, dim=72, vdim=128, size=33, pool=5, scale=0.1), None),
                   (K.latent(heads=17, dim=128, rot_dim=64, vdim=128, kv_rank=512, size=130, scale=0.07), K.dense(136)),
                   (K.full(heads=2, kv_heads=2, dim=40, vdim=64, scale=0.15, softcap=30.0, coef=0.5, every=100), K.dense(256))], width=128, vocab=200)


def _bf16_errors_ok(errors, spread):
    """Errors of logit rows relative to the logits' spread: bf16 rounding; a wrong row is off by about 1."""
    e = torch.cat(errors) / spread
    return float(e.median()) < 0.03 and float(e.quantile(0.95)) < 0.08 and float(e.max()) < 0.5


def test_tensor_core_shapes_whole_and_decoded():
    w = K.weights(TENSOR, 31, torch.bfloat16)
    sizes = (300, 1, 129, 64)
    reqs = [K.tokens(TENSOR, n + 12, n) for n in sizes]
    want = [O.forward(t, TENSOR, w) for t in reqs]
    eng = K.engine(TENSOR, w, DEV, torch.bfloat16, page_size=64, max_tokens=1024)
    spread = float(want[0].std(-1).mean())
    prompts, steps = [], []
    err = lambda a, b: (a.double().cpu() - b).pow(2).mean(-1).sqrt()
    for i, (t, n) in enumerate(zip(reqs, sizes)):              # alone, equal lengths (one flash launch for the batch)
        lg = eng.step(["x", "y"], [t[:n], t[:n]], [list(range(n))] * 2)
        prompts.append(err(lg, torch.cat([want[i][:n]] * 2)))
        for s in range(12):
            steps.append(err(eng.decode(["x", "y"], [t[n + s]] * 2), torch.stack([want[i][n + s]] * 2)))
        eng.release("x")
        eng.release("y")
    assert _bf16_errors_ok(prompts, spread) and _bf16_errors_ok(steps, spread)
    ids = list("abcd")
    steps = []
    lg = eng.step(ids, [t[:n] for t, n in zip(reqs, sizes)])
    steps.append(err(lg, torch.stack([x[n - 1] for x, n in zip(want, sizes)])))
    for s in range(12):
        if s == 6:
            eng.release(ids.pop(1))
            reqs.pop(1), want.pop(1)
            sizes = (300, 129, 64)
        lg = eng.decode(ids, [t[n + s] for t, n in zip(reqs, sizes)])
        steps.append(err(lg, torch.stack([x[n + s] for x, n in zip(want, sizes)])))
    assert _bf16_errors_ok(steps, spread)


def test_tensor_core_shapes_continued_prompt_and_long_decode():
    w = K.weights(TENSOR, 32, torch.bfloat16)
    toks = K.tokens(TENSOR, 270, 33)
    want = O.forward(toks, TENSOR, w)
    eng = K.engine(TENSOR, w, DEV, torch.bfloat16, page_size=64, max_tokens=1024)
    for name, cuts in (("a", [130, 2, 128, 10]), ("b", [20] + [1] * 250)):
        got = K.run(eng, name, toks, cuts).double().cpu()
        assert _bf16_errors_ok([(got - want).pow(2).mean(-1).sqrt()], float(want.std(-1).mean())), name
