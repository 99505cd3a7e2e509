"""Munazen on a B200: kernels, engine (eager and captured steps) and generation against munazen_oracle.py; fp32 on the any-size
kernels, bf16 also on the tensor-core kernels (padded flash attention, paged decode with wider values, recurrent units in blocks of
multiples of 16, linear-attention keys of 64 / 128)."""
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import munazen_cases as K  # noqa: E402
import munazen_oracle as O  # noqa: E402

pytestmark = pytest.mark.gpu
TOL = 5e-4
DEV = "cuda"


@pytest.fixture(autouse=True)
def _needs_gpu(cuda_device):
    yield


def rel(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return float((a - b).norm() / b.norm().clamp_min(1e-12))


def begin(ids, lens, starts, max_len=4096):
    """A packed batch whose sequences start at the given positions."""
    from jax_gpt_b200.ops.packed import PackedBatch, seq_begin
    b = PackedBatch.make(ids, lens, not any(starts), max_len, DEV)
    have = torch.zeros(max(ids) + 1, dtype=torch.int32)
    for i, s in zip(ids, starts):
        have[i] = s
    seq_begin(b, torch.zeros(b.n_tok, dtype=torch.int32, device=DEV), have.to(DEV), torch.zeros_like(have).to(DEV))
    return b


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


def test_one_key_stands_out():
    K.check_one_key_stands_out(DEV, 1e-4)


@pytest.mark.parametrize("H,G,d,dv,dims", [(4, 2, 64, 64, 64), (4, 1, 64, 128, 16), (3, 1, 40, 72, 24), (2, 1, 128, 128, 128), (2, 2, 136, 120, 8),
                                           (8, 1, 128, 256, 64), (2, 1, 200, 256, 200)])
def test_one_key_stands_out_on_tensor_cores(H, G, d, dv, dims):
    K.check_one_key_stands_out(DEV, 0.05, torch.bfloat16, H, G, d, dv, dims, n=150, ps=64)


def test_far_tokens():
    K.check_far_tokens(DEV, TOL)


def test_state_carries():
    K.check_state_carries(DEV, TOL)


def test_long_decode():
    K.check_long_decode(DEV, TOL)


def test_loop_passes_keep_their_own_state():
    K.check_loop_passes_keep_their_own_state(DEV, TOL)


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


# ---- tensor-core shapes ----------------------------------------------------------------------------------------------------
TENSOR = K.config([(K.gla(heads=2, dim=128, vdim=128, tau=10.0), None),
                   (K.par(heads=8, kv_heads=2, dim=64, rot_dims=32, vdim=128, scale=0.2, width=256, blocks=2, conv=4), K.dense(512)),
                   (K.gla(heads=3, dim=64, vdim=64, tau=2.0), None),
                   (K.par(heads=3, kv_heads=1, dim=72, rot_dims=72, vdim=88, scale=0.1, width=96, blocks=2, conv=3), None),
                   (K.par(heads=2, kv_heads=1, dim=128, rot_dims=64, vdim=128, scale=0.1, width=320, blocks=1, conv=2), K.dense(136))],
                  width=128, groups=1, vocab=200, streams=2, loop=(1, 3, 2))


def _bf16_errors_ok(errors, spread):
    """Errors of logit rows relative to the logits' spread: bf16 rounding; a wrong row is off by about 1."""
    e = torch.cat(errors) / spread
    return float(e.median()) < 0.02 and float(e.quantile(0.95)) < 0.06 and float(e.max()) < 0.5


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


def test_tensor_core_shapes_continued_prompt():
    w = K.weights(TENSOR, 32, torch.bfloat16)
    toks = K.tokens(TENSOR, 270, 33)
    want = O.forward(toks, TENSOR, w)
    eng = K.engine(TENSOR, w, DEV, torch.bfloat16, page_size=64, max_tokens=512)
    got = K.run(eng, "a", toks, [130, 2, 128, 10]).double().cpu()
    assert _bf16_errors_ok([(got - want).pow(2).mean(-1).sqrt()], float(want.std(-1).mean()))


# ---- gated linear recurrent unit -------------------------------------------------------------------------------------------
LENS, SLOTS = [63, 64, 65, 1, 200, 2, 128], [5, 0, 3, 1, 2, 4, 6]


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("W,blocks,taps", [(256, 2, 4), (64, 4, 4), (96, 2, 3), (48, 1, 2), (320, 1, 4), (30, 3, 5), (24, 24, 1), (40, 5, 6), (512, 1, 1)])
def test_gated_lru(W, blocks, taps, dtype):
    """Chunk edges, tails, carried states and convolution inputs; slow, fast and mixed decays; a first token that dominates."""
    from jax_gpt_b200.ops.gated_lru import LruWeights, gated_lru, lru_decay
    g = torch.Generator().manual_seed(W + taps)
    r = lambda *s: torch.randn(*s, generator=g)
    n, wb = sum(LENS), W // blocks
    wide = r(n, 2 * W + 16)
    first = 0
    for k in LENS:
        wide[first, :W] *= 20
        first += k
    wide = wide.to(dtype)
    x, y = wide[:, :W], wide[:, W + 8:2 * W + 8]
    xb, yb, conv, cb = r(W), r(W), r(W, taps), 0.3 * r(W)
    ra, ri = ((2 * r(blocks, wb, wb) * wb ** -0.5).to(dtype) for _ in range(2))
    rab, rib, lam = r(blocks, wb), r(blocks, wb), torch.linspace(-9, 2, W)[torch.randperm(W, generator=g)]
    dv = lambda t: t.contiguous().to(DEV)
    w = LruWeights(dv(xb), dv(yb), dv(conv), dv(cb), dv(torch.stack([ra, ri], 1)), dv(torch.stack([rab, rib], 1)), dv(lru_decay(lam)))
    D = lambda t: t.double()
    wd = wide.to(DEV)
    tol_state, tol_out = (1e-4, 4e-3) if dtype == torch.bfloat16 else (3e-6, 3e-6)
    for start in (0, 7):
        s0, ring0 = 3 * r(7, W), r(7, taps, W)
        state, ring = s0.to(DEV), ring0.to(DEV)
        out = torch.zeros(n, W + 24, dtype=dtype, device=DEV)
        gated_lru(begin(SLOTS, LENS, [start] * 7), wd[:, :W], wd[:, W + 8:2 * W + 8], w, ring, state, 0.6, out[:, 8:W + 8])
        assert float(out[:, :8].abs().max()) == 0 and float(out[:, W + 8:].abs().max()) == 0
        c0 = 0
        for k, slot in zip(LENS, SLOTS):
            xin = D(x[c0:c0 + k].float() + xb)
            past = torch.stack([D(ring0[slot, p % taps]) for p in range(start - taps + 1, start)]) if start and taps > 1 else xin[:0]
            u = O.causal_conv(torch.cat([past, xin]), D(conv), D(cb))[len(past):]
            S, last = O.rglru_recurrence(u, O.sigmoid(O.block_linear(u, D(ra), D(rab))), O.sigmoid(O.block_linear(u, D(ri), D(rib))), D(lam),
                                         D(s0[slot]) if start else None)
            want = 0.6 * S * O.gelu_tanh(D(y[c0:c0 + k].float() + yb))
            assert rel(out[c0:c0 + k, 8:W + 8], want) < tol_out, (k, start)
            assert rel(state[slot], last) < tol_state, (k, start)
            for p in range(max(start, start + k - taps + 1), start + k):
                assert rel(ring[slot, p % taps], xin[p - start]) < 1e-6, (k, start, p)
            c0 += k


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("W,blocks,taps", [(256, 2, 4), (30, 3, 5), (1024, 8, 4), (24, 24, 1), (96, 2, 3), (1024, 2, 1), (48, 3, 6)])
@pytest.mark.parametrize("B", [1, 3, 8, 19])
def test_gated_lru_one_token_steps(W, blocks, taps, B, dtype):
    """Steps from position 0 on against the recurrence over the whole sequence."""
    from jax_gpt_b200.ops.gated_lru import LruWeights, gated_lru, lru_decay
    g = torch.Generator().manual_seed(W + B)
    r = lambda *s: torch.randn(*s, generator=g)
    T, wb = 9, W // blocks
    x, y = r(T, B, W).to(dtype), r(T, B, W).to(dtype)
    xb, yb, conv, cb, lam = r(W), r(W), r(W, taps), r(W), -4 + 2 * r(W)
    ra, ri = ((2 * r(blocks, wb, wb) * wb ** -0.5).to(dtype) for _ in range(2))
    rab, rib = r(blocks, wb), r(blocks, wb)
    dv = lambda t: t.contiguous().to(DEV)
    w = LruWeights(dv(xb), dv(yb), dv(conv), dv(cb), dv(torch.stack([ra, ri], 1)), dv(torch.stack([rab, rib], 1)), dv(lru_decay(lam)))
    state, ring = torch.full((B, W), 1e4, device=DEV), torch.full((B, taps, W), 1e4, device=DEV)
    slots = torch.randperm(B, generator=g).tolist()
    got = []
    for t in range(T):
        out = torch.empty(B, W, dtype=dtype, device=DEV)
        gated_lru(begin(slots, [1] * B, [t] * B), x[t].to(DEV), y[t].to(DEV), w, ring, state, 1.5, out)
        got.append(out.cpu())
    D = lambda t: t.double()
    for b in range(B):
        u = O.causal_conv(D(x[:, b].float() + xb), D(conv), D(cb))
        S, last = O.rglru_recurrence(u, O.sigmoid(O.block_linear(u, D(ra), D(rab))), O.sigmoid(O.block_linear(u, D(ri), D(rib))), D(lam))
        assert rel(torch.stack(got)[:, b], 1.5 * S * O.gelu_tanh(D(y[:, b].float() + yb))) < (4e-3 if dtype == torch.bfloat16 else 2e-6)
        assert rel(state[slots[b]], last) < (1e-5 if dtype == torch.bfloat16 else 2e-6)


# ---- linear attention with a decay per key channel -------------------------------------------------------------------------
def _gla_case(H, N, P, R, lens, dtype, g, low_scale=1.0, shift=1.0):
    x = torch.randn(sum(lens), H * (2 * N + P) + 8, generator=g) * 0.5
    first = 0
    for k in lens:
        x[first] *= 12                                         # the first token of every sequence dominates the state
        first += k
    low = low_scale * torch.randn(sum(lens), R + 8, generator=g)
    w2, b2 = (torch.randn(H * N, R, generator=g) * R ** -0.5).to(dtype), shift + torch.randn(H * N, generator=g)
    return x.to(dtype), low.to(dtype), w2, b2


def _log_alpha(low, w2, b2, tau, H, N):
    return O.log_sigmoid(low.double() @ w2.double().T + b2.double()).reshape(len(low), H, N) / tau


@pytest.mark.parametrize("kind", ["auto", "tokens"])
@pytest.mark.parametrize("H,N,P,R", [(3, 128, 64, 16), (2, 128, 128, 16), (1, 64, 192, 8), (4, 64, 64, 24), (2, 32, 48, 16), (2, 48, 80, 5), (1, 256, 64, 16)])
@pytest.mark.parametrize("tau,shift,scale", [(16.0, 1.0, 1.0), (1.0, 4.0, 2.0), (0.3, -3.0, 6.0)])
def test_channel_decay_scan(H, N, P, R, tau, shift, scale, kind):
    """Slow decays, mixed ones, and decays far below what a chunk's products could hold; chunk edges, tails, carried state."""
    from jax_gpt_b200.ops import linear_attention as LIN
    g = torch.Generator().manual_seed(N + P)
    x, low, w2, b2 = _gla_case(H, N, P, R, LENS, torch.bfloat16, g, scale, shift)
    w = H * (2 * N + P)
    xd, ld = x.to(DEV), low.to(DEV)
    for start in (0, 7):
        s0 = torch.randn(7, H, N, P, generator=g)
        state = s0.to(DEV)
        ch = LIN.ChannelDecay(ld[:, :R], w2.to(DEV), b2.to(DEV), tau)
        y = LIN.linear_scan(begin(SLOTS, LENS, [start] * 7), xd[:, :w], state, channels=ch, q_scale=0.7, kind=None if kind == "auto" else LIN.TOKENS).y
        c0 = 0
        for k, slot in zip(LENS, SLOTS):
            q, kk, v = [t.reshape(k, H, -1) for t in x[c0:c0 + k, :w].double().split([H * N, H * N, H * P], -1)]
            want, S = O.channel_decay_recurrence(0.7 * q, kk, v, _log_alpha(low[c0:c0 + k, :R], w2, b2, tau, H, N), s0[slot].double() if start else None)
            for h in range(H):
                assert rel(y[c0:c0 + k].reshape(k, H, P)[:, h], want[:, h]) < 6e-3, (k, start, h)
                assert rel(state[slot, h], S[h]) < 3e-5, (k, start, h)
            c0 += k


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("H,N,P,R", [(3, 16, 24, 4), (2, 128, 128, 16), (1, 5, 67, 3), (2, 300, 40, 1), (4, 1, 1, 2)])
def test_channel_decay_steps_of_any_size(H, N, P, R, dtype):
    """Token-by-token scan of a portion, then one-token steps from its state, norm and SiLU gate behind."""
    from jax_gpt_b200.ops import linear_attention as LIN
    g = torch.Generator().manual_seed(N)
    n, steps = 19, 4
    x, low, w2, b2 = _gla_case(H, N, P, R, [n + steps] * 2, dtype, g)
    w = H * (2 * N + P)
    x, low = x[:, :w].reshape(2, n + steps, w), low[:, :R].reshape(2, n + steps, R)
    state = torch.full((3, H, N, P), 1e4, device=DEV)
    z, gamma = torch.randn(2, n + steps, H * P, generator=g).to(dtype), torch.rand(P, generator=g) + 0.5
    got = []
    for at, k in [(0, n)] + [(n + t, 1) for t in range(steps)]:
        b = begin([2, 0], [k, k], [at, at])
        flat = lambda t: t[:, at:at + k].reshape(2 * k, -1).contiguous().to(DEV)
        s = LIN.linear_scan(b, flat(x), state, channels=LIN.ChannelDecay(flat(low), w2.to(DEV), b2.to(DEV), 3.0), q_scale=0.5)
        o = LIN.head_norm_gate(b, s, flat(z), gamma.repeat(H).to(DEV), H, 1e-3, dtype, silu=True)
        got.append(o.reshape(2, k, H * P))
    got = torch.cat(got, 1)
    for r in range(2):
        q, k, v = [t.reshape(n + steps, H, -1) for t in x[r].double().split([H * N, H * N, H * P], -1)]
        o, _ = O.channel_decay_recurrence(q * 0.5, k, v, _log_alpha(low[r], w2, b2, 3.0, H, N))
        want = (O.unit_rms(o, 1e-3) * gamma.double()).reshape(n + steps, -1) * O.silu(z[r].double())
        assert rel(got[r], want) < (2e-2 if dtype == torch.bfloat16 else 2e-5), r


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_slow_decays_do_not_drift(dtype):
    """Thousands of tokens with decays close to 1: a systematic error of the decay would add up to far more than rounding."""
    from jax_gpt_b200.ops import linear_attention as LIN
    from jax_gpt_b200.ops.gated_lru import LruWeights, gated_lru, lru_decay
    g = torch.Generator().manual_seed(9)
    n, W = 3000, 64
    r = lambda *s: torch.randn(*s, generator=g)
    x, y = (0.1 * r(n, W) + 1).to(dtype), r(n, W).to(dtype)
    ra, ri, rab, rib, lam = (r(1, W, W) * 0.02).to(dtype), (r(1, W, W) * 0.02).to(dtype), r(1, W), 3 + r(1, W), -9 + 0.3 * r(W)
    conv, zero = torch.ones(W, 1), torch.zeros(W)
    dv = lambda t: t.contiguous().to(DEV)
    w = LruWeights(dv(zero), dv(zero), dv(conv), dv(zero), dv(torch.stack([ra, ri], 1)), dv(torch.stack([rab, rib], 1)), dv(lru_decay(lam)))
    state, out = torch.zeros(1, W, device=DEV), torch.empty(n, W, dtype=dtype, device=DEV)
    gated_lru(begin([0], [n], [0]), dv(x), dv(y), w, torch.zeros(1, 1, W, device=DEV), state, 1.0, out)
    D = lambda t: t.double()
    _, last = O.rglru_recurrence(D(x), O.sigmoid(O.block_linear(D(x), D(ra), D(rab))), O.sigmoid(O.block_linear(D(x), D(ri), D(rib))), D(lam))
    assert rel(state[0], last) < 3e-6
    H, N, P = 1, 16, 16
    qkv = (0.1 * r(n, H * (2 * N + P)) + 1).to(dtype)
    low, w2, b2 = r(n, 4).to(dtype), (0.1 * r(H * N, 4)).to(dtype), 4 + r(H * N)
    S = torch.zeros(1, H, N, P, device=DEV)
    LIN.linear_scan(begin([0], [n], [0]), dv(qkv), S, channels=LIN.ChannelDecay(dv(low), dv(w2), dv(b2), 20.0))
    q, k, v = [t.reshape(n, H, -1) for t in D(qkv).split([H * N, H * N, H * P], -1)]
    _, want = O.channel_decay_recurrence(q, k, v, _log_alpha(low, w2, b2, 20.0, H, N))
    assert rel(S[0], want) < (2e-5 if dtype == torch.bfloat16 else 3e-6)


# ---- attention operands -----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("H,G,dk,dv,dims,dense", [(8, 2, 128, 128, 128, (128, 128)), (3, 3, 40, 72, 24, (128, 128)), (4, 1, 12, 20, 6, None),
                                                  (2, 1, 7, 2, 4, (64, 64)), (2, 2, 64, 128, 64, None), (1, 1, 250, 130, 2, (256, 256))])
def test_rotated_operands(H, G, dk, dv, dims, dense, dtype):
    from jax_gpt_b200.cache.paged import PagedCache
    from jax_gpt_b200.ops import rotated_kv as RKV
    from jax_gpt_b200.ops.rope import rope_tables
    g = torch.Generator().manual_seed(dk)
    rot = K.rot(dims)
    cache = PagedCache(2, [3, G * (dk + dv)], 20, 8, 3, 8, dtype, DEV)
    ids, lens, starts = [2, 0], [13, 1], [5, 9]
    cache.begin_step(ids, [s + n for s, n in zip(starts, lens)])
    b = begin(ids, lens, starts, 64)
    up8 = lambda n: (n + 7) // 8 * 8
    cols = (0, up8(H * dk), up8(H * dk) + up8(G * dk))
    y = torch.randn(14, up8(cols[2] + G * dv) + 8, generator=g).to(dtype)
    sizes = (H * dk, G * dk, G * dv)
    bias = torch.randn(sum(sizes), generator=g)
    tables = lambda d, sc: rope_tables(d, rot["base"], 64, sc, DEV)
    q, k, v = RKV.qkv_rotate(b, y.to(DEV), cols, bias.to(DEV), H, G, dk, dv, tables(dims, rot["scaling"]), tables(dv, None), cache, 1, dense)
    pos = list(range(5, 18)) + [9]
    parts = [(y[:, c:c + n].double() + bb.double()).reshape(14, -1, d) for c, n, bb, d in zip(cols, sizes, bias.split(sizes), (dk, dk, dv))]
    f, amp = O.rotary_frequencies(rot)
    wq, wk, wv = O.turn_pairs(parts[0], pos, f, amp), O.turn_pairs(parts[1], pos, f, amp), O.turn_pairs(parts[2], pos, O.value_frequencies(rot["base"], dv))
    tol = 5e-3 if dtype == torch.bfloat16 else 2e-6
    assert rel(q[..., :dk], wq) < tol
    if dense:
        assert rel(k[..., :dk], wk) < tol and rel(v[..., :dv], wv) < tol
        assert all(float(t[..., d:].abs().sum()) == 0 for t, d in ((q, dk), (k, dk), (v, dv)))
    for slot, c0, n, s in ((2, 0, 13, 5), (0, 13, 1, 9)):
        pages, offs = cache.slots(slot, s, n)
        rows = cache.pool[1][pages, offs].double().cpu()
        assert rel(rows[:, :G * dk], wk[c0:c0 + n].reshape(n, -1)) < tol and rel(rows[:, G * dk:], wv[c0:c0 + n].reshape(n, -1)) < tol
    o = torch.randn(14, H, (dense or (0, dv))[1], generator=g).to(dtype)
    gate = torch.randn(14, H + 3, generator=g).to(dtype)
    out = torch.zeros(14, H * dv + 16, dtype=dtype, device=DEV)
    RKV.turn_back_gate(b, o.to(DEV), gate.to(DEV)[:, :H], tables(dv, None), 1.7, out[:, 8:8 + H * dv])
    want = O.turn_pairs(o[..., :dv].double(), [-p for p in pos], O.value_frequencies(rot["base"], dv)) * 1.7 * O.sigmoid(gate[:, :H].double())[:, :, None]
    assert rel(out[:, 8:8 + H * dv], want.reshape(14, -1)) < tol
    assert float(out[:, :8].abs().sum()) == 0 and float(out[:, 8 + H * dv:].abs().sum()) == 0


# ---- streams, norms, activations --------------------------------------------------------------------------------------------
@pytest.mark.parametrize("y_dtype,dtype", [(torch.bfloat16, torch.bfloat16), (torch.float32, torch.bfloat16), (torch.float32, torch.float32)])
@pytest.mark.parametrize("rows,S,D,groups", [(3, 3, 30, 3), (70, 2, 256, 8), (2, 4, 1000, 5), (5, 2, 2048, 4), (3, 1, 4096, 1), (2, 3, 8192, 64),
                                             (2, 2, 9000, 9), (4, 2, 384, 3), (3, 6, 64, 2), (2, 4, 12288, 4), (1, 16, 20, 20), (3, 2, 1024, 256)])
def test_stream_norm(rows, S, D, groups, y_dtype, dtype):
    from jax_gpt_b200.ops.streams import Connection, group_norm_rows, stream_norm
    g = torch.Generator().manual_seed(D + S)
    r = lambda *s: torch.randn(*s, generator=g)
    y, xs, bias = r(rows, D).to(y_dtype), 5 * r(rows, S, D), r(D)
    mix, wo, wi, gamma = r(S, S), r(S), r(S), r(D)
    xs[..., :D // groups] *= 30                                 # one group far from the others
    d = lambda t: t.to(DEV)
    for first in (False, True):
        got = d(xs)
        h, u = stream_norm(d(y), got, Connection(d(wi), None if first else d(mix), d(wo)), d(wi), d(gamma), groups, 1e-3, dtype, bias=d(bias), want_u=True)
        new = O.streams_out(0 * xs.double() if first else xs.double(), y.double() + bias.double(), mix.double(), wo.double())
        want = O.streams_in(new, wi.double())
        assert rel(got, new) < 1e-6 and rel(u, want) < 2e-6
        assert rel(h, O.group_norm(want, gamma.double(), groups, 1e-3)) < (4e-3 if dtype == torch.bfloat16 else 3e-6)
    x = r(rows, D)
    assert rel(group_norm_rows(d(x), d(gamma), groups, 1e-3, dtype), O.group_norm(x.double(), gamma.double(), groups, 1e-3)) < (
        4e-3 if dtype == torch.bfloat16 else 1e-6)


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("rows,N", [(3, 7), (2, 320), (40, 1024), (3, 2000), (2, 4096), (3, 8192), (2, 11008), (1, 20480), (2, 33000)])
def test_poly_norm(rows, N, dtype):
    from jax_gpt_b200.ops.streams import poly_norm
    g = torch.Generator().manual_seed(N)
    z = (3 * torch.randn(rows, N + 8, generator=g)).to(dtype)
    coef = torch.tensor([0.7, -0.5, 1.3, 0.2])
    assert rel(poly_norm(z.to(DEV)[:, :N], coef.to(DEV), 1e-4), O.poly_norm(z[:, :N].double(), coef.double(), 1e-4)) < (
        4e-3 if dtype == torch.bfloat16 else 1e-6)


# ---- engine ----------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("cfg", [K.CONFIGS["mixed_odd"], TENSOR], ids=["mixed_odd", "tensor"])
def test_captured_steps_equal_eager_steps(cfg):
    """Graph replays over changing batches, slots and block tables against the eager engine, bit by bit."""
    w = K.weights(cfg, 40, torch.bfloat16)
    a = K.engine(cfg, w, DEV, torch.bfloat16, max_seqs=4, max_tokens=400)
    e = K.engine(cfg, w, DEV, torch.bfloat16, max_seqs=4, max_tokens=400, use_cuda_graph=False)
    reqs = {s: K.tokens(cfg, 60, i) for i, s in enumerate("pqrs")}
    at = {}
    for rnd, live in enumerate(("pq", "pqr", "qr", "rs", "s", "pqrs")):
        for s in live:
            if s not in at:
                at[s] = 3 + rnd
                for eng in (a, e):
                    eng.step([s], [reqs[s][:at[s]]])
        for s in [s for s in at if s not in live]:
            at.pop(s)
            for eng in (a, e):
                eng.release(s)
        for _ in range(5):
            nxt = [reqs[s][at[s]] for s in live]
            assert torch.equal(a.decode(list(live), nxt), e.decode(list(live), nxt)), (rnd, live)
            for s in live:
                at[s] += 1
    assert sum(d.graph is not None for d in a._decode.values()) >= 3


def test_trace_runner(tmp_path):
    import json
    import subprocess
    from safetensors.torch import save_file
    cfg = K.CONFIGS["mixed_odd"]
    w = K.weights(cfg, 41, torch.bfloat16)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.contiguous() for k, v in w.items()}, str(tmp_path / "model.safetensors"))
    reqs = {"a": K.tokens(cfg, 14, 1), "b": K.tokens(cfg, 6, 2)}
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": reqs["a"][:10], "want": [0, 9]}, {"id": "b", "tokens": reqs["b"][:5], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": reqs["a"][10:11], "want": []}, {"id": "b", "tokens": reqs["b"][5:], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": reqs["a"][11:12], "want": []}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": reqs["a"][12:13], "want": [0]}], "end": ["a"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path),
                        "--max-tokens", "24"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    want = {k: O.forward(t, cfg, w) for k, t in reqs.items()}
    read = lambda i: torch.frombuffer(bytearray((tmp_path / f"{i}.f32").read_bytes()), dtype=torch.float32).reshape(-1, cfg["vocab"])
    assert K.error(read(0), want["a"][[0, 9]]) < TOL and K.error(read(1), want["b"][5:6]) < TOL and K.error(read(3), want["a"][12:13]) < TOL
    assert not (tmp_path / "2.f32").exists()
