"""Fovudra on a B200: kernels, engine (eager and captured steps) and generation against fovudra_oracle.py; fp32 on the any-size
kernels, bf16 also on the tensor-core kernels (attention heads of 64 / 128 / 256, recurrent keys of 128)."""
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import fovudra_cases as K  # noqa: E402
import fovudra_oracle as O  # noqa: E402

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


def test_far_tokens_show_where_the_mask_lets_them():
    K.check_far_tokens(DEV, TOL)


def test_state_carries():
    K.check_state_carries(DEV, TOL)


def test_long_decode():
    K.check_long_decode(DEV, TOL)


@pytest.mark.parametrize("name", sorted(K.CONFIGS))
def test_bf16_any_size(name):
    cfg = K.CONFIGS[name]
    w = K.weights(cfg, 1, torch.bfloat16)
    for k in w:                                   # close routing calls would compare different experts
        if k.endswith("router"):
            w[k] = w[k] * 8
    toks = K.tokens(cfg, 45, 2)
    want = O.forward(toks, cfg, w)
    eng = K.engine(cfg, w, DEV, torch.bfloat16)
    spread = want.std(-1).mean()
    for k, cuts in enumerate(([45], [30] + [1] * 15, [20, 25])):
        d = (K.run(eng, f"s{k}", toks, cuts).double().cpu() - want).pow(2).mean(-1).sqrt() / spread
        assert float(d.median()) < 0.12, (name, cuts)
        eng.release(f"s{k}")


# ---- tensor-core shapes ----------------------------------------------------------------------------------------------------
TENSOR = K.config([(K.mlstm(heads=2, dim=128, vdim=128, cap=9.0), None),
                   (K.attn(heads=8, kv_heads=2, dim=64, rot_dims=32, size=100, keep_first=17, scale=0.2), K.moe(ff=64, experts=6, top=6, shared=72)),
                   (K.lightning(heads=3, dim=128, vdim=64, decay=(0.8, 0.97, 0.999)), None),
                   (K.attn(heads=6, kv_heads=1, dim=128, rot_dims=128, size=130, keep_first=140, scale=0.1), None),
                   (K.mlstm(heads=1, dim=128, vdim=192, cap=15.0), K.moe(ff=32, experts=1, top=1, shared=16)),
                   (K.attn(heads=2, kv_heads=1, dim=256, rot_dims=64, size=33, keep_first=0, scale=0.06), None)], width=128, vocab=200)


def _bf16_errors_ok(errors, spread):
    """Errors of logit rows relative to the logits' spread: bf16 rounding everywhere, more only where a recurrent head's
    output is a small difference of large terms (its norm then magnifies the rounding); a wrong row is off by about 1."""
    e = torch.cat(errors) / spread
    return float(e.median()) < 0.012 and float(e.quantile(0.95)) < 0.05 and float(e.max()) < 0.5


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


# ---- recurrences -----------------------------------------------------------------------------------------------------------
LENS, SLOTS = [127, 128, 129, 1, 400, 2], [5, 0, 3, 1, 2, 4]


def _qkv(H, N, P, g, lens):
    x = torch.randn(sum(lens), H * (2 * N + P) + 8, generator=g) * 0.5
    first = 0
    for k in lens:
        x[first] *= 12                                         # the first token of every sequence dominates the state
        first += k
    return x.bfloat16()[:, :H * (2 * N + P)]                   # a strided slice, as in the model


def _parts(x, H, N, P):
    return [t.reshape(len(x), H, -1) for t in x.double().split([H * N, H * N, H * P], -1)]


@pytest.mark.parametrize("kind", ["chunked", "tokens"])
@pytest.mark.parametrize("P,H", [(64, 3), (128, 2), (192, 1)])
def test_fixed_decay_scan(P, H, kind):
    """Chunk edges, tails, carried state; slow and fast decays."""
    from jax_gpt_b200.ops import linear_attention as LIN
    N = 128
    g = torch.Generator().manual_seed(P)
    x = _qkv(H, N, P, g, LENS)
    decay = torch.tensor([0.999, 0.4, 0.95])[:H].contiguous()
    for start in (0, 7):
        s0 = torch.randn(6, H, N, P, generator=g)
        state = s0.to(DEV)
        b = begin(SLOTS, LENS, [start] * 6)
        xd = torch.zeros(x.shape[0], x.shape[1] + 8, dtype=torch.bfloat16)
        xd[:, :x.shape[1]] = x
        y = LIN.linear_scan(b, xd.to(DEV)[:, :x.shape[1]], state, decay=decay.to(DEV), q_scale=0.7,
                            kind=LIN.CHUNKED if kind == "chunked" else LIN.TOKENS).y
        c0 = 0
        for k, slot in zip(LENS, SLOTS):
            q, kk, v = _parts(x[c0:c0 + k], H, N, P)
            want, S = O.decay_recurrence(0.7 * q, kk, v, decay.double(), s0[slot].double() if start else None)
            assert rel(y[c0:c0 + k], want.reshape(k, -1)) < 4e-3, (k, start)
            assert rel(state[slot], S) < 2e-5, (k, start)
            c0 += k


@pytest.mark.parametrize("kind", ["chunked", "tokens"])
@pytest.mark.parametrize("P,H", [(64, 3), (128, 2), (192, 1)])
def test_gated_scan(P, H, kind):
    """Open, closed and mixed gates; outputs, state, normaliser and running maximum, carried over portions and slots."""
    from jax_gpt_b200.ops import linear_attention as LIN
    N, cap = 128, 11.0
    g = torch.Generator().manual_seed(P + 1)
    x = _qkv(H, N, P, g, LENS)
    n = x.shape[0]
    raw = 3 * torch.randn(n, 2 * H, generator=g)
    bias = torch.cat([torch.tensor([0.0, -9.0, 5.0])[:H], torch.tensor([4.0, 1.0, 9.0])[:H]])
    z, gamma = torch.randn(n, H * P, generator=g).bfloat16(), torch.rand(H * P, generator=g) + 0.5
    for start in (0, 7):
        s0, v0 = torch.randn(6, H, N, P, generator=g), torch.randn(6, H, N + 1, generator=g)
        state, vec = s0.to(DEV), v0.to(DEV)
        b = begin(SLOTS, LENS, [start] * 6)
        xd = x.to(DEV)
        s = LIN.linear_scan(b, xd, state, gates=LIN.Gates(raw.to(DEV), bias.to(DEV), cap, vec), q_scale=N ** -0.5,
                            kind=LIN.CHUNKED if kind == "chunked" else LIN.TOKENS)
        den = s.den.cpu().double()
        o = s.y.cpu().double().reshape(n, H, P) / (torch.maximum((den[..., 0] + den[..., 1]).abs(), den[..., 2]) + 1e-6)[..., None]
        out = LIN.head_norm_gate(b, s, z.to(DEV), gamma.to(DEV), H, 1e-5, torch.bfloat16)
        c0 = 0
        for k, slot in zip(LENS, SLOTS):
            q, kk, v = _parts(x[c0:c0 + k], H, N, P)
            i = O.soft_cap(raw[c0:c0 + k, :H].double() + bias[:H], cap)
            f = O.log_sigmoid(O.soft_cap(raw[c0:c0 + k, H:].double() + bias[H:], cap))
            carried = (s0[slot].double(), v0[slot, :, :N].double(), v0[slot, :, N].double()) if start else None
            want, (S, nv, m) = O.mlstm_recurrence(q * N ** -0.5, kk, v, i, f, carried)
            for h in range(H):
                assert rel(o[c0:c0 + k, h], want[:, h]) < 6e-3, (k, start, h)
                assert rel(state[slot, h], S[h]) < 3e-5, (k, start, h)
                assert rel(vec[slot, h, :N], nv[h]) < 3e-5 and abs(float(vec[slot, h, N]) - float(m[h])) < 1e-4, (k, start, h)
            full = O.unit_rms(want, 1e-5).reshape(k, -1) * gamma.double() * O.sigmoid(z[c0:c0 + k].double())
            assert rel(out[c0:c0 + k], full) < 8e-3, (k, start)
            c0 += k


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("H,N,P", [(3, 16, 24), (2, 128, 128), (1, 5, 67), (2, 300, 40), (4, 1, 1)])
def test_one_token_step_and_scan_of_any_size(H, N, P, dtype):
    """Token-by-token scan of a portion, then one-token steps from its state, both gate kinds, SiLU applied on the way in."""
    from jax_gpt_b200.ops import linear_attention as LIN
    g = torch.Generator().manual_seed(N)
    n, steps = 19, 4
    x = torch.randn(2, n + steps, H * (2 * N + P), generator=g).to(dtype)
    raw, bias = 2 * torch.randn(2, n + steps, 2 * H, generator=g), torch.cat([torch.randn(H, generator=g), 2 + torch.randn(H, generator=g)])
    decay = torch.rand(H, generator=g) * 0.9 + 0.1
    tol = 2e-2 if dtype == torch.bfloat16 else 2e-5
    for gated in (False, True):
        state, vec = torch.full((3, H, N, P), 1e4, device=DEV), torch.full((3, H, N + 1), 1e4, device=DEV)
        got = []
        for at, k in [(0, n)] + [(n + t, 1) for t in range(steps)]:
            b = begin([2, 0], [k, k], [at, at])
            xd, rd = x[:, at:at + k].reshape(2 * k, -1).to(DEV), raw[:, at:at + k].reshape(2 * k, -1).contiguous().to(DEV)
            s = LIN.linear_scan(b, xd, state, decay=None if gated else decay.to(DEV), gates=LIN.Gates(rd, bias.to(DEV), 5.0, vec) if gated else None,
                                q_scale=0.5, silu=not gated)
            big = torch.full((2 * k, H * P), 60.0, dtype=dtype, device=DEV)
            o = LIN.head_norm_gate(b, s, big, torch.ones(H * P, device=DEV), H if gated else 1, 1e-3, dtype)
            got.append(o.reshape(2, k, H * P))
        got = torch.cat(got, 1)
        for r in range(2):
            q, k, v = _parts(x[r], H, N, P) if gated else [O.silu(t) for t in _parts(x[r], H, N, P)]
            if gated:
                i = O.soft_cap(raw[r, :, :H].double() + bias[:H], 5.0)
                f = O.log_sigmoid(O.soft_cap(raw[r, :, H:].double() + bias[H:], 5.0))
                want = O.unit_rms(O.mlstm_recurrence(q * 0.5, k, v, i, f)[0], 1e-3).reshape(n + steps, -1)
            else:
                want = O.unit_rms(O.decay_recurrence(q * 0.5, k, v, decay.double())[0].reshape(n + steps, -1), 1e-3)
            assert rel(got[r], want) < tol, (gated, r)


# ---- attention -------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("D", [64, 128, 256])
def test_flash_and_paged_kernels_take_a_window(D):
    """One key stands out for every query: on both sides of the window's and the kept tokens' edges and of tile borders."""
    from jax_gpt_b200.cache.paged import PagedCache
    from jax_gpt_b200.ops import attention as A
    g = torch.Generator().manual_seed(D)
    B, T, H, G = 1, 300, 4, 2
    k = torch.randn(T, G, D, generator=g)
    k = (k / k.norm(dim=-1, keepdim=True)).bfloat16()
    v = torch.randn(T, G, D, generator=g).bfloat16()
    cache = PagedCache(1, 2 * G * D, 8, 64, 2, 6, torch.bfloat16, DEV)
    cache.append(0, [1], torch.cat([k.reshape(1, T, -1), v.reshape(1, T, -1)], -1).to(DEV), commit=True)
    for size, keep in ((100, 20), (128, 128), (129, 1), (1, 0), (7, 130), (64, 300), (1000, 5)):
        mask = O.window_mask(T, size, keep)
        for shift in (size - 1, size, size + 1, 0):             # every query i asks for key i - shift, ...
            target = (torch.arange(T) - shift).clamp(0, T - 1)
            for fixed in (None, keep - 1, keep):                # ... or all of them for one of the first keys
                if fixed is not None and not 0 <= fixed < T or (fixed is not None and shift):
                    continue
                t = target if fixed is None else torch.full((T,), fixed)
                q = (30.0 * k[t].float()).repeat_interleave(H // G, 1).bfloat16()
                want = O.masked_softmax_attention(q.double(), k.double(), v.double(), mask, 0.5)
                o, _ = A.attn_fwd(q[None].to(DEV), k[None].to(DEV), v[None].to(DEV), True, 0.5, window=size, keep_first=keep)
                assert rel(o[0], want) < 1.2e-2, (size, keep, shift, fixed)
                for i in (T - 1, 150, 127, 128, 0):
                    lens = torch.full((2,), i + 1, dtype=torch.int32, device=DEV)
                    for splits in (1, 5):
                        sc = (torch.empty(1, H, splits, D, device=DEV), torch.empty(1, H, splits, 2, device=DEV))
                        o1 = A.attention_decode_paged(q[i:i + 1].to(DEV), cache.pool[0], cache.block_table, torch.tensor([1], dtype=torch.int32, device=DEV),
                                                      lens, G, 0, 0.5, scratch=sc, window=size, keep_first=keep)
                        assert rel(o1[0], want[i]) < 1.2e-2, (size, keep, shift, fixed, i, splits)


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("H,G,D,dims", [(8, 2, 128, 128), (3, 3, 64, 32), (4, 1, 96, 64), (2, 1, 20, 12), (2, 2, 256, 16), (1, 1, 512, 512), (5, 1, 7, 2)])
def test_attention_operands(H, G, D, dims, dtype):
    from jax_gpt_b200.cache.paged import PagedCache
    from jax_gpt_b200.ops import window_attention as WA
    from jax_gpt_b200.ops.rope import rope_tables
    g = torch.Generator().manual_seed(D)
    rot = K.rot(dims)
    cache = PagedCache(2, [3, 2 * G * D], 20, 8, 3, 8, dtype, DEV)
    ids, lens, starts = [2, 0], [13, 1], [5, 9]
    cache.begin_step(ids, [s + n for s, n in zip(starts, lens)])
    b = begin(ids, lens, starts, 64)
    y = torch.randn(14, (H + G) * D + 8, generator=g).to(dtype)
    bias = torch.randn((H + G) * D, generator=g)
    tables = rope_tables(dims, rot["base"], 64, rot["scaling"], DEV)
    q, k, v = WA.qk_prepare(b, y.to(DEV)[:, :(H + G) * D], bias.to(DEV), H, G, D, True, 1e-3, tables, cache, 1, dense=True)
    x = (y[:, :(H + G) * D].double() + bias.double()).reshape(14, H + G, D)
    pos = list(range(5, 18)) + [9]
    r = O.unit_rms(O.rotate_half(x, pos, rot), 1e-3)
    tol = 5e-3 if dtype == torch.bfloat16 else 2e-6
    assert rel(q, r[:, :H]) < tol and rel(k, r[:, H:]) < tol and rel(v, x[:, H:]) < tol
    for slot, c0, n, s in ((2, 0, 13, 5), (0, 13, 1, 9)):
        pages, offs = cache.slots(slot, s, n)
        rows = cache.pool[1][pages, offs]
        assert torch.equal(rows[:, :G * D], k[c0:c0 + n].reshape(n, -1)) and torch.equal(rows[:, G * D:], v[c0:c0 + n].reshape(n, -1))


# ---- norms, linear layers, experts ----------------------------------------------------------------------------------------
@pytest.mark.parametrize("y_dtype,dtype", [(torch.bfloat16, torch.bfloat16), (torch.float32, torch.bfloat16), (torch.float32, torch.float32)])
@pytest.mark.parametrize("rows,D", [(3, 30), (70, 256), (2, 1000), (5, 2048), (3, 4096), (1, 8192), (2, 9000)])
def test_residual_norm(rows, D, y_dtype, dtype):
    from jax_gpt_b200.ops.packed import residual_norm_rows
    g = torch.Generator().manual_seed(D)
    y, x = torch.randn(rows, D, generator=g).to(y_dtype), 5 * torch.randn(rows, D, generator=g)
    a, c = torch.rand(D, generator=g), torch.rand(D, generator=g)
    for add in (True, False):
        xd = x.to(DEV)
        h = residual_norm_rows(y.to(DEV), 1 + a.to(DEV), xd, 1 + c.to(DEV), 1e-3, dtype, add)
        want = O.rms_norm_zero_centred(y.double(), a.double(), 1e-3) + (x.double() if add else 0)
        assert rel(xd, want) < 1e-6
        assert rel(h, O.rms_norm_zero_centred(want, c.double(), 1e-3)) < (4e-3 if dtype == torch.bfloat16 else 1e-6)


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_linear_with_silu_glu_and_fp32_tail(dtype):
    from jax_gpt_b200.ops.gemm import linear_rows, linear_rows_f32_tail, silu_glu_rows
    g = torch.Generator().manual_seed(6)
    tol = 6e-3 if dtype == torch.bfloat16 else 5e-6
    for M in (1, 2, 7, 9, 20, 32, 130):
        for Kd, N in ((256, 120), (100, 78), (1024, 2400), (6, 6)):
            x, w = torch.randn(M, Kd, generator=g).to(dtype), (torch.randn(N, Kd, generator=g) * Kd ** -0.5).to(dtype)
            full = x.double() @ w.double().T
            xd, wd = x.to(DEV), w.to(DEV)
            assert rel(linear_rows(xd, wd, act="silu"), O.silu(full)) < tol, (M, Kd, N)
            up = full[:, N // 2:]
            assert rel(silu_glu_rows(xd, wd), O.silu(full[:, :N // 2]) * up) < 2 * tol, (M, Kd, N)
            y, tail = linear_rows_f32_tail(xd, wd, 4)
            assert tail.dtype == torch.float32 and y.dtype == dtype
            assert rel(y, full[:, :-4]) < tol and rel(tail, full[:, -4:]) < 5e-6, (M, Kd, N)


@pytest.mark.parametrize("M", [1, 5, 200])
@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("D,I,E,top,S", [(64, 48, 6, 3, 32), (30, 7, 3, 1, 9), (40, 8, 1, 1, 16), (64, 16, 70, 8, 24)])
def test_sigmoid_experts(M, dtype, D, I, E, top, S):
    from jax_gpt_b200.ops.sigmoid_moe import sigmoid_moe, sigmoid_topk
    g = torch.Generator().manual_seed(7)
    h = torch.randn(M, D, generator=g).to(dtype)
    mat = lambda *s: torch.randn(*s, generator=g) * s[-1] ** -0.5
    router = (4 * mat(E, D)).to(dtype)
    gate, up, down = (2 * mat(E, I, D)).to(dtype), (2 * mat(E, I, D)).to(dtype), mat(E, D, I).to(dtype)
    sg, su, sd = (2 * mat(S, D)).to(dtype), (2 * mat(S, D)).to(dtype), mat(D, S).to(dtype)
    w = {"router": router, "shared.gate": sg, "shared.up": su, "shared.down": sd}
    for e in range(E):
        w.update({f"e{e}.gate": gate[e], f"e{e}.up": up[e], f"e{e}.down": down[e]})
    want = O.moe(h.double(), {"router": {"top": top}}, {k: t.double() for k, t in w.items()}, "")
    dv = lambda t: t.contiguous().to(DEV)
    out = sigmoid_moe(dv(h), dv(router), top, dv(torch.cat([gate, up], 1)), dv(down), dv(torch.cat([sg, su])), dv(sd))
    assert rel(out, want) < (1e-2 if dtype == torch.bfloat16 else 1e-5)
    z = h.float() @ router.float().T
    ids, s = sigmoid_topk(z.to(DEV), top)
    order, score = O.choose_experts(z.double(), top)
    assert torch.equal(ids.cpu().long(), order) and rel(s, score) < 1e-6


# ---- engine ----------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", ["mixed_odd", "aligned"])
def test_captured_steps_equal_eager_steps(name):
    """Graph replays over changing batches, slots and block tables against the eager engine, bit by bit."""
    cfg = K.CONFIGS[name]
    w = K.weights(cfg, 40, torch.bfloat16)
    a = K.engine(cfg, w, DEV, torch.bfloat16, max_seqs=4)
    e = K.engine(cfg, w, DEV, torch.bfloat16, max_seqs=4, use_cuda_graph=False)
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
