"""Vobunex on a B200: kernels, engine (eager and captured steps) and generation against vobunex_oracle.py; fp32 on the
any-size kernels, bf16 also on the tensor-core kernels (heads of 128 + 64, latent 512, state 128)."""
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import vobunex_cases as K  # noqa: E402
import vobunex_oracle as O  # noqa: E402

pytestmark = pytest.mark.gpu
TOL = 5e-4
DEV = "cuda"


@pytest.fixture(autouse=True)
def _needs_gpu(cuda_device):
    yield


def rel(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return float((a - b).norm() / b.norm().clamp_min(1e-12))


# ---- the whole model in fp32 ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", sorted(K.CONFIGS))
def test_prompts_and_cuts(name):
    K.check_prompts_and_cuts(name, DEV, TOL)


@pytest.mark.parametrize("name", sorted(K.CONFIGS))
def test_layers(name):
    K.check_layers(name, DEV, TOL)


@pytest.mark.parametrize("name", ["mixed_odd", "aligned", "mamba_only"])
def test_batches_slots_and_pages_reused(name):
    K.check_batch_and_reuse(name, DEV, TOL)


def test_mixed_step():
    K.check_mixed_step(DEV, TOL)


def test_greedy_and_sampled_generation():
    K.check_generate(DEV, TOL)


def test_one_key_stands_out():
    K.check_one_key_stands_out(DEV, 1e-4)


def test_far_token_and_sink_show_in_the_logits():
    K.check_far_token(DEV, TOL)


def test_long_decode():
    K.check_long_decode(DEV, TOL)


@pytest.mark.parametrize("name", sorted(K.CONFIGS))
def test_bf16_any_size(name):
    cfg = K.CONFIGS[name]
    w = K.weights(cfg, 1, torch.bfloat16)
    toks = K.tokens(cfg, 45, 2)
    want = O.forward(toks, cfg, w)
    eng = K.engine(cfg, w, DEV, torch.bfloat16)
    spread = want.std(-1).mean()
    for k, cuts in enumerate(([45], [30] + [1] * 15, [20, 25])):
        d = K.run(eng, f"s{k}", toks, cuts).double().cpu() - want
        assert float(d.pow(2).mean().sqrt() / spread) < 0.1, (name, cuts)
        eng.release(f"s{k}")


# ---- tensor-core shapes ----------------------------------------------------------------------------------------------------
TENSOR = K.config([(K.mamba(heads=4, vdim=64, state=128, groups=2, conv=4, norm_groups=2), K.moe(ff=64, experts=6, top=2, limit=1.2)),
                   (K.attn(heads=3, dim=128, rot_dim=64, vdim=128, q_rank=96, kv_rank=512, scale=0.09), K.dense(160)),
                   (K.mamba(heads=2, vdim=128, state=128, groups=1, conv=4, norm_groups=1), None),
                   (K.attn(heads=20, dim=128, rot_dim=64, vdim=128, q_rank=96, kv_rank=512, scale=0.09), K.moe(ff=32, experts=3, top=3))],
                  width=128, vocab=200, bigram=(101, 17, 3))


def test_tensor_core_shapes_whole_and_decoded():
    w = K.weights(TENSOR, 31, torch.bfloat16)
    sizes = (300, 1, 129, 64)
    reqs = [K.tokens(TENSOR, n + 12, n) for n in sizes]
    want = [O.forward(t, TENSOR, w) for t in reqs]
    eng = K.engine(TENSOR, w, DEV, torch.bfloat16, page_size=64, max_tokens=1024)
    spread = float(want[0].std(-1).mean())
    err = lambda a, b: float((a.double().cpu() - b).pow(2).mean(-1).sqrt().max()) / spread
    for i, (t, n) in enumerate(zip(reqs, sizes)):              # alone, equal lengths (one flash launch for the batch)
        lg = eng.step(["x", "y"], [t[:n], t[:n]], [list(range(n))] * 2)
        assert err(lg, torch.cat([want[i][:n]] * 2)) < 0.12, n
        for s in range(12):
            lg = eng.decode(["x", "y"], [t[n + s]] * 2)
            assert err(lg, torch.stack([want[i][n + s]] * 2)) < 0.12, (n, s)
        eng.release("x")
        eng.release("y")
    ids = list("abcd")
    lg = eng.step(ids, [t[:n] for t, n in zip(reqs, sizes)])
    assert err(lg, torch.stack([x[n - 1] for x, n in zip(want, sizes)])) < 0.12
    for s in range(12):
        if s == 6:
            eng.release(ids.pop(1))
            reqs.pop(1), want.pop(1)
            sizes = (300, 129, 64)
        lg = eng.decode(ids, [t[n + s] for t, n in zip(reqs, sizes)])
        assert err(lg, torch.stack([x[n + s] for x, n in zip(want, sizes)])) < 0.12, s


def test_tensor_core_shapes_continued_prompt():
    w = K.weights(TENSOR, 32, torch.bfloat16)
    toks = K.tokens(TENSOR, 270, 33)
    want = O.forward(toks, TENSOR, w)
    eng = K.engine(TENSOR, w, DEV, torch.bfloat16, page_size=64, max_tokens=512)
    got = K.run(eng, "a", toks, [130, 2, 128, 10]).double().cpu()
    assert float((got - want).pow(2).mean(-1).sqrt().max() / want.std(-1).mean()) < 0.12


@pytest.mark.parametrize("P,H,G", [(64, 6, 3), (128, 2, 1), (192, 2, 2)])
def test_chunked_scan(P, H, G):
    """Chunk edges, tails, carried state; decays slow enough that an early token stays in the state across chunks."""
    from jax_gpt_b200.ops import ssm
    from jax_gpt_b200.ops.packed import PackedBatch, seq_begin
    N = 128
    g = torch.Generator().manual_seed(P)
    lens = [127, 128, 129, 1, 700, 2]
    b = PackedBatch.make([5, 0, 3, 1, 2, 4], lens, True, 800, DEV)
    n, C = sum(lens), H * P + 2 * G * N
    xbc = torch.randn(n, C, generator=g).bfloat16()
    first = 0
    for k in lens:
        xbc[first] *= 30                                      # the first token of every sequence dominates the state
        first += k
    zxd = torch.randn(n, C + H, generator=g).bfloat16()
    db, al, D = torch.rand(H, generator=g) * 3 - 4, torch.log(torch.rand(H, generator=g) * 0.2 + 0.001), torch.randn(H, generator=g)
    for start in (0, 7):
        s0 = torch.randn(6, H, N, P, generator=g)
        state = s0.to(DEV)
        lensd = torch.full((6,), start, dtype=torch.int32, device=DEV)
        seq_begin(b, torch.zeros(n, dtype=torch.int32, device=DEV), lensd, torch.zeros(6, dtype=torch.int32, device=DEV))
        y = ssm.ssd_scan(b, xbc.to(DEV), zxd.to(DEV)[:, C:], db.to(DEV), al.to(DEV), D.to(DEV), state, G, chunked=True)
        c0 = 0
        for k, slot in zip(lens, [5, 0, 3, 1, 2, 4]):
            x, B, Cc = xbc[c0:c0 + k].double().split([H * P, G * N, G * N], -1)
            dt = torch.nn.functional.softplus(zxd[c0:c0 + k, C:].double() + db.double())
            want, S = O.ssd_recurrence(x.reshape(k, H, P), B.reshape(k, G, N), Cc.reshape(k, G, N), dt, al.double(), D.double(),
                                       s0[slot].double() if start else None)
            assert rel(y[c0:c0 + k], want.reshape(k, -1)) < 4e-3, (k, start)       # bf16 output
            assert rel(state[slot], S) < 2e-5, (k, start)
            c0 += k


def test_flash_and_paged_kernels_take_a_sink():
    from jax_gpt_b200.cache.paged import PagedCache
    from jax_gpt_b200.ops import attention as A
    from jax_gpt_b200.ops.mla_decode import mla_paged_decode
    g = torch.Generator().manual_seed(5)
    B, T, H = 2, 200, 3
    sink = torch.tensor([-3.0, 1.0, 8.0])
    for d, dv in ((192, 128), (64, 64), (128, 128)):
        q, k, v = (torch.randn(B, T, H, n, generator=g).bfloat16() for n in (d, d, dv))
        o, _ = A.attn_fwd(q.to(DEV), k.to(DEV), v.to(DEV), True, 0.1, sink=sink.to(DEV))
        s = torch.einsum("bthd,bshd->bhts", q.double(), k.double()) * 0.1
        s = s.masked_fill(~torch.ones(T, T, dtype=torch.bool).tril(), -float("inf"))
        want = torch.einsum("bhts,bshd->bthd", O.sink_softmax(s, sink.double()[None, :, None, None].expand(B, H, T, 1)), v.double())
        assert rel(o, want) < 6e-3, (d, dv)
    cache = PagedCache(1, 576, 12, 64, 2, 6, torch.bfloat16, DEV)
    lens = (150, 65)
    rows = [torch.randn(n, 576, generator=g).bfloat16() for n in lens]
    for i, r in enumerate(rows):
        cache.append(0, [i], r[None].to(DEV), commit=True)
    for H in (16, 40):
        q = torch.randn(2, H, 576, generator=g).bfloat16()
        sink = torch.randn(H, generator=g) * 4
        o = mla_paged_decode(q.to(DEV), cache, 0, [0, 1], 0.08, sink=sink.to(DEV))
        for i, r in enumerate(rows):
            s = (q[i].double() @ r.double().T) * 0.08
            assert rel(o[i], O.sink_softmax(s, sink.double()[:, None]) @ r[:, :512].double()) < 8e-3, (H, i)


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_few_row_and_wide_linear(dtype):
    from jax_gpt_b200.ops.gemm import linear_rows
    g = torch.Generator().manual_seed(6)
    tol = 5e-3 if dtype == torch.bfloat16 else 5e-6
    for M in (1, 2, 3, 7, 8, 9, 130):
        for Kd, N in ((256, 120), (100, 77), (2048, 9600), (6, 5)):
            x, w = torch.randn(M, Kd, generator=g).to(dtype), (torch.randn(N, Kd, generator=g) * Kd ** -0.5).to(dtype)
            want = x.double() @ w.double().T
            xd, wd = x.to(DEV), w.to(DEV)
            res = torch.randn(M, N, generator=g)
            acc = linear_rows(xd, wd, out=res.to(DEV), accumulate=True)
            assert rel(acc, want + res.double()) < tol, (M, Kd, N)
            assert rel(linear_rows(xd, wd, act="relu2"), want.clamp_min(0) ** 2) < tol, (M, Kd, N)
            out = linear_rows(xd, wd, f32_out=True)
            assert out.dtype == torch.float32 and rel(out, want) < tol, (M, Kd, N)


@pytest.mark.parametrize("M", [1, 5, 200])
@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("D,I,E,top", [(64, 48, 6, 3), (30, 7, 3, 1), (40, 8, 1, 1)])
def test_table_experts(M, dtype, D, I, E, top):
    from jax_gpt_b200.ops.table_moe import table_moe
    g = torch.Generator().manual_seed(7)
    V = 50
    h = torch.randn(M, D, generator=g).to(dtype)
    tok = torch.randint(0, V, (M,), generator=g)
    table = torch.rand(V, E, generator=g).argsort(-1)[:, :top].int().contiguous()
    gate, up = ((torch.randn(E, I, D, generator=g) * 2 * D ** -0.5).to(dtype) for _ in range(2))
    down = (torch.randn(E, D, I, generator=g) * I ** -0.5).to(dtype)
    w = {"table": table}
    for e in range(E):
        w.update({f"e{e}.gate": gate[e].double(), f"e{e}.up": up[e].double(), f"e{e}.down": down[e].double()})
    want = O.table_moe(h.double(), tok.tolist(), {"router": {"top": top}, "expert": {"limit": 0.9}}, w, "")
    res = torch.randn(M, D, generator=g)
    out = table_moe(h.to(DEV), tok.int().to(DEV), table.to(DEV), torch.cat([gate, up], 1).contiguous().to(DEV), down.to(DEV), 0.9,
                    1.702, res.to(DEV))
    assert rel(out.cpu() - res, want) < (8e-3 if dtype == torch.bfloat16 else 1e-5)


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("rows,D,parts", [(5, 96, 4), (3, 4096, 2), (2, 10240, 1), (4, 33, 3), (70, 512, 8)])
def test_gated_group_norm(dtype, rows, D, parts):
    from jax_gpt_b200.ops.ssm import gated_group_norm
    g = torch.Generator().manual_seed(8)
    zy = torch.randn(rows, 2 * D, generator=g).to(dtype)
    z, y = zy[:, :D], zy[:, D:].contiguous()
    y[:, :D // parts] *= 50                                   # pieces of very different size keep their own mean square
    gamma = torch.randn(D, generator=g)
    gated = y.double() * O.silu(z.double())
    want = O.grouped_rms_norm(gated, gamma.double(), parts, 1e-5)
    tol = 5e-3 if dtype == torch.bfloat16 else 1e-5
    zd = zy.to(DEV)[:, :D]
    assert rel(gated_group_norm(y.to(DEV), zd, gamma.to(DEV), parts, 1e-5, dtype), want) < tol
    assert rel(gated_group_norm(gated.float().to(DEV), None, gamma.to(DEV), parts, 1e-5, dtype), want) < tol


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("C,taps", [(64, 4), (64, 3), (21, 4), (40, 1), (16, 6)])
def test_convolution_carries_its_inputs(dtype, C, taps):
    from jax_gpt_b200.ops.packed import PackedBatch, seq_begin
    from jax_gpt_b200.ops.ssm import ssm_conv
    g = torch.Generator().manual_seed(9)
    lens, slots = [37, 1, 18], [2, 0, 1]
    xs = [torch.randn(n, C, generator=g).to(dtype) for n in lens]
    w, bias = torch.randn(C, taps, generator=g), torch.randn(C, generator=g)
    ring = torch.full((3, taps, C), 1e4, device=DEV)
    lensd, prev = torch.zeros(3, dtype=torch.int32, device=DEV), torch.zeros(3, dtype=torch.int32, device=DEV)
    got = [[] for _ in lens]
    at = [0, 0, 0]
    for cut in ((5, 1, 2), (2, 0, 14), (17, 0, 1), (13, 0, 1)):
        live = [i for i in range(3) if cut[i]]
        b = PackedBatch.make([slots[i] for i in live], [cut[i] for i in live], False, 64, DEV)
        pad = torch.cat([xs[i][at[i]:at[i] + cut[i]] for i in live])
        x = torch.cat([torch.zeros(pad.shape[0], 8).to(dtype), pad], 1).to(DEV)[:, 8:]
        seq_begin(b, torch.zeros(b.n_tok, dtype=torch.int32, device=DEV), lensd, prev)
        y = ssm_conv(b, x, w.to(DEV), bias.to(DEV), ring)
        c0 = 0
        for i in live:
            got[i].append(y[c0:c0 + cut[i]])
            at[i] += cut[i]
            c0 += cut[i]
    for i in range(3):
        want = O.causal_conv_silu(xs[i].double(), w.double(), bias.double())
        assert rel(torch.cat(got[i]), want) < (5e-3 if dtype == torch.bfloat16 else 1e-5), i


def test_captured_steps_equal_eager_steps():
    """Graph replays over changing batches, slots and block tables against the eager engine, bit by bit."""
    cfg = K.CONFIGS["aligned"]
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
