"""Munazen on CPU: every operation's restatement, the engine's batching, cache and bookkeeping, and greedy generation, against the
plain implementation of munazen_oracle.py."""
import json
import math
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import munazen_cases as K  # noqa: E402
import munazen_oracle as O  # noqa: E402

from jax_gpt_b200.models import registry  # noqa: E402
from jax_gpt_b200.models.munazen import MunazenConfig, MunazenEngine, forward, init_params, random_state_dict  # noqa: E402
from jax_gpt_b200.models.munazen.weight_loader import expected_shapes, load_from_state_dict  # noqa: E402
from jax_gpt_b200.ops import linear_attention as LIN  # noqa: E402
from jax_gpt_b200.ops.gated_lru import LruWeights, gated_lru, lru_decay  # noqa: E402
from jax_gpt_b200.ops.packed import PackedBatch, seq_begin  # noqa: E402
from jax_gpt_b200.ops.rope import rope_tables, rotate_interleaved, yarn_frequencies  # noqa: E402
from jax_gpt_b200.ops.streams import Connection, group_norm_rows, poly_norm, stream_norm  # noqa: E402

TOL = 3e-4


@pytest.mark.parametrize("name", sorted(K.CONFIGS))
def test_prompts_and_cuts(name):
    K.check_prompts_and_cuts(name, "cpu", TOL)


@pytest.mark.parametrize("name", sorted(K.CONFIGS))
def test_layers(name):
    K.check_layers(name, "cpu", TOL)


@pytest.mark.parametrize("name", ["mixed_odd", "gla_only"])
def test_batches_slots_and_pages_reused(name):
    K.check_batch_and_reuse(name, "cpu", TOL)


def test_mixed_step():
    K.check_mixed_step("cpu", TOL)


def test_greedy_and_sampled_generation():
    K.check_generate("cpu", TOL)


def test_one_key_stands_out():
    K.check_one_key_stands_out("cpu", 1e-4)


def test_far_tokens():
    K.check_far_tokens("cpu", TOL)


def test_state_carries():
    K.check_state_carries("cpu", TOL)


def test_long_decode():
    K.check_long_decode("cpu", TOL)


def test_loop_passes_keep_their_own_state():
    K.check_loop_passes_keep_their_own_state("cpu", TOL)


# ---- mechanisms alone --------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("rot", [K.rot(8), K.rot(8, scaling=False), K.rot(16, base=1e6), K.rot(2), K.rot(12, base=40.0),
                                 {"base": 1e4, "dims": 6, "scaling": {"factor": 4.0, "fast": 2.0, "slow": 2.0, "original": 50}}])
def test_rotation(rot):
    f, amp = yarn_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    of, oamp = O.rotary_frequencies(rot)
    assert f == pytest.approx(of) and amp == pytest.approx(oamp)
    x = torch.randn(9, 2, rot["dims"] + 3, dtype=torch.float64)
    pos = torch.tensor([0, 1, 2, 63, 64, 500, 7, 8, 999])
    got = rotate_interleaved(x, pos, rope_tables(rot["dims"], rot["base"], 1000, rot.get("scaling")))
    assert torch.allclose(got, O.turn_pairs(x, pos.tolist(), of, oamp), atol=1e-5)


def test_rotated_values_depend_on_distance_only():
    """Turning values by their positions and the sum back by the query's equals turning each value by the distance."""
    T, dv = 9, 6
    q, k, v = torch.randn(T, 2, 4, dtype=torch.float64), torch.randn(T, 1, 4, dtype=torch.float64), torch.randn(T, 1, dv, dtype=torch.float64)
    f = O.value_frequencies(50.0, dv)
    mask = O.causal_mask(T)
    o = O.turn_pairs(O.masked_softmax_attention(q, k, O.turn_pairs(v, range(T), f), mask, 0.7), [-p for p in range(T)], f)
    i = 6
    rel = O.turn_pairs(v, [j - i for j in range(T)], f)
    assert torch.allclose(o[i], O.masked_softmax_attention(q[i:i + 1], k, rel, mask[i:i + 1], 0.7)[0])


def test_group_norm_and_streams():
    g = torch.Generator().manual_seed(1)
    N, S, D, G, eps = 4, 3, 12, 3, 1e-3
    xs, y, b = torch.randn(N, S, D, generator=g), torch.randn(N, D, generator=g), torch.randn(D, generator=g)
    mix, wo, wi, gamma = (torch.randn(*s, generator=g) for s in ((S, S), (S,), (S,), (D,)))
    new = O.streams_out(xs.double(), (y + b).double(), mix.double(), wo.double())
    u = O.streams_in(new, wi.double())
    got = xs.clone()
    h, uu = stream_norm(y, got, Connection(None, mix, wo), wi, gamma, G, eps, torch.float32, bias=b, want_u=True)
    assert torch.allclose(got.double(), new, atol=1e-5) and torch.allclose(uu.double(), u, atol=1e-5)
    assert torch.allclose(h.double(), O.group_norm(u, gamma.double(), G, eps), atol=1e-5)
    # the streams start: every stream holds the row, whatever was there before
    got.fill_(float("nan"))
    one = torch.ones(S)
    h, _ = stream_norm(y, got, Connection(one, None, one), wi, gamma, G, eps, torch.float32)
    assert torch.equal(got, y[:, None].expand(N, S, D)) and torch.allclose(h, O.group_norm(wi.sum() * y, gamma, G, eps), atol=1e-5)
    assert torch.allclose(group_norm_rows(y, gamma, G, eps, torch.float32), O.group_norm(y, gamma, G, eps), atol=1e-6)


def test_mix_is_indexed_from_to():
    xs = torch.tensor([[[1.0], [10.0]]])
    mix = torch.tensor([[0.0, 1.0], [0.0, 0.0]])               # stream 0 goes to stream 1
    assert O.streams_out(xs, torch.zeros(1, 1), mix, torch.zeros(2)).flatten().tolist() == [0.0, 1.0]


def test_poly_norm():
    z, coef = torch.randn(5, 9), torch.tensor([0.7, -0.4, 1.1, 0.2])
    assert torch.allclose(poly_norm(z, coef, 1e-4), O.poly_norm(z, coef, 1e-4), atol=1e-6)
    v = torch.tensor([[2.0, 0.0]])                             # N(z) = (sqrt 2, 0) without eps, N(z^2) and N(z^3) likewise
    r = math.sqrt(2)
    assert torch.allclose(O.poly_norm(v, [1.0, 10.0, 100.0, 5.0], 0.0), torch.tensor([[111 * r + 5, 5.0]]))


def test_log_sigmoid_and_softplus_far_out():
    x = torch.tensor([-300.0, -20.0, 0.0, 20.0, 300.0], dtype=torch.float64)
    assert torch.allclose(O.log_sigmoid(x), torch.nn.functional.logsigmoid(x)) and torch.allclose(O.softplus(x), torch.nn.functional.softplus(x, threshold=1e9))
    assert torch.allclose(O.sigmoid(x), torch.sigmoid(x))


def _portions(n, cuts, slots=3, slot=2):
    """Packed batches of one sequence, portion by portion."""
    lens, prev = torch.zeros(slots, dtype=torch.int32), torch.zeros(slots, dtype=torch.int32)
    at = 0
    for c in cuts:
        b = PackedBatch.make([slot], [c], at == 0, n, "cpu")
        seq_begin(b, torch.zeros(c, dtype=torch.int32), lens, prev)
        yield b, at, at + c
        at += c


def test_gated_lru_restatement():
    g = torch.Generator().manual_seed(3)
    n, W, nb, taps = 14, 12, 3, 4
    r = lambda *s: torch.randn(*s, generator=g)
    x, y, xb, yb, conv, cb = r(n, W), r(n, W), r(W), r(W), r(W, taps), r(W)
    ra, ri, rab, rib, lam = r(nb, 4, 4), r(nb, 4, 4), r(nb, 4), r(nb, 4), r(W)
    w = LruWeights(xb, yb, conv, cb, torch.stack([ra, ri], 1), torch.stack([rab, rib], 1), lru_decay(lam))
    D = lambda t: t.double()
    u = O.causal_conv(D(x + xb), D(conv), D(cb))
    S, last = O.rglru_recurrence(u, O.sigmoid(O.block_linear(u, D(ra), D(rab))), O.sigmoid(O.block_linear(u, D(ri), D(rib))), D(lam))
    want = 0.6 * S * O.gelu_tanh(D(y + yb))
    for cuts in ([14], [1] * 14, [2, 5, 1, 6]):
        ring, state, out = torch.full((3, taps, W), 1e3), torch.full((3, W), 1e3), torch.empty(n, W)
        for b, c0, c1 in _portions(n, cuts):
            gated_lru(b, x[c0:c1], y[c0:c1], w, ring, state, 0.6, out[c0:c1])
        assert torch.allclose(out.double(), want, atol=1e-5) and torch.allclose(state[2].double(), last, atol=1e-5)


def test_lru_first_token_and_bias_before_the_start():
    """The first token is like any other (factor sqrt(1 - a^2)), and what lies before the start is zero, not the bias."""
    x, conv = torch.zeros(1, 1, dtype=torch.float64), torch.tensor([[5.0, 2.0]], dtype=torch.float64)
    u = O.causal_conv(x + 3.0, conv, torch.zeros(1, dtype=torch.float64))
    assert float(u) == pytest.approx(6.0)
    half = torch.full((1, 1), 0.5, dtype=torch.float64)
    S, _ = O.rglru_recurrence(u, half, half, torch.zeros(1, dtype=torch.float64))
    a = math.exp(-4 * math.log(2))
    assert float(S) == pytest.approx(math.sqrt(1 - a * a) * 0.5 * 6.0)


@pytest.mark.parametrize("tau", [1.0, 16.0, 0.25])
def test_channel_decay_restatement(tau):
    g = torch.Generator().manual_seed(4)
    H, N, P, n, R = 2, 5, 4, 13, 3
    qkv, low = torch.randn(n, H * (2 * N + P), generator=g), torch.randn(n, R, generator=g)
    w2, b2 = torch.randn(H * N, R, generator=g), 1 + torch.randn(H * N, generator=g)
    state = torch.full((3, H, N, P), 1e3)
    q, k, v = [t.reshape(n, H, -1).double() for t in qkv.split([H * N, H * N, H * P], -1)]
    la = O.log_sigmoid(low.double() @ w2.double().T + b2.double()).reshape(n, H, N) / tau
    want, last = O.channel_decay_recurrence(q * 0.3, k, v, la)
    ys = [LIN.linear_scan(b, qkv[c0:c1], state, channels=LIN.ChannelDecay(low[c0:c1], w2, b2, tau), q_scale=0.3).y
          for b, c0, c1 in _portions(n, [6, 1, 6])]
    assert torch.allclose(torch.cat(ys).double(), want.reshape(n, -1), atol=1e-4) and torch.allclose(state[2].double(), last, atol=1e-4)


def test_head_norm_with_silu_gate():
    N, H, P = 3, 2, 4
    y, z, gamma = torch.randn(N, H * P), torch.randn(N, H * P), torch.rand(P)
    b = PackedBatch.make([0], [N], True, N, "cpu")
    got = LIN.head_norm_gate(b, LIN.Numerators(y), z, gamma.repeat(H), H, 1e-4, torch.float32, silu=True)
    assert torch.allclose(got, (O.unit_rms(y.reshape(N, H, P), 1e-4) * gamma).reshape(N, -1) * O.silu(z), atol=1e-6)


# ---- the framework around it --------------------------------------------------------------------------------------------
def test_forward_matches_other_families_signature():
    cfg = K.CONFIGS["aligned"]
    w = K.weights(cfg, 20)
    c = MunazenConfig.from_dict(cfg)
    tok = torch.tensor([K.tokens(cfg, 9, 1), K.tokens(cfg, 9, 2)])
    got = forward(load_from_state_dict(w, c, torch.float32), tok, c)
    want = torch.stack([O.forward(t, cfg, w) for t in tok.tolist()])
    assert got.shape == want.shape and K.error(got, want) < TOL


def test_loader_checks_names_and_shapes():
    cfg = K.CONFIGS["mixed_odd"]
    c = MunazenConfig.from_dict(cfg)
    w = K.weights(cfg, 22)
    rankless = lambda s: {k: v for k, v in s.items() if not k.endswith((".a1", ".a2"))}
    assert rankless({k: tuple(v.shape) for k, v in w.items()}) == rankless(expected_shapes(c)) and set(w) == set(expected_shapes(c))
    with pytest.raises(KeyError):
        load_from_state_dict({k: v for k, v in w.items() if k != "l1.mix.a2.b"}, c)
    with pytest.raises(ValueError):
        load_from_state_dict(dict(w, head=w["head"][:-1]), c)
    with pytest.raises(ValueError):
        load_from_state_dict(dict(w, **{"l1.mix.a2": w["l1.mix.a2"][:, :-1]}), c)
    p = load_from_state_dict(w, c, torch.bfloat16)
    assert p["layers"][0]["mix"]["in"].dtype == torch.bfloat16 and p["layers"][0]["norm1"].dtype == torch.float32
    assert p["layers"][0]["mix"]["lru"].gates.dtype == torch.bfloat16 and p["layers"][0]["mix"]["lru"].decay.dtype == torch.float32
    (q0, k0, v0, x0, y0, g0), total = c.layers[0].mixer.segments()
    assert p["layers"][0]["mix"]["in"].shape[0] == total and all(s % 8 == 0 for s in (q0, k0, v0, x0, y0, g0, total))
    assert torch.equal(p["layers"][0]["mix"]["in"][g0:g0 + 6], w["l0.mix.left.g"].bfloat16())


def test_config_rejects_what_the_design_does_not_have():
    cfg = K.CONFIGS["aligned"]
    layer = lambda l, m=None: {"layers": [dict(l, mlp=m)], "loop": None}
    for change in ({"architecture": "Other"}, {"layers": [dict(cfg["layers"][0], type="window")]}, {"streams": 0},
                   {"norm": {"eps": 1e-5, "groups": 5}}, {"loop": {"start": 1, "stop": 9, "times": 2}},
                   layer(K.gla(), {"kind": "moe", "ff": 3}), layer(K.par(heads=3, kv_heads=2)), layer(K.par(rot_dims=12)),
                   layer(K.par(vdim=5)), layer(K.par(width=10, blocks=3)), layer(K.gla(tau=0.0))):
        with pytest.raises(ValueError):
            MunazenConfig.from_dict(dict(cfg, **change))


def test_runs_of_a_loop():
    c = MunazenConfig.from_dict(K.config([(K.gla(), None)] * 4, loop=(1, 3, 3)))
    assert c.runs == (0, 1, 2, 1, 2, 1, 2, 3)
    assert MunazenConfig.from_dict(K.config([(K.gla(), None)] * 3)).runs == (0, 1, 2)


def test_registry_loads_a_folder(tmp_path):
    from safetensors.torch import save_file
    cfg = K.CONFIGS["mixed_odd"]
    w = K.weights(cfg, 23, torch.bfloat16)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.contiguous() for k, v in w.items()}, str(tmp_path / "model.safetensors"))
    eng = registry.load_engine(str(tmp_path), torch.float32, "cpu", max_tokens=64, max_seqs=2)
    assert isinstance(eng, MunazenEngine)
    toks = K.tokens(cfg, 12, 3)
    assert K.error(K.run(eng, "a", toks, [12]), O.forward(toks, cfg, w)) < TOL


def test_presets_run():
    c = MunazenConfig.tiny()
    assert set(random_state_dict(c)) == set(expected_shapes(c))
    eng = MunazenEngine(init_params(c, 1), c, max_tokens=64, max_seqs=2)
    assert torch.isfinite(eng.step(["a"], [[1, 2, 3, 4, 5]])).all()
    s = MunazenConfig.serving()
    assert len(s.layers) == 8 and len({type(l.mixer) for l in s.layers}) == 2


def test_engine_refuses_bad_steps_and_stays_usable():
    cfg = K.CONFIGS["gla_only"]
    w = K.weights(cfg, 24)
    eng = K.engine(cfg, w, max_tokens=32, max_seqs=1)
    with pytest.raises(ValueError):
        eng.step(["a"], [[cfg["vocab"]]])
    toks = K.tokens(cfg, 6, 7)
    eng.step(["a"], [toks[:3]])
    with pytest.raises(MemoryError):
        eng.step(["b"], [[1]])
    assert K.error(eng.step(["a"], [toks[3:]]), O.forward(toks, cfg, w)[-1:]) < TOL


def test_sample_script_continues_token_ids(tmp_path):
    import subprocess
    from safetensors.torch import save_file
    cfg = K.CONFIGS["aligned"]
    w = K.weights(cfg, 50)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.contiguous() for k, v in w.items()}, str(tmp_path / "model.safetensors"))
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    prompt = K.tokens(cfg, 7, 1)
    r = subprocess.run([sys.executable, "scripts/sample.py", "--model-dir", str(tmp_path), "--dtype", "float32", "--temperature", "0", "--new_tokens",
                        "5", "--prompt-ids", ",".join(map(str, prompt))], cwd=root, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    got = [list(map(int, l.split(","))) for l in r.stdout.splitlines() if l and not l.startswith("---")][0]
    assert len(got) == 5
    for n, t in enumerate(got):
        lg = O.forward(prompt + got[:n], cfg, w)[-1]
        assert float(lg.max() - lg[t]) < 1e-3
