"""Fovudra on CPU: every operation's restatement, the engine's batching, cache and bookkeeping, and greedy generation, against
the plain implementation of fovudra_oracle.py."""
import json
import math
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import fovudra_cases as K  # noqa: E402
import fovudra_oracle as O  # noqa: E402

from jax_gpt_b200.models import registry  # noqa: E402
from jax_gpt_b200.models.fovudra import FovudraConfig, FovudraEngine, forward, init_params, random_state_dict  # noqa: E402
from jax_gpt_b200.models.fovudra.weight_loader import expected_shapes, load_from_state_dict  # noqa: E402
from jax_gpt_b200.ops import linear_attention as LIN  # noqa: E402
from jax_gpt_b200.ops.packed import PackedBatch, residual_norm_rows, seq_begin  # noqa: E402
from jax_gpt_b200.ops.rope import banded_frequencies, rope_tables, rotate_half_split  # noqa: E402
from jax_gpt_b200.ops.sigmoid_moe import sigmoid_topk  # noqa: E402

TOL = 3e-4


@pytest.mark.parametrize("name", sorted(K.CONFIGS))
def test_prompts_and_cuts(name):
    K.check_prompts_and_cuts(name, "cpu", TOL)


@pytest.mark.parametrize("name", sorted(K.CONFIGS))
def test_layers(name):
    K.check_layers(name, "cpu", TOL)


@pytest.mark.parametrize("name", ["mixed_odd", "recurrent_only"])
def test_batches_slots_and_pages_reused(name):
    K.check_batch_and_reuse(name, "cpu", TOL)


def test_mixed_step():
    K.check_mixed_step("cpu", TOL)


def test_greedy_and_sampled_generation():
    K.check_generate("cpu", TOL)


def test_one_key_stands_out():
    K.check_one_key_stands_out("cpu", 1e-4)


def test_far_tokens_show_where_the_mask_lets_them():
    K.check_far_tokens("cpu", TOL)


def test_state_carries():
    K.check_state_carries("cpu", TOL)


def test_long_decode():
    K.check_long_decode("cpu", TOL)


# ---- mechanisms alone --------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("rot", [K.rot(8), K.rot(8, scaling=False), K.rot(16, base=1e6), K.rot(2), K.rot(12, base=40.0),
                                 {"base": 1e4, "dims": 6, "scaling": {"factor": 4.0, "low": 2.0, "high": 2.0, "original": 50}}])
def test_rotation(rot):
    f = banded_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    assert f == pytest.approx(O.rotary_frequencies(rot))
    x = torch.randn(9, 2, rot["dims"] + 3, dtype=torch.float64)
    pos = torch.tensor([0, 1, 2, 63, 64, 500, 7, 8, 999])
    got = rotate_half_split(x, pos, rope_tables(rot["dims"], rot["base"], 1000, rot.get("scaling")))
    assert torch.allclose(got, O.rotate_half(x, pos.tolist(), rot), atol=1e-5)


def test_frequency_bands_by_hand():
    # base e^2, 6 dims: f = 1, e^(-2/3), e^(-4/3); original / wavelength = 8, 8 e^(-2/3) = 4.107, 8 e^(-4/3) = 2.109
    sc = {"factor": 10.0, "low": 3.0, "high": 5.0, "original": 16 * math.pi}
    f = banded_frequencies(6, math.exp(2.0), sc)
    s = (8 * math.exp(-2 / 3) - 3) / 2
    assert f[0] == pytest.approx(1.0) and f[2] == pytest.approx(math.exp(-4 / 3) / 10)
    assert f[1] == pytest.approx(math.exp(-2 / 3) * ((1 - s) / 10 + s))


def test_window_by_hand():
    rows = ["1000000", "1100000", "1110000", "1111000", "1101100", "1100110", "1100011"]
    m = O.window_mask(7, 2, 2)           # a window of two and two kept tokens
    assert ["".join(str(int(x)) for x in r) for r in m] == rows


@pytest.mark.parametrize("gated", [False, True])
def test_recurrence_restatement(gated):
    g = torch.Generator().manual_seed(3)
    H, N, P, n, cap = 2, 5, 4, 13, 4.0
    qkv = torch.randn(n, H * (2 * N + P), generator=g)
    split = lambda x: [t.reshape(len(x), H, -1).double() for t in x.split([H * N, H * N, H * P], -1)]
    raw, bias = 3 * torch.randn(n, 2 * H, generator=g), torch.randn(2 * H, generator=g)
    state, vec = torch.full((3, H, N, P), 1e3), torch.full((3, H, N + 1), 1e3)
    lens, prev = torch.zeros(3, dtype=torch.int32), torch.zeros(3, dtype=torch.int32)
    decay = torch.tensor([0.6, 0.97])
    ys = []
    for c0, c1 in ((0, 6), (6, 7), (7, 13)):
        b = PackedBatch.make([2], [c1 - c0], c0 == 0, 20, "cpu")
        seq_begin(b, torch.zeros(c1 - c0, dtype=torch.int32), lens, prev)
        gates = LIN.Gates(raw[c0:c1], bias, cap, vec) if gated else None
        s = LIN.linear_scan(b, qkv[c0:c1], state, decay=None if gated else decay, gates=gates, q_scale=0.3)
        ys.append(LIN.head_norm_gate(b, s, torch.full((c1 - c0, H * P), 50.0), torch.ones(H * P), H, 1e-5, torch.float32))
    q, k, v = split(qkv)
    if gated:
        i = O.soft_cap(raw[:, :H].double() + bias[:H], cap)
        f = O.log_sigmoid(O.soft_cap(raw[:, H:].double() + bias[H:], cap))
        want, (S, nv, m) = O.mlstm_recurrence(q * 0.3, k, v, i, f)
        assert torch.allclose(vec[2].double(), torch.cat([nv, m[:, None]], -1), atol=1e-4)
    else:
        want, S = O.decay_recurrence(q * 0.3, k, v, decay.double())
    assert torch.allclose(state[2].double(), S, atol=1e-4)
    assert torch.allclose(torch.cat(ys).double(), O.unit_rms(want, 1e-5).reshape(n, -1), atol=1e-4)


def test_running_maximum_starts_at_zero():
    """With closed input gates the denominator's floor exp(-m) is what divides, and m falls from 0 with the forget gate."""
    q = k = torch.ones(2, 1, 1, dtype=torch.float64)
    v = torch.full((2, 1, 1), 2.0, dtype=torch.float64)
    i, f = torch.full((2, 1), -5.0, dtype=torch.float64), torch.full((2, 1), -0.5, dtype=torch.float64)
    o, (S, n, m) = O.mlstm_recurrence(q, k, v, i, f)
    assert float(m[0]) == pytest.approx(-1.0)
    # m_1 = -0.5, S_1 = 2 e^(-4.5); floor e^(0.5)
    assert float(o[0]) == pytest.approx(2 * math.exp(-4.5) / (math.exp(0.5) + 1e-6))


def test_router_takes_the_largest_scores():
    z = torch.tensor([[0.1, 3.0, -2.0, 1.0], [-5.0, -4.0, -9.0, -4.5]])
    ids, s = sigmoid_topk(z, 2)
    assert ids.tolist() == [[1, 3], [1, 3]] and torch.allclose(s, torch.sigmoid(torch.tensor([[3.0, 1.0], [-4.0, -4.5]])))
    order, w = O.choose_experts(z, 2)
    assert torch.equal(order, ids.long()) and torch.allclose(w, s)


def test_residual_norm():
    y, x, a, b = torch.randn(3, 10), torch.randn(3, 10), torch.rand(10), torch.rand(10)
    xx = x.clone()
    h = residual_norm_rows(y, 1 + a, xx, 1 + b, 1e-5, torch.float32)
    want = x + O.rms_norm_zero_centred(y, a, 1e-5)
    assert torch.allclose(xx, want, atol=1e-6) and torch.allclose(h, O.rms_norm_zero_centred(want, b, 1e-5), atol=1e-6)
    assert residual_norm_rows(y, 1 + a, xx, None, 1e-5, torch.float32, add=False) is None
    assert torch.allclose(xx, O.rms_norm_zero_centred(y, a, 1e-5), atol=1e-6)


# ---- the framework around it --------------------------------------------------------------------------------------------
def test_forward_matches_other_families_signature():
    cfg = K.CONFIGS["aligned"]
    w = K.weights(cfg, 20)
    c = FovudraConfig.from_dict(cfg)
    tok = torch.tensor([K.tokens(cfg, 9, 1), K.tokens(cfg, 9, 2)])
    got = forward(load_from_state_dict(w, c, torch.float32), tok, c)
    want = torch.stack([O.forward(t, cfg, w) for t in tok.tolist()])
    assert got.shape == want.shape and K.error(got, want) < TOL


def test_loader_checks_names_and_shapes():
    cfg = K.CONFIGS["mixed_odd"]
    c = FovudraConfig.from_dict(cfg)
    w = K.weights(cfg, 22)
    assert {k: tuple(v.shape) for k, v in w.items()} == expected_shapes(c)
    with pytest.raises(KeyError):
        load_from_state_dict({k: v for k, v in w.items() if k != "l1.mix.i.b"}, c)
    with pytest.raises(ValueError):
        load_from_state_dict(dict(w, head=w["head"][:-1]), c)
    p = load_from_state_dict(w, c, torch.bfloat16)
    assert p["layers"][1]["mix"]["in"].dtype == torch.bfloat16 and p["layers"][0]["norm1"].dtype == torch.float32
    assert p["layers"][1]["mix"]["gate_b"].dtype == torch.float32


def test_config_rejects_what_the_design_does_not_have():
    cfg = K.CONFIGS["aligned"]
    bad_v = K.attn()
    bad_v["mixer"]["vdim"] = 9
    for change in ({"architecture": "Other"}, {"layers": [dict(cfg["layers"][0], type="window")]},
                   {"layers": [dict(cfg["layers"][0], mlp={"kind": "dense", "ff": 3})]}, {"layers": [dict(bad_v, mlp=None)]},
                   {"layers": [dict(K.lightning(decay=(0.5,)), mlp=None)]}, {"layers": [dict(K.mlstm(), mlp=K.moe(experts=2, top=3))]}):
        with pytest.raises(ValueError):
            FovudraConfig.from_dict(dict(cfg, **change))


def test_registry_loads_a_folder(tmp_path):
    from safetensors.torch import save_file
    cfg = K.CONFIGS["mixed_odd"]
    w = K.weights(cfg, 23, torch.bfloat16)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.contiguous() for k, v in w.items()}, str(tmp_path / "model.safetensors"))
    eng = registry.load_engine(str(tmp_path), torch.float32, "cpu", max_tokens=64, max_seqs=2)
    assert isinstance(eng, FovudraEngine)
    toks = K.tokens(cfg, 12, 3)
    assert K.error(K.run(eng, "a", toks, [12]), O.forward(toks, cfg, w)) < TOL


def test_presets_run():
    c = FovudraConfig.tiny()
    assert set(random_state_dict(c)) == set(expected_shapes(c))
    eng = FovudraEngine(init_params(c, 1), c, max_tokens=64, max_seqs=2)
    assert torch.isfinite(eng.step(["a"], [[1, 2, 3, 4, 5]])).all()
    s = FovudraConfig.serving()
    assert len(s.layers) == 8 and len(s.attention_layers) == 2
    assert len({type(s.layers[i].mixer) for i in s.recurrent_layers}) == 2


def test_engine_refuses_bad_steps_and_stays_usable():
    cfg = K.CONFIGS["recurrent_only"]
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
