"""Mopalorn on CPU: every operation's restatement, the engine's batching, cache and bookkeeping, and greedy generation, against the
plain implementation of mopalorn_oracle.py."""
import json
import math
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import mopalorn_cases as K  # noqa: E402
import mopalorn_oracle as O  # noqa: E402

from jax_gpt_b200.models import registry  # noqa: E402
from jax_gpt_b200.models.mopalorn import MopalornConfig, MopalornEngine, forward, init_params, random_state_dict  # noqa: E402
from jax_gpt_b200.models.mopalorn.weight_loader import expected_shapes, load_from_state_dict  # noqa: E402
from jax_gpt_b200.ops.gemm import linear_rows, xielu  # noqa: E402
from jax_gpt_b200.ops.mixed_kv import query_factors  # noqa: E402
from jax_gpt_b200.ops.rope import pair_order, rope_tables, rotate_interleaved  # noqa: E402

TOL = 3e-4


@pytest.fixture(autouse=True)
def _one_thread():
    """The tensors are tiny: threads would only wait for one another."""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


@pytest.mark.parametrize("name", sorted(K.CONFIGS))
def test_prompts_and_cuts(name):
    K.check_prompts_and_cuts(name, "cpu", TOL)


@pytest.mark.parametrize("name", sorted(K.CONFIGS))
def test_layers(name):
    K.check_layers(name, "cpu", TOL)


@pytest.mark.parametrize("name", ["mixed_odd", "blocks_beyond_pages"])
def test_batches_slots_and_pages_reused(name):
    K.check_batch_and_reuse(name, "cpu", TOL)


def test_mixed_step():
    K.check_mixed_step("cpu", TOL)


def test_greedy_and_sampled_generation():
    K.check_generate("cpu", TOL)


def test_long_decode():
    K.check_long_decode("cpu", TOL)


def test_far_tokens():
    K.check_far_tokens("cpu", TOL)


def test_one_key_stands_out():
    K.check_one_key_stands_out("cpu", 1e-4)
    K.check_one_key_stands_out("cpu", 1e-4, masks=((0, 0),), softcap=9.0)


def test_one_latent_stands_out():
    K.check_one_latent_stands_out("cpu", 1e-4)


@pytest.mark.parametrize("P,ps", [(4, 8), (5, 8), (8, 8), (19, 8), (1, 8), (16, 64), (24, 16)])
def test_block_means_follow_the_rows(P, ps):
    K.check_block_means("cpu", torch.float32, 1e-6, P, ps)


def test_activation():
    K.check_activation(linear_rows, "cpu", torch.float32, 1e-4, ((3, 16, 9), (40, 24, 16)))
    z = torch.tensor([0.0, -1e-6, 1e-6, -30.0, 30.0])
    assert torch.allclose(xielu(z, 2.0, 1.5).double(), torch.where(z > 0, 2.0 * z * z + z / 2, 1.5 * (torch.expm1(z) - z) + z / 2).double())


# ---- mechanisms alone --------------------------------------------------------------------------------------------------
def test_query_factors_step_with_the_context():
    f = query_factors(0.5, 4, 12)
    assert f[:3].tolist() == [1.0] * 3 and f[3] == f[6] == pytest.approx(1 + 0.5 * math.log(2)) and f[7] == pytest.approx(1 + 0.5 * math.log(3))
    assert f.tolist() == pytest.approx([O.query_factor(p, 0.5, 4) for p in range(12)])


@pytest.mark.parametrize("width,dims,base", [(8, 8, 500.0), (6, 6, 1e4), (2, 2, 9.0)])
def test_reordered_pairs_give_the_same_scores(width, dims, base):
    """Half-split rotation of the stored order and neighbour rotation of the reordered features: equal up to the order."""
    x, pos = torch.randn(5, 3, width, dtype=torch.float64), [0, 1, 7, 400, 33]
    want = O.turn_halves(x, base, pos)
    got = rotate_interleaved(x[..., pair_order(width, dims)], torch.tensor(pos), rope_tables(dims, base, 500))
    assert torch.allclose(got, want[..., pair_order(width, dims)], atol=1e-5)
    assert sorted(pair_order(9, 6).tolist()) == list(range(9)) and pair_order(9, 6).tolist()[6:] == [6, 7, 8]


def test_which_blocks_are_seen():
    """Window 3, blocks of 2: position 4 sees tokens 2 .. 4 and the block of tokens 0, 1; position 5 no block more (token 2 has left the
    window, its block has not)."""
    seen = O.seen_blocks(8, 2, 3)
    assert seen.long().sum(1).tolist() == [0, 0, 0, 0, 1, 1, 2, 2]
    assert O.seen_tokens(8, 3)[5].nonzero().flatten().tolist() == [3, 4, 5]


def test_sink_takes_weight_and_nothing_else():
    s = torch.tensor([[0.0, 0.0]], dtype=torch.float64)
    a = O.weights_of(s, torch.tensor([[True, True]]), torch.tensor([[math.log(2.0)]], dtype=torch.float64))
    assert torch.allclose(a, torch.full((1, 2), 0.25, dtype=torch.float64))


# ---- the framework around it --------------------------------------------------------------------------------------------
def test_forward_matches_other_families_signature():
    cfg = K.CONFIGS["aligned"]
    w = K.weights(cfg, 20)
    c = MopalornConfig.from_dict(cfg)
    tok = torch.tensor([K.tokens(cfg, 9, 1), K.tokens(cfg, 9, 2)])
    got = forward(load_from_state_dict(w, c, torch.float32), tok, c)
    want = torch.stack([O.forward(t, cfg, w) for t in tok.tolist()])
    assert got.shape == want.shape and K.error(got, want) < TOL


def test_first_mixing_layer_gives_its_values():
    """The mixing weight of the first such layer does nothing, the later ones' do; a layer without mixing is passed over."""
    cfg = K.config([(K.full(v_mix=False, vdim=3), None), (K.pooled(), None), (K.latent(), None), (K.full(), None)])
    w = K.weights(cfg, 21)
    toks = K.tokens(cfg, 14, 1)
    c = MopalornConfig.from_dict(cfg)
    assert c.first_values == 1
    lg = lambda ww: K.run(K.engine(cfg, ww), "a", toks, [9, 1, 4])
    base = lg(w)
    assert K.error(base, O.forward(toks, cfg, w)) < TOL
    assert torch.equal(lg(dict(w, **{"l1.mix.vmix": torch.tensor(9.0)})), base)
    assert K.error(lg(dict(w, **{"l3.mix.vmix": torch.tensor(0.0)})), base) > 100 * TOL


def test_loader_checks_names_and_shapes():
    cfg = K.CONFIGS["mixed_odd"]
    c = MopalornConfig.from_dict(cfg)
    w = K.weights(cfg, 22)
    assert {k: tuple(v.shape) for k, v in w.items()} == expected_shapes(c)
    with pytest.raises(KeyError):
        load_from_state_dict({k: v for k, v in w.items() if k != "l0.mix.sink"}, c)
    with pytest.raises(ValueError):
        load_from_state_dict(dict(w, embed=w["embed"][:-1]), c)
    p = load_from_state_dict(w, c, torch.bfloat16)
    assert p["layers"][0]["mix"]["in"].dtype == torch.bfloat16 and p["layers"][0]["norm1"].dtype == torch.float32
    assert p["layers"][0]["mix"]["sink"].dtype == torch.float32
    (q0, k0, v0), total = c.layers[0].mixer.segments()
    assert p["layers"][0]["mix"]["in"].shape[0] == total and all(s % 8 == 0 for s in (q0, k0, v0, total))
    assert torch.equal(p["layers"][0]["mix"]["in"][v0:v0 + 10], w["l0.mix.v"].bfloat16())


def test_config_rejects_what_the_design_does_not_have():
    cfg = K.CONFIGS["aligned"]
    layer = lambda l, m=None: {"layers": [dict(l, mlp=m)]}
    odd = K.latent()
    odd["mixer"]["rot"]["dims"] = 5
    for change in ({"architecture": "Other"}, {"layers": [dict(cfg["layers"][0], type="window")]}, layer(K.full(), {"kind": "moe", "ff": 3}),
                   layer(K.full(heads=3, kv_heads=2)), layer(K.pooled(size=0)), layer(odd), layer(K.full(every=0)),
                   {"layers": [dict(K.full(vdim=3), mlp=None), dict(K.pooled(vdim=4), mlp=None)]}):
        with pytest.raises(ValueError):
            MopalornConfig.from_dict(dict(cfg, **change))


def test_registry_loads_a_folder(tmp_path):
    from safetensors.torch import save_file
    cfg = K.CONFIGS["mixed_odd"]
    w = K.weights(cfg, 23, torch.bfloat16)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.contiguous() for k, v in w.items()}, str(tmp_path / "model.safetensors"))
    eng = registry.load_engine(str(tmp_path), torch.float32, "cpu", max_tokens=64, max_seqs=2)
    assert isinstance(eng, MopalornEngine)
    toks = K.tokens(cfg, 12, 3)
    assert K.error(K.run(eng, "a", toks, [12]), O.forward(toks, cfg, w)) < TOL


def test_presets_run():
    c = MopalornConfig.tiny()
    assert set(random_state_dict(c)) == set(expected_shapes(c))
    eng = MopalornEngine(init_params(c, 1), c, max_tokens=64, max_seqs=2)
    assert torch.isfinite(eng.step(["a"], [[1, 2, 3, 4, 5]])).all()
    s = MopalornConfig.serving()
    assert len(s.layers) == 8 and [bool(getattr(l.mixer, "pool", 0)) for l in s.layers].count(True) == 2


def test_engine_refuses_bad_steps_and_stays_usable():
    cfg = K.CONFIGS["grouped_only"]
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
