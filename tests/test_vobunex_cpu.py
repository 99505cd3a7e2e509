"""Vobunex on CPU: every operation's restatement, the engine's batching, cache and bookkeeping, and greedy generation,
against the plain implementation of vobunex_oracle.py."""
import json
import math
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import vobunex_cases as K  # noqa: E402
import vobunex_oracle as O  # noqa: E402

from jax_gpt_b200.models import registry  # noqa: E402
from jax_gpt_b200.models.vobunex import VobunexConfig, VobunexEngine, forward, init_params, random_state_dict  # noqa: E402
from jax_gpt_b200.models.vobunex.weight_loader import expected_shapes, load_from_state_dict  # noqa: E402
from jax_gpt_b200.ops.rope import rope_tables, rotate_interleaved, yarn_frequencies  # noqa: E402

TOL = 2e-4


@pytest.mark.parametrize("name", sorted(K.CONFIGS))
def test_prompts_and_cuts(name):
    K.check_prompts_and_cuts(name, "cpu", TOL)


@pytest.mark.parametrize("name", sorted(K.CONFIGS))
def test_layers(name):
    K.check_layers(name, "cpu", TOL)


@pytest.mark.parametrize("name", ["mixed_odd", "mamba_only"])
def test_batches_slots_and_pages_reused(name):
    K.check_batch_and_reuse(name, "cpu", TOL)


def test_mixed_step():
    K.check_mixed_step("cpu", TOL)


def test_greedy_and_sampled_generation():
    K.check_generate("cpu", TOL)


def test_one_key_stands_out():
    K.check_one_key_stands_out("cpu", 1e-4)


def test_far_token_and_sink_show_in_the_logits():
    K.check_far_token("cpu", TOL)


def test_long_decode():
    K.check_long_decode("cpu", TOL)


@pytest.mark.parametrize("rot", [K.rot(8), K.rot(8, scaling=False), K.rot(16, base=1e6), K.rot(2), K.rot(12, base=40.0),
                                 {"base": 1e4, "dims": 6, "scaling": {"factor": 1.0, "original": 16, "fast": 8.0, "slow": 8.0}}])
def test_rotation(rot):
    f, amp = yarn_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    g, amp2 = O.rotary_frequencies(rot)
    assert amp == pytest.approx(amp2) and f == pytest.approx(g)
    x = torch.randn(9, 2, rot["dims"] + 3, dtype=torch.float64)
    pos = torch.tensor([0, 1, 2, 63, 64, 500, 7, 8, 999])
    got = rotate_interleaved(x, pos, rope_tables(rot["dims"], rot["base"], 1000, rot.get("scaling")))
    want = torch.cat([O.rotate(x[..., :rot["dims"]], pos.tolist(), rot), x[..., rot["dims"]:]], -1)
    assert torch.allclose(got, want, atol=1e-5)


def test_yarn_ramp_by_hand():
    # base e^2, 4 dims: dim(t) = ln(original / (2 pi t)); original = 2 pi e^3 -> dim(1) = 3, dim(e^2) = 1
    f, amp = yarn_frequencies(4, math.exp(2.0), {"factor": 5.0, "original": 2 * math.pi * math.exp(3.0), "fast": math.exp(2.0) * 1.0001,
                                                 "slow": 1.0001})
    assert f[0] == pytest.approx(1.0) and amp == pytest.approx(1 + 0.1 * math.log(5))
    assert f[1] == pytest.approx(math.exp(-1.0) * (1 / 3 / 5 + 2 / 3), rel=1e-3)      # lo = 0, hi = 3, ramp(1) = 1/3


def test_forward_matches_other_families_signature():
    cfg = K.CONFIGS["aligned"]
    w = K.weights(cfg, 20)
    c = VobunexConfig.from_dict(cfg)
    tok = torch.tensor([K.tokens(cfg, 9, 1), K.tokens(cfg, 9, 2)])
    got = forward(load_from_state_dict(w, c, torch.float32), tok, c)
    want = torch.stack([O.forward(t, cfg, w) for t in tok.tolist()])
    assert got.shape == want.shape and K.error(got, want) < TOL


def test_bigram_row_by_hand():
    cfg = K.config([(K.mamba(), None)], bigram=(10, 7, 3), vocab=20)
    w = K.weights(cfg, 21)
    x = O.embed(torch.tensor([4, 9, 4]), cfg, w)
    assert torch.allclose(x[0], w["embed"][4] + w["bigram"][10])
    assert torch.allclose(x[1], w["embed"][9] + w["bigram"][(4 * 7 + 9 * 3) % 10])
    assert torch.allclose(x[2], w["embed"][4] + w["bigram"][(9 * 7 + 4 * 3) % 10])


def test_loader_checks_names_shapes_and_tables():
    cfg = K.CONFIGS["mixed_odd"]
    c = VobunexConfig.from_dict(cfg)
    w = K.weights(cfg, 22)
    assert {k: tuple(v.shape) for k, v in w.items()} == expected_shapes(c)
    with pytest.raises(KeyError):
        load_from_state_dict({k: v for k, v in w.items() if k != "l1.mix.D"}, c)
    with pytest.raises(ValueError):
        load_from_state_dict(dict(w, head=w["head"][:-1]), c)
    bad = w["l0.mlp.table"].clone()
    bad[3, 1] = 5
    with pytest.raises(ValueError):
        load_from_state_dict(dict(w, **{"l0.mlp.table": bad}), c)
    p = load_from_state_dict(w, c, torch.bfloat16)
    assert p["layers"][0]["mix"]["ukv"].dtype == torch.bfloat16 and p["layers"][0]["norm1"].dtype == torch.float32


def test_config_rejects_what_the_design_does_not_have():
    cfg = K.CONFIGS["aligned"]
    for change in ({"architecture": "Other"}, {"layers": [dict(cfg["layers"][0], type="window")]},
                   {"layers": [dict(cfg["layers"][0], mlp={"kind": "shared", "ff": 3})]}):
        with pytest.raises(ValueError):
            VobunexConfig.from_dict(dict(cfg, **change))


def test_registry_loads_a_folder(tmp_path):
    from safetensors.torch import save_file
    cfg = K.CONFIGS["mixed_odd"]
    w = K.weights(cfg, 23, torch.bfloat16)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.contiguous() for k, v in w.items()}, str(tmp_path / "model.safetensors"))
    eng = registry.load_engine(str(tmp_path), torch.float32, "cpu", max_tokens=64, max_seqs=2)
    toks = K.tokens(cfg, 19, 5)
    assert isinstance(eng, VobunexEngine)
    assert K.error(eng.step(["x"], [toks], [list(range(19))]), O.forward(toks, cfg, w)) < TOL
    assert registry.family_for_config({"model_type": "deepseek_v3"}).name == "deepseek_v3"
    with pytest.raises(KeyError):
        registry.family_for_config({"architecture": "nothing"})


def test_engine_refuses_bad_steps_and_stays_usable():
    cfg = K.CONFIGS["aligned"]
    eng = K.engine(cfg, K.weights(cfg, 24), max_tokens=32, max_seqs=2)
    for seqs, toks, want in ((["a"], [[]], None), (["a"], [[cfg["vocab"]]], None), (["a"], [[-1]], None), (["a", "a"], [[1], [2]], None),
                             (["a"], [[1, 2]], [[2]])):
        with pytest.raises(ValueError):
            eng.step(seqs, toks, want)
    with pytest.raises((MemoryError, ValueError)):
        eng.step(["big"], [[1] * 500])
    assert "big" not in eng.cache
    eng.step(["a", "b"], [[1, 2], [3]])
    with pytest.raises(MemoryError):
        eng.step(["c"], [[1]])
    eng.release("a")
    assert eng.step(["c"], [[1]]).shape == (1, cfg["vocab"])


def test_presets():
    for c in (VobunexConfig.tiny(), VobunexConfig.serving(width=128, experts=4, top=2, ff=32, vocab=64)):
        sd = random_state_dict(c, 1)
        assert {k: tuple(v.shape) for k, v in sd.items()} == expected_shapes(c)
    c = VobunexConfig.tiny()
    lg = forward(init_params(c, 0), torch.arange(12)[None], c)
    assert lg.shape == (1, 12, c.vocab_size) and torch.isfinite(lg).all()


def test_sample_script_continues_token_ids(tmp_path):
    import subprocess
    from safetensors.torch import save_file
    cfg = K.CONFIGS["aligned"]
    w = K.weights(cfg, 50)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.contiguous() for k, v in w.items()}, str(tmp_path / "model.safetensors"))
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    prompts = [K.tokens(cfg, 7, 1), K.tokens(cfg, 3, 2)]
    args = [sys.executable, "scripts/sample.py", "--model-dir", str(tmp_path), "--dtype", "float32", "--temperature", "0", "--new_tokens", "5"]
    for p in prompts:
        args += ["--prompt-ids", ",".join(map(str, p))]
    r = subprocess.run(args, cwd=root, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    rows = [list(map(int, l.split(","))) for l in r.stdout.splitlines() if l and not l.startswith("---")]
    for p, got in zip(prompts, rows):
        for n, t in enumerate(got):
            lg = O.forward(p + got[:n], cfg, w)[-1]
            assert float(lg.max() - lg[t]) < 1e-3
