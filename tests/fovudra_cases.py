"""Small Fovudra configurations and random weights for the tests (the dictionaries of a ``config.json``, tensors by checkpoint
name), and the comparisons that the CPU and the GPU tests share."""
import torch

import fovudra_oracle as O


def rot(dims, base=700.0, scaling=True):
    r = {"base": base, "dims": dims}
    if scaling:
        r["scaling"] = {"factor": 3.0, "low": 1.0, "high": 5.0, "original": 90}
    return r


def attn(heads=6, kv_heads=2, dim=10, rot_dims=6, size=7, keep_first=3, scale=0.4, scaling=True, base=700.0):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale,
                                           "mask": {"size": size, "keep_first": keep_first}, "rot": rot(rot_dims, base, scaling)}}


def mlstm(heads=3, dim=7, vdim=5, cap=6.0):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def lightning(heads=2, dim=9, vdim=6, decay=(0.5, 0.99)):
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}}


def moe(ff=14, experts=5, top=3, shared=11):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, "shared": {"ff": shared}}


def config(layers, vocab=61, width=30, eps=1e-5):
    return {"architecture": "Fovudra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": [dict(l, mlp=m) for l, m in layers]}


# every branch of the design, in several orders and sizes (odd widths take the kernels' scalar paths)
CONFIGS = {
    "mixed_odd": config([(attn(), moe()), (mlstm(), None), (lightning(), moe(top=1)), (mlstm(heads=2, dim=12, vdim=9, cap=2.0), moe(top=5)),
                         (attn(heads=3, kv_heads=3, dim=5, rot_dims=4, size=11, keep_first=0, scaling=False), None)]),
    "aligned": config([(lightning(heads=3, dim=16, vdim=24, decay=(0.7, 0.95, 0.999)), moe(ff=24, experts=9, top=2, shared=40)),
                       (attn(heads=8, kv_heads=1, dim=32, rot_dims=32, size=20, keep_first=9), moe(ff=16, experts=4, top=1, shared=8)),
                       (mlstm(heads=2, dim=32, vdim=16, cap=10.0), moe(ff=32, experts=6, top=4, shared=24))], width=48, vocab=80, eps=1e-4),
    "ones": config([(mlstm(heads=1, dim=1, vdim=1, cap=1.0), moe(ff=1, experts=1, top=1, shared=1)),
                    (attn(heads=1, kv_heads=1, dim=3, rot_dims=2, size=1, keep_first=1), moe(ff=2, experts=2, top=2, shared=1)),
                    (lightning(heads=1, dim=1, vdim=2, decay=(1.0,)), None)], width=7, vocab=11),
    "attention_only": config([(attn(heads=5, kv_heads=1, size=16, keep_first=8), None), (attn(heads=4, kv_heads=4, size=200, keep_first=300), None)]),
    "recurrent_only": config([(mlstm(heads=5, cap=15.0), None), (lightning(heads=4, dim=3, vdim=12, decay=(0.2, 0.9, 0.97, 0.6)), moe(experts=40, top=7))],
                             vocab=37),
}


def weights(cfg, seed=0, dtype=torch.float32):
    """Random tensors under the checkpoint names, matrices scaled by their fan-in; input gates from closed to wide open."""
    g = torch.Generator().manual_seed(seed)
    n = lambda *s: torch.randn(*s, generator=g)
    mat = lambda o, i: n(o, i) * i ** -0.5
    V, D = cfg["vocab"], cfg["width"]
    w = {"embed": n(V, D), "embed.norm": 0.2 * n(D), "head": mat(V, D), "final.norm": 0.2 * n(D)}
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer["mlp"]
        for k in ("norm1", "norm1b") + (("norm2", "norm2b") if f else ()):
            w[p + k] = 0.3 * n(D)
        H, d = m["heads"], m["dim"]
        if layer["type"] == "attention":
            G = m["kv_heads"]
            w.update({p + "mix.q": mat(H * d, D), p + "mix.q.b": n(H * d), p + "mix.k": mat(G * d, D), p + "mix.k.b": n(G * d),
                      p + "mix.o": mat(D, H * d)})
        else:
            v = m["vdim"]
            w.update({p + "mix.q": mat(H * d, D), p + "mix.k": mat(H * d, D), p + "mix.v": mat(H * v, D), p + "mix.g": mat(H * v, D),
                      p + "mix.norm": 1 + 0.3 * n(H * v), p + "mix.o": mat(D, H * v)})
        if layer["type"] == "mlstm":
            w.update({p + "mix.i": 2 * mat(H, D), p + "mix.i.b": 3 * n(H), p + "mix.f": 2 * mat(H, D), p + "mix.f.b": 2 + 2 * n(H)})
        if f:
            E, ff = f["router"]["experts"], f["expert"]["ff"]
            w[p + "mlp.router"] = 2 * mat(E, D)
            for e, ff in [(f"e{e}", ff) for e in range(E)] + [("shared", f["shared"]["ff"])]:
                w.update({f"{p}mlp.{e}.gate": 2 * mat(ff, D), f"{p}mlp.{e}.up": 2 * mat(ff, D), f"{p}mlp.{e}.down": mat(D, ff)})
    return {k: v.to(dtype) for k, v in w.items()}


def tokens(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def engine(cfg, w, device="cpu", dtype=torch.float32, page_size=8, max_tokens=256, max_seqs=6, poison=True, **kw):
    """Step engine over a configuration; ``poison`` fills state and pages with large garbage that must never be read."""
    from jax_gpt_b200.models.fovudra import FovudraConfig, FovudraEngine, load_from_state_dict
    c = FovudraConfig.from_dict(cfg, page_size=page_size)
    eng = FovudraEngine(load_from_state_dict(w, c, dtype, device), c, max_tokens=max_tokens, max_seqs=max_seqs, **kw)
    if poison:
        for t in eng.cache.states + [v for v in eng.cache.vecs if v is not None] + list(eng.cache.paged.pool):
            t.fill_(1e4)
    return eng


def error(got, want):
    """Largest difference of logits with their mean taken off, relative to the logits' spread."""
    got, want = got.double().cpu(), want.double().cpu()
    d = (got - got.mean(-1, keepdim=True)) - (want - want.mean(-1, keepdim=True))
    return float(d.abs().max() / want.std(-1).mean().clamp_min(1e-3))


def run(eng, seq, toks, cuts):
    """Feeds one sequence in portions of the given sizes; returns the logits of every position."""
    out, at = [], 0
    for n in cuts:
        out.append(eng.step([seq], [toks[at:at + n]], [list(range(n))]).clone())
        at += n
    assert at == len(toks)
    return torch.cat(out)


# ---- comparisons shared by the CPU and the GPU tests -------------------------------------------------------------------
def check_prompts_and_cuts(name, device, tol, dtype=torch.float32):
    """Whole prompts, token by token, and portions of several sizes against the plain forward pass."""
    cfg = CONFIGS[name]
    w = weights(cfg, 1)
    toks = tokens(cfg, 45, 2)
    want = O.forward(toks, cfg, w)
    eng = engine(cfg, w, device, dtype)
    for k, cuts in enumerate(([45], [1] * 45, [44, 1], [2] * 22 + [1], [1, 44], [7, 8, 9, 16, 5], [17, 1, 1, 26])):
        got = run(eng, f"s{k}", toks, cuts)
        assert error(got, want) < tol, (name, cuts)
        eng.release(f"s{k}")


def check_layers(name, device, tol):
    cfg = CONFIGS[name]
    w = weights(cfg, 3)
    toks = tokens(cfg, 21, 4)
    want, got = [], []
    O.forward(toks, cfg, w, want)
    engine(cfg, w, device).step(["a"], [toks], layers_out=got)
    assert len(want) == len(got)
    for i, (a, b) in enumerate(zip(got, want)):
        assert float((a.double().cpu() - b).abs().max() / b.abs().max()) < tol, i


def check_batch_and_reuse(name, device, tol):
    """Unequal requests in one batch against each alone; later requests take freed slots and pages."""
    cfg = CONFIGS[name]
    w = weights(cfg, 5)
    eng = engine(cfg, w, device, max_tokens=72, max_seqs=3)     # small: every later round reuses slots and pages
    free = eng.cache.paged.alloc.n_free
    for rnd, sizes in enumerate(((1, 9, 30), (17, 8), (33, 1, 2), (16, 24, 7))):
        reqs = [tokens(cfg, n + 6, 10 * rnd + i) for i, n in enumerate(sizes)]
        want = [O.forward(t, cfg, w) for t in reqs]
        ids = [f"{rnd}.{i}" for i in range(len(reqs))]
        lg = eng.step(ids, [t[:n] for t, n in zip(reqs, sizes)], [[0, n - 1] if n > 1 else [0] for n in sizes])
        expect = torch.cat([x[[0, n - 1]] if n > 1 else x[:1] for x, n in zip(want, sizes)])
        assert error(lg, expect) < tol, (name, rnd)
        live = list(range(len(reqs)))
        for t in range(6):                                      # decode together; the first request ends earlier
            if t == 3 and len(live) > 1:
                eng.release(ids[live.pop(0)])
            lg = eng.step([ids[i] for i in live], [[reqs[i][sizes[i] + t]] for i in live])
            assert error(lg, torch.stack([want[i][sizes[i] + t] for i in live])) < tol, (name, rnd, t)
        for i in live:
            eng.release(ids[i])
        assert eng.cache.paged.alloc.n_free == free and eng.cache.n_free_slots == 3


def check_mixed_step(device, tol):
    """One step with a new prompt, a continued prompt and single tokens."""
    cfg = CONFIGS["mixed_odd"]
    w = weights(cfg, 6)
    reqs = [tokens(cfg, n, n) for n in (20, 13, 31)]
    want = [O.forward(t, cfg, w) for t in reqs]
    eng = engine(cfg, w, device)
    eng.step(["a", "b"], [reqs[0][:12], reqs[1][:12]])
    lg = eng.step(["c", "a", "b"], [reqs[2], reqs[0][12:], reqs[1][12:]])
    assert error(lg, torch.stack([want[2][-1], want[0][-1], want[1][-1]])) < tol


def check_generate(device, tol):
    """Greedy continuation through the package's entry point against the plain forward pass, past page borders."""
    from jax_gpt_b200.models.fovudra import FovudraConfig, generate, load_from_state_dict
    cfg = CONFIGS["aligned"]
    w = weights(cfg, 7)
    c = FovudraConfig.from_dict(cfg, page_size=8)
    p = load_from_state_dict(w, c, torch.float32, device)
    prompts = [tokens(cfg, n, 70 + n) for n in (5, 1, 12)]
    out = generate(p, prompts, c, 30).tolist()
    for pr, cont in zip(prompts, out):
        lg = O.forward(pr + cont[:-1], cfg, w)[len(pr) - 1:]
        top = lg.max(-1).values - lg[torch.arange(30), torch.tensor(cont)]
        assert float(top.max()) < tol * float(lg.std())          # the greedy choice up to rounding ties
    again = generate(p, prompts, c, 6, temperature=0.8, top_k=5, key=3)
    assert torch.equal(again, generate(p, prompts, c, 6, temperature=0.8, top_k=5, key=3)) and again.shape == (3, 6)


def edges(qpos, size, keep_first, page):
    """Key positions worth asking for from ``qpos``: both sides of the window's and the kept tokens' edges, page borders."""
    at = {0, 1, keep_first - 1, keep_first, keep_first + 1, qpos - size - 1, qpos - size, qpos - size + 1, qpos - size + 2, qpos - 1, qpos,
          page - 1, page, 31, 32, 33, 63, 64, 127, 128}
    return sorted(j for j in at if 0 <= j <= qpos)


def check_one_key_stands_out(device, tol):
    """A query that matches one chosen key far above the rest, just inside and just outside the window and the kept tokens
    and around page borders: a key that is lost, doubled, wrongly seen or read from a wrong page changes the output wholly."""
    from jax_gpt_b200.cache.paged import PagedCache
    from jax_gpt_b200.ops import window_attention as WA
    from jax_gpt_b200.ops.packed import PackedBatch, seq_begin
    g = torch.Generator().manual_seed(11)
    H, G, D, n, ps = 6, 2, 12, 75, 8
    cache = PagedCache(2, [5, 2 * G * D], 40, ps, 4, 12, torch.float32, device)
    for layer in range(2):
        cache.pool[layer].fill_(1e3)
    cache.reserve(3, 20)
    cache.reserve(1, n)
    cache.release(3)                     # the pages of sequence 1 do not start at page 0
    cache.reserve(2, 9)
    k, v = torch.randn(n, G, D, generator=g), torch.randn(n, G, D, generator=g)
    k = k / k.norm(dim=-1, keepdim=True)
    pages, offs = cache.slots(1, 0, n)
    cache.pool[1][pages, offs] = torch.cat([k.reshape(n, -1), v.reshape(n, -1)], -1).to(device)
    for size, keep in ((20, 5), (33, 8), (8, 0), (1, 1), (64, 32), (1, 0), (7, 75), (100, 3)):
        for qpos in sorted({0, size - 1, size, size + keep, 31, 32, 40, n - 1} & set(range(n))):
            for target in edges(qpos, size, keep, ps):
                for start in {0, qpos, max(0, qpos - 3)}:           # as part of a prompt, a decode step, a short portion
                    q = torch.zeros(qpos - start + 1, H, D)
                    q[-1] = 40.0 * k[target].repeat_interleave(H // G, 0)
                    b = PackedBatch.make([1], [qpos - start + 1], start == 0, n, device)
                    lens = torch.zeros(4, dtype=torch.int32)
                    lens[1] = start
                    seq_begin(b, torch.zeros(b.n_tok, dtype=torch.int32, device=device), lens.to(device),
                              torch.zeros(4, dtype=torch.int32, device=device))
                    mask = torch.tensor([[O.visible(qpos, j, size, keep) for j in range(qpos + 1)]])
                    want = O.masked_softmax_attention(q[-1:].double(), k[:qpos + 1].double(), v[:qpos + 1].double(), mask, 0.5)[0]
                    for splits in (1, 3) if device != "cpu" and start else (0,):
                        got = WA.window_attention_any(b, q.to(device), cache, 1, G, size, keep, 0.5, n_splits=splits)
                        assert float((got[-1].double().cpu() - want).abs().max()) < tol, (size, keep, target, qpos, start, splits)


def check_far_tokens(device, tol):
    """In the whole model, with values that dominate the residual: a changed early token shows in later logits exactly where
    the window or the kept tokens let it, in prompts and in decoding; elsewhere nothing changes."""
    cfg = config([(attn(heads=4, kv_heads=2, dim=8, rot_dims=8, size=12, keep_first=5, scale=0.05), None)], width=24)
    w = weights(cfg, 12)
    w["l0.norm1b"] += 4.0
    toks = tokens(cfg, 60, 13)
    want = O.forward(toks, cfg, w)
    eng = engine(cfg, w, device)
    for name, cuts in (("a", [60]), ("b", [30] + [1] * 30), ("c", [2] * 30)):
        assert error(run(eng, name, toks, cuts), want) < tol
        eng.release(name)
    for at in (0, 4, 5, 7, 8, 15, 16, 29, 30, 31, 40):
        other = toks[:at] + [(toks[at] + 1) % cfg["vocab"]] + toks[at + 1:]
        plain = O.forward(other, cfg, w)
        got = run(eng, f"t{at}", other, [30] + [1] * 30)
        eng.release(f"t{at}")
        assert error(got, plain) < tol
        inside, outside = at + 12 - 1, at + 12
        assert error(plain[inside:inside + 1], want[inside:inside + 1]) > 100 * tol
        changed = error(got[outside:outside + 1], want[outside:outside + 1])
        assert changed > 100 * tol if at < 5 else changed < tol, at


def check_state_carries(device, tol):
    """Slow decays and open forget gates: a token of the first portion still shows hundreds of positions later, far above the
    tolerance, and the framework follows it through prompts cut at odd places."""
    for layer in (mlstm(heads=2, dim=8, vdim=8, cap=20.0), lightning(heads=2, dim=8, vdim=8, decay=(0.9999, 0.999))):
        cfg = config([(layer, None)], width=24)
        w = weights(cfg, 16)
        if layer["type"] == "mlstm":
            w["l0.mix.f.b"].fill_(9.0)
            w["l0.mix.f"] *= 0.1
        toks = tokens(cfg, 150, 17)
        want = O.forward(toks, cfg, w)
        eng = engine(cfg, w, device)
        assert error(run(eng, "a", toks, [5, 2, 64, 1, 1, 57, 20]), want) < tol
        other = O.forward(toks[:1] + [(toks[1] + 1) % cfg["vocab"]] + toks[2:], cfg, w)
        assert error(other[100:], want[100:]) > 10 * tol


def check_long_decode(device, tol):
    """A short prompt and a few hundred decode steps over slow decays (state) and many pages and windows (attention)."""
    cfg = CONFIGS["aligned"]
    w = weights(cfg, 14)
    w["l2.mix.f.b"].fill_(8.0)
    toks = tokens(cfg, 230, 15)
    want = O.forward(toks, cfg, w)
    eng = engine(cfg, w, device, max_tokens=240)
    assert error(run(eng, "a", toks, [3] + [1] * 227), want) < tol
