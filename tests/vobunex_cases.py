"""Small Vobunex configurations and random weights for the tests (the dictionaries of a ``config.json``, tensors by
checkpoint name), and the comparisons that the CPU and the GPU tests share."""
import torch

import vobunex_oracle as O


def rot(dims, base=500.0, scaling=True):
    r = {"base": base, "dims": dims}
    if scaling:
        r["scaling"] = {"factor": 3.0, "original": 40, "fast": 3.0, "slow": 0.4}
    return r


def attn(heads=3, dim=10, rot_dim=6, vdim=7, q_rank=18, kv_rank=13, scale=0.3, scaling=True):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank,
                                                  "kv_rank": kv_rank, "scale": scale, "rot": rot(rot_dim, scaling=scaling)}}


def mamba(heads=6, vdim=5, state=9, groups=3, conv=3, norm_groups=2):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                        "norm_groups": norm_groups}}


def dense(ff=33):
    return {"kind": "dense", "ff": ff}


def moe(ff=14, limit=0.8, experts=5, top=3):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def config(layers, vocab=61, width=30, eps=1e-5, bigram=(23, 19, 5)):
    out = {"architecture": "Vobunex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {},
           "layers": [dict(l, mlp=m) for l, m in layers]}
    if bigram:
        out["embedding"] = {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))}
    return out


# every branch of the design, in several orders and sizes (odd widths take the kernels' scalar paths)
CONFIGS = {
    "mixed_odd": config([(attn(), moe()), (mamba(), None), (mamba(heads=4, vdim=6, state=7, groups=1, conv=5, norm_groups=4), dense()),
                         (attn(heads=2, dim=8, rot_dim=4, vdim=9, q_rank=11, kv_rank=20, scaling=False), moe(top=1))]),
    "aligned": config([(mamba(heads=8, vdim=16, state=32, groups=2, conv=4, norm_groups=1), moe(ff=32, experts=7, top=2, limit=2.0)),
                       (attn(heads=4, dim=24, rot_dim=8, vdim=16, q_rank=32, kv_rank=40), dense(80))], width=48, vocab=80),
    "ones": config([(mamba(heads=1, vdim=3, state=1, groups=1, conv=1, norm_groups=1), dense(1)),
                    (attn(heads=1, dim=3, rot_dim=2, vdim=1, q_rank=1, kv_rank=2), moe(ff=1, experts=1, top=1))],
                   width=7, vocab=11, bigram=(1, 3, 2)),
    "attention_only": config([(attn(heads=5), None), (attn(heads=1, kv_rank=6), dense())], bigram=None),
    "mamba_only": config([(mamba(groups=6), None), (mamba(groups=1, conv=2, norm_groups=6), moe(experts=9, top=4))], vocab=37),
}


def weights(cfg, seed=0, dtype=torch.float32):
    """Random tensors under the checkpoint names, matrices scaled by their fan-in."""
    g = torch.Generator().manual_seed(seed)
    n = lambda *s: torch.randn(*s, generator=g)
    mat = lambda o, i: n(o, i) * i ** -0.5
    V, D = cfg["vocab"], cfg["width"]
    w = {"embed": n(V, D), "head": mat(V, D), "final.norm": 1 + 0.2 * n(D), "final.norm.b": 0.2 * n(D)}
    big = cfg["embedding"].get("bigram")
    if big:
        w["bigram"] = n(big["buckets"] + 1, D)
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer["mlp"]
        for k in ("norm1", "norm2") if f else ("norm1",):
            w[p + k], w[p + k + ".b"] = 1 + 0.2 * n(D), 0.2 * n(D)
        if layer["type"] == "latent_attention":
            H, r = m["heads"], m["kv_rank"]
            w.update({p + "mix.dq": mat(m["q_rank"], D), p + "mix.dq.norm": 1 + 0.2 * n(m["q_rank"]),
                      p + "mix.uq": mat(H * (m["dim"] + m["rot_dim"]), m["q_rank"]), p + "mix.dkv": mat(r + m["rot_dim"], D),
                      p + "mix.dkv.norm": 1 + 0.2 * n(r), p + "mix.uk": mat(H * m["dim"], r), p + "mix.uv": mat(H * m["vdim"], r),
                      p + "mix.sink": n(H) + 0.5, p + "mix.o": mat(D, H * m["vdim"])})
        else:
            H, inner = m["heads"], m["heads"] * m["vdim"]
            C = inner + 2 * m["groups"] * m["state"]
            w.update({p + "mix.in": mat(inner + C + H, D), p + "mix.conv": n(C, m["conv"]) * m["conv"] ** -0.5,
                      p + "mix.conv.b": 0.2 * n(C), p + "mix.dt_bias": torch.rand(H, generator=g) * 3 - 3,
                      p + "mix.A_log": torch.log(torch.rand(H, generator=g) * 3 + 0.05), p + "mix.D": n(H),
                      p + "mix.norm": 1 + 0.2 * n(inner), p + "mix.o": mat(D, inner)})
        if f and f["kind"] == "dense":
            w.update({p + "mlp.up": mat(f["ff"], D), p + "mlp.down": mat(D, f["ff"])})
        elif f:
            E, top, ff = f["router"]["experts"], f["router"]["top"], f["expert"]["ff"]
            w[p + "mlp.table"] = torch.rand(V, E, generator=g).argsort(-1)[:, :top].to(torch.int32)
            for e in range(E):
                w.update({f"{p}mlp.e{e}.gate": 2 * mat(ff, D), f"{p}mlp.e{e}.up": 2 * mat(ff, D), f"{p}mlp.e{e}.down": mat(D, ff)})
    return {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in w.items()}


def tokens(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def engine(cfg, w, device="cpu", dtype=torch.float32, page_size=8, max_tokens=256, max_seqs=6, poison=True, **kw):
    """Step engine over a configuration; ``poison`` fills state and pages with large garbage that must never be read."""
    from jax_gpt_b200.models.vobunex import VobunexConfig, VobunexEngine, load_from_state_dict
    c = VobunexConfig.from_dict(cfg, page_size=page_size)
    eng = VobunexEngine(load_from_state_dict(w, c, dtype, device), c, max_tokens=max_tokens, max_seqs=max_seqs, **kw)
    if poison:
        for t in eng.cache.states + eng.cache.rings + list(eng.cache.paged.pool):
            t.fill_(1e4)
        eng.cache.prev.fill_(1)
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
    from jax_gpt_b200.models.vobunex import VobunexConfig, generate, load_from_state_dict
    cfg = CONFIGS["aligned"]
    w = weights(cfg, 7)
    c = VobunexConfig.from_dict(cfg, page_size=8)
    p = load_from_state_dict(w, c, torch.float32, device)
    prompts = [tokens(cfg, n, 70 + n) for n in (5, 1, 12)]
    out = generate(p, prompts, c, 20).tolist()
    for pr, cont in zip(prompts, out):
        lg = O.forward(pr + cont[:-1], cfg, w)[len(pr) - 1:]
        top = lg.max(-1).values - lg[torch.arange(20), torch.tensor(cont)]
        assert float(top.max()) < tol * float(lg.std())          # the greedy choice up to rounding ties
    torch.manual_seed(0)
    again = generate(p, prompts, c, 6, temperature=0.8, top_k=5, key=3)
    assert torch.equal(again, generate(p, prompts, c, 6, temperature=0.8, top_k=5, key=3)) and again.shape == (3, 6)


def check_one_key_stands_out(device, tol):
    """A query that matches one chosen key far above the rest: first, page-border, farthest and own positions, and a sink
    that swallows everything else. A key that is lost, doubled or read from a wrong page changes the output wholly."""
    from jax_gpt_b200.cache.paged import PagedCache
    from jax_gpt_b200.ops import latent_attention as LA
    from jax_gpt_b200.ops.packed import PackedBatch, seq_begin
    g = torch.Generator().manual_seed(11)
    R, dr, H, n, ps = 12, 4, 2, 75, 8
    cache = PagedCache(2, [5, R + dr], 40, ps, 4, 12, torch.float32, device)
    for layer in range(2):
        cache.pool[layer].fill_(1e3)
    cache.reserve(3, 20)
    cache.reserve(1, n)
    cache.release(3)                     # the pages of sequence 1 do not start at page 0
    cache.reserve(2, 9)
    rows = torch.randn(n, R + dr, generator=g)
    rows = rows / rows.norm(dim=-1, keepdim=True)
    pages, offs = cache.slots(1, 0, n)
    cache.pool[1][pages, offs] = rows.to(device)
    sink = torch.tensor([4.0, -2.0])
    for target in (0, 1, ps - 1, ps, 2 * ps - 1, 31, 32, 33, 63, 64, n - 2, n - 1):
        for qpos in sorted({target, min(target + 1, n - 1), n - 1}):
            for start in {0, qpos}:                     # as part of a prompt, and as a decode step
                q = torch.zeros(qpos - start + 1, H, R + dr)
                q[-1] = 40.0 * rows[target]
                b = PackedBatch.make([1], [qpos - start + 1], start == 0, n, device)
                lens = torch.zeros(4, dtype=torch.int32)
                lens[1] = start
                seq_begin(b, torch.zeros(b.n_tok, dtype=torch.int32, device=device), lens.to(device),
                          torch.zeros(4, dtype=torch.int32, device=device))
                s = (q[-1].double() @ rows[:qpos + 1].double().T) * 0.5
                want = O.sink_softmax(s, sink.double()[:, None]) @ rows[:qpos + 1, :R].double()
                for splits in (1, 3) if device != "cpu" and start else (0,):
                    got = LA.latent_attention(b, q.to(device), cache, 1, R, 0.5, sink.to(device), n_splits=splits)
                    assert float((got[-1].double().cpu() - want).abs().max()) < tol, (target, qpos, start, splits)


def check_far_token(device, tol):
    """In the whole model: values dominate the residual, so every early token, page borders included, shows in the logits
    of positions decoded much later, and so does the sink; both by far more than the tolerance."""
    cfg = config([(attn(heads=2, dim=8, rot_dim=4, vdim=8, q_rank=16, kv_rank=16, scale=1.0), None)], bigram=None, width=24)
    w = weights(cfg, 12)
    w["l0.mix.uv"] *= 8
    toks = tokens(cfg, 70, 13)
    want = O.forward(toks, cfg, w)
    got = run(engine(cfg, w, device), "a", toks, [40] + [1] * 30)
    assert error(got, want) < tol
    for at in (0, 7, 8, 15, 16, 31, 32, 39):
        other = O.forward(toks[:at] + [(toks[at] + 1) % cfg["vocab"]] + toks[at + 1:], cfg, w)
        assert error(other[41:], want[41:]) > 100 * tol
    no_sink = O.forward(toks, cfg, dict(w, **{"l0.mix.sink": torch.full((2,), -100.0)}))
    assert error(no_sink[41:], want[41:]) > 50 * tol


def check_long_decode(device, tol):
    """A short prompt and a few hundred decode steps over slow decays (state) and many pages (attention)."""
    cfg = CONFIGS["aligned"]
    w = weights(cfg, 14)
    w["l0.mix.A_log"].fill_(-5.0)
    toks = tokens(cfg, 230, 15)
    want = O.forward(toks, cfg, w)
    eng = engine(cfg, w, device, max_tokens=240)
    got = run(eng, "a", toks, [3] + [1] * 227)
    assert error(got, want) < tol
