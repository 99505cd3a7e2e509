"""Small Munazen configurations and random weights for the tests (the dictionaries of a ``config.json``, tensors by checkpoint name),
and the comparisons that the CPU and the GPU tests share."""
import torch

import munazen_oracle as O


def rot(dims, base=700.0, scaling=True):
    r = {"base": base, "dims": dims}
    if scaling:
        r["scaling"] = {"factor": 3.0, "fast": 8.0, "slow": 1.0, "original": 90}
    return r


def par(heads=6, kv_heads=2, dim=10, rot_dims=6, vdim=14, scale=0.4, scaling=True, base=700.0, width=20, blocks=4, conv=3, left_scale=0.8,
        right_scale=1.3):
    return {"type": "parallel", "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": rot(rot_dims, base, scaling)},
        "right": {"width": width, "blocks": blocks, "conv": conv}, "left_scale": left_scale, "right_scale": right_scale}}


def gla(heads=3, dim=7, vdim=5, tau=6.0):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}}


def dense(ff=23):
    return {"kind": "dense", "ff": ff}


def config(layers, vocab=61, width=30, groups=3, eps=1e-5, streams=3, loop=None):
    c = {"architecture": "Munazen", "vocab": vocab, "width": width, "norm": {"eps": eps, "groups": groups}, "streams": streams,
         "layers": [dict(l, mlp=m) for l, m in layers]}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


# every branch of the design, in several orders and sizes (odd widths take the kernels' scalar paths)
CONFIGS = {
    "mixed_odd": config([(par(), dense()), (gla(), None), (par(heads=3, kv_heads=3, dim=5, rot_dims=4, vdim=2, scaling=False, width=9, blocks=3,
                                                              conv=5, left_scale=1.5, right_scale=0.4), None), (gla(heads=2, dim=12, vdim=9, tau=1.0), dense(31))],
                        loop=(1, 3, 2)),
    "aligned": config([(gla(heads=3, dim=16, vdim=24, tau=12.0), dense(72)),
                       (par(heads=8, kv_heads=1, dim=32, rot_dims=16, vdim=16, width=48, blocks=2, conv=4), dense(40)),
                       (par(heads=4, kv_heads=2, dim=16, rot_dims=16, vdim=32, width=64, blocks=1, conv=2, base=9000.0), None)],
                      width=64, groups=2, vocab=80, eps=1e-4, streams=2, loop=(0, 2, 3)),
    "ones": config([(par(heads=1, kv_heads=1, dim=2, rot_dims=2, vdim=2, width=1, blocks=1, conv=1), dense(1)), (gla(heads=1, dim=1, vdim=1, tau=1.0), dense(2)),
                    (par(heads=2, kv_heads=1, dim=3, rot_dims=2, vdim=4, width=4, blocks=4, conv=2), None)], width=7, groups=1, vocab=11, streams=1,
                   loop=(2, 3, 1)),
    "parallel_only": config([(par(heads=5, kv_heads=1, dim=6, rot_dims=6, vdim=8, conv=7), None), (par(heads=4, kv_heads=4, blocks=1), dense(17))],
                            streams=4, groups=1, loop=(0, 2, 2)),
    "gla_only": config([(gla(heads=5, tau=16.0), None), (gla(heads=4, dim=3, vdim=12, tau=0.5), dense(50))], vocab=37, streams=5, groups=2),
}


def weights(cfg, seed=0, dtype=torch.float32):
    """Random tensors under the checkpoint names, matrices scaled by their fan-in; decays from short to long memory."""
    g = torch.Generator().manual_seed(seed)
    n = lambda *s: torch.randn(*s, generator=g)
    mat = lambda o, i: n(o, i) * i ** -0.5
    V, D, S = cfg["vocab"], cfg["width"], cfg["streams"]
    w = {"embed": n(V, D), "head": mat(V, D), "final.norm": 1 + 0.2 * n(D)}
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer["mlp"]
        for q in (1, 2) if f else (1,):
            w.update({f"{p}norm{q}": 1 + 0.3 * n(D), f"{p}hc{q}.in": 0.5 + 0.5 * n(S), f"{p}hc{q}.out": 0.5 + 0.5 * n(S),
                      f"{p}hc{q}.mix": (0.8 * torch.eye(S) + 0.3 * n(S, S)) / (1 + 0.1 * S)})
        x = p + "mix."
        if layer["type"] == "parallel":
            a, r = m["left"], m["right"]
            H, G, W, nb = a["heads"], a["kv_heads"], r["width"], r["blocks"]
            for k, rows in (("q", H * a["dim"]), ("k", G * a["dim"]), ("v", G * a["vdim"])):
                w.update({f"{x}left.{k}": mat(rows, D), f"{x}left.{k}.b": n(rows)})
            w.update({x + "left.g": 2 * mat(H, D), x + "left.o": mat(D, H * a["vdim"]), x + "left.o.b": n(D)})
            for k in ("y", "x"):
                w.update({f"{x}right.{k}": mat(W, D), f"{x}right.{k}.b": n(W)})
            for k in ("ra", "ri"):
                w.update({f"{x}right.{k}": 2 * n(nb, W // nb, W // nb) * (W // nb) ** -0.5, f"{x}right.{k}.b": n(nb, W // nb)})
            w.update({x + "right.conv": n(W, r["conv"]) * r["conv"] ** -0.5, x + "right.conv.b": 0.5 * n(W), x + "right.lam": -3 + 2 * n(W),
                      x + "right.o": mat(D, W)})
        else:
            k, v = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            R = 4 + i                                       # the rank comes with the tensors
            w.update({x + "q": 2 * mat(k, D), x + "k": mat(k, D), x + "v": mat(v, D), x + "g": mat(v, D), x + "o": mat(D, v),
                      x + "norm": 1 + 0.3 * n(m["vdim"]), x + "a1": mat(R, D), x + "a2": 2 * mat(k, R), x + "a2.b": 1 + 2 * n(k)})
        if f:
            w.update({p + "mlp.up": 2 * mat(f["ff"], D), p + "mlp.down": mat(D, f["ff"]), p + "mlp.act": n(4)})
    return {k: v.to(dtype) for k, v in w.items()}


def tokens(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def engine(cfg, w, device="cpu", dtype=torch.float32, page_size=8, max_tokens=256, max_seqs=6, poison=True, **kw):
    """Step engine over a configuration; ``poison`` fills state and pages with large garbage that must never be read."""
    from jax_gpt_b200.models.munazen import MunazenConfig, MunazenEngine, load_from_state_dict
    c = MunazenConfig.from_dict(cfg, page_size=page_size)
    eng = MunazenEngine(load_from_state_dict(w, c, dtype, device), c, max_tokens=max_tokens, max_seqs=max_seqs, **kw)
    if poison:
        for t in eng.cache.states + [r for r in eng.cache.rings if r is not None] + list(eng.cache.paged.pool):
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
    assert len(want) == len(got) == len(O.layer_runs(cfg))
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
    from jax_gpt_b200.models.munazen import MunazenConfig, generate, load_from_state_dict
    cfg = CONFIGS["aligned"]
    w = weights(cfg, 7)
    c = MunazenConfig.from_dict(cfg, page_size=8)
    p = load_from_state_dict(w, c, torch.float32, device)
    prompts = [tokens(cfg, n, 70 + n) for n in (5, 1, 12)]
    out = generate(p, prompts, c, 30).tolist()
    for pr, cont in zip(prompts, out):
        lg = O.forward(pr + cont[:-1], cfg, w)[len(pr) - 1:]
        top = lg.max(-1).values - lg[torch.arange(30), torch.tensor(cont)]
        assert float(top.max()) < tol * float(lg.std())          # the greedy choice up to rounding ties
    again = generate(p, prompts, c, 6, temperature=0.8, top_k=5, key=3)
    assert torch.equal(again, generate(p, prompts, c, 6, temperature=0.8, top_k=5, key=3)) and again.shape == (3, 6)


def check_one_key_stands_out(device, tol, dtype=torch.float32, H=6, G=2, d=12, dv=10, rot_dims=8, n=75, ps=8):
    """Operands, cache rows, attention and the turn back of the output against the plain functions, with a query that matches one
    chosen key far above the rest: first positions, page borders, its own and distant places. A key that is lost, read from a wrong
    page or turned by a wrong angle changes the output wholly."""
    from jax_gpt_b200.cache.paged import PagedCache
    from jax_gpt_b200.ops import rotated_kv as RKV
    from jax_gpt_b200.ops.packed import PackedBatch, seq_begin
    from jax_gpt_b200.ops.rope import rope_tables
    g = torch.Generator().manual_seed(11)
    r = rot(rot_dims, 300.0)
    pages = (n + ps - 1) // ps
    cache = PagedCache(2, [5, G * (d + dv)], 5 * pages, ps, 4, pages + 2, dtype, device)
    for layer in range(2):
        cache.pool[layer].fill_(1e3)
    cache.reserve(3, 20)
    cache.reserve(1, n)
    cache.release(3)                     # the pages of sequence 1 do not start at page 0
    cache.reserve(2, 9)
    rope = rope_tables(rot_dims, r["base"], n + 9, r["scaling"], device)
    vrope = rope_tables(dv, r["base"], n + 9, None, device)
    gap = 8                              # columns between the parts, as alignment leaves them
    widths = (H * d, G * d, G * dv)
    cols = (gap, 2 * gap + widths[0], 3 * gap + widths[0] + widths[1])
    bias = 0.3 * torch.randn(sum(widths), generator=g)
    k = torch.randn(n, G, d, generator=g)
    k = k / k.norm(dim=-1, keepdim=True)
    v = torch.randn(n, G, dv, generator=g)
    gate = torch.randn(n, H, generator=g)
    freqs, amp = O.rotary_frequencies(r)
    vf = O.value_frequencies(r["base"], dv)
    rnd = lambda t: t.to(dtype).double()

    def rows(q, k, v):
        m = q.shape[0]
        y = torch.full((m, cols[2] + widths[2] + 3), 7e3)
        for c, t, b in zip(cols, (q, k, v), bias.split(widths)):
            y[:, c:c + b.numel()] = t.reshape(m, -1) - b
        return y.to(dtype).to(device)

    def batch(start, m):
        b = PackedBatch.make([1], [m], start == 0, n + 9, device)
        lens = torch.zeros(4, dtype=torch.int32)
        lens[1] = start
        seq_begin(b, torch.zeros(m, dtype=torch.int32, device=device), lens.to(device), torch.zeros(4, dtype=torch.int32, device=device))
        cache.seq_lens.zero_()
        cache.seq_lens[1] = start + m
        return b

    rope64 = lambda t, pos, f, a=1.0: O.turn_pairs(t.double(), pos, f, a)
    kt = rnd(rope64(k, range(n), freqs, amp))
    vt = rnd(rope64(v, range(n), vf))
    for qpos in sorted({0, 1, ps - 1, ps, 31, 32, 40, n - 1} & set(range(n))):
        near = {0, 1, 2, qpos, qpos - 1, qpos - 2, ps - 1, ps, 2 * ps - 1, 31, 32, 33, 63, 64}
        for target in sorted(j for j in near if 0 <= j <= qpos):
            for start in {0, qpos, max(0, qpos - 3)}:           # as part of a prompt, a decode step, a short portion
                m = qpos - start + 1
                if start:
                    b0 = batch(0, start)
                    RKV.qkv_rotate(b0, rows(torch.zeros(start, H, d), k[:start], v[:start]), cols, bias.to(device), H, G, d, dv, rope, vrope, cache, 1, None)
                q = torch.zeros(m, H, d)
                want_q = rope64(k[target:target + 1], [target], freqs, amp) * 60       # turned key; the query before its own turn:
                q[-1] = (O.turn_pairs(want_q, [-qpos], freqs, 1 / amp)).repeat_interleave(H // G, 1)[0].float()
                b = batch(start, m)
                wide = RKV.flash_widths(b, dtype, device != "cpu", d, dv)
                qo, ko, vo = RKV.qkv_rotate(b, rows(q, k[start:qpos + 1], v[start:qpos + 1]), cols, bias.to(device), H, G, d, dv, rope, vrope,
                                            cache, 1, wide)
                o = RKV.causal_attention(b, qo, ko, vo, cache, 1, G, dv, 0.5)
                out = torch.zeros(m, H * dv + 5, dtype=dtype, device=device)
                RKV.turn_back_gate(b, o, gate[start:qpos + 1].to(dtype).to(device), vrope, 0.7, out[:, :H * dv])
                qt = rnd(O.turn_pairs(q[-1:].double(), [qpos], freqs, amp))
                w = O.masked_softmax_attention(qt, kt[:qpos + 1], vt[:qpos + 1], torch.ones(1, qpos + 1, dtype=torch.bool), 0.5)
                w = O.turn_pairs(w, [-qpos], vf) * 0.7 * O.sigmoid(rnd(gate[qpos:qpos + 1]))[:, :, None]
                got = out[-1, :H * dv].double().cpu().reshape(1, H, dv)
                assert float((got - w).abs().max()) < tol, (target, qpos, start)
                assert float(out[:, H * dv:].abs().max()) == 0


def check_far_tokens(device, tol):
    """In the whole model: queries and keys made so that a repeated token finds its first occurrence across a long distance; changing
    what follows that place changes the late logits, far above the tolerance, in prompts, portions and decoding."""
    cfg = config([(par(heads=2, kv_heads=1, dim=8, rot_dims=2, vdim=6, scale=1.0, base=1e5, left_scale=3.0, right_scale=0.1), None)], width=24,
                 groups=1, streams=1)
    w = weights(cfg, 12)
    w["l0.mix.left.k"] = w["l0.mix.left.q"][:8] * 1.0           # matching tokens score highest
    w["l0.mix.left.q"] = torch.cat([w["l0.mix.left.k"]] * 2) * 3
    for b in ("q", "k"):
        w[f"l0.mix.left.{b}.b"] *= 0
    toks = [t % (cfg["vocab"] - 1) for t in tokens(cfg, 90, 13)]
    rare = cfg["vocab"] - 1
    for at in (0, 1, 7, 8, 31, 32):
        this = toks[:at] + [rare] + toks[at + 1:-1] + [rare]
        want = O.forward(this, cfg, w)
        other = this[:at] + [toks[-2]] + this[at + 1:]
        plain = O.forward(other, cfg, w)
        assert error(plain[-1:], want[-1:]) > 100 * tol, at
        eng = engine(cfg, w, device)
        for name, cuts in (("a", [90]), ("b", [60] + [1] * 30), ("c", [2] * 45)):
            assert error(run(eng, name, this, cuts), want) < tol, (at, name)
            assert error(run(eng, name + "o", other, cuts), plain) < tol, (at, name)
            eng.release(name)
            eng.release(name + "o")


def check_state_carries(device, tol):
    """Slow decays: a token of the first portion still shows a hundred positions later, far above the tolerance, and the framework
    follows it through prompts cut at odd places."""
    for layer in (par(heads=1, kv_heads=1, dim=2, rot_dims=2, vdim=2, width=16, blocks=2, conv=4, left_scale=0.0), gla(heads=2, dim=8, vdim=8, tau=50.0)):
        cfg = config([(layer, None)], width=24, groups=2, streams=2)
        w = weights(cfg, 16)
        if layer["type"] == "parallel":
            w["l0.mix.right.lam"].fill_(-9.0)
        else:
            w["l0.mix.a2.b"].fill_(6.0)
        toks = tokens(cfg, 150, 17)
        want = O.forward(toks, cfg, w)
        eng = engine(cfg, w, device)
        assert error(run(eng, "a", toks, [5, 2, 64, 1, 1, 57, 20]), want) < tol
        other = O.forward(toks[:1] + [(toks[1] + 1) % cfg["vocab"]] + toks[2:], cfg, w)
        assert error(other[100:], want[100:]) > 10 * tol


def check_long_decode(device, tol):
    """A short prompt and a few hundred decode steps over slow decays (state) and many pages (attention)."""
    cfg = CONFIGS["aligned"]
    w = weights(cfg, 14)
    w["l1.mix.right.lam"].fill_(-8.0)
    w["l0.mix.a2.b"].fill_(5.0)
    toks = tokens(cfg, 230, 15)
    want = O.forward(toks, cfg, w)
    eng = engine(cfg, w, device, max_tokens=240)
    assert error(run(eng, "a", toks, [3] + [1] * 227), want) < tol


def check_loop_passes_keep_their_own_state(device, tol):
    """A looped layer against the same layers written out with copied weights; and the passes must not share caches: decoding after a
    prompt gives what the whole prompt gives."""
    cfg = config([(par(), dense()), (gla(), None), (par(heads=2, kv_heads=1), dense(9))], loop=(0, 2, 3))
    w = weights(cfg, 18)
    flat = config([(cfg["layers"][i], cfg["layers"][i]["mlp"]) for i in (0, 1, 0, 1, 0, 1, 2)])
    wf = {k: v for k, v in w.items() if not k.startswith("l")}
    for j, i in enumerate((0, 1, 0, 1, 0, 1, 2)):
        wf.update({f"l{j}." + k.split(".", 1)[1]: v for k, v in w.items() if k.startswith(f"l{i}.")})
    toks = tokens(cfg, 33, 19)
    got = run(engine(cfg, w, device), "a", toks, [20] + [1] * 13)
    assert error(got, O.forward(toks, flat, wf)) < tol
    assert error(run(engine(flat, wf, device), "a", toks, [20] + [1] * 13), got) < tol
