"""Small Mopalorn configurations and random weights for the tests (the dictionaries of a ``config.json``, tensors by checkpoint name),
and the comparisons that the CPU and the GPU tests share."""
import math

import torch

import mopalorn_oracle as O


def latent(heads=3, dim=7, rot_dim=6, vdim=5, kv_rank=11, size=10, scale=0.45, base=600.0):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
                                                  "mask": {"size": size}, "rot": {"base": base, "dims": rot_dim}}}


def full(heads=6, kv_heads=2, dim=9, vdim=5, scale=0.5, softcap=4.0, coef=0.6, every=5, v_mix=True):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": softcap,
                                           "q_temp": {"coef": coef, "every": every}, "v_mix": v_mix}}


def pooled(heads=4, kv_heads=2, dim=7, vdim=5, scale=0.6, size=9, pool=4, v_mix=True):
    return {"type": "attention_2", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                                             "mask": {"size": size, "pool": pool}, "v_mix": v_mix}}


def dense(ff=23):
    return {"kind": "dense", "ff": ff}


def config(layers, vocab=61, width=30, eps=1e-5, logit_scale=0.3):
    return {"architecture": "Mopalorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale,
            "layers": [dict(l, mlp=m) for l, m in layers]}


# every branch of the design, in several orders and sizes (odd widths take the kernels' scalar paths)
CONFIGS = {
    "mixed_odd": config([(pooled(), dense()), (latent(), None), (full(), dense(31)), (pooled(heads=2, kv_heads=1, dim=3, vdim=10, size=3, pool=7), None),
                         (latent(heads=1, dim=4, rot_dim=2, vdim=3, kv_rank=5, size=25), dense(9))]),
    "aligned": config([(latent(heads=4, dim=16, rot_dim=8, vdim=16, kv_rank=24, size=17), dense(72)), (full(heads=8, kv_heads=1, dim=32, vdim=16), dense(40)),
                       (pooled(heads=4, kv_heads=2, dim=16, vdim=8, size=16, pool=8), None), (full(heads=2, kv_heads=2, dim=8, vdim=8, every=16), dense(64))],
                      width=64, vocab=80, eps=1e-4, logit_scale=1.7),
    "ones": config([(full(heads=1, kv_heads=1, dim=1, vdim=1, every=1, softcap=1.0), dense(1)), (pooled(heads=1, kv_heads=1, dim=1, vdim=1, size=1, pool=1), None),
                    (latent(heads=1, dim=1, rot_dim=2, vdim=1, kv_rank=1, size=1), dense(2))], width=7, vocab=11, logit_scale=1.0),
    "latent_only": config([(latent(heads=5, size=200), None), (latent(size=8), dense(17)), (latent(size=1), dense(8))]),
    "grouped_only": config([(full(v_mix=False), dense(19)), (pooled(size=8, pool=8, vdim=6), None), (pooled(kv_heads=4, vdim=3, size=12, pool=11), dense(13)),
                            (full(heads=3, kv_heads=1, vdim=12, softcap=30.0, every=1000), None), (pooled(v_mix=False, size=40, pool=3), None)]),
    "blocks_beyond_pages": config([(pooled(heads=2, kv_heads=2, size=2, pool=19), None), (pooled(heads=2, kv_heads=2, size=5, pool=1), dense())]),
}


def weights(cfg, seed=0, dtype=torch.float32):
    """Random tensors under the checkpoint names, matrices scaled by their fan-in."""
    g = torch.Generator().manual_seed(seed)
    n = lambda *s: torch.randn(*s, generator=g)
    mat = lambda o, i: n(o, i) * i ** -0.5
    V, D = cfg["vocab"], cfg["width"]
    w = {"embed": n(V, D), "final.norm": 1 + 0.2 * n(D)}
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer["mlp"]
        for name in ("norm1", "norm1b") + (("norm2", "norm2b") if f else ()):
            w[p + name] = 1 + 0.3 * n(D)
        x, H = p + "mix.", m["heads"]
        w[x + "o"] = mat(D, H * m["vdim"])
        if layer["type"] == "latent_attention":
            R = m["kv_rank"]
            w.update({x + "q": 2 * mat(H * (m["dim"] + m["rot_dim"]), D), x + "dkv": mat(R + m["rot_dim"], D), x + "dkv.norm": 1 + 0.3 * n(R),
                      x + "uk": mat(H * m["dim"], R), x + "uv": mat(H * m["vdim"], R), x + "g": 2 * mat(H * m["vdim"], D)})
        else:
            G = m["kv_heads"]
            w.update({x + "q": 2 * mat(H * m["dim"], D), x + "k": mat(G * m["dim"], D), x + "v": mat(G * m["vdim"], D)})
            if m["v_mix"]:
                w[x + "vmix"] = 0.6 + 0.5 * n(1)[0]
            if layer["type"] == "attention_2":
                w[x + "sink"] = 1.5 * n(H)
        if f:
            w.update({p + "mlp.up": 2 * mat(f["ff"], D), p + "mlp.down": mat(D, f["ff"]), p + "mlp.act": n(2)})
    return {k: v.to(dtype) for k, v in w.items()}


def tokens(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def engine(cfg, w, device="cpu", dtype=torch.float32, page_size=8, max_tokens=256, max_seqs=6, poison=True, **kw):
    """Step engine over a configuration; ``poison`` fills rows and block means with large garbage that must never be read."""
    from jax_gpt_b200.models.mopalorn import MopalornConfig, MopalornEngine, load_from_state_dict
    c = MopalornConfig.from_dict(cfg, page_size=page_size)
    eng = MopalornEngine(load_from_state_dict(w, c, dtype, device), c, max_tokens=max_tokens, max_seqs=max_seqs, **kw)
    if poison:
        for t in list(eng.cache.paged.pool) + [p for p in eng.cache.paged.pooled if p is not None]:
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
    assert len(want) == len(got) == len(cfg["layers"])
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
    """Greedy continuation through the package's entry point against the plain forward pass, past page and window borders."""
    from jax_gpt_b200.models.mopalorn import MopalornConfig, generate, load_from_state_dict
    cfg = CONFIGS["aligned"]
    w = weights(cfg, 7)
    c = MopalornConfig.from_dict(cfg, page_size=8)
    p = load_from_state_dict(w, c, torch.float32, device)
    prompts = [tokens(cfg, n, 70 + n) for n in (5, 1, 12)]
    out = generate(p, prompts, c, 30).tolist()
    for pr, cont in zip(prompts, out):
        lg = O.forward(pr + cont[:-1], cfg, w)[len(pr) - 1:]
        top = lg.max(-1).values - lg[torch.arange(30), torch.tensor(cont)]
        assert float(top.max()) < tol * float(lg.std())          # the greedy choice up to rounding ties
    again = generate(p, prompts, c, 6, temperature=0.8, top_k=5, key=3)
    assert torch.equal(again, generate(p, prompts, c, 6, temperature=0.8, top_k=5, key=3)) and again.shape == (3, 6)


def check_long_decode(device, tol):
    """A short prompt and a few hundred decode steps over many pages, windows and blocks."""
    cfg = CONFIGS["aligned"]
    w = weights(cfg, 14)
    toks = tokens(cfg, 230, 15)
    want = O.forward(toks, cfg, w)
    eng = engine(cfg, w, device, max_tokens=240)
    assert error(run(eng, "a", toks, [3] + [1] * 227), want) < tol


def begin(cache, slot, start, m, n_pos, device):
    """A packed batch with m tokens of one sequence from ``start`` on; the cache's lengths include them, as within a step."""
    from jax_gpt_b200.ops.packed import PackedBatch, seq_begin
    b = PackedBatch.make([slot], [m], start == 0, n_pos, device)
    slots = cache.seq_lens.numel()
    lens = torch.zeros(slots, dtype=torch.int32)
    lens[slot] = start
    seq_begin(b, torch.zeros(m, dtype=torch.int32, device=device), lens.to(device), torch.zeros(slots, dtype=torch.int32, device=device))
    cache.seq_lens.zero_()
    cache.seq_lens[slot] = start + m
    return b


def scattered_cache(widths, n, ps, dtype, device, blocks=()):
    """A cache whose sequence 1 holds n positions in pages that are neither first nor in order, full of garbage."""
    from jax_gpt_b200.cache.paged import PagedCache
    pages = (n + ps - 1) // ps
    cache = PagedCache(len(widths), widths, 5 * pages + 4, ps, 4, pages + 2, dtype, device, blocks=blocks)
    for t in list(cache.pool) + [p for p in cache.pooled if p is not None]:
        t.fill_(1e3)
    cache.reserve(3, 2 * ps)
    cache.reserve(1, min(n, ps))
    cache.release(3)
    cache.reserve(2, 1)
    cache.reserve(1, n)
    return cache


def edges(qpos, size, P, ps):
    """Key positions worth asking for from ``qpos``: both sides of the window's edge, of a block that is just seen, page borders."""
    out = qpos - size                                          # the last token outside the window
    last = (max(0, out + 1) // P) * P                          # the first token of no seen block
    at = {0, 1, out - 1, out, out + 1, out + 2, last - P - 1, last - P, last - 1, last, last + 1, qpos - 1, qpos, ps - 1, ps, 31, 32, 63, 64, 127, 128}
    return sorted(j for j in at if 0 <= j <= qpos)


def grouped_reference(q, k, v, qpos, scale, size=None, P=0, softcap=0.0, sink=None, hide=None, rnd=lambda t: t):
    """Output (H, dv) of one query (H, d) at qpos over keys (T, H, d): tokens, or tokens in a window and the blocks before it. ``hide`` =
    ("token" | "block", index) flips what the query sees there. ``rnd`` rounds the means as the cache does."""
    T = k.shape[0]
    seen = O.seen_tokens(T, size)[qpos]
    if P:
        k, v = torch.cat([k, rnd(O.block_means(k, P))]), torch.cat([v, rnd(O.block_means(v, P))])
        seen = torch.cat([seen, O.seen_blocks(T, P, size)[qpos]])
    if hide:
        i = hide[1] + (T if hide[0] == "block" else 0)
        seen = seen.clone()
        seen[i] = ~seen[i]
    s = torch.einsum("hd,jhd->hj", q, k) * scale
    s = O.cap(s, softcap) if softcap else s
    a = O.weights_of(s, seen[None], sink[:, None] if sink is not None else None)
    return torch.einsum("hj,jhd->hd", a, v)


def check_one_key_stands_out(device, tol, dtype=torch.float32, H=6, G=2, d=12, dv=10, n=75, ps=8,
                             masks=((20, 5), (9, 8), (8, 16), (1, 1), (3, 11), (40, 1), (30, 25), (64, 4)), softcap=0.0):
    """Operands, cache rows, block means and attention against the plain functions, with a query that matches one chosen key and its block
    far above the rest: both sides of the window's edge, blocks that are just seen or not yet, page borders, first positions. Flipping what
    the query sees at that place changes the expected output by far more than the tolerance."""
    from jax_gpt_b200.ops import window_attention as WA
    from jax_gpt_b200.ops.mixed_kv import mixed_kv, query_factors
    g = torch.Generator().manual_seed(11)
    gap = 8
    widths = (H * d, G * d, G * dv)
    cols = (gap, 2 * gap + (widths[0] + 7) // 8 * 8, 3 * gap + sum((x + 7) // 8 * 8 for x in widths[:2]))
    rnd = lambda t: t.to(dtype).double()
    factors, lam = query_factors(0.5, 7, n + 9, device), 0.7
    vf = torch.randn(n, G * dv, generator=g).to(dtype)
    sink = torch.randn(H, generator=g)
    of = torch.arange(H) // (H // G)

    def rows(q, k, v):
        m = q.shape[0]
        y = torch.full((m, cols[2] + (widths[2] + 7) // 8 * 8), 7e3)
        for c, t in zip(cols, (q, k, v)):
            y[:, c:c + t[0].numel()] = t.reshape(m, -1)
        return y.to(dtype).to(device)

    for size, P in masks:
        window = size or WA.NO_WINDOW
        dirs = torch.randn(n // max(P, 1) + 1, G, d, generator=g)
        k = dirs[torch.arange(n) // max(P, 1)] + 0.5 * torch.randn(n, G, d, generator=g)
        k = k / k.norm(dim=-1, keepdim=True)
        v = torch.randn(n, G, dv, generator=g)
        kt, vt = rnd(k), rnd(O.mixed_values(rnd(v), rnd(vf).reshape(n, G, dv), lam))
        cache = scattered_cache([5, G * (d + dv)], n, ps, dtype, device, blocks=[0, P])
        for qpos in sorted({0, size - 1, size, size + P - 1, size + P, size + 2 * P, 31, 32, 40, n - 2, n - 1} & set(range(n))):
            for target in edges(qpos, size or n, max(P, 1), ps):
                q = torch.zeros(n, H, d)
                q[qpos] = (25.0 * k[target])[of]
                f = O.query_factor(qpos, 0.5, 7)
                qt = rnd(rnd(q[qpos]) * f)
                ref = lambda **kw: grouped_reference(qt, kt[:qpos + 1][:, of], vt[:qpos + 1][:, of], qpos, 0.5, size or None, P, softcap, sink.double(), rnd=rnd, **kw)
                want = ref()
                flips = [("token", target)] if target < qpos and P != 1 else []     # blocks of one token are that token
                if P > 1 and qpos - target >= size and target // P < (qpos + 1) // P:
                    flips.append(("block", target // P))
                for hide in flips:
                    # (tokens of the block that are still in the window take most of the weight: there only fp32 shows it)
                    beside = hide[0] == "block" and qpos - (target // P * P + P - 1) < size
                    if not (beside and dtype == torch.bfloat16):
                        assert float((ref(hide=hide) - want).abs().max()) > 3 * tol, ("the case does not show", size, P, qpos, target, hide)
                for start in sorted({0, qpos, max(0, qpos - 3)}):           # as part of a prompt, a decode step, a short portion
                    put = lambda a, b: mixed_kv(begin(cache, 1, a, b - a, n + 9, device), rows(q[a:b], k[a:b], v[a:b]), cols, H, G, d, dv, cache, 1,
                                                None, factors, vf[a:b].to(device), lam, window)
                    if start:
                        put(0, start)
                    b = begin(cache, 1, start, qpos + 1 - start, n + 9, device)
                    wide = WA.flash_widths(b, dtype, device != "cpu", d, dv)
                    qo, ko, vo = mixed_kv(b, rows(q[start:qpos + 1], k[start:qpos + 1], v[start:qpos + 1]), cols, H, G, d, dv, cache, 1, wide,
                                          factors, vf[start:qpos + 1].to(device), lam, window)
                    o = WA.grouped_attention(b, qo, ko, vo, cache, 1, G, dv, 0.5, window, softcap=softcap, sink=sink.to(device), pool=P)
                    got = o[-1, :, :dv].double().cpu()
                    assert float((got - want).abs().max()) < tol, (size, P, qpos, target, start)


def check_one_latent_stands_out(device, tol, dtype=torch.float32, H=5, dn=6, dr=4, dv=7, R=9, n=75, ps=8, sizes=(20, 8, 1, 33, 75)):
    """Latent attention over a window with an output gate: a query that matches one chosen key far above the rest, on both sides of the
    window's edge, at page borders and at first positions; as part of a prompt, a decode step and a short portion."""
    from jax_gpt_b200.ops import latent_attention as LA
    from jax_gpt_b200.ops.rope import rope_tables
    g = torch.Generator().manual_seed(12)
    base, eps, scale = 300.0, 1e-4, 0.5
    rep = 13.0 / (scale * (4 * dn ** 0.5 + dr))                 # the matching key scores about 13
    pairs = torch.tensor([x for i in range(dr // 2) for x in (i, i + dr // 2)])    # the kernels turn neighbours
    rnd = lambda t: t.to(dtype).double()
    y = torch.randn(n, R + dr, generator=g)
    gamma = 1 + 0.3 * torch.randn(R, generator=g)
    w_uk, w_uv = torch.randn(H * dn, R, generator=g) * R ** -0.5, torch.randn(H * dv, R, generator=g) * R ** -0.5
    gate = torch.randn(n, H * dv, generator=g).to(dtype)
    w = torch.cat([w_uk, w_uv]).to(dtype)
    c = O.rms(rnd(y)[:, :R], eps) * gamma.double()
    kn, kr = (rnd(c) @ rnd(w_uk).T).reshape(n, H, dn), O.turn_halves(rnd(y)[:, R:], base)
    vals = (rnd(c) @ rnd(w_uv).T).reshape(n, H, dv)
    rope = rope_tables(dr, base, n + 9, None, device)
    yk = torch.cat([y[:, :R], y[:, R:][:, pairs]], 1)
    cache = scattered_cache([5, R + dr], n, ps, dtype, device)
    for size in sizes:
        for qpos in sorted({0, size - 1, size, size + 1, 31, 32, 40, n - 1} & set(range(n))):
            for target in edges(qpos, size, 16, ps):
                q = torch.zeros(n, H, dn + dr, dtype=torch.float64)
                q[qpos, :, :dn] = rep * kn[target] / kn[target].norm(dim=-1, keepdim=True) * 4
                q[qpos, :, dn:] = rep * O.turn_halves(rnd(y)[target:target + 1, R:], base, [target - qpos])
                qt = rnd(q[qpos].float())
                qr = O.turn_halves(qt[None, :, dn:], base, [qpos])[0]
                s = (torch.einsum("hd,jhd->hj", qt[:, :dn], kn[:qpos + 1]) + torch.einsum("hd,jd->hj", qr, kr[:qpos + 1])) * scale
                seen = O.seen_tokens(qpos + 1, size)[qpos][None]
                out = lambda m: torch.einsum("hj,jhd->hd", O.weights_of(s, m), vals[:qpos + 1]) * torch.sigmoid(rnd(gate[qpos]).reshape(H, dv))
                want = out(seen)
                if 0 <= target < qpos:
                    other = seen.clone()
                    other[:, target] = ~other[:, target]
                    assert float((out(other) - want).abs().max()) > 3 * tol, ("the case does not show", size, qpos, target)
                turned = torch.cat([q[..., :dn], q[..., dn:][..., pairs]], -1).to(dtype)
                for start in sorted({0, qpos, max(0, qpos - 3)}):
                    def part(a, b, attend):
                        bt = begin(cache, 1, a, b - a, n + 9, device)
                        flash = attend and LA.flash_ok(bt, yk.to(dtype).to(device), dn, dr, dv, R)
                        wide = torch.full((b - a, 8 + R + dr + 8), 5e3)
                        wide[:, 8:8 + R + dr] = yk[a:b]
                        _, lat = LA.mla_prepare(bt, wide.to(dtype).to(device)[:, 8:8 + R + dr], None, gamma.to(device), eps, rope, cache, 1, flash)
                        if not attend:
                            return None
                        row = torch.zeros(b - a, H * (dn + dr) + 8, dtype=dtype)
                        row[:, :H * (dn + dr)] = turned[a:b].reshape(b - a, -1)
                        qv = row.to(device)[:, :H * (dn + dr)].unflatten(-1, (H, dn + dr))
                        return LA.attend(bt, qv, lat, w.to(device), R, dv, rope, cache, 1, scale, window=size, gate=gate[a:b].to(device))
                    if start:
                        part(0, start, False)
                    got = part(start, qpos + 1, True)[-1].double().cpu().reshape(H, dv)
                    assert float((got - want).abs().max()) < tol, (size, qpos, target, start)


def check_far_tokens(device, tol):
    """In the whole model: query weights made so that one token asks for another one (or for the block that repeats it) across a long
    distance; changing what stands there changes the late logits, far above the tolerance, in prompts, portions and decoding."""
    for layer, run_len, places in ((full(heads=2, kv_heads=1, dim=8, vdim=6, scale=1.0, softcap=40.0), 1, (0, 1, 7, 8, 31, 32)),
                                   (pooled(heads=2, kv_heads=1, dim=8, vdim=6, scale=1.0, size=11, pool=5), 5, (0, 5, 30, 70))):
        cfg = config([(layer, None)], width=24)
        w = weights(cfg, 12)
        asks, rare = cfg["vocab"] - 2, cfg["vocab"] - 1
        h = (O.rms(w["embed"].double(), 1e-5) * w["l0.norm1"].double()).float()
        want_q = 3 * (w["l0.mix.k"] @ h[rare])
        w["l0.mix.q"] = torch.cat([torch.outer(want_q, h[asks]) / h[asks].square().sum()] * 2)
        toks = [t % asks for t in tokens(cfg, 90, 13)]
        for at in places:
            this = toks[:at] + [rare] * run_len + toks[at + run_len:-1] + [asks]
            want = O.forward(this, cfg, w)
            other = this[:at] + toks[at:at + run_len] + this[at + run_len:]
            plain = O.forward(other, cfg, w)
            assert error(plain[-1:], want[-1:]) > 50 * tol, (layer["type"], at)
            eng = engine(cfg, w, device)
            for name, seq, expect, cuts in (("a", this, want, [90]), ("b", this, want, [60] + [1] * 30), ("c", this, want, [2] * 45), ("d", other, plain, [72, 18])):
                assert error(run(eng, name, seq, cuts), expect) < tol, (at, name)
                eng.release(name)


def check_block_means(device, dtype, tol, P, ps, G=2, d=6, dv=4):
    """Means beside the pages are those of the cached rows, however the tokens came in."""
    from jax_gpt_b200.ops.mixed_kv import mixed_kv
    n = 60
    g = torch.Generator().manual_seed(P)
    y = torch.randn(n, G * (2 * d + dv), generator=g).to(dtype)
    for cuts in ([60], [1] * 60, [7, 1, 30, 2, 20]):
        cache = scattered_cache([G * (d + dv)], n, ps, dtype, device, blocks=[P])
        at = 0
        for m in cuts:
            mixed_kv(begin(cache, 1, at, m, n, device), y[at:at + m].to(device), (0, G * d, 2 * G * d), G, G, d, dv, cache, 0)
            at += m
            whole = at // P
            rows = cache.gather(0, 1, at).double().cpu()
            assert torch.equal(rows, y[:at, G * d:].double())
            if whole:
                got = cache.gather_pooled(0, 1, whole).double().cpu()
                assert float((got - O.block_means(rows, P)).abs().max()) < tol, (P, ps, at)


def check_activation(linear, device, dtype, tol, sizes):
    """The up projection's activation against the plain function, positive, negative, tiny and large inputs."""
    g = torch.Generator().manual_seed(5)
    p, q = 0.7, -1.2
    sp = lambda t: math.log1p(math.exp(t))
    for M, K, N in sizes:
        x, w = torch.randn(M, K, generator=g).to(dtype), (3 * torch.randn(N, K, generator=g) * K ** -0.5).to(dtype)
        w[0] *= 1e-4
        want = O.xielu(x.double() @ w.double().T, p, q)
        got = linear(x.to(device), w.to(device), act="xielu", act_args=(sp(p), 0.5 + sp(q))).double().cpu()
        assert float(((got - want).abs() / (1e-6 + want.abs() + (x.double().abs() @ w.double().abs().T) * 1e-2)).max()) < tol, (M, K, N)
