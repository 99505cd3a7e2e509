"""Munazen checkpoint names -> parameter tree, and random trees.

Linear weights stay (out, in) as stored. Projections that share an input are one matrix whose parts start at multiples of 8 rows (zero
rows between); the two output projections of a parallel layer are one matrix over [heads | recurrent channels], its bias scaled by
``left_scale``. Norm gains, biases, connections, convolutions and decays are kept in fp32, matrices and embeddings in the serving
dtype::

    embed (V, D)  final_norm (D)  head (V, D)  ones (streams)
    layers[i].norm1 [, norm2], hc1 [, hc2]: Connection
    layers[i].mix   parallel: in ([q | k | v | x | y | g], D)  qkv_b  lru: LruWeights  o (D, H vdim + W)  o_b (D)
                    gla:      in ([q | k | v | g | a1], D)  a2 (H dim, rank)  a2_b (H dim)  norm (H vdim)  o (D, H vdim)
    layers[i].mlp   up (ff, D)  down (D, ff)  act (4)
"""
from __future__ import annotations

import torch

from ...ops.gated_lru import LruWeights, lru_decay
from ...ops.streams import Connection
from .config import LRU_RATE, MunazenConfig, Parallel


def expected_shapes(c: MunazenConfig) -> dict:
    """Checkpoint tensor names and shapes of a configuration; the rank of the decay projection is ``c.decay_rank`` here and
    whatever the tensors have when loading."""
    D, V, S, R = c.width, c.vocab_size, c.streams, c.decay_rank
    s = {"embed": (V, D), "head": (V, D), "final.norm": (D,)}
    for i, layer in enumerate(c.layers):
        p, m, f = f"l{i}.", layer.mixer, layer.mlp
        for q in (1, 2) if f else (1,):
            s.update({f"{p}norm{q}": (D,), f"{p}hc{q}.in": (S,), f"{p}hc{q}.out": (S,), f"{p}hc{q}.mix": (S, S)})
        x = p + "mix."
        if isinstance(m, Parallel):
            a, r = m.left, m.right
            q, k, v, W, wb = a.heads * a.dim, a.kv_heads * a.dim, a.kv_heads * a.vdim, r.width, r.width // r.blocks
            o = a.heads * a.vdim
            for n, w in (("q", q), ("k", k), ("v", v)):
                s.update({f"{x}left.{n}": (w, D), f"{x}left.{n}.b": (w,)})
            s.update({x + "left.g": (a.heads, D), x + "left.o": (D, o), x + "left.o.b": (D,)})
            for n in ("y", "x"):
                s.update({f"{x}right.{n}": (W, D), f"{x}right.{n}.b": (W,)})
            s.update({x + "right.conv": (W, r.conv), x + "right.conv.b": (W,), x + "right.lam": (W,), x + "right.o": (D, W)})
            for n in ("ra", "ri"):
                s.update({f"{x}right.{n}": (r.blocks, wb, wb), f"{x}right.{n}.b": (r.blocks, wb)})
        else:
            k, v = m.heads * m.dim, m.heads * m.vdim
            s.update({x + "q": (k, D), x + "k": (k, D), x + "v": (v, D), x + "g": (v, D), x + "o": (D, v), x + "norm": (m.vdim,),
                      x + "a1": (R, D), x + "a2": (k, R), x + "a2.b": (k,)})
        if f:
            s.update({p + "mlp.up": (f.ff, D), p + "mlp.down": (D, f.ff), p + "mlp.act": (4,)})
    return s


def load_from_state_dict(sd, config: MunazenConfig, dtype=torch.bfloat16, device="cpu") -> dict:
    """``sd``: mapping of checkpoint names to tensors (lazy mappings work: each key is read once)."""
    c = config
    shapes = expected_shapes(c)
    missing = [k for k in shapes if k not in sd]
    if missing:
        raise KeyError(f"checkpoint lacks {len(missing)} tensor(s), e.g. {missing[:4]}")

    def raw(k, shape=None):
        t, want = sd[k], shape or shapes[k]
        if len(t.shape) != len(want) or any(w is not None and n != w for n, w in zip(t.shape, want)):
            raise ValueError(f"{k}: shape {tuple(t.shape)}, the configuration says {want}")
        return t.detach()
    cast = lambda t: t.to(device=device, dtype=dtype).contiguous()
    mat = lambda k: cast(raw(k))
    vec = lambda *ks: torch.cat([raw(k).to(device=device, dtype=torch.float32).reshape(-1) for k in ks]).contiguous()
    f32 = lambda k: raw(k).to(device=device, dtype=torch.float32).contiguous()

    def rows(*mats):
        """Matrices over one input below each other, each padded with zero rows to a multiple of 8."""
        return torch.cat([torch.nn.functional.pad(t, (0, 0, 0, -t.shape[0] % 8)) for t in mats]).contiguous()

    layers = []
    for i, layer in enumerate(c.layers):
        p, m = f"l{i}.", layer.mixer
        x = p + "mix."
        lp = {}
        for q in (1, 2) if layer.mlp else (1,):
            lp[f"norm{q}"] = vec(f"{p}norm{q}")
            lp[f"hc{q}"] = Connection(vec(f"{p}hc{q}.in"), f32(f"{p}hc{q}.mix"), vec(f"{p}hc{q}.out"))
        if isinstance(m, Parallel):
            l, r = x + "left.", x + "right."
            lru = LruWeights(x_bias=vec(r + "x.b"), y_bias=vec(r + "y.b"), conv=f32(r + "conv"), conv_bias=vec(r + "conv.b"),
                             gates=torch.stack([mat(r + "ra"), mat(r + "ri")], 1).contiguous(),
                             gates_bias=torch.stack([f32(r + "ra.b"), f32(r + "ri.b")], 1).contiguous(),
                             decay=lru_decay(vec(r + "lam"), LRU_RATE))
            lp["mix"] = {"in": rows(mat(l + "q"), mat(l + "k"), mat(l + "v"), mat(r + "x"), mat(r + "y"), mat(l + "g")),
                         "qkv_b": vec(l + "q.b", l + "k.b", l + "v.b"), "lru": lru,
                         "o": torch.cat([mat(l + "o"), mat(r + "o")], 1).contiguous(), "o_b": m.left_scale * vec(l + "o.b")}
        else:
            a1 = cast(raw(x + "a1", (None, c.width)))
            lp["mix"] = {"in": rows(torch.cat([mat(x + n) for n in "qkv"]), mat(x + "g"), a1),
                         "a2": cast(raw(x + "a2", (m.heads * m.dim, a1.shape[0]))), "a2_b": vec(x + "a2.b"),
                         "norm": vec(x + "norm").repeat(m.heads), "o": mat(x + "o")}
        if layer.mlp is not None:
            lp["mlp"] = {"up": mat(p + "mlp.up"), "down": mat(p + "mlp.down"), "act": vec(p + "mlp.act")}
        layers.append(lp)
    return {"embed": mat("embed"), "layers": layers, "final_norm": vec("final.norm"), "head": mat("head"),
            "ones": torch.ones(c.streams, dtype=torch.float32, device=device)}


def random_state_dict(config: MunazenConfig, seed: int = 0, dtype=torch.float32, device="cpu") -> dict:
    """Random checkpoint of a configuration: matrices N(0, 1 / fan_in), gains near one, decays of the recurrent units between 0.9 and
    0.999 at an open gate, streams near a plain residual sum."""
    g = torch.Generator(device=device).manual_seed(seed)
    n = lambda *s: torch.randn(*s, generator=g, device=device)
    sd = {}
    for k, s in expected_shapes(config).items():
        leaf = k.rsplit(".", 1)[-1]
        if leaf.startswith("norm"):
            t = 1.0 + 0.1 * n(*s)
        elif leaf == "lam":
            a = 0.9 + 0.099 * torch.rand(*s, generator=g, device=device)
            t = torch.log(torch.expm1(-torch.log(a) / LRU_RATE))
        elif leaf == "mix":
            t = torch.eye(s[0], device=device) + 0.1 * n(*s)
        elif leaf in ("in", "out") and ".hc" in k:
            t = 1.0 / s[0] + 0.1 * n(*s)
        elif leaf == "act":
            t = torch.tensor([0.6, 0.3, 0.3, 0.0], device=device) + 0.1 * n(*s)
        elif leaf == "b":
            t = 0.1 * n(*s) + (2.0 if k.endswith("a2.b") else 0.0)
        elif k == "embed":
            t = n(*s)
        else:
            t = n(*s) * s[-1] ** -0.5
        sd[k] = t.to(dtype)
    return sd
