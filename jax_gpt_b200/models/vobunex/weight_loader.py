"""Vobunex checkpoint names -> parameter tree, and the way back for random trees.

Linear weights stay (out, in) as stored; projections that share an input are concatenated (query and kv latents, key and
value up-projections, the experts' gate and up), experts are stacked on a leading axis. Everything that enters a norm,
the convolution, the recurrence or the softmax is kept in fp32, matrices and embeddings in the serving dtype::

    embed (V, D)  bigram (buckets + 1, D) | None  final_norm, final_norm_b (D)  head (V, D)
    layers[i].norm1, norm1_b [, norm2, norm2_b]
    layers[i].mix   latent attention: down (q_rank + kv_rank + rot, D)  q_norm  kv_norm  uq (H (dn + dr), q_rank)
                                      ukv (H dn + H dv, kv_rank)  sink (H)  o (D, H dv)
                    mamba2:           in (2 inner + 2 G N + H, D)  conv (C, taps)  conv_b (C)  dt_bias, A_log, D (H)
                                      norm (inner)  o (D, inner)
    layers[i].mlp   dense: up (ff, D)  down (D, ff)      experts: gate_up (E, 2 ff, D)  down (E, D, ff)  table (V, top)
"""
from __future__ import annotations

import torch

from .config import DenseMlp, LatentAttention, TableMoe, VobunexConfig


def expected_shapes(c: VobunexConfig) -> dict:
    """Checkpoint tensor names and shapes of a configuration."""
    D, V = c.width, c.vocab_size
    s = {"embed": (V, D), "head": (V, D), "final.norm": (D,), "final.norm.b": (D,)}
    if c.bigram:
        s["bigram"] = (c.bigram.buckets + 1, D)
    for i, layer in enumerate(c.layers):
        p, m, f = f"l{i}.", layer.mixer, layer.mlp
        for n in ("norm1", "norm2") if f else ("norm1",):
            s[p + n] = s[p + n + ".b"] = (D,)
        if isinstance(m, LatentAttention):
            H = m.heads
            s.update({p + "mix.dq": (m.q_rank, D), p + "mix.dq.norm": (m.q_rank,), p + "mix.uq": (H * (m.dim + m.rot_dim), m.q_rank),
                      p + "mix.dkv": (m.width, D), p + "mix.dkv.norm": (m.kv_rank,), p + "mix.uk": (H * m.dim, m.kv_rank),
                      p + "mix.uv": (H * m.vdim, m.kv_rank), p + "mix.sink": (H,), p + "mix.o": (D, H * m.vdim)})
        else:
            s.update({p + "mix.in": (m.inner + m.conv_dim + m.heads, D), p + "mix.conv": (m.conv_dim, m.conv),
                      p + "mix.conv.b": (m.conv_dim,), p + "mix.dt_bias": (m.heads,), p + "mix.A_log": (m.heads,),
                      p + "mix.D": (m.heads,), p + "mix.norm": (m.inner,), p + "mix.o": (D, m.inner)})
        if isinstance(f, DenseMlp):
            s.update({p + "mlp.up": (f.ff, D), p + "mlp.down": (D, f.ff)})
        elif isinstance(f, TableMoe):
            s[p + "mlp.table"] = (V, f.top)
            for e in range(f.experts):
                s.update({f"{p}mlp.e{e}.gate": (f.ff, D), f"{p}mlp.e{e}.up": (f.ff, D), f"{p}mlp.e{e}.down": (D, f.ff)})
    return s


def load_from_state_dict(sd, config: VobunexConfig, dtype=torch.bfloat16, device="cpu") -> dict:
    """``sd``: mapping of checkpoint names to tensors (lazy mappings work: each key is read once)."""
    c = config
    shapes = expected_shapes(c)
    missing = [k for k in shapes if k not in sd]
    if missing:
        raise KeyError(f"checkpoint lacks {len(missing)} tensor(s), e.g. {missing[:4]}")

    def raw(k):
        t = sd[k]
        if tuple(t.shape) != shapes[k]:
            raise ValueError(f"{k}: shape {tuple(t.shape)}, the configuration says {shapes[k]}")
        return t.detach()
    mat = lambda k: raw(k).to(device=device, dtype=dtype).contiguous()
    vec = lambda k: raw(k).to(device=device, dtype=torch.float32).contiguous()
    cat = lambda *ks: torch.cat([mat(k) for k in ks]).contiguous()

    layers = []
    for i, layer in enumerate(c.layers):
        p, m, f = f"l{i}.", layer.mixer, layer.mlp
        lp = {"norm1": vec(p + "norm1"), "norm1_b": vec(p + "norm1.b")}
        if isinstance(m, LatentAttention):
            lp["mix"] = {"down": cat(p + "mix.dq", p + "mix.dkv"), "q_norm": vec(p + "mix.dq.norm"), "kv_norm": vec(p + "mix.dkv.norm"),
                         "uq": mat(p + "mix.uq"), "ukv": cat(p + "mix.uk", p + "mix.uv"), "sink": vec(p + "mix.sink"), "o": mat(p + "mix.o")}
        else:
            lp["mix"] = {"in": mat(p + "mix.in"), "conv": vec(p + "mix.conv"), "conv_b": vec(p + "mix.conv.b"),
                         "dt_bias": vec(p + "mix.dt_bias"), "A_log": vec(p + "mix.A_log"), "D": vec(p + "mix.D"),
                         "norm": vec(p + "mix.norm"), "o": mat(p + "mix.o")}
        if f is not None:
            lp["norm2"], lp["norm2_b"] = vec(p + "norm2"), vec(p + "norm2.b")
        if isinstance(f, DenseMlp):
            lp["mlp"] = {"up": mat(p + "mlp.up"), "down": mat(p + "mlp.down")}
        elif isinstance(f, TableMoe):
            table = raw(p + "mlp.table")
            if int(table.min()) < 0 or int(table.max()) >= f.experts:
                raise ValueError(f"{p}mlp.table names experts outside 0 .. {f.experts - 1}")
            lp["mlp"] = {"gate_up": torch.stack([cat(f"{p}mlp.e{e}.gate", f"{p}mlp.e{e}.up") for e in range(f.experts)]),
                         "down": torch.stack([mat(f"{p}mlp.e{e}.down") for e in range(f.experts)]),
                         "table": table.to(device=device, dtype=torch.int32).contiguous()}
        layers.append(lp)
    return {"embed": mat("embed"), "bigram": mat("bigram") if c.bigram else None, "layers": layers,
            "final_norm": vec("final.norm"), "final_norm_b": vec("final.norm.b"), "head": mat("head")}


def random_state_dict(config: VobunexConfig, seed: int = 0, dtype=torch.float32, device="cpu") -> dict:
    """Random checkpoint of a configuration: matrices N(0, 1 / fan_in), norms near 1, decays and step sizes in the range
    of trained state-space layers, tables of distinct experts."""
    g = torch.Generator(device=device).manual_seed(seed)
    n = lambda *s: torch.randn(*s, generator=g, device=device)
    sd = {}
    for k, s in expected_shapes(config).items():
        name = k.rsplit(".", 1)[-1]
        if name == "table":
            E = config.layers[int(k[1:k.index(".")])].mlp.experts
            sd[k] = torch.rand(s[0], E, generator=g, device=device).argsort(-1)[:, :s[1]].to(torch.int32)
            continue
        if name == "A_log":
            t = torch.log(torch.rand(s, generator=g, device=device) * 7.0 + 0.5)
        elif name == "dt_bias":
            t = torch.rand(s, generator=g, device=device) * 3.0 - 4.0
        elif name in ("D", "norm", "norm1", "norm2"):
            t = 1.0 + 0.1 * n(*s)
        elif name == "b" or name == "sink":
            t = 0.1 * n(*s) if name == "b" else 0.5 * n(*s)
        elif name == "conv":
            t = n(*s) * s[1] ** -0.5
        elif name in ("embed", "bigram"):
            t = n(*s)
        else:
            t = n(*s) * s[-1] ** -0.5
        sd[k] = t.to(dtype)
    return sd
