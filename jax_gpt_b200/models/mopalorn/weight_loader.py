"""Mopalorn checkpoint names -> parameter tree, and random trees.

Linear weights stay (out, in) as stored. Projections that share an input are one matrix whose parts start at multiples of 8 rows (zero
rows between). Checkpoints rotate features i and i + dims / 2 together; the rotated rows of the query and key weights are reordered to
the neighbouring pairs that the latent-attention kernels turn, which leaves the scores as they are. The logits' scale is part of the final
norm's gain. Gains and sinks are fp32, matrices and embeddings have the serving dtype::

    embed (V, D)  final_norm (D)
    layers[i].norm1, norm1b [, norm2, norm2b]
    layers[i].mix   latent attention:  in ([q | latent, rotary key | gate], D)  kv_norm (R)  ukv (H dn + H dv, R)  o (D, H dv)
                    grouped attention: in ([q | k | v], D)  o (D, H dv)  vmix: float  sink (H) | None
    layers[i].mlp   up (ff, D)  down (D, ff)  act: (a, b) of ``ops.gemm.xielu``
"""
from __future__ import annotations

import math

import torch

from ...ops.rope import pair_order
from .config import LatentAttention, MopalornConfig


def expected_shapes(c: MopalornConfig) -> dict:
    """Checkpoint tensor names and shapes of a configuration."""
    D = c.width
    s = {"embed": (c.vocab_size, D), "final.norm": (D,)}
    for i, layer in enumerate(c.layers):
        p, m, f = f"l{i}.", layer.mixer, layer.mlp
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if f else ()):
            s[p + n] = (D,)
        x, H = p + "mix.", m.heads
        s[x + "o"] = (D, H * m.vdim)
        if isinstance(m, LatentAttention):
            s.update({x + "q": (H * (m.dim + m.rot_dim), D), x + "dkv": (m.width, D), x + "dkv.norm": (m.kv_rank,),
                      x + "uk": (H * m.dim, m.kv_rank), x + "uv": (H * m.vdim, m.kv_rank), x + "g": (H * m.vdim, D)})
        else:
            s.update({x + "q": (H * m.dim, D), x + "k": (m.kv_heads * m.dim, D), x + "v": (m.kv_heads * m.vdim, D)})
            if m.v_mix:
                s[x + "vmix"] = ()
            if m.sink:
                s[x + "sink"] = (H,)
        if f:
            s.update({p + "mlp.up": (f.ff, D), p + "mlp.down": (D, f.ff), p + "mlp.act": (2,)})
    return s


def softplus(x: float) -> float:
    return max(x, 0.0) + math.log1p(math.exp(-abs(x)))


def load_from_state_dict(sd, config: MopalornConfig, dtype=torch.bfloat16, device="cpu") -> dict:
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

    def rows(*mats):
        """Matrices over one input below each other, each padded with zero rows to a multiple of 8."""
        return torch.cat([torch.nn.functional.pad(t, (0, 0, 0, -t.shape[0] % 8)) for t in mats]).contiguous()

    layers = []
    for i, layer in enumerate(c.layers):
        p, m = f"l{i}.", layer.mixer
        x = p + "mix."
        lp = {n: vec(p + n) for n in ("norm1", "norm1b") + (("norm2", "norm2b") if layer.mlp else ())}
        if isinstance(m, LatentAttention):
            turn = pair_order(m.rot_dim, m.rot.dims)
            head = torch.cat([torch.arange(m.dim), m.dim + turn])
            q_rows = (torch.arange(m.heads)[:, None] * (m.dim + m.rot_dim) + head).flatten().to(device)
            kv_rows = torch.cat([torch.arange(m.kv_rank), m.kv_rank + turn]).to(device)
            lp["mix"] = {"in": rows(mat(x + "q")[q_rows], mat(x + "dkv")[kv_rows], mat(x + "g")), "kv_norm": vec(x + "dkv.norm"),
                         "ukv": torch.cat([mat(x + "uk"), mat(x + "uv")]).contiguous(), "o": mat(x + "o")}
        else:
            lp["mix"] = {"in": rows(mat(x + "q"), mat(x + "k"), mat(x + "v")), "o": mat(x + "o"),
                         "vmix": float(raw(x + "vmix")) if m.v_mix else 0.0, "sink": vec(x + "sink") if m.sink else None}
        if layer.mlp is not None:
            a, b = (softplus(float(t)) for t in raw(p + "mlp.act"))
            lp["mlp"] = {"up": mat(p + "mlp.up"), "down": mat(p + "mlp.down"), "act": (a, 0.5 + b)}
        layers.append(lp)
    return {"embed": mat("embed"), "layers": layers, "final_norm": c.logit_scale * vec("final.norm")}


def random_state_dict(config: MopalornConfig, seed: int = 0, dtype=torch.float32, device="cpu") -> dict:
    """Random checkpoint of a configuration: matrices N(0, 1 / fan_in), gains near one."""
    g = torch.Generator(device=device).manual_seed(seed)
    n = lambda *s: torch.randn(*s, generator=g, device=device)
    sd = {}
    for k, s in expected_shapes(config).items():
        leaf = k.rsplit(".", 1)[-1]
        if leaf.startswith("norm"):
            t = 1.0 + 0.1 * n(*s)
        elif leaf == "vmix":
            t = 0.5 + 0.1 * n(1)[0]
        elif leaf in ("sink", "act"):
            t = 0.5 * n(*s)
        elif k == "embed":
            t = n(*s)
        else:
            t = n(*s) * s[-1] ** -0.5
        sd[k] = t.to(dtype)
    return sd
