"""Fovudra checkpoint names -> parameter tree, and random trees.

Linear weights stay (out, in) as stored; projections that share an input are concatenated, experts are stacked on a leading
axis. Norm gains, biases, gate biases and decays are kept in fp32 (gains stored around zero get their 1 here), matrices and
embeddings in the serving dtype::

    embed (V, D)  embed_norm, final_norm (D)  head (V, D)
    layers[i].norm1, norm1b [, norm2, norm2b]
    layers[i].mix   attention: qk ((H + G) dim, D)  qk_b ((H + G) dim)  o (D, H dim)
                    mlstm:     in ([q | k | v | g | i | f], D)  gate_b (2 H)  norm (H vdim)  o (D, H vdim)
                    lightning: in ([q | k | v | g], D)  decay (H)  norm (H vdim)  o (D, H vdim)
    layers[i].mlp   router (E, D)  gate_up (E, 2 ff, D)  down (E, D, ff)  shared_gate_up (2 ff', D)  shared_down (D, ff')
"""
from __future__ import annotations

import torch

from .config import FovudraConfig, Lightning, MLstm, WindowAttention


def expected_shapes(c: FovudraConfig) -> dict:
    """Checkpoint tensor names and shapes of a configuration."""
    D, V = c.width, c.vocab_size
    s = {"embed": (V, D), "embed.norm": (D,), "head": (V, D), "final.norm": (D,)}
    for i, layer in enumerate(c.layers):
        p, m, f = f"l{i}.", layer.mixer, layer.mlp
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if f else ()):
            s[p + n] = (D,)
        if isinstance(m, WindowAttention):
            q, k = m.heads * m.dim, m.kv_heads * m.dim
            s.update({p + "mix.q": (q, D), p + "mix.q.b": (q,), p + "mix.k": (k, D), p + "mix.k.b": (k,), p + "mix.o": (D, q)})
        else:
            qk, v = m.heads * m.dim, m.heads * m.vdim
            s.update({p + "mix.q": (qk, D), p + "mix.k": (qk, D), p + "mix.v": (v, D), p + "mix.g": (v, D), p + "mix.o": (D, v),
                      p + "mix.norm": (v,)})
            if isinstance(m, MLstm):
                s.update({p + "mix.i": (m.heads, D), p + "mix.i.b": (m.heads,), p + "mix.f": (m.heads, D), p + "mix.f.b": (m.heads,)})
        if f:
            s[p + "mlp.router"] = (f.experts, D)
            for e, ff in [(f"e{e}", f.ff) for e in range(f.experts)] + [("shared", f.shared_ff)]:
                s.update({f"{p}mlp.{e}.gate": (ff, D), f"{p}mlp.{e}.up": (ff, D), f"{p}mlp.{e}.down": (D, ff)})
    return s


def load_from_state_dict(sd, config: FovudraConfig, dtype=torch.bfloat16, device="cpu") -> dict:
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
    vec = lambda *ks: torch.cat([raw(k).to(device=device, dtype=torch.float32) for k in ks]).contiguous()
    gain = lambda k: 1.0 + vec(k)
    cat = lambda *ks: torch.cat([mat(k) for k in ks]).contiguous()

    layers = []
    for i, layer in enumerate(c.layers):
        p, m, f = f"l{i}.", layer.mixer, layer.mlp
        x = p + "mix."
        lp = {"norm1": gain(p + "norm1"), "norm1b": gain(p + "norm1b")}
        if isinstance(m, WindowAttention):
            lp["mix"] = {"qk": cat(x + "q", x + "k"), "qk_b": vec(x + "q.b", x + "k.b"), "o": mat(x + "o")}
        elif isinstance(m, MLstm):
            lp["mix"] = {"in": cat(x + "q", x + "k", x + "v", x + "g", x + "i", x + "f"), "gate_b": vec(x + "i.b", x + "f.b"),
                         "norm": vec(x + "norm"), "o": mat(x + "o")}
        else:
            lp["mix"] = {"in": cat(x + "q", x + "k", x + "v", x + "g"), "decay": torch.tensor(m.decay, dtype=torch.float32, device=device),
                         "norm": vec(x + "norm"), "o": mat(x + "o")}
        if f is not None:
            lp["norm2"], lp["norm2b"] = gain(p + "norm2"), gain(p + "norm2b")
            e = lambda k: f"{p}mlp.{k}."
            lp["mlp"] = {"router": mat(p + "mlp.router"),
                         "gate_up": torch.stack([cat(e(f"e{k}") + "gate", e(f"e{k}") + "up") for k in range(f.experts)]),
                         "down": torch.stack([mat(e(f"e{k}") + "down") for k in range(f.experts)]),
                         "shared_gate_up": cat(e("shared") + "gate", e("shared") + "up"), "shared_down": mat(e("shared") + "down")}
        layers.append(lp)
    return {"embed": mat("embed"), "embed_norm": gain("embed.norm"), "layers": layers, "final_norm": gain("final.norm"), "head": mat("head")}


def random_state_dict(config: FovudraConfig, seed: int = 0, dtype=torch.float32, device="cpu") -> dict:
    """Random checkpoint of a configuration: matrices N(0, 1 / fan_in), norm weights near their neutral value, forget gates
    mostly open."""
    g = torch.Generator(device=device).manual_seed(seed)
    n = lambda *s: torch.randn(*s, generator=g, device=device)
    sd = {}
    for k, s in expected_shapes(config).items():
        if k.endswith(".norm") and ".mix." in k:
            t = 1.0 + 0.1 * n(*s)
        elif k.endswith(".f.b"):
            t = 3.0 + n(*s)
        elif len(s) == 1:
            t = 0.1 * n(*s)
        elif k == "embed":
            t = n(*s)
        else:
            t = n(*s) * s[-1] ** -0.5
        sd[k] = t.to(dtype)
    return sd
