"""Configuration of Munazen: a decoder-only model over several residual streams whose layer list mixes parallel layers (attention with
rotated values beside a gated linear recurrent unit) and gated-linear-attention layers, each with its own sizes and with a dense or no
feed-forward; a span of layers may run several times with the same weights.

``MunazenConfig.from_dict`` reads the published ``config.json``; every size and constant comes from there.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, replace
from typing import Optional, Tuple, Union

ARCHITECTURE = "Munazen"
LRU_RATE = 8.0             # log a = -LRU_RATE * softplus(lam) * recurrence gate, fixed by the design
YARN_KEYS = ("factor", "fast", "original", "slow")


@dataclass(frozen=True)
class Rotary:
    base: float
    dims: int
    scaling: Optional[Tuple[Tuple[str, float], ...]] = None   # YaRN: factor, fast, original, slow; keys and queries only


@dataclass(frozen=True)
class RotatedAttention:
    """Causal grouped-query attention with interleaved rotary pairs, rotated values and a sigmoid gate per head."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Rotary

    @property
    def width(self) -> int:
        """One cached token: keys and values of every kv head."""
        return self.kv_heads * (self.dim + self.vdim)


@dataclass(frozen=True)
class GatedLru:
    width: int
    blocks: int
    conv: int


@dataclass(frozen=True)
class Parallel:
    left: RotatedAttention
    right: GatedLru
    left_scale: float
    right_scale: float

    def segments(self):
        """(first column of q, k, v, x, y, g; all columns) of the fused input projection."""
        a, r = self.left, self.right
        return segments(a.heads * a.dim, a.kv_heads * a.dim, a.kv_heads * a.vdim, r.width, r.width, a.heads)


@dataclass(frozen=True)
class GatedLinear:
    """Linear attention with a decay per key channel, alpha = sigmoid(z)^(1 / tau)."""
    heads: int
    dim: int
    vdim: int
    tau: float


@dataclass(frozen=True)
class PolyMlp:
    ff: int


@dataclass(frozen=True)
class Layer:
    mixer: Union[Parallel, GatedLinear]
    mlp: Optional[PolyMlp]


@dataclass(frozen=True)
class MunazenConfig:
    vocab_size: int
    width: int
    norm_eps: float
    norm_groups: int
    streams: int
    layers: Tuple[Layer, ...]
    loop: Optional[Tuple[int, int, int]] = None     # (start, stop, times)
    decay_rank: int = 16                            # of random checkpoints; loaded ones have their tensors' rank
    page_size: int = 64
    dtype: str = "bfloat16"

    @property
    def n_layers(self) -> int:
        return len(self.layers)

    @property
    def runs(self) -> Tuple[int, ...]:
        """Layer indices in the order they run; every run has its own cache or state."""
        n = len(self.layers)
        a, b, times = self.loop or (0, 0, 1)
        return tuple(range(a)) + tuple(range(a, b)) * times + tuple(range(b, n))

    def replace(self, **kw) -> "MunazenConfig":
        return replace(self, **kw)

    @staticmethod
    def from_dict(d: dict, **kw) -> "MunazenConfig":
        if d.get("architecture") != ARCHITECTURE:
            raise ValueError(f"not a {ARCHITECTURE} configuration: architecture {d.get('architecture')!r}")
        lo = d.get("loop")
        c = MunazenConfig(vocab_size=int(d["vocab"]), width=int(d["width"]), norm_eps=float(d["norm"]["eps"]),
                          norm_groups=int(d["norm"]["groups"]), streams=int(d["streams"]), layers=tuple(_layer(l) for l in d["layers"]),
                          loop=(int(lo["start"]), int(lo["stop"]), int(lo["times"])) if lo else None, **kw)
        if c.norm_groups < 1 or c.width % c.norm_groups:
            raise ValueError("norm.groups must divide width")
        if c.streams < 1:
            raise ValueError("streams must be positive")
        if c.loop and not (0 <= c.loop[0] <= c.loop[1] <= c.n_layers and c.loop[2] >= 0):
            raise ValueError(f"loop {lo} does not fit {c.n_layers} layers")
        return c

    @staticmethod
    def from_dir(path: str, **kw) -> "MunazenConfig":
        with open(os.path.join(path, "config.json")) as f:
            return MunazenConfig.from_dict(json.load(f), **kw)

    # ---- presets (random weights: tests, benchmarks) ----
    @staticmethod
    def tiny() -> "MunazenConfig":
        rot = Rotary(2000.0, 8, (("factor", 3.0), ("fast", 6.0), ("original", 96.0), ("slow", 1.0)))
        p = Parallel(RotatedAttention(4, 2, 12, 10, 0.3, rot), GatedLru(24, 3, 4), 0.9, 0.6)
        return MunazenConfig(vocab_size=89, width=36, norm_eps=1e-5, norm_groups=3, streams=3, decay_rank=5, page_size=16, loop=(1, 2, 2),
                             layers=(Layer(p, PolyMlp(40)), Layer(GatedLinear(2, 9, 14, 8.0), PolyMlp(20)), Layer(p, None)))

    @staticmethod
    def serving(width: int = 2048, n_parallel: int = 6, n_gla: int = 2, streams: int = 2, heads: int = 16, kv_heads: int = 2, dim: int = 128,
                vdim: int = 128, lru_block: int = 128, gla_dim: int = 128, gla_vdim: int = 128, ff: Optional[int] = None,
                loop: Optional[Tuple[int, int, int]] = None, vocab: int = 65536) -> "MunazenConfig":
        """Layers with the widths of a real model: attention heads of 128, recurrent units over the model width in blocks of 128,
        linear-attention heads of 128 over the model width, gated-linear layers spread evenly."""
        rot = Rotary(1e6, dim, (("factor", 4.0), ("fast", 32.0), ("original", 8192.0), ("slow", 1.0)))
        p = Parallel(RotatedAttention(heads, kv_heads, dim, vdim, dim ** -0.5, rot), GatedLru(width, width // lru_block, 4), 1.0, 1.0)
        g = GatedLinear(width // gla_vdim, gla_dim, gla_vdim, 16.0)
        n = n_parallel + n_gla
        every = max(1, n // max(1, n_gla))
        mlp = PolyMlp(ff or 4 * width)
        mixers = [g if n_gla > 0 and i % every == every - 1 and i // every < n_gla else p for i in range(n)]
        return MunazenConfig(vocab_size=vocab, width=width, norm_eps=1e-5, norm_groups=8, streams=streams, loop=loop,
                             layers=tuple(Layer(m, mlp) for m in mixers))


def segments(*sizes: int):
    """Columns of a fused projection: (first column of every part, all columns); parts start at multiples of 8 (16-byte loads)."""
    at, firsts = 0, []
    for n in sizes:
        firsts.append(at)
        at += (n + 7) // 8 * 8
    return tuple(firsts), at


def _rotary(d: dict) -> Rotary:
    sc = d.get("scaling")
    return Rotary(float(d["base"]), int(d["dims"]), tuple((k, float(sc[k])) for k in YARN_KEYS) if sc else None)


def _layer(d: dict) -> Layer:
    m, kind = d["mixer"], d["type"]
    if kind == "parallel":
        a, r = m["left"], m["right"]
        left = RotatedAttention(heads=int(a["heads"]), kv_heads=int(a["kv_heads"]), dim=int(a["dim"]), vdim=int(a["vdim"]),
                                scale=float(a["scale"]), rot=_rotary(a["rot"]))
        if left.rot.dims > left.dim or left.rot.dims % 2 or left.vdim % 2:
            raise ValueError(f"parallel: rot.dims {left.rot.dims} must be even and fit dim {left.dim}, vdim must be even")
        if left.heads % left.kv_heads:
            raise ValueError("parallel: heads must divide into kv_heads")
        right = GatedLru(width=int(r["width"]), blocks=int(r["blocks"]), conv=int(r["conv"]))
        if right.blocks < 1 or right.width % right.blocks or right.conv < 1:
            raise ValueError("parallel: right.blocks must divide right.width, right.conv must be positive")
        mixer = Parallel(left, right, float(m["left_scale"]), float(m["right_scale"]))
    elif kind == "gla":
        mixer = GatedLinear(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), tau=float(m["tau"]))
        if mixer.tau <= 0:
            raise ValueError("gla: tau must be positive")
    else:
        raise ValueError(f"unknown mixer type {kind!r}")
    f = d.get("mlp")
    if not f:
        mlp = None
    elif f["kind"] == "dense":
        mlp = PolyMlp(int(f["ff"]))
    else:
        raise ValueError(f"unknown feed-forward kind {f['kind']!r}")
    return Layer(mixer, mlp)
