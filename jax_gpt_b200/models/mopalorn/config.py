"""Configuration of Mopalorn: a decoder-only model whose layer list mixes windowed latent attention with an output gate, soft-capped full
attention and windowed attention over tokens and block means, each with its own sizes and with a dense or no feed-forward; norms before
and after every sublayer, values mixed with those of the first such layer, embeddings tied to the output.

``MopalornConfig.from_dict`` reads the published ``config.json``; every size and constant comes from there.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, replace
from typing import Optional, Tuple, Union

ARCHITECTURE = "Mopalorn"


@dataclass(frozen=True)
class Rotary:
    base: float
    dims: int


@dataclass(frozen=True)
class LatentAttention:
    """Latent attention over a sliding window, queries projected directly, a sigmoid gate on the output's features."""
    heads: int
    dim: int               # unrotated query / key features per head
    rot_dim: int           # rotated features per head (half-split pairs); the key part is shared by all heads
    vdim: int
    kv_rank: int
    scale: float
    rot: Rotary
    window: Optional[int]

    @property
    def width(self) -> int:
        """One cached token: the normed latent and the rotated key part."""
        return self.kv_rank + self.rot_dim

    def segments(self):
        """(first column of q, latent and rotary key, gate; all columns) of the fused input projection."""
        return segments(self.heads * (self.dim + self.rot_dim), self.width, self.heads * self.vdim)


@dataclass(frozen=True)
class GroupedAttention:
    """Grouped-query attention without rotation: all keys, or a sliding window and the means of the blocks before it."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    v_mix: bool
    softcap: float = 0.0                              # 0: none
    q_temp: Optional[Tuple[float, int]] = None        # (coef, every): factor of the query by its position
    window: Optional[int] = None
    pool: int = 0                                     # tokens per block, 0: no blocks
    sink: bool = False

    @property
    def width(self) -> int:
        """One cached token: keys and values of every kv head."""
        return self.kv_heads * (self.dim + self.vdim)

    def segments(self):
        """(first column of q, k, v; all columns) of the fused input projection."""
        return segments(self.heads * self.dim, self.kv_heads * self.dim, self.kv_heads * self.vdim)


@dataclass(frozen=True)
class XieluMlp:
    ff: int


@dataclass(frozen=True)
class Layer:
    mixer: Union[LatentAttention, GroupedAttention]
    mlp: Optional[XieluMlp]


@dataclass(frozen=True)
class MopalornConfig:
    vocab_size: int
    width: int
    norm_eps: float
    logit_scale: float
    layers: Tuple[Layer, ...]
    page_size: int = 64
    dtype: str = "bfloat16"

    @property
    def n_layers(self) -> int:
        return len(self.layers)

    @property
    def first_values(self) -> Optional[int]:
        """The layer whose values the later mixing layers take."""
        return next((i for i, l in enumerate(self.layers) if mixes_values(l.mixer)), None)

    def replace(self, **kw) -> "MopalornConfig":
        return replace(self, **kw)

    @staticmethod
    def from_dict(d: dict, **kw) -> "MopalornConfig":
        if d.get("architecture") != ARCHITECTURE:
            raise ValueError(f"not a {ARCHITECTURE} configuration: architecture {d.get('architecture')!r}")
        c = MopalornConfig(vocab_size=int(d["vocab"]), width=int(d["width"]), norm_eps=float(d["norm"]["eps"]),
                           logit_scale=float(d["logit_scale"]), layers=tuple(_layer(l) for l in d["layers"]), **kw)
        if len({l.mixer.kv_heads * l.mixer.vdim for l in c.layers if mixes_values(l.mixer)}) > 1:
            raise ValueError("layers with v_mix must have values of one width")
        return c

    @staticmethod
    def from_dir(path: str, **kw) -> "MopalornConfig":
        with open(os.path.join(path, "config.json")) as f:
            return MopalornConfig.from_dict(json.load(f), **kw)

    # ---- presets (random weights: tests, benchmarks) ----
    @staticmethod
    def tiny() -> "MopalornConfig":
        lat = LatentAttention(3, 10, 6, 9, 14, 0.25, Rotary(900.0, 6), 11)
        full = GroupedAttention(4, 2, 12, 8, 0.3, True, softcap=6.0, q_temp=(0.4, 7))
        pooled = GroupedAttention(6, 2, 10, 8, 0.32, True, window=9, pool=5, sink=True)
        return MopalornConfig(vocab_size=83, width=36, norm_eps=1e-5, logit_scale=0.4, page_size=16,
                              layers=(Layer(pooled, XieluMlp(40)), Layer(lat, None), Layer(full, XieluMlp(28)), Layer(pooled, XieluMlp(20))))

    @staticmethod
    def serving(width: int = 2048, n_latent: int = 4, n_full: int = 2, n_pooled: int = 2, heads: int = 16, kv_heads: int = 2, dim: int = 128,
                vdim: int = 128, kv_rank: int = 512, rot_dim: int = 64, window: int = 1024, pool: int = 16, ff: Optional[int] = None,
                vocab: int = 65536) -> "MopalornConfig":
        """Layers with the widths of a real model: latent attention with heads of 128 + 64 and a latent of 512, grouped attention with
        heads of 128; the grouped layers spread evenly, full and pooled ones in turn."""
        lat = LatentAttention(heads, dim, rot_dim, vdim, kv_rank, (dim + rot_dim) ** -0.5, Rotary(50000.0, rot_dim), window)
        full = GroupedAttention(heads, kv_heads, dim, vdim, dim ** -0.5, True, softcap=50.0, q_temp=(0.1, 8192))
        pooled = GroupedAttention(heads, kv_heads, dim, vdim, dim ** -0.5, True, window=window, pool=pool, sink=True)
        grouped = [m for pair in zip([full] * n_full + [None] * n_pooled, [pooled] * n_pooled + [None] * n_full) for m in pair if m]
        n = n_latent + len(grouped)
        every = max(1, n // max(1, len(grouped)))
        mixers = [grouped[i // every] if i % every == every - 1 and i // every < len(grouped) else lat for i in range(n)]
        mlp = XieluMlp(ff or 4 * width)
        return MopalornConfig(vocab_size=vocab, width=width, norm_eps=1e-5, logit_scale=width ** -0.5, layers=tuple(Layer(m, mlp) for m in mixers))


def mixes_values(m) -> bool:
    return isinstance(m, GroupedAttention) and m.v_mix


def segments(*sizes: int):
    """Columns of a fused projection: (first column of every part, all columns); parts start at multiples of 8 (16-byte loads)."""
    at, firsts = 0, []
    for n in sizes:
        firsts.append(at)
        at += (n + 7) // 8 * 8
    return tuple(firsts), at


def _mask(kind: str, m: dict) -> Tuple[Optional[int], int]:
    """(window, tokens per block)."""
    mask = m.get("mask")
    if not mask:
        return None, 0
    size, pool = int(mask["size"]), int(mask.get("pool") or 0)
    if size < 1 or pool < 0:
        raise ValueError(f"{kind}: mask.size and mask.pool must be positive")
    return size, pool


def _layer(d: dict) -> Layer:
    m, kind = d["mixer"], d["type"]
    if kind == "latent_attention":
        rot = Rotary(float(m["rot"]["base"]), int(m["rot"].get("dims", m["rot_dim"])))
        mixer = LatentAttention(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]),
                                kv_rank=int(m["kv_rank"]), scale=float(m["scale"]), rot=rot, window=_mask(kind, m)[0])
        if rot.dims > mixer.rot_dim or rot.dims % 2:
            raise ValueError(f"latent_attention: rot.dims {rot.dims} must be even and fit rot_dim {mixer.rot_dim}")
    elif kind in ("attention", "attention_2"):
        shape = dict(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), scale=float(m["scale"]),
                     v_mix=bool(m.get("v_mix", False)))
        if shape["heads"] % shape["kv_heads"]:
            raise ValueError(f"{kind}: heads must divide into kv_heads")
        if kind == "attention":
            t = m.get("q_temp")
            mixer = GroupedAttention(**shape, softcap=float(m.get("softcap") or 0.0), q_temp=(float(t["coef"]), int(t["every"])) if t else None)
            if mixer.softcap < 0 or (mixer.q_temp and mixer.q_temp[1] < 1):
                raise ValueError("attention: softcap and q_temp.every must be positive")
        else:
            window, pool = _mask(kind, m)
            mixer = GroupedAttention(**shape, window=window, pool=pool, sink=True)
    else:
        raise ValueError(f"unknown mixer type {kind!r}")
    f = d.get("mlp")
    if not f:
        mlp = None
    elif f["kind"] == "dense":
        mlp = XieluMlp(int(f["ff"]))
    else:
        raise ValueError(f"unknown feed-forward kind {f['kind']!r}")
    return Layer(mixer, mlp)
