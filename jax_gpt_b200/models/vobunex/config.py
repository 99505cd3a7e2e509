"""Configuration of Vobunex: a decoder-only model whose layer list mixes Mamba-2 and latent-attention layers, each with
its own sizes and with a dense, an expert or no feed-forward; token and bigram embeddings, pre-norm with layer norms.

``VobunexConfig.from_dict`` reads the published ``config.json``; every size and constant comes from there.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, replace
from typing import Optional, Tuple, Union

ARCHITECTURE = "Vobunex"
GLU_ALPHA = 1.702          # slope inside the experts' sigmoid, fixed by the design


@dataclass(frozen=True)
class Rotary:
    base: float
    dims: int
    scaling: Optional[Tuple[Tuple[str, float], ...]] = None   # YaRN: factor, original, fast, slow


@dataclass(frozen=True)
class LatentAttention:
    heads: int
    dim: int               # unrotated query / key features per head
    rot_dim: int           # rotated features per head; the key part is shared by all heads
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: Rotary

    @property
    def width(self) -> int:
        """One cached token: the normed latent and the rotated key part."""
        return self.kv_rank + self.rot_dim


@dataclass(frozen=True)
class Mamba2:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int              # taps
    norm_groups: int

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def conv_dim(self) -> int:
        return self.inner + 2 * self.groups * self.state


@dataclass(frozen=True)
class DenseMlp:
    ff: int


@dataclass(frozen=True)
class TableMoe:
    ff: int
    limit: float
    experts: int
    top: int


@dataclass(frozen=True)
class Layer:
    mixer: Union[LatentAttention, Mamba2]
    mlp: Optional[Union[DenseMlp, TableMoe]]


@dataclass(frozen=True)
class Bigram:
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class VobunexConfig:
    vocab_size: int
    width: int
    norm_eps: float
    layers: Tuple[Layer, ...]
    bigram: Optional[Bigram] = None
    page_size: int = 64
    dtype: str = "bfloat16"

    @property
    def n_layers(self) -> int:
        return len(self.layers)

    @property
    def attention_layers(self):
        return [i for i, l in enumerate(self.layers) if isinstance(l.mixer, LatentAttention)]

    @property
    def ssm_layers(self):
        return [i for i, l in enumerate(self.layers) if isinstance(l.mixer, Mamba2)]

    def replace(self, **kw) -> "VobunexConfig":
        return replace(self, **kw)

    @staticmethod
    def from_dict(d: dict, **kw) -> "VobunexConfig":
        if d.get("architecture") != ARCHITECTURE:
            raise ValueError(f"not a {ARCHITECTURE} configuration: architecture {d.get('architecture')!r}")
        big = (d.get("embedding") or {}).get("bigram")
        bigram = Bigram(int(big["buckets"]), int(big["mul_prev"]), int(big["mul_cur"])) if big else None
        return VobunexConfig(vocab_size=int(d["vocab"]), width=int(d["width"]), norm_eps=float(d["norm"]["eps"]),
                             layers=tuple(_layer(l) for l in d["layers"]), bigram=bigram, **kw)

    @staticmethod
    def from_dir(path: str, **kw) -> "VobunexConfig":
        with open(os.path.join(path, "config.json")) as f:
            return VobunexConfig.from_dict(json.load(f), **kw)

    # ---- presets (random weights: tests, benchmarks) ----
    @staticmethod
    def tiny() -> "VobunexConfig":
        rot = Rotary(10000.0, 8, (("factor", 4.0), ("fast", 4.0), ("original", 32), ("slow", 0.5)))
        m = Mamba2(heads=6, vdim=8, state=12, groups=3, conv=3, norm_groups=2)
        a = LatentAttention(heads=3, dim=12, rot_dim=8, vdim=10, q_rank=20, kv_rank=14, scale=0.21, rot=rot)
        return VobunexConfig(vocab_size=97, width=40, norm_eps=1e-5, bigram=Bigram(53, 31, 7), page_size=16,
                             layers=(Layer(a, TableMoe(24, 0.9, 5, 3)), Layer(m, None), Layer(m, TableMoe(20, 1.1, 4, 1)),
                                     Layer(a, DenseMlp(56))))

    @staticmethod
    def serving(width: int = 2048, n_mamba: int = 6, n_attention: int = 2, experts: int = 64, top: int = 6, ff: int = 1024,
                heads: int = 16, vocab: int = 65536) -> "VobunexConfig":
        """Layers with the widths of a real model: Mamba-2 inner 2 x width in heads of 64 with state 128, latent attention
        with heads of 128 + 64 and a latent of 512, tabled experts; attention layers spread evenly."""
        rot = Rotary(10000.0, 64, (("factor", 4.0), ("fast", 32.0), ("original", 4096), ("slow", 1.0)))
        m = Mamba2(heads=2 * width // 64, vdim=64, state=128, groups=8, conv=4, norm_groups=8)
        a = LatentAttention(heads=heads, dim=128, rot_dim=64, vdim=128, q_rank=1536 if width > 4096 else 768, kv_rank=512,
                            scale=192 ** -0.5, rot=rot)
        n = n_mamba + n_attention
        every = max(1, n // max(1, n_attention))
        kinds = [n_attention > 0 and i % every == every - 1 and i // every < n_attention for i in range(n)]
        mlp = TableMoe(ff, 7.0, experts, top)
        return VobunexConfig(vocab_size=vocab, width=width, norm_eps=1e-5, bigram=Bigram(4 * vocab - 1, 31337, 271),
                             layers=tuple(Layer(a if k else m, mlp) for k in kinds))


def _rotary(d: dict) -> Rotary:
    sc = d.get("scaling")
    return Rotary(float(d["base"]), int(d["dims"]), tuple(sorted((k, float(v)) for k, v in sc.items())) if sc else None)


def _layer(d: dict) -> Layer:
    m = d["mixer"]
    if d["type"] == "latent_attention":
        mixer = LatentAttention(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]),
                                q_rank=int(m["q_rank"]), kv_rank=int(m["kv_rank"]), scale=float(m["scale"]), rot=_rotary(m["rot"]))
        if mixer.rot.dims > mixer.rot_dim or mixer.rot.dims % 2:
            raise ValueError(f"rot.dims {mixer.rot.dims} does not fit rot_dim {mixer.rot_dim}")
    elif d["type"] == "mamba2":
        mixer = Mamba2(heads=int(m["heads"]), vdim=int(m["vdim"]), state=int(m["state"]), groups=int(m["groups"]),
                       conv=int(m["conv"]), norm_groups=int(m["norm_groups"]))
        if mixer.heads % mixer.groups or mixer.inner % mixer.norm_groups:
            raise ValueError("mamba2: heads must divide into groups and the inner width into norm_groups")
    else:
        raise ValueError(f"unknown mixer type {d['type']!r}")
    f = d.get("mlp")
    if not f:
        mlp = None
    elif f["kind"] == "dense":
        mlp = DenseMlp(int(f["ff"]))
    elif f["kind"] == "moe":
        mlp = TableMoe(int(f["expert"]["ff"]), float(f["expert"]["limit"]), int(f["router"]["experts"]), int(f["router"]["top"]))
    else:
        raise ValueError(f"unknown feed-forward kind {f['kind']!r}")
    return Layer(mixer, mlp)
