"""Configuration of Fovudra: a decoder-only model whose layer list mixes windowed attention, mLSTM and lightning-attention
layers, each with its own sizes and with an expert or no feed-forward; norms before and after every sublayer.

``FovudraConfig.from_dict`` reads the published ``config.json``; every size and constant comes from there.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, replace
from typing import Optional, Tuple, Union

ARCHITECTURE = "Fovudra"
DEN_EPS = 1e-6             # added to the mLSTM denominator, fixed by the design


@dataclass(frozen=True)
class Rotary:
    base: float
    dims: int
    scaling: Optional[Tuple[Tuple[str, float], ...]] = None   # wavelength bands: factor, low, high, original


@dataclass(frozen=True)
class WindowAttention:
    """Grouped-query attention over a sliding window and the first tokens; projected keys double as values."""
    heads: int
    kv_heads: int
    dim: int
    scale: float
    rot: Rotary
    window: int
    keep_first: int

    @property
    def width(self) -> int:
        """One cached token: keys and values of every kv head."""
        return 2 * self.kv_heads * self.dim


@dataclass(frozen=True)
class MLstm:
    heads: int
    dim: int               # query / key width per head
    vdim: int
    gate_cap: float


@dataclass(frozen=True)
class Lightning:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]


@dataclass(frozen=True)
class SigmoidMoe:
    ff: int
    experts: int
    top: int
    shared_ff: int


@dataclass(frozen=True)
class Layer:
    mixer: Union[WindowAttention, MLstm, Lightning]
    mlp: Optional[SigmoidMoe]


@dataclass(frozen=True)
class FovudraConfig:
    vocab_size: int
    width: int
    norm_eps: float
    layers: Tuple[Layer, ...]
    page_size: int = 64
    dtype: str = "bfloat16"

    @property
    def n_layers(self) -> int:
        return len(self.layers)

    @property
    def attention_layers(self):
        return [i for i, l in enumerate(self.layers) if isinstance(l.mixer, WindowAttention)]

    @property
    def recurrent_layers(self):
        return [i for i, l in enumerate(self.layers) if not isinstance(l.mixer, WindowAttention)]

    def replace(self, **kw) -> "FovudraConfig":
        return replace(self, **kw)

    @staticmethod
    def from_dict(d: dict, **kw) -> "FovudraConfig":
        if d.get("architecture") != ARCHITECTURE:
            raise ValueError(f"not a {ARCHITECTURE} configuration: architecture {d.get('architecture')!r}")
        return FovudraConfig(vocab_size=int(d["vocab"]), width=int(d["width"]), norm_eps=float(d["norm"]["eps"]),
                             layers=tuple(_layer(l) for l in d["layers"]), **kw)

    @staticmethod
    def from_dir(path: str, **kw) -> "FovudraConfig":
        with open(os.path.join(path, "config.json")) as f:
            return FovudraConfig.from_dict(json.load(f), **kw)

    # ---- presets (random weights: tests, benchmarks) ----
    @staticmethod
    def tiny() -> "FovudraConfig":
        rot = Rotary(1000.0, 8, (("factor", 4.0), ("high", 3.0), ("low", 1.0), ("original", 64.0)))
        a = WindowAttention(heads=4, kv_heads=2, dim=12, scale=0.3, rot=rot, window=9, keep_first=3)
        m, l = MLstm(3, 10, 14, 12.0), Lightning(2, 9, 11, (0.7, 0.98))
        return FovudraConfig(vocab_size=97, width=40, norm_eps=1e-5, page_size=16,
                             layers=(Layer(a, SigmoidMoe(24, 5, 3, 20)), Layer(m, None), Layer(l, SigmoidMoe(20, 4, 1, 30)),
                                     Layer(m, SigmoidMoe(12, 3, 2, 8))))

    @staticmethod
    def serving(width: int = 2048, n_mlstm: int = 3, n_lightning: int = 3, n_attention: int = 2, experts: int = 64, top: int = 6,
                ff: int = 1024, shared_ff: int = 128, heads: int = 16, kv_heads: int = 2, window: int = 1024, keep_first: int = 64,
                vocab: int = 65536) -> "FovudraConfig":
        """Layers with the widths of a real model: recurrent heads of 128 over the model width, attention heads of 128 over a
        window with kept first tokens, routed experts and a shared one; attention layers spread evenly."""
        rot = Rotary(500000.0, 128, (("factor", 8.0), ("high", 4.0), ("low", 1.0), ("original", 8192.0)))
        a = WindowAttention(heads, kv_heads, 128, 128 ** -0.5, rot, window, keep_first)
        H = width // 128
        m = MLstm(H, 128, 128, 15.0)
        l = Lightning(H, 128, 128, tuple(1.0 - 2.0 ** (-5 - 8 * h / H) for h in range(H)))
        n = n_mlstm + n_lightning + n_attention
        every = max(1, n // max(1, n_attention))
        mixers, rec = [], [m] * n_mlstm + [l] * n_lightning
        rec = [rec[i // 2 + (i % 2) * n_mlstm] for i in range(len(rec))] if n_mlstm == n_lightning else rec
        for i in range(n):
            attn = n_attention > 0 and i % every == every - 1 and i // every < n_attention
            mixers.append(a if attn else rec.pop(0))
        mlp = SigmoidMoe(ff, experts, top, shared_ff)
        return FovudraConfig(vocab_size=vocab, width=width, norm_eps=1e-5, layers=tuple(Layer(x, mlp) for x in mixers))


def _rotary(d: dict) -> Rotary:
    sc = d.get("scaling")
    return Rotary(float(d["base"]), int(d["dims"]), tuple(sorted((k, float(sc[k])) for k in ("factor", "low", "high", "original"))) if sc else None)


def _layer(d: dict) -> Layer:
    m, kind = d["mixer"], d["type"]
    if kind == "attention":
        mask = m["mask"]
        mixer = WindowAttention(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), scale=float(m["scale"]),
                                rot=_rotary(m["rot"]), window=int(mask["size"]), keep_first=int(mask["keep_first"]))
        if mixer.rot.dims > mixer.dim or mixer.rot.dims % 2:
            raise ValueError(f"rot.dims {mixer.rot.dims} does not fit dim {mixer.dim}")
        if mixer.heads % mixer.kv_heads or int(m.get("vdim", mixer.dim)) != mixer.dim:
            raise ValueError("attention: heads must divide into kv_heads, and keys double as values (vdim = dim)")
        if mixer.window < 1 or mixer.keep_first < 0:
            raise ValueError("attention: mask.size must be positive and mask.keep_first not negative")
    elif kind == "mlstm":
        mixer = MLstm(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), gate_cap=float(m["gate_cap"]))
    elif kind == "lightning":
        mixer = Lightning(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), decay=tuple(float(x) for x in m["decay"]))
        if len(mixer.decay) != mixer.heads or min(mixer.decay) <= 0:
            raise ValueError("lightning: one positive decay per head")
    else:
        raise ValueError(f"unknown mixer type {kind!r}")
    f = d.get("mlp")
    if not f:
        mlp = None
    elif f["kind"] == "moe":
        mlp = SigmoidMoe(int(f["expert"]["ff"]), int(f["router"]["experts"]), int(f["router"]["top"]), int(f["shared"]["ff"]))
        if not 1 <= mlp.top <= mlp.experts:
            raise ValueError("moe: router.top must be between 1 and router.experts")
    else:
        raise ValueError(f"unknown feed-forward kind {f['kind']!r}")
    return Layer(mixer, mlp)
