"""Configuration of a Nilatar model: read from the checkpoint folder's config.json (keys as the checkpoints carry them).

Every size and constant comes from here; nothing is specialised to one checkpoint.  A layer's mixer is one of
  latent_attention   keys and values of all heads from one small latent per token, queries from a latent of their own, a rotated key part
                     shared by the heads whose long waves are slowed down
  lightning          linear attention with a constant decay per head
  attention          windowed attention without positions, with a sink; with kv_from it reads an earlier layer's keys and values
(a numbered type such as "attention_2" is the same mechanism with sizes of its own), its feed-forward is dense or absent.
`runs` is the execution order (one run per layer); caches and states are keyed by run."""
from __future__ import annotations

import json
import math
import os
from dataclasses import dataclass, field
from typing import List, Optional

from ..nelovik.config import Run, _base_kind


@dataclass
class RotScaling:
    factor: float
    original: float
    fast: float
    slow: float


@dataclass
class LatentConfig:
    heads: int
    dim: int                       # unrotated query / key entries per head
    rot_dim: int                   # rotated ones
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    rot_dims: int = 0              # leading entries of a rotated part that are turned
    rot_base: float = 10000.0
    rot_scaling: Optional[RotScaling] = None
    window: int = 0                # 0: every earlier key
    kind: str = "latent_attention"

    def frequencies(self) -> List[float]:
        """Angle per position of every pair.  With scaling, pair i keeps its frequency below the pair that makes `fast` turns within the
        original length, turns `factor` times slower above the one that makes `slow` turns, with a linear blend in i between the two."""
        n, s = self.rot_dims, self.rot_scaling
        plain = [self.rot_base ** (-2.0 * i / n) for i in range(n // 2)]
        if s is None:
            return plain
        pair_of = lambda turns: n * math.log(s.original / (2.0 * math.pi * turns)) / (2.0 * math.log(self.rot_base))
        lo, hi = max(math.floor(pair_of(s.fast)), 0), min(math.ceil(pair_of(s.slow)), n - 1)
        out = []
        for i, f in enumerate(plain):
            ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            out.append(f / s.factor * ramp + f * (1.0 - ramp))
        return out

    @property
    def rot_len(self) -> float:
        """Length of a turned vector: cosines and sines are multiplied by it."""
        return 0.1 * math.log(self.rot_scaling.factor) + 1.0 if self.rot_scaling is not None else 1.0


@dataclass
class LightningConfig:
    heads: int
    dim: int
    vdim: int
    decay: List[float]
    kind: str = "lightning"


@dataclass
class WindowConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int = 0                # positions a query sees, itself included (0: every earlier key)
    kv_from: Optional[int] = None  # layer whose keys and values this one reads
    kind: str = "attention"


@dataclass
class LayerConfig:
    mixer: object
    ff: int = 0                    # hidden size of the feed-forward (0: none)


def _latent(m: dict) -> LatentConfig:
    rot = m.get("rot") or {}
    s = rot.get("scaling")
    rot_dim = int(m.get("rot_dim") or 0)
    c = LatentConfig(int(m["heads"]), int(m["dim"]), rot_dim, int(m["vdim"]), int(m["kv_rank"]), int(m["q_rank"]), float(m["scale"]),
                     int(rot.get("dims", rot_dim) or 0) if rot else 0, float(rot.get("base", 10000.0)),
                     RotScaling(float(s["factor"]), float(s["original"]), float(s["fast"]), float(s["slow"])) if s else None,
                     int((m.get("mask") or {}).get("size", 0) or 0))
    if c.rot_dim % 2 or c.rot_dims % 2 or c.rot_dims > c.rot_dim:
        raise ValueError(f"rot.dims ({c.rot_dims}) must be even and at most rot_dim ({c.rot_dim}), which must be even")
    return c


def _lightning(m: dict) -> LightningConfig:
    c = LightningConfig(int(m["heads"]), int(m["dim"]), int(m["vdim"]), [float(v) for v in m["decay"]])
    if len(c.decay) != c.heads:
        raise ValueError(f"{len(c.decay)} decays for {c.heads} heads")
    return c


def _window(m: dict) -> WindowConfig:
    heads = int(m["heads"])
    src = m.get("kv_from")
    c = WindowConfig(heads, int(m.get("kv_heads") or heads), int(m["dim"]), int(m["vdim"]), float(m["scale"]),
                     int((m.get("mask") or {}).get("size", 0) or 0), None if src is None else int(src))
    if c.heads % c.kv_heads:
        raise ValueError(f"{c.heads} query heads do not split over {c.kv_heads} key/value heads")
    return c


_MIXERS = {"latent_attention": _latent, "lightning": _lightning, "attention": _window}


@dataclass
class NilatarConfig:
    vocab_size: int
    width: int
    layers: List[LayerConfig]
    eps: float
    embed_scale: float = 1.0
    max_seqlen: int = 8192
    max_batch_size: int = 1
    runs: List[Run] = field(default_factory=list)

    def __post_init__(self):
        self.runs = [Run(i) for i in range(len(self.layers))]
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            if m.kind != "attention" or m.kv_from is None:
                continue
            j = m.kv_from
            src = self.layers[j].mixer if 0 <= j < i else None
            if src is None or src.kind != "attention" or src.kv_from is not None:
                raise ValueError(f"layer {i} reads the keys and values of layer {j}, which is no earlier attention layer with projections of its own")
            if (src.kv_heads, src.dim, src.vdim) != (m.kv_heads, m.dim, m.vdim):
                raise ValueError(f"layer {i} and layer {j}, whose keys and values it reads, differ in their head sizes")

    def get(self, key, default=None):
        return getattr(self, key, default)

    @classmethod
    def from_dict(cls, d: dict) -> "NilatarConfig":
        layers = []
        for entry in d["layers"]:
            kind = _base_kind(entry["type"])
            if kind not in _MIXERS:
                raise NotImplementedError(f"mixer type {entry['type']!r}")
            mlp = entry.get("mlp")
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise NotImplementedError(f"feed-forward kind {mlp.get('kind')!r}")
            layers.append(LayerConfig(_MIXERS[kind](entry["mixer"]), int(mlp["ff"]) if mlp is not None else 0))
        return cls(vocab_size=int(d["vocab"]), width=int(d["width"]), layers=layers, eps=float(d["norm"]["eps"]),
                   embed_scale=float((d.get("embedding") or {}).get("scale", 1.0)), max_seqlen=int(d.get("max_seqlen", 8192)))

    @classmethod
    def from_dir(cls, model_dir: str) -> "NilatarConfig":
        with open(os.path.join(model_dir, "config.json")) as f:
            return cls.from_dict(json.load(f))

    @property
    def unused_tensor_names(self):
        """Tensors a checkpoint may carry although this configuration never reads them (norm and scale of an absent feed-forward)."""
        return tuple(f"l{i}.{n}" for i, layer in enumerate(self.layers) if not layer.ff for n in ("norm2", "ls2"))

    def tensor_shapes(self) -> dict:
        """checkpoint tensor name -> shape, in checkpoint naming."""
        d, out = self.width, {"embed": (self.vocab_size, self.width)}
        for i, layer in enumerate(self.layers):
            m, p = layer.mixer, f"l{i}."
            x, inner = p + "mix.", m.heads * m.vdim
            out.update({p + "norm1": (d,), p + "ls1": (d,), x + "g": (inner, d), x + "o": (d, inner)})
            if m.kind == "attention":
                out.update({x + "q": (m.heads * m.dim, d), x + "sink": (m.heads,)})
                if m.kv_from is None:
                    out.update({x + "k": (m.kv_heads * m.dim, d), x + "v": (m.kv_heads * m.vdim, d)})
            elif m.kind == "latent_attention":
                out.update({x + "dq": (m.q_rank, d), x + "dq.norm": (m.q_rank,), x + "uq": (m.heads * (m.dim + m.rot_dim), m.q_rank),
                            x + "dkv": (m.kv_rank + m.rot_dim, d), x + "dkv.norm": (m.kv_rank,), x + "uk": (m.heads * m.dim, m.kv_rank), x + "uv": (inner, m.kv_rank)})
            else:
                out.update({x + "q": (m.heads * m.dim, d), x + "k": (m.heads * m.dim, d), x + "v": (inner, d), x + "norm": (inner,)})
            if layer.ff:
                out.update({p + "norm2": (d,), p + "ls2": (d,), p + "mlp.gate": (layer.ff, d), p + "mlp.up": (layer.ff, d), p + "mlp.down": (d, layer.ff)})
        out["final.norm"] = (d,)
        out["head"] = (self.vocab_size, d)
        return out
