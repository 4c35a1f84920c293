"""Configuration of a Gagotar model: read from the checkpoint folder's config.json (keys as the checkpoints carry them).

Every size and constant comes from here or from a tensor's shape (the rank of the decay projection is only in the latter: `shapes`);
nothing is specialised to one checkpoint.  Every layer's mixer is a pair run side by side,
  left   attention with whole-row query / key norms, rotation with slowed-down long waves, mixed head scores and a chunked causal mask
  right  gated linear attention with a decay per key channel
(a numbered type such as "parallel_2" is the same mechanism with sizes of its own) and its feed-forward is a mixture of experts or absent.
`runs` is the execution order (one run per layer); caches and states are keyed by run."""
from __future__ import annotations

import json
import math
import os
from dataclasses import dataclass, field
from typing import List, Optional

from ..nelovik.config import Run, _base_kind

DECAY_RANK = 16                    # rank of the decay projection when no tensor shapes are given (random initialisation)


@dataclass
class RotScaling:
    factor: float
    low: float
    high: float
    original: float


@dataclass
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int = 0                 # positions per chunk (0: plain causal)
    rot_dims: int = 0              # leading entries of a head that are rotated (0: none)
    rot_base: float = 10000.0
    rot_scaling: Optional[RotScaling] = None

    def frequencies(self) -> List[float]:
        """Angle per position of every rotated pair.  With scaling, waves longer than original / low turn `factor` times slower, waves
        shorter than original / high are kept, and between the two the frequency is blended linearly in original / wavelength."""
        out = []
        for i in range(self.rot_dims // 2):
            f = self.rot_base ** (-2.0 * i / self.rot_dims)
            s = self.rot_scaling
            if s is not None:
                turns = s.original * f / (2.0 * math.pi)              # turns within the original length
                if turns < s.low:
                    f = f / s.factor
                elif turns <= s.high:
                    t = (turns - s.low) / (s.high - s.low) if s.high > s.low else 1.0
                    f = (1.0 - t) * f / s.factor + t * f
            out.append(f)
        return out


@dataclass
class LinearAttentionConfig:
    heads: int
    dim: int
    vdim: int
    tau: float
    rank: int


@dataclass
class MlpConfig:
    ff: int                        # hidden size of one expert
    limit: float                   # bound of the gate (above) and of the up value (both sides)
    experts: int
    top: int


@dataclass
class LayerConfig:
    left: AttentionConfig
    right: LinearAttentionConfig
    mlp: Optional[MlpConfig] = None


def _attention(a: dict) -> AttentionConfig:
    rot, mask = a.get("rot") or {}, a.get("mask") or {}
    s = rot.get("scaling")
    heads, dim = int(a["heads"]), int(a["dim"])
    c = AttentionConfig(heads, int(a.get("kv_heads") or heads), dim, int(a.get("vdim") or dim), float(a.get("scale", dim ** -0.5)), int(mask.get("size", 0) or 0),
                        int(rot.get("dims", dim) or 0) if rot else 0, float(rot.get("base", 10000.0)),
                        RotScaling(float(s["factor"]), float(s["low"]), float(s["high"]), float(s["original"])) if s else None)
    if c.heads % c.kv_heads:
        raise ValueError(f"{c.heads} query heads do not split over {c.kv_heads} key/value heads")
    if c.rot_dims % 2 or c.rot_dims > c.dim:
        raise ValueError(f"rot.dims ({c.rot_dims}) must be even and at most dim ({c.dim})")
    return c


def _mlp(mlp: Optional[dict]) -> Optional[MlpConfig]:
    if mlp is None:
        return None
    if mlp.get("kind", "moe") != "moe":
        raise NotImplementedError(f"feed-forward kind {mlp.get('kind')!r}")
    e, r = mlp["expert"], mlp["router"]
    f = MlpConfig(int(e["ff"]), float(e["limit"]), int(r["experts"]), int(r["top"]))
    if not 0 < f.top <= f.experts:
        raise ValueError(f"router picks {f.top} of {f.experts} experts")
    if not f.limit > 0.0:
        raise ValueError(f"expert.limit ({f.limit}) must be positive")
    return f


@dataclass
class GagotarConfig:
    needs_shapes = True            # from_dict wants the stored tensors' shapes (see models._load_flat)

    vocab_size: int
    width: int
    layers: List[LayerConfig]
    eps: float
    max_seqlen: int = 8192
    max_batch_size: int = 1
    runs: List[Run] = field(default_factory=list)

    def __post_init__(self):
        self.runs = [Run(i) for i in range(len(self.layers))]

    def get(self, key, default=None):
        return getattr(self, key, default)

    @classmethod
    def from_dict(cls, d: dict, shapes: Optional[dict] = None) -> "GagotarConfig":
        layers = []
        for i, entry in enumerate(d["layers"]):
            kind, m = entry["type"], entry["mixer"]
            if _base_kind(kind) != "parallel":
                raise NotImplementedError(f"mixer type {kind!r}")
            s = m["right"]
            a1 = (shapes or {}).get(f"l{i}.mix.right.a1")
            right = LinearAttentionConfig(int(s["heads"]), int(s["dim"]), int(s["vdim"]), float(s["tau"]), int(a1[0]) if a1 is not None else DECAY_RANK)
            layers.append(LayerConfig(_attention(m["left"]), right, _mlp(entry.get("mlp"))))
        return cls(vocab_size=int(d["vocab"]), width=int(d["width"]), layers=layers, eps=float(d["norm"]["eps"]), max_seqlen=int(d.get("max_seqlen", 8192)))

    @classmethod
    def from_dir(cls, model_dir: str) -> "GagotarConfig":
        from ..ingest import stored_shapes
        with open(os.path.join(model_dir, "config.json")) as f:
            return cls.from_dict(json.load(f), stored_shapes(model_dir))

    @property
    def unused_tensor_names(self):
        """Tensors a checkpoint may carry although this configuration never reads them (norm and scale of an absent feed-forward)."""
        return tuple(f"l{i}.{n}" for i, layer in enumerate(self.layers) if layer.mlp is None for n in ("norm2", "ls2"))

    def tensor_shapes(self) -> dict:
        """checkpoint tensor name -> shape, in checkpoint naming."""
        d, out = self.width, {"embed": (self.vocab_size, self.width)}
        for i, layer in enumerate(self.layers):
            p = f"l{i}."
            a, s, f = layer.left, layer.right, layer.mlp
            l, r = p + "mix.left.", p + "mix.right."
            qw, kw, vw = a.heads * a.dim, a.kv_heads * a.dim, a.kv_heads * a.vdim
            out.update({p + "norm1": (d,), p + "ls1": (d,)})
            out.update({l + "q": (qw, d), l + "q.b": (qw,), l + "k": (kw, d), l + "k.b": (kw,), l + "v": (vw, d), l + "v.b": (vw,), l + "q.norm": (qw,), l + "k.norm": (kw,),
                        l + "talk": (a.heads, a.heads), l + "temp": (a.heads,), l + "g": (a.heads, d), l + "o": (d, a.heads * a.vdim), l + "out": (d,)})
            qk, vv = s.heads * s.dim, s.heads * s.vdim
            out.update({r + "q": (qk, d), r + "k": (qk, d), r + "v": (vv, d), r + "g": (vv, d), r + "o": (d, vv), r + "norm": (s.vdim,),
                        r + "a1": (s.rank, d), r + "a2": (qk, s.rank), r + "a2.b": (qk,), r + "out": (d,)})
            if f is not None:
                out.update({p + "norm2": (d,), p + "ls2": (d,), p + "mlp.router": (f.experts, d)})
                for e in range(f.experts):
                    out.update({f"{p}mlp.e{e}.gate": (f.ff, d), f"{p}mlp.e{e}.up": (f.ff, d), f"{p}mlp.e{e}.down": (d, f.ff)})
        out["final.norm"] = (d,)
        out["head"] = (self.vocab_size, d)
        return out
