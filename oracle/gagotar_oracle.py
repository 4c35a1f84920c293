"""Plain, slow statement of the Gagotar design in PyTorch, one function per mechanism, whole sequences only, float64 by default.
It shares no code with evo_b200: the product is compared against it.

Notation: T tokens, D width, H heads, G key/value heads, dk / dv per-head key / value sizes, positions 0 .. T-1.
  rms(u)         = u / sqrt(mean(u^2) + eps)
  layer i        : x <- x + ls1 * mixer(rms(x) n1);  x <- x + ls2 * experts(rms(x) n2)
  mixer          : (rms(left(h)) w_l + rms(right(h)) w_r) / 2
  left           : a_g = scale * temp_g * q_g.k_g for every head g;  s_h = sum_g talk[h, g] a_g;  softmax over the keys of the query's own
                   chunk up to the query;  each head's output times sigmoid of one gate number
  right          : S_t = diag(alpha_t) S_{t-1} + k_t v_t^T;  o_t = S_t^T q_t dk^{-1/2};  alpha = sigmoid(A2 (A1 h) + b)^(1/tau)
  experts        : softmax over the chosen experts' logits;  expert: c = min(gate, limit), u = clamp(up, -limit, limit),
                   down (c sigmoid(slope c) (u + 1))
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

SLOPE = 1.702


def rms(u, eps):
    return u / torch.sqrt((u * u).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def rotation_frequencies(rot: dict) -> List[float]:
    """Angle per position of every rotated pair; the long waves are slowed down by `factor`, the short ones kept, a linear blend between."""
    dims, base = int(rot["dims"]), float(rot["base"])
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        s = rot.get("scaling")
        if s:
            wave = 2.0 * math.pi / f
            if wave > s["original"] / s["low"]:
                f = f / s["factor"]
            elif wave >= s["original"] / s["high"]:
                t = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
                f = (1.0 - t) * f / s["factor"] + t * f
        out.append(f)
    return out


def rotate(x, pos, rot: Optional[dict]):
    """x (T, heads, d): entry i of a head's first `dims` entries is turned with entry i + dims/2."""
    if not rot or not rot["dims"]:
        return x
    dims = int(rot["dims"])
    half = dims // 2
    a = pos.to(x.dtype)[:, None] * torch.tensor(rotation_frequencies(rot), dtype=x.dtype)[None, :]
    cos, sin = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], -1)


def visible(i: int, chunk: int) -> int:
    """First key that position i sees."""
    return i // chunk * chunk if chunk > 0 else 0


def mixed_head_attention(q, k, v, scale, temp, talk, chunk, pos0=0):
    """q (L, H, dk) at positions pos0 ..;  k, v (pos0 + L, G, d) -> (L, H, dv), ungated."""
    L, H, _ = q.shape
    G = k.shape[1]
    head_of = torch.arange(H) // (H // G)
    out = torch.zeros(L, H, v.shape[2], dtype=q.dtype)
    for t in range(L):
        i = pos0 + t
        lo = visible(i, chunk)
        a = torch.einsum("hd,jhd->hj", q[t], k[lo:i + 1][:, head_of]) * scale * temp[:, None]
        p = torch.softmax(talk @ a, -1)
        out[t] = torch.einsum("hj,jhd->hd", p, v[lo:i + 1][:, head_of])
    return out


def left_mixer(h, w, m, eps):
    """h (T, D) -> (T, D)."""
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q = rms(h @ w["q"].T + w["q.b"], eps) * w["q.norm"]
    k = rms(h @ w["k"].T + w["k.b"], eps) * w["k.norm"]
    v = (h @ w["v"].T + w["v.b"]).view(T, G, dv)
    q, k = rotate(q.view(T, H, dk), pos, m.get("rot")), rotate(k.view(T, G, dk), pos, m.get("rot"))
    o = mixed_head_attention(q, k, v, m["scale"], w["temp"], w["talk"], int((m.get("mask") or {}).get("size", 0)))
    o = o * torch.sigmoid(h @ w["g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ w["o"].T


def decay_scan(q, k, v, alpha):
    """q, k, alpha (T, H, dk), v (T, H, dv) -> read-outs (T, H, dv)."""
    T, H, dk = q.shape
    S = torch.zeros(H, dk, v.shape[2], dtype=q.dtype)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hkv,hk->hv", S, q[t])
    return out


def right_mixer(h, w, m, eps):
    """h (T, D) -> (T, D)."""
    T = h.shape[0]
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T).view(T, H, dk) * dk ** -0.5
    k = (h @ w["k"].T).view(T, H, dk)
    v = (h @ w["v"].T).view(T, H, dv)
    z = (h @ w["a1"].T) @ w["a2"].T + w["a2.b"]
    alpha = (torch.sigmoid(z) ** (1.0 / m["tau"])).view(T, H, dk)
    o = rms(decay_scan(q, k, v, alpha), eps) * w["norm"]
    return (o.reshape(T, H * dv) * silu(h @ w["g"].T)) @ w["o"].T


def _under(w, pre):
    return {k[len(pre):]: t for k, t in w.items() if k.startswith(pre)}


def parallel_mixer(h, w, m, eps):
    left = rms(left_mixer(h, _under(w, "left."), m["left"], eps), eps) * w["left.out"]
    right = rms(right_mixer(h, _under(w, "right."), m["right"], eps), eps) * w["right.out"]
    return 0.5 * (left + right)


def route(h, w_router, top):
    """h (T, D) -> (T, experts): softmax over the `top` largest logits, zero elsewhere."""
    z = h @ w_router.T
    val, idx = z.topk(top, -1)
    return torch.zeros_like(z).scatter_(1, idx, torch.softmax(val, -1))


def limited_glu(gate, up, limit):
    c = torch.clamp(gate, max=limit)
    return c * torch.sigmoid(SLOPE * c) * (torch.clamp(up, -limit, limit) + 1.0)


def experts_ff(h, w, f):
    wts = route(h, w["router"], int(f["router"]["top"]))
    out = torch.zeros_like(h)
    for e in range(int(f["router"]["experts"])):
        p = f"e{e}."
        out = out + wts[:, e:e + 1] * (limited_glu(h @ w[p + "gate"].T, h @ w[p + "up"].T, float(f["expert"]["limit"])) @ w[p + "down"].T)
    return out


def forward(tokens: List[int], W: Dict[str, torch.Tensor], cfg: dict, dtype=torch.float64, taps: Optional[list] = None):
    """Logits (T, V) of a whole sequence.  taps: receives the stream after every layer."""
    W = {k: t.to(dtype) for k, t in W.items()}
    eps = float(cfg["norm"]["eps"])
    x = W["embed"][torch.tensor(tokens)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + W[p + "ls1"] * parallel_mixer(rms(x, eps) * W[p + "norm1"], _under(W, p + "mix."), layer["mixer"], eps)
        if layer.get("mlp") is not None:
            x = x + W[p + "ls2"] * experts_ff(rms(x, eps) * W[p + "norm2"], _under(W, p + "mlp."), layer["mlp"])
        if taps is not None:
            taps.append(x)
    return (rms(x, eps) * W["final.norm"]) @ W["head"].T


def make_config(mlps=("moe", "moe"), width=64, vocab=97, eps=1e-5, heads=4, kv_heads=2, dim=16, vdim=12, scale=0.3, chunk=24,
                rot_dims=8, rot_base=1000.0, scaling=(8.0, 1.0, 4.0, 64), lin_heads=2, lin_dim=12, lin_vdim=20, tau=8.0,
                experts=6, top=2, expert_ff=24, limit=1.2) -> dict:
    """A small configuration in the checkpoints' own keys; every layer gets the same sizes (tests change single entries)."""
    out = []
    for mlp in mlps:
        left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
        if chunk:
            left["mask"] = {"size": chunk}
        if rot_dims:
            left["rot"] = {"base": rot_base, "dims": rot_dims}
            if scaling:
                left["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
        m = {"left": left, "right": {"heads": lin_heads, "dim": lin_dim, "vdim": lin_vdim, "tau": tau}}
        f = {"kind": "moe", "expert": {"ff": expert_ff, "limit": limit}, "router": {"experts": experts, "top": top}} if mlp == "moe" else None
        out.append({"type": "parallel", "mixer": m, "mlp": f})
    return {"architecture": "Gagotar", "layers": out, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def tensor_shapes(cfg: dict, rank: int = 5) -> Dict[str, tuple]:
    """Checkpoint tensor name -> shape for a configuration; rank: of the decay projection (no entry of the configuration gives it)."""
    d, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, d)}
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        a, s = layer["mixer"]["left"], layer["mixer"]["right"]
        H, G, dk, dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
        l, r = p + "mix.left.", p + "mix.right."
        out.update({p + "norm1": (d,), p + "ls1": (d,), l + "q": (H * dk, d), l + "q.b": (H * dk,), l + "k": (G * dk, d), l + "k.b": (G * dk,), l + "v": (G * dv, d),
                    l + "v.b": (G * dv,), l + "q.norm": (H * dk,), l + "k.norm": (G * dk,), l + "talk": (H, H), l + "temp": (H,), l + "g": (H, d), l + "o": (d, H * dv), l + "out": (d,)})
        H, dk, dv = s["heads"], s["dim"], s["vdim"]
        out.update({r + "q": (H * dk, d), r + "k": (H * dk, d), r + "v": (H * dv, d), r + "g": (H * dv, d), r + "o": (d, H * dv), r + "norm": (dv,),
                    r + "a1": (rank, d), r + "a2": (H * dk, rank), r + "a2.b": (H * dk,), r + "out": (d,)})
        f = layer.get("mlp")
        if f is not None:
            e = f["expert"]["ff"]
            out.update({p + "norm2": (d,), p + "ls2": (d,), p + "mlp.router": (f["router"]["experts"], d)})
            for k in range(f["router"]["experts"]):
                out.update({f"{p}mlp.e{k}.gate": (e, d), f"{p}mlp.e{k}.up": (e, d), f"{p}mlp.e{k}.down": (d, e)})
    out["final.norm"] = (d,)
    out["head"] = (V, d)
    return out


def random_weights(cfg: dict, seed: int = 0, rank: int = 5) -> Dict[str, torch.Tensor]:
    """Random bf16-representable weights of a usable scale."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg, rank).items():
        leaf = name.split(".")[-1]
        if leaf in ("norm1", "norm2", "norm", "out"):
            v = 1.0 + torch.randn(shape, generator=g) * 0.1
        elif name.endswith("a2.b"):
            v = torch.randn(shape, generator=g)
        elif leaf == "b":
            v = torch.randn(shape, generator=g) * 0.3
        elif leaf in ("ls1", "ls2"):
            v = 0.5 + torch.rand(shape, generator=g)
        elif leaf == "temp":
            v = 0.6 + 0.8 * torch.rand(shape, generator=g)
        elif leaf == "talk":
            v = torch.eye(shape[0]) + torch.randn(shape, generator=g) * 0.5
        elif name == "embed":
            v = torch.randn(shape, generator=g)
        elif leaf in ("gate", "up"):
            v = torch.randn(shape, generator=g) * 1.5 / math.sqrt(shape[-1])          # the limits are reached
        elif leaf in ("a1", "a2"):
            v = torch.randn(shape, generator=g) * 1.5 / math.sqrt(shape[-1])
        else:
            v = torch.randn(shape, generator=g) / math.sqrt(shape[-1])
        out[name] = v.to(torch.bfloat16)
    return out
