"""Plain, slow statement of the Nilatar design in PyTorch, one function per mechanism, whole sequences only, float64 by default.
It shares no code with evo_b200: the product is compared against it.

Notation: T tokens, D width, H heads, positions 0 .. T-1.
  rms(u, w)      = u / sqrt(mean(u^2) + eps) * w
  layer i        : x <- x + ls1 * mixer(rms(x, n1));  with a feed-forward also x <- x + ls2 * ff(rms(x, n2))
  latent mixer   : q = Uq rms(Dq h), per head [plain | turned];  [c' | r] = Dkv h, c = rms(c');  per head key [Uk c | turned r], value Uv c
  lightning mixer: q, k, v through silu;  S_t = decay S_{t-1} + k_t v_t^T;  o_t = S_t^T q_t;  one norm over all heads, sigmoid gate
  attention mixer: no rotation, a sliding window, a sink in the softmax denominator, sigmoid gate; a layer may read an earlier layer's keys
  ff             : down (gelu_tanh(gate h) * (up h))
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional, Tuple

import torch


def rms(u, w, eps):
    return u / torch.sqrt((u * u).mean(-1, keepdim=True) + eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def turn_frequencies(rot: dict) -> List[float]:
    """Angle per position of every rotated pair.  With scaling, pair i keeps its frequency while it makes at least `fast` turns within the
    original length, has it divided by `factor` when it makes `slow` turns or fewer, and is blended linearly in i in between."""
    dims, base = int(rot["dims"]), float(rot["base"])
    s = rot.get("scaling")
    out = []
    if s:
        at = lambda turns: dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
        lo, hi = max(math.floor(at(s["fast"])), 0), min(math.ceil(at(s["slow"])), dims - 1)
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if s:
            ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            f = f / s["factor"] * ramp + f * (1.0 - ramp)
        out.append(f)
    return out


def turn_length(rot: dict) -> float:
    """What cosine and sine are multiplied by."""
    s = rot.get("scaling")
    return 0.1 * math.log(s["factor"]) + 1.0 if s else 1.0


def turn(x, rot: Optional[dict], pos0=0):
    """x (T, heads, d): entries 2i and 2i+1 of the first `dims` are a pair, turned by (pos0 + t) * f_i; the rest passes."""
    if not rot or not rot["dims"]:
        return x
    dims = int(rot["dims"])
    pos = torch.arange(pos0, pos0 + x.shape[0], dtype=x.dtype)
    a = pos[:, None] * torch.tensor(turn_frequencies(rot), dtype=x.dtype)
    c, s = (turn_length(rot) * torch.cos(a))[:, None, :], (turn_length(rot) * torch.sin(a))[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2], out[..., 1:dims:2] = u * c - v * s, v * c + u * s
    return out


def softmax_attention(q, k, v, scale, window=0, sink=None, pos0=0):
    """q (L, H, dk) at positions pos0 ..;  k (pos0 + L, G, dk), v (pos0 + L, G, dv) -> (L, H, dv).  window 0: every earlier key."""
    L, H, _ = q.shape
    head = torch.arange(H) // (H // k.shape[1])
    out = torch.zeros(L, H, v.shape[2], dtype=q.dtype)
    for t in range(L):
        i = pos0 + t
        lo = max(0, i - window + 1) if window > 0 else 0
        s = torch.einsum("hd,jhd->hj", q[t], k[lo:i + 1][:, head]) * scale
        if sink is not None:
            s = torch.cat([s, sink.to(s.dtype)[:, None]], 1)
        p = torch.softmax(s, -1)[:, :i + 1 - lo]
        out[t] = torch.einsum("hj,jhd->hd", p, v[lo:i + 1][:, head])
    return out


def window_mixer(h, w, m, eps, kv=None):
    """h (T, D) -> ((T, D), (k, v)).  kv: another layer's keys and values."""
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T).view(T, H, dk)
    if kv is None:
        kv = (h @ w["k"].T).view(T, G, dk), (h @ w["v"].T).view(T, G, dv)
    o = softmax_attention(q, kv[0], kv[1], m["scale"], int((m.get("mask") or {}).get("size", 0)), w["sink"])
    return (o.reshape(T, H * dv) * torch.sigmoid(h @ w["g"].T)) @ w["o"].T, kv


def latent_mixer(h, w, m, eps):
    T = h.shape[0]
    H, dim, rd, dv, rank, rot = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m.get("rot")
    q = (rms(h @ w["dq"].T, w["dq.norm"], eps) @ w["uq"].T).view(T, H, dim + rd)
    q = torch.cat([q[..., :dim], turn(q[..., dim:], rot)], -1)
    down = h @ w["dkv"].T
    c = rms(down[:, :rank], w["dkv.norm"], eps)
    shared = turn(down[:, None, rank:], rot)
    k = torch.cat([(c @ w["uk"].T).view(T, H, dim), shared.expand(T, H, rd)], -1)
    o = softmax_attention(q, k, (c @ w["uv"].T).view(T, H, dv), m["scale"])
    return (o.reshape(T, H * dv) * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def decay_scan(q, k, v, decay, state=None):
    """q, k (T, H, dk), v (T, H, dv), decay (H) -> read-outs (T, H, dv), last state (H, dk, dv)."""
    T, H, dk = q.shape
    S = torch.zeros(H, dk, v.shape[2], dtype=q.dtype) if state is None else state
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hkv,hk->hv", S, q[t])
    return out, S


def lightning_mixer(h, w, m, eps):
    T = h.shape[0]
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    q, k, v = silu(h @ w["q"].T).view(T, H, dk), silu(h @ w["k"].T).view(T, H, dk), silu(h @ w["v"].T).view(T, H, dv)
    o, _ = decay_scan(q, k, v, torch.tensor(m["decay"], dtype=h.dtype))
    return (rms(o.reshape(T, H * dv), w["norm"], eps) * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def dense_ff(h, w):
    return (gelu_tanh(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def _under(w, pre):
    return {k[len(pre):]: t for k, t in w.items() if k.startswith(pre)}


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float64) -> Tuple[torch.Tensor, List[torch.Tensor]]:
    """-> logits (T, V), the stream after every layer."""
    w = {k: t.to(dtype) for k, t in weights.items()}
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][torch.as_tensor(tokens)] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    taps, held = [], {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        lw = _under(w, p)
        h, mw = rms(x, lw["norm1"], eps), _under(lw, "mix.")
        kind = layer["type"].rstrip("0123456789_")
        if kind == "attention":
            y, held[i] = window_mixer(h, mw, m, eps, held[m["kv_from"]] if m.get("kv_from") is not None else None)
        else:
            y = {"latent_attention": latent_mixer, "lightning": lightning_mixer}[kind](h, mw, m, eps)
        x = x + y * lw["ls1"]
        if layer["mlp"] is not None:
            x = x + dense_ff(rms(x, lw["norm2"], eps), _under(lw, "mlp.")) * lw["ls2"]
        taps.append(x)
    return rms(x, w["final.norm"], eps) @ w["head"].T, taps


def generate_greedy(cfg, weights, prompt, n, dtype=torch.float64):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(cfg, weights, toks, dtype)[0][-1].argmax()))
    return toks[len(prompt):]


def make_weights(cfg: dict, seed: int = 0) -> Dict[str, torch.Tensor]:
    """Random bf16 weights of a usable scale under the checkpoint's names."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g)
    lin = lambda n, k: rnd(n, k) / math.sqrt(k)
    gain = lambda n: 1.0 + 0.2 * rnd(n)
    D, V = cfg["width"], cfg["vocab"]
    w = {"embed": rnd(V, D) / float((cfg.get("embedding") or {}).get("scale", 1.0))}
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer["mlp"]
        kind, x, H, dv = layer["type"].rstrip("0123456789_"), f"l{i}.mix.", layer["mixer"]["heads"], layer["mixer"]["vdim"]
        w[p + "norm1"], w[p + "ls1"] = gain(D), 0.5 + torch.rand(D, generator=g)
        w[x + "g"], w[x + "o"] = lin(H * dv, D), lin(D, H * dv)
        if kind == "attention":
            w[x + "q"], w[x + "sink"] = 2.0 * lin(H * m["dim"], D), 1.0 + rnd(H)
            if m.get("kv_from") is None:
                w[x + "k"], w[x + "v"] = lin(m["kv_heads"] * m["dim"], D), lin(m["kv_heads"] * dv, D)
        elif kind == "latent_attention":
            rank, qr = m["kv_rank"], m["q_rank"]
            w[x + "dq"], w[x + "dq.norm"], w[x + "uq"] = lin(qr, D), gain(qr), 2.0 * lin(H * (m["dim"] + m["rot_dim"]), qr)
            w[x + "dkv"], w[x + "dkv.norm"] = lin(rank + m["rot_dim"], D), gain(rank)
            w[x + "uk"], w[x + "uv"] = lin(H * m["dim"], rank), lin(H * dv, rank)
        else:
            w[x + "q"], w[x + "k"], w[x + "v"], w[x + "norm"] = lin(H * m["dim"], D), lin(H * m["dim"], D), lin(H * dv, D), gain(H * dv)
        if f is not None:
            w[p + "norm2"], w[p + "ls2"] = gain(D), 0.5 + torch.rand(D, generator=g)
            w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"] = lin(f["ff"], D), lin(f["ff"], D), lin(D, f["ff"])
    w["final.norm"], w["head"] = gain(D), lin(V, D)
    return {k: t.to(torch.bfloat16) for k, t in w.items()}


def make_config(kinds=("attention", "latent_attention", "lightning", "shared"), ff=(40, 40, 0, 40), width=64, vocab=101, eps=1e-5, embed_scale=4.0,
                heads=4, kv_heads=2, dim=16, vdim=12, window=24, scale=0.3,
                lat_heads=3, lat_dim=8, rot_dim=12, lat_vdim=20, kv_rank=24, q_rank=28, lat_scale=0.25, rot_base=1000.0, scaling=(4.0, 64, 8.0, 1.0),
                lin_heads=2, lin_dim=12, lin_vdim=24, decay=None) -> dict:
    """A small configuration; "shared" is an attention layer that reads the keys and values of the last attention layer before it."""
    decay = decay or [1.0 - 0.5 ** (h + 1) for h in range(lin_heads)]
    layers, source = [], None
    for i, kind in enumerate(kinds):
        if kind == "latent_attention":
            rot = {"base": rot_base, "dims": rot_dim}
            if scaling:
                rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
            m = {"heads": lat_heads, "dim": lat_dim, "rot_dim": rot_dim, "vdim": lat_vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": lat_scale, "rot": rot}
        elif kind == "lightning":
            m = {"heads": lin_heads, "dim": lin_dim, "vdim": lin_vdim, "decay": list(decay)}
        else:
            m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": window}}
            if kind == "shared":
                m["kv_from"] = source
            else:
                source = i
        layers.append({"type": "attention" if kind == "shared" else kind, "mixer": m, "mlp": {"kind": "dense", "ff": ff[i]} if ff[i] else None})
    return {"architecture": "Nilatar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embed_scale}, "layers": layers}
