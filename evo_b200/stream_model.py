"""Shared base of the model families that keep the residual stream in fp32 and are described by a flat table of checkpoint
tensors (Zaverax, Movalorn, Nelovik, Gakupel, Gagotar, Nilatar): weight holding and strict loading, the padded GEMM weights, the linear-layer dispatch
(tcgen05 GEMMs for bf16 activations, the CUDA-core fp32 GEMM for the all-fp32 mode), the inference-state holders, the
forward protocol and the on-device generation loop.  A family provides `_ensure_packed()` and
`_body(ids, B, L, state, offset, pos_dev=None, rows=None) -> fp32 logits`; everything that drives a model -- the generation loop,
the scheduler, the trace replay, the command line -- talks to the methods defined here.

Protocol (the same as StripedHyena's):
    model(ids) -> (logits, None)                          stateless, whole sequences
    model(ids, inference_params_dict=d) -> (logits, d)    continues from the caches in d at d["mha"].seqlen_offset
    model.initialize_inference_params()                   the framework's two state holders
    model.decode_loop(...)                                one CUDA graph per generated token
State is keyed by RUN index (a looped layer has one entry per pass): d["mha"].key_value_memory_dict[r] for caches that grow
with the sequence, d["hyena"].state_dict[r] / fir_state_dict[r] for fixed-size recurrent state.
"""
from __future__ import annotations

import ctypes as C
import os
from typing import Dict, Optional

import torch
import torch.nn as nn

from . import _lib
from ._lib import (EPI_GELU_TANH_GATE, EPI_NONE, EPI_SILU_COLS, ConvActParams, GatedDeltaParams, GluActParams, LatentDecodeParams, LatentPrepParams, MoeRouteParams, SumNormParams, WindowAttnParams,
                   check, ptr)
from .engine import KernelOps
from .stripedhyena.cache import InferenceParams, RecurrentInferenceParams


ABSORBED_MAX_ROWS = 4         # latent attention: portions up to this many tokens attend straight from the latent cache


def _round_up(x: int, m: int) -> int:
    return (x + m - 1) // m * m


class _Packed:
    """A linear layer's weight in the GEMMs' layout: (Np, Kp) bf16, zero rows / columns past (N, K)."""

    def __init__(self, w: torch.Tensor, k_tile: int = 64):
        self.N, self.K = w.shape
        self.Np, self.Kp = _round_up(self.N, 256), _round_up(self.K, k_tile)
        self.w = torch.zeros(self.Np, self.Kp, dtype=torch.bfloat16, device=w.device)
        self.w[:self.N, :self.K] = w.to(torch.bfloat16)


class _PackedGate(_Packed):
    """The gate and up weights of a gated feed-forward, (F, K) each, as one linear layer whose rows alternate in runs of RUN, [gate | up]:
    both halves of a product land in one tile of the GEMM, whose epilogue can then store act(gate) * up, (M, Fp)."""
    RUN = 128

    def __init__(self, gate: torch.Tensor, up: torch.Tensor):
        self.F, K = gate.shape
        self.Fp, self.Kp = _round_up(self.F, self.RUN), _round_up(K, 64)
        self.N = self.Np = 2 * self.Fp
        self.K = K
        self.w = torch.zeros(self.Np, self.Kp, dtype=torch.bfloat16, device=gate.device)
        runs = self.w.view(self.Fp // self.RUN, 2, self.RUN, self.Kp)
        for half, src in enumerate((gate, up)):
            full = torch.zeros(self.Fp, self.Kp, dtype=torch.bfloat16, device=gate.device)
            full[:self.F, :K] = src.to(torch.bfloat16)
            runs[:, half] = full.view(-1, self.RUN, self.Kp)


class StreamDecoder(KernelOps, nn.Module):
    architecture = None
    gemm_env = "EVO_B200_STREAM_GEMM"          # "simt": linear layers of the bf16 path on the CUDA-core GEMM (comparator)
    fir_taps = 0                               # taps of a short convolution whose carried rows live in the recurrent holder

    def __init__(self, config, dtype: torch.dtype = torch.bfloat16):
        super().__init__()
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("activation dtype must be torch.bfloat16 or torch.float32")
        self.config = config
        self.act_dtype = dtype
        self.weights: Dict[str, torch.Tensor] = {}
        for name, shape in config.tensor_shapes().items():
            self.weights[name] = torch.zeros(shape, dtype=torch.bfloat16)
        self._packed = None
        # linear layers of the bf16 path: "tc" = tcgen05 GEMMs, "simt" = the CUDA-core GEMM (comparator)
        self.gemm_path = os.environ.get(self.gemm_env, "tc")
        self.gemm_variant = int(os.environ.get("EVO_B200_GEMM_VARIANT", "0"))
        self.gemm_variant_gate = self.gemm_variant
        # few-row latent attention: "shared" = heads share each tile of latents (three launches), "head" = one CTA per (query, head)
        self.latent_decode_path = os.environ.get("EVO_B200_LATENT_DECODE", "shared")
        self.decode_graph = os.environ.get("EVO_B200_DECODE_GRAPH", "1") != "0"
        self._smallm_ws = None
        self._decode = None
        self._loop = None
        self._prof = None
        self._tap = None          # set to a list: receives the fp32 stream after every run (bring-up / tests)

    # ---- parameters ----------------------------------------------------------------------------
    def state_dict(self, *a, **kw):
        return dict(self.weights)

    def load_state_dict(self, state_dict, strict: bool = True, **kw):
        missing = [k for k in self.weights if k not in state_dict]
        unexpected = [k for k in state_dict if k not in self.weights]
        errors = []
        for k, v in state_dict.items():
            if k in self.weights:
                if tuple(v.shape) != tuple(self.weights[k].shape):
                    errors.append(f"size mismatch for {k}: checkpoint {tuple(v.shape)}, model {tuple(self.weights[k].shape)}")
                else:
                    self.weights[k] = v.to(device=self.weights[k].device, dtype=torch.bfloat16).contiguous()
        if errors or (strict and (missing or unexpected)):
            raise RuntimeError(f"Error(s) in loading state_dict for {type(self).__name__}: missing {missing}, unexpected {unexpected}, {errors}")
        self._invalidate()
        return missing, unexpected

    def _invalidate(self):
        self._packed = None
        self._decode = None
        self._loop = None

    def _apply(self, fn, *a, **kw):
        out = super()._apply(fn, *a, **kw)
        for k, v in self.weights.items():
            moved = fn(v)
            self.weights[k] = moved if moved.dtype == torch.bfloat16 else moved.to(torch.bfloat16)      # .float() / .half() do not apply to the checkpoint's bf16
        self._invalidate()
        return out

    @property
    def device(self):
        return self.weights["embed"].device

    def eval(self):
        return self

    def _ensure_packed(self):
        raise NotImplementedError

    def _body(self, ids, B, L, ipd, off: int, pos_dev=None, rows=None):
        raise NotImplementedError

    # ---- state -----------------------------------------------------------------------------------
    def initialize_inference_params(self, max_seqlen: Optional[int] = None, max_batch_size: Optional[int] = None):
        return {
            "mha": InferenceParams(max_seqlen=max_seqlen or self.config.max_seqlen, max_batch_size=max_batch_size or self.config.max_batch_size, seqlen_offset=0),
            "hyena": RecurrentInferenceParams(fir_filter_length=self.fir_taps, state_dim=0, seqlen_offset=0),
        }

    def _kv_rows(self, ip: InferenceParams, r: int, width: int, B: int, off: int, L: int, pos_dev=None):
        """The cache of run r, (max_batch, max_seqlen, width) in the activation dtype, zero-filled: allocated on first use and
        doubled (outside a captured step) when rows [off, off + L) would not fit.  Rows are never overwritten or moved within a
        sequence, so a window only limits what the kernels read."""
        cache = ip.key_value_memory_dict.get(r)
        dev = self.device
        if cache is None:
            cache = ip.key_value_memory_dict[r] = torch.zeros(ip.max_batch_size, max(ip.max_seqlen, off + L), width, dtype=self.act_dtype, device=dev)
        if B > cache.shape[0]:
            raise _lib.EvoError(f"KV cache too small: batch {B} > {cache.shape[0]}")
        if off + L > cache.shape[1]:
            if pos_dev is not None:             # inside a captured step the cache cannot move
                raise _lib.EvoError(f"KV cache too small: length {off + L} > {cache.shape[1]}")
            grown = torch.zeros(cache.shape[0], max(off + L, 2 * cache.shape[1]), width, dtype=self.act_dtype, device=dev)
            grown[:, :off] = cache[:, :off]
            cache = ip.key_value_memory_dict[r] = grown
            ip.max_seqlen = max(ip.max_seqlen, cache.shape[1])
        return cache

    def _cache_tokens(self, key, cache) -> int:
        """Tokens of a sequence that the cache under `key` has room for (a family that keeps one row per several tokens overrides this)."""
        return cache.shape[1]

    # ---- kernels ---------------------------------------------------------------------------------
    @property
    def _dt(self) -> int:
        return 1 if self.act_dtype == torch.float32 else 0

    @property
    def _fused(self) -> bool:
        """Whether linear layers run on the tensor-core GEMMs, whose epilogues can apply an activation."""
        return not self._dt and self.gemm_path != "simt"

    def _linear(self, a, pk: _Packed, M: int, out=None, silu_cols=0):
        """(M, Kp) activations -> (M, Np): rows of A are padded with zeros up to Kp by their producers.  out: rows of a (.., Np) buffer to fill.
        silu_cols: the first columns go through silu in the GEMM's epilogue (only where self._fused; other callers apply it themselves)."""
        assert not silu_cols or self._fused
        epi = EPI_SILU_COLS if silu_cols else EPI_NONE
        if out is None:
            out = torch.empty(M, pk.Np, dtype=self.act_dtype, device=a.device)
        if self._dt or self.gemm_path == "simt":
            self._record(f"gemm_simt/{pk.N}x{pk.K}", 2.0 * M * pk.N * pk.K, lambda: check(_lib.lib().evo_gemm_simt(
                ptr(a), pk.Kp, ptr(pk.w), pk.Kp, ptr(out), pk.Np, M, pk.N, pk.K, self._dt, self._stream()), "evo_gemm_simt"))
        elif M <= 64:
            self._gemm_smallm(a, pk.w, out, M, pk.Np, pk.Kp, epi, act_cols=silu_cols)
        else:
            self._gemm(a, pk.w, out, M, pk.Np, pk.Kp, epi, variant=2 if M <= 512 else self.gemm_variant, act_cols=silu_cols)
        return out

    def _gelu_gate(self, h, pk: _PackedGate, M: int):
        """gelu_tanh(gate h) * (up h) -> (M, Fp), columns past F zero: in the GEMM's epilogue, or by a second kernel behind the fp32 / comparator GEMM."""
        a = torch.empty(M, pk.Fp, dtype=self.act_dtype, device=h.device)
        if not self._fused:
            z = self._linear(h, pk, M)
            self._glu(z.data_ptr(), z.data_ptr() + pk.RUN * z.element_size(), pk.Np, a, pk.Fp, M, pk.F, 0, interleave=pk.RUN)
        elif M <= 64:
            self._gemm_smallm(h, pk.w, a, M, pk.Np, pk.Kp, EPI_GELU_TANH_GATE)
        else:
            self._gemm(h, pk.w, a, M, pk.Np, pk.Kp, EPI_GELU_TANH_GATE, ldc=pk.Fp, variant=1 if M <= 512 else self.gemm_variant)
        return a

    # ---- row kernels and mixers shared by several families -----------------------------------------
    def _sum_norm(self, x, branches, outs, rows, gather=None, col_scale=None):
        """x += col_scale * sum of the branches (y, ldy, norm weight or None, scale); outs: [(buffer, weight)] normed copies of the new x."""
        cfg = self.config
        p = SumNormParams(x=x.data_ptr(), n_branches=len(branches), eps=cfg.eps, dtype=self._dt, rows=rows, D=cfg.width,
                          gather=gather.data_ptr() if gather is not None else None, ldo=_round_up(cfg.width, 64),
                          col_scale=col_scale.data_ptr() if col_scale is not None else None)
        for b, (y, ldy, nw, scale) in enumerate(branches):
            p.y[b], p.ldy[b], p.norm_w[b], p.scale[b] = y.data_ptr(), ldy, (nw.data_ptr() if nw is not None else None), scale
        for n, (o, wt) in enumerate(outs):
            p.out[n], p.w[n] = o.data_ptr(), wt.data_ptr()
        esz = 4 if self._dt else 2
        nbytes = rows * cfg.width * (8.0 + esz * (len(branches) + len(outs)))
        self._record("sum_norm", nbytes, lambda: check(_lib.lib().evo_sum_norm(C.byref(p), self._stream()), "evo_sum_norm"))

    def _glu(self, z_ptr, up_ptr, ld, out, ldo, rows, F, act, limit=0.0, slope=1.0, route=None, group=0, n_groups=0, tail_w=0, interleave=0):
        """out (rows, ldo) = act(gate) * up [* routing weight of the column's expert] (see evo_glu_act)."""
        p = GluActParams(gate=z_ptr, up=up_ptr, ld=ld, out=out.data_ptr(), ldo=ldo, rows=rows, F=F, act=act, dtype=self._dt, limit=limit, slope=slope, interleave=interleave)
        if route is not None:
            p.group_w, p.ldw, p.group, p.n_groups, p.tail_w = route.data_ptr(), route.shape[1], group, n_groups, tail_w
        self._record("glu_act", 3.0 * out.element_size() * rows * F, lambda: check(_lib.lib().evo_glu_act_ex(C.byref(p), self._stream()), "evo_glu_act"))

    def _moe_route(self, h, M, router_w, E, top, correction=None, chosen=None, **kw):
        """Routing weights (M, E + n_extra) fp32 from rows h (M, Kp); kw: further fields of evo_moe_route_params."""
        n_extra = kw.get("n_extra", 0)
        route = torch.empty(M, E + n_extra, dtype=torch.float32, device=h.device)
        rp = MoeRouteParams(h=h.data_ptr(), ldh=h.shape[1], router_w=router_w.data_ptr(), correction=correction.data_ptr() if correction is not None else None,
                            weights=route.data_ptr(), ldw=E + n_extra, chosen=chosen.data_ptr() if chosen is not None else None,
                            rows=M, D=self.config.width, E=E, top=top, dtype=self._dt, **kw)
        self._record("moe_route", float(M) * self.config.width * h.element_size(), lambda: check(_lib.lib().evo_moe_route_ex(C.byref(rp), self._stream()), "evo_moe_route"))
        return route

    def _conv(self, r, src_ptr, ld, weight, bias, channels, taps, B, L, rec, fresh):
        """SiLU(short convolution) of `channels` columns starting at src_ptr -> (B*L, channels); the carried inputs live in rec.fir_state_dict[r]."""
        dev = weight.device
        out = torch.empty(B * L, channels, dtype=self.act_dtype, device=dev)
        carry, zero = None, 1
        if taps > 1:
            carry = rec.fir_state_dict.get(r)
            zero = 0
            if carry is None or fresh:
                if carry is None:
                    carry = rec.fir_state_dict[r] = torch.empty(B, taps - 1, channels, dtype=torch.float32, device=dev)
                zero = 1
        cp = ConvActParams(inp=src_ptr, ld=ld, weight=weight.data_ptr(), bias=bias.data_ptr() if bias is not None else None,
                           carry=carry.data_ptr() if carry is not None else None, zero_start=zero, out=out.data_ptr(), ldo=channels,
                           B=B, L=L, C=channels, taps=taps, act=1, dtype=self._dt)
        self._record("conv_act", 2.0 * out.element_size() * B * L * channels, lambda: check(_lib.lib().evo_conv_act(C.byref(cp), self._stream()), "evo_conv_act"))
        return out

    def _matrix_state(self, r, rec, B, H, dk, dv, fresh):
        state = rec.state_dict.get(r)
        if state is None:
            state = rec.state_dict[r] = torch.empty(B, H, dk, dv, dtype=torch.float32, device=self.device)
            return state, 1
        return state, 1 if fresh else 0

    def _delta_mixer(self, r, i, m, h, B, L, rec, fresh):
        """Gated delta rule of layer i (tensors l<i>.mix.*; m: heads, kv_heads, dim, vdim, taps) on h (M, Kp) -> (output projection, its row stride)."""
        pk = self._packed["layers"][i]
        M, dev = B * L, h.device
        w = self.weights
        z = self._linear(h, pk["in"], M)
        esz, ldz = z.element_size(), pk["in"].Np
        qk, vw = m.kv_heads * m.dim, m.heads * m.vdim
        cw = 2 * qk + vw
        c = self._conv(r, z.data_ptr(), ldz, pk["conv"], None, cw, m.taps, B, L, rec, fresh)
        state, zero = self._matrix_state(r, rec, B, m.heads, m.dim, m.vdim, fresh)
        ldo = _round_up(vw, 64)
        out = torch.empty(M, ldo, dtype=self.act_dtype, device=dev)
        p = f"l{i}.mix."
        gp = GatedDeltaParams(q=c.data_ptr(), k=c.data_ptr() + qk * esz, v=c.data_ptr() + 2 * qk * esz, ld=cw,
                              b=z.data_ptr() + (cw + vw) * esz, a=z.data_ptr() + (cw + vw + m.heads) * esz, gate=z.data_ptr() + cw * esz, ldz=ldz,
                              A_log=w[p + "A_log"].data_ptr(), dt_bias=w[p + "dt_bias"].data_ptr(), norm_w=w[p + "norm"].data_ptr(),
                              eps=self.config.eps, unit_eps=1e-6, q_scale=m.dim ** -0.5, state=state.data_ptr(), zero_start=zero,
                              out=out.data_ptr(), ldo=ldo, dtype=self._dt, B=B, L=L, H=m.heads, G=m.kv_heads, dk=m.dim, dv=m.vdim)
        nws = _lib.lib().evo_gated_delta_workspace(C.byref(gp))
        ws = torch.empty(nws, dtype=torch.uint8, device=dev) if nws else None
        self._record("gated_delta", 4.0 * M * m.heads * m.dim * m.vdim, lambda: check(_lib.lib().evo_gated_delta_fwd(C.byref(gp), ptr(ws), nws, self._stream()), "evo_gated_delta_fwd"))
        return self._linear(out, pk["out"], M), pk["out"].Np

    # ---- latent attention: m has heads, dim, rot_dim, vdim, kv_rank, rot_dims, scale, window (0: every earlier key)
    def _pack_latent(self, m, uk, uv):
        """Expansion of cache rows [latent | 0.. | rotated key part] into per-head keys [Uk_h c | rotated part] and values Uv_h c as one
        linear layer: identity rows carry the shared rotated part into every head's key."""
        dev, hd, rank_pad = uk.device, m.dim + m.rot_dim, _round_up(m.kv_rank, 8)
        up = torch.zeros(m.heads * hd + m.heads * m.vdim, rank_pad + m.rot_dim, dtype=torch.bfloat16, device=dev)
        for h in range(m.heads):
            up[h * hd:h * hd + m.dim, :m.kv_rank] = uk[h * m.dim:(h + 1) * m.dim]
            up[h * hd + m.dim:(h + 1) * hd, rank_pad:] = torch.eye(m.rot_dim, dtype=torch.bfloat16, device=dev)
        up[m.heads * hd:, :m.kv_rank] = uv
        expand = _Packed(up)
        return {"expand": expand, "rank_pad": rank_pad, "cache_row": expand.Kp}

    def _latent_prep(self, m, freq, rot_len, B, L, off, pos_dev, **part):
        pp = LatentPrepParams(eps=self.config.eps, freq=freq.data_ptr() if freq is not None else None, rot_len=rot_len, B=B, L=L, H=m.heads, dim=m.dim, rot=m.rot_dim,
                              rank=m.kv_rank, pos0=off, pos_dev=pos_dev.data_ptr() if pos_dev is not None else None, dtype=self._dt, rot_dims=m.rot_dims, **part)
        hd, esz = m.dim + m.rot_dim, 4 if self._dt else 2
        moved = (m.heads * (hd if part.get("dkv") else 2 * m.rot_dim) if part.get("q") else 0) + (2 * (m.kv_rank + m.rot_dim) if part.get("dkv") else 0) + 2 * part.get("q_rank", 0)
        self._record("latent_prep", float(B * L) * moved * esz, lambda: check(_lib.lib().evo_latent_prep(C.byref(pp), self._stream()), "evo_latent_prep"))

    def _latent_rows(self, r, m, lat, dkv_ptr, ld_dkv, norm_w, freq, rot_len, B, L, ip, off, pos_dev, q=None, query=None):
        """Latents (normed) and turned key parts of the call's tokens -> rows of run r's cache, which is returned.  q (pointer, row
        stride): queries whose rotated parts are turned in the same launch; query (pointer, row stride, norm weight, rank, out): the
        queries' own latent, normed into out."""
        row = lat["cache_row"]
        cache = torch.zeros(B, L, row, dtype=self.act_dtype, device=self.device) if ip is None else self._kv_rows(ip, r, row, B, off, L, pos_dev)
        part = dict(dkv=dkv_ptr, ld_dkv=ld_dkv, norm_w=norm_w.data_ptr(), cache=cache.data_ptr(), cache_row=row, cache_batch_stride=cache.shape[1] * row, rank_pad=lat["rank_pad"])
        if q is not None:
            part.update(q=q[0], ldq=q[1])
        if query is not None:
            part.update(dq=query[0], ld_dq=query[1], dq_norm_w=query[2].data_ptr(), q_rank=query[3], cq=query[4].data_ptr(), ld_cq=query[4].shape[1])
        self._latent_prep(m, freq, rot_len, B, L, off, pos_dev, **part)
        return cache

    def _latent_turn(self, m, q, ldq, freq, rot_len, B, L, off, pos_dev):
        """Turns the rotated parts of queries that were not there yet when the cache rows were written."""
        if m.rot_dims:
            self._latent_prep(m, freq, rot_len, B, L, off, pos_dev, q=q.data_ptr(), ldq=ldq)

    @staticmethod
    def _mean_keys(off, L, window):
        """Keys that a query at positions off .. off + L - 1 sees on average."""
        if window <= 0 or off + L <= window:
            return off + (L + 1) / 2.0
        ramp = max(0, min(L, window - off))           # queries whose window still reaches the sequence's start
        return (ramp * (off + (ramp + 1) / 2.0) + (L - ramp) * float(window)) / L

    def _latent_attend(self, m, lat, q_ptr, ldq, cache, uk, uv, gate_ptr, ld_gate, gate_per_channel, B, L, off, pos_dev):
        """Prepared queries against the latent cache -> (B*L, heads*vdim padded), gated.  Steps and short portions stay in the latent space
        (absorbed form); longer ones expand the visible rows into keys and values first."""
        lib, dev, esz, M = _lib.lib(), cache.device, cache.element_size(), B * L
        row, bstride, hd = lat["cache_row"], cache.shape[1] * lat["cache_row"], m.dim + m.rot_dim
        pos_ptr = pos_dev.data_ptr() if pos_dev is not None else None
        ldo = _round_up(m.heads * m.vdim, 64)
        out = torch.empty(M, ldo, dtype=self.act_dtype, device=dev)
        span = self._mean_keys(off, L, m.window)
        if L <= ABSORBED_MAX_ROWS or pos_dev is not None:
            dp = LatentDecodeParams(q=q_ptr, ldq=ldq, cache=cache.data_ptr(), cache_row=row, cache_batch_stride=bstride, rank_pad=lat["rank_pad"],
                                    uk=uk.data_ptr(), uv=uv.data_ptr(), gate=gate_ptr, ld_gate=ld_gate, gate_per_channel=int(gate_per_channel),
                                    out=out.data_ptr(), ldo=ldo, B=B, Lq=L, H=m.heads, dim=m.dim, rot=m.rot_dim, rank=m.kv_rank, vdim=m.vdim,
                                    pos0=off, pos_dev=pos_ptr, window=m.window, scale=m.scale, dtype=self._dt,
                                    max_keys=cache.shape[1] if pos_dev is not None else off + L)
            nws = lib.evo_latent_attn_decode_workspace(C.byref(dp)) if self.latent_decode_path == "shared" else 0
            ws = torch.empty(nws, dtype=torch.uint8, device=dev) if nws else None
            # roofline bytes: each sequence's visible latents once (all heads share them)
            self._record("latent_decode", float(M) * span * (m.kv_rank + m.rot_dim) * esz,
                         lambda: check(lib.evo_latent_attn_decode(C.byref(dp), ptr(ws), nws, self._stream()), "evo_latent_attn_decode"))
            return out
        lo = max(0, off - (m.window - 1)) if m.window > 0 else 0
        n, ex = off + L - lo, lat["expand"]
        kv = torch.empty(B, n, ex.Np, dtype=self.act_dtype, device=dev)
        for b in range(B):
            self._linear(cache[b, lo:off + L], ex, n, out=kv[b])
        ap = WindowAttnParams(q=q_ptr, q_tok_stride=ldq, gate=gate_ptr, gate_tok_stride=ld_gate, gate_per_head=0 if gate_per_channel else 1,
                              k=kv.data_ptr() - lo * ex.Np * esz, v=kv.data_ptr() + (m.heads * hd - lo * ex.Np) * esz,
                              k_tok_stride=ex.Np, v_tok_stride=ex.Np, k_batch_stride=n * ex.Np, v_batch_stride=n * ex.Np,
                              out=out.data_ptr(), ldo=ldo, dtype=self._dt, B=B, Lq=L, H=m.heads, G=m.heads, dk=hd, dv=m.vdim, n_maps=1,
                              q_pos0=off, window=m.window, keep_first=0, scale=m.scale, norm_eps=self.config.eps, out_scale=1.0)
        self._record("window_attn", 2.0 * M * m.heads * span * (hd + m.vdim),
                     lambda: check(lib.evo_window_attn_fwd(C.byref(ap), self._stream()), "evo_window_attn_fwd"))
        return out

    def _run_chosen_experts(self, h, M, chosen, experts, ff, E, top, **act):
        """Only the chosen experts of a mixture: the (token, choice) pairs of `chosen` (M, top) int32 are sorted by expert, and every
        expert ([gate ; up] and down weights, packed, hidden size ff; act: form and constants of the gate, SiLU by default) runs on its slice of the gathered rows of h (M, Kp).
        Returns (ys, slot_of): the experts' outputs in sorted order and the slot of every pair, for evo_moe_combine.  The per-expert
        row counts come back to the host (one round trip), so this does not run inside a captured step."""
        dev, lib = h.device, _lib.lib()
        n, esz = M * top, h.element_size()
        counts = torch.zeros(2, E, dtype=torch.int32, device=dev)                      # row 0: counts, row 1: the scatter's cursors
        check(lib.evo_moe_count(ptr(chosen), n, E, ptr(counts), self._stream()), "evo_moe_count")
        cnt = counts[0].cpu()                                                           # the one host round trip of the layer
        off = torch.zeros(E + 1, dtype=torch.int64)
        off[1:] = torch.cumsum(cnt.to(torch.int64), 0)
        offsets = off[:E].to(torch.int32).to(dev)
        total = int(off[E])
        perm = torch.empty(max(total, 1), dtype=torch.int32, device=dev)
        slot_of = torch.empty(M, top, dtype=torch.int32, device=dev)
        check(lib.evo_moe_scatter(ptr(chosen), n, top, E, ptr(offsets), C.c_void_p(counts.data_ptr() + 4 * E), ptr(perm), ptr(slot_of), self._stream()), "evo_moe_scatter")
        Kp = h.shape[1]
        hs = torch.empty(max(total, 1), Kp, dtype=self.act_dtype, device=dev)
        self._record("moe_gather", 2.0 * total * Kp * esz, lambda: check(lib.evo_gather_rows(ptr(h), Kp * esz, ptr(hs), Kp * esz, ptr(perm), total, Kp * esz, self._stream()), "evo_gather_rows"))
        down0 = experts[0][1]
        ys = torch.empty(max(total, 1), down0.Np, dtype=self.act_dtype, device=dev)
        for e in range(E):
            lo, ne = int(off[e]), int(cnt[e])
            if ne == 0:
                continue
            up, down = experts[e]
            z = self._linear(hs[lo:lo + ne], up, ne)
            a = torch.empty(ne, down.Kp, dtype=self.act_dtype, device=dev)
            self._glu(z.data_ptr(), z.data_ptr() + ff * esz, up.Np, a, down.Kp, ne, ff, **(act or {"act": 1}))
            self._linear(a, down, ne, out=ys[lo:lo + ne])
        return ys, slot_of

    # ---- forward ---------------------------------------------------------------------------------
    def forward(self, x, inference_params_dict=None, padding_mask=None, logits_rows=None):
        """ids (B, L) -> (fp32 logits (B, L, V), state).  With a state dict the call continues every sequence at
        state["mha"].seqlen_offset (the caller advances it, as the framework's generation loop does).
        logits_rows: flat indices into the (B*L) rows whose logits are wanted -> logits (len, V)."""
        if padding_mask is not None:
            raise NotImplementedError("padding_mask is not supported")
        if x.dim() != 2 or x.dtype not in (torch.int32, torch.int64):
            raise TypeError("input ids must be (batch, length) int32/int64")
        self._ensure_packed()
        dev = self.device
        if x.device != dev:
            raise _lib.EvoError(f"input ids on {x.device}, model on {dev}")
        x = x.contiguous()
        B, L = x.shape
        off = int(inference_params_dict["mha"].seqlen_offset) if inference_params_dict is not None else 0
        with torch.cuda.device(dev), torch.no_grad():
            rows = None
            if logits_rows is not None:
                rows = torch.as_tensor(logits_rows, dtype=torch.int64, device=dev).contiguous()
            logits = self._body(x, B, L, inference_params_dict, off, rows=rows)
        if rows is not None:
            return logits, inference_params_dict
        return logits.view(B, L, -1), inference_params_dict

    # ---- on-device generation loop: the whole step + token pick as one CUDA graph ------------------
    def decode_loop(self, first_token, ipd, n_steps, start_pos, *, top_k=1, top_p=0.0, temperature=1.0, forced=None, n_out=None, seed=None):
        """`n_steps` single-token steps without returning to the host: same contract as StripedHyena.decode_loop
        (step i feeds the token of step i-1; forced[:, i] while i < forced.shape[1], then picked on the device)."""
        lib = _lib.lib()
        dev = self.device
        x = first_token.reshape(-1, 1).contiguous()
        B, V = x.shape[0], self.config.vocab_size
        if V > 1024:
            raise _lib.EvoError("the device sampler handles vocabularies up to 1024; use the per-token host loop")
        mha_ip, rec = ipd["mha"], ipd["hyena"]
        n_forced = 0 if forced is None else int(forced.shape[1])
        n_out = n_steps - n_forced if n_out is None else n_out
        if n_out < 0:
            raise ValueError("more forced tokens than steps")
        for k, c in mha_ip.key_value_memory_dict.items():
            if start_pos + n_steps > self._cache_tokens(k, c):
                raise _lib.EvoError(f"sequence length {start_pos + n_steps} exceeds the KV cache ({self._cache_tokens(k, c)})")
        with torch.cuda.device(dev), torch.no_grad():
            self._ensure_packed()
            picked = torch.empty(B, max(n_out, 1), dtype=torch.long, device=dev)
            kept = torch.empty(B, max(n_out, 1), V, dtype=torch.float32, device=dev)
            forced_c = forced.to(dev, torch.long).contiguous() if n_forced else None
            if seed is None:
                seed = int(torch.randint(0, 2 ** 62, (1,)).item())
            lp = _lib.LoopParams(forced=forced_c.data_ptr() if n_forced else None, n_forced=n_forced, forced_stride=n_forced,
                                 picked=picked.data_ptr(), picked_stride=picked.shape[1], kept_logits=kept.data_ptr(), n_out=n_out,
                                 top_k=int(top_k), top_p=float(top_p), temperature=float(temperature), seed=seed, step0=0)
            key = ("loop", B, tuple((k, t.data_ptr()) for k, t in sorted(rec.state_dict.items())),
                   tuple((k, t.data_ptr()) for k, t in sorted(rec.fir_state_dict.items())),
                   tuple((k, t.data_ptr(), t.shape[1]) for k, t in sorted(mha_ip.key_value_memory_dict.items())))
            st = self._loop
            if st is None or st["key"] != key:
                st = {"key": key, "graph": None, "x": torch.empty(B, 1, dtype=torch.long, device=dev), "pos": torch.zeros(1, dtype=torch.int64, device=dev),
                      "step": torch.zeros(1, dtype=torch.int64, device=dev), "lp": torch.zeros(C.sizeof(_lib.LoopParams), dtype=torch.uint8, device=dev)}
                self._loop = st
            host = torch.frombuffer(bytearray(bytes(lp)), dtype=torch.uint8)
            st["lp"].copy_(host)
            st["pos"].fill_(int(start_pos))
            st["step"].zero_()
            st["x"].copy_(x.to(torch.long))

            def one_step():
                logits = self._body(st["x"], B, 1, ipd, 0, pos_dev=st["pos"])
                l16 = logits.to(torch.bfloat16)
                check(lib.evo_sample_step(ptr(l16), ptr(st["x"]), B, V, ptr(st["lp"]), ptr(st["step"]), self._stream()), "evo_sample_step")
                check(lib.evo_advance_counters(ptr(st["pos"]), ptr(st["step"]), 1, self._stream()), "evo_advance_counters")

            done = 0
            if st["graph"] is None or st.get("ws") != (self._smallm_ws.data_ptr() if self._smallm_ws is not None else 0):
                one_step()                      # eager step: allocates the workspaces the capture must not
                done = 1
                st["graph"] = None
                if self.decode_graph and n_steps > 1:
                    g = torch.cuda.CUDAGraph()
                    torch.cuda.synchronize()
                    n0 = lib.evo_launch_count()
                    with torch.cuda.graph(g):
                        one_step()
                    st["graph"], st["launches"] = g, lib.evo_launch_count() - n0
                    st["ws"] = self._smallm_ws.data_ptr() if self._smallm_ws is not None else 0
                    lib.evo_note_graph_replay(-st["launches"])
            for _ in range(done, n_steps):
                if st["graph"] is not None:
                    st["graph"].replay()
                    lib.evo_note_graph_replay(st["launches"])
                else:
                    one_step()
            mha_ip.seqlen_offset = rec.seqlen_offset = int(start_pos) + n_steps - 1
            return picked[:, :n_out], kept[:, :n_out]
