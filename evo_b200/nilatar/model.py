"""Nilatar: a decoder-only pre-norm model with an fp32 residual stream and per-column layer scales,
x <- x + ls1 * mixer(rms(x) n1), x <- x + ls2 * down(gelu(gate h) * (up h)), h = rms(x) n2 (where a layer has a feed-forward).  Three kinds
of mixer: latent attention whose queries come out of a latent of their own, with a shared rotated key part and a gate per output channel;
linear attention with a constant decay per head, normed over all heads; and windowed attention without positions, with a sink, some of
whose layers read an earlier layer's keys and values.  Executed by libevo_b200.so.

It follows the object protocol of the framework's other models (see stream_model.StreamDecoder), so the same generation loop, scheduler,
trace replay and command line drive it.  State, keyed by RUN index r:
    d["mha"].key_value_memory_dict[r]   latent attention: (B, max_seqlen, row) with rows [latent | 0.. | turned key part | 0..];
                                        attention: (B, max_seqlen, G*dim + G*vdim), keys, then values; a layer that reads an earlier
                                        layer's keys and values has no entry
    d["hyena"].state_dict[r]            (B, heads, dim, vdim) fp32: the linear attention's matrix state
Cache rows stay where they are; the window only limits what the kernels read.  Closing one sublayer and opening the next is ONE row kernel
(evo_sum_norm), all projections that read the mixer's input are one GEMM, and the feed-forward's gate and the linear attention's silu sit
in their GEMMs' epilogues.  Linear layers: bf16 activations -> the framework's tcgen05
GEMMs (weights zero-padded once to their tiles); fp32 activations (dtype=torch.float32) -> evo_gemm_simt, true fp32 multiply-add.
"""
from __future__ import annotations

import ctypes as C
import math

import torch

from .. import _lib
from .._lib import DecayScanParams, WindowAttnParams, check, ptr
from ..stream_model import StreamDecoder, _Packed, _PackedGate, _round_up
from .config import NilatarConfig


class Nilatar(StreamDecoder):
    architecture = "Nilatar"
    gemm_env = "EVO_B200_NILATAR_GEMM"

    def __init__(self, config: NilatarConfig, dtype: torch.dtype = torch.bfloat16):
        super().__init__(config, dtype)
        self.decay_recurrent = 0                   # 1: the linear attention token by token for prompts as well (comparisons)

    # ---- parameters ----------------------------------------------------------------------------
    def init_random(self, seed: int = 0, device=None) -> "Nilatar":
        """Random weights of a usable scale (benchmarks, tests)."""
        g = torch.Generator().manual_seed(seed)
        for name, t in self.weights.items():
            shape = t.shape
            leaf = name.split(".")[-1]
            if leaf in ("norm1", "norm2", "norm"):
                v = 1.0 + torch.randn(shape, generator=g) * 0.1
            elif leaf in ("ls1", "ls2"):
                v = 0.5 + torch.rand(shape, generator=g)
            elif leaf == "sink":
                v = torch.randn(shape, generator=g)
            elif name == "embed":
                v = torch.randn(shape, generator=g) / max(self.config.embed_scale, 1e-6)
            else:
                v = torch.randn(shape, generator=g) / math.sqrt(shape[-1])
            self.weights[name] = v.to(torch.bfloat16)
        self._invalidate()
        return self.to(device) if device is not None else self

    # ---- packing -------------------------------------------------------------------------------
    def _ensure_packed(self):
        if self._packed is not None:
            return self._packed
        dev = self.device
        if dev.type != "cuda":
            raise _lib.EvoError("evo_b200 runs on CUDA (sm_100a) only: move the model with .to('cuda:N'); there is no CPU path")
        w = self.weights
        packed = {"head": _Packed(w["head"]), "layers": []}
        for i, layer in enumerate(self.config.layers):
            m, p = layer.mixer, f"l{i}.mix."
            if m.kind == "latent_attention":
                names = ["dq", "dkv", "g"]
            else:
                names = ["q", "g"] if m.kind == "attention" and m.kv_from is not None else ["q", "k", "v", "g"]
            # one projection for everything that reads the mixer's input
            col, e = 0, {"col": {}}
            for n in names:
                e["col"][n] = col
                col += w[p + n].shape[0]
            e["in"], e["out"] = _Packed(torch.cat([w[p + n] for n in names], 0)), _Packed(w[p + "o"])
            if m.kind == "latent_attention":
                e["uq"] = _Packed(w[p + "uq"])
                e["latent"] = self._pack_latent(m, w[p + "uk"], w[p + "uv"])
                e["freq"] = torch.tensor(m.frequencies(), dtype=torch.float64).to(torch.float32).to(dev) if m.rot_dims else None
            elif m.kind == "lightning":
                e["decay"] = torch.tensor(m.decay, dtype=torch.float64).to(torch.float32).to(dev)
            if layer.ff:
                q = f"l{i}.mlp."
                e["up"], e["down"] = _PackedGate(w[q + "gate"], w[q + "up"]), _Packed(w[q + "down"], _PackedGate.RUN)
            packed["layers"].append(e)
        self._packed = packed
        return packed

    # ---- mixers ----------------------------------------------------------------------------------
    def _window_attention(self, r, i, m, h, B, L, ip, off, pos_dev):
        """Cache rows (unless another layer's are read), then windowed attention over them with sink and gate -> output projection."""
        pk, w, lib = self._packed["layers"][i], self.weights, _lib.lib()
        M, dev = B * L, h.device
        z = self._linear(h, pk["in"], M)
        esz, ldz, col = z.element_size(), pk["in"].Np, pk["col"]
        kw, vw = m.kv_heads * m.dim, m.kv_heads * m.vdim
        cw = kw + vw
        pos_ptr = pos_dev.data_ptr() if pos_dev is not None else None
        at = lambda n: z.data_ptr() + col[n] * esz
        if m.kv_from is None:
            cache = self._kv_rows(ip, r, cw, B, off, L, pos_dev)
            self._record("copy_rows", 2.0 * M * cw * esz, lambda: check(lib.evo_copy_rows(
                C.c_void_p(at("k")), ldz, ptr(cache), cw, cache.shape[1] * cw, B, L, cw, off, pos_ptr, self._dt, self._stream()), "evo_copy_rows"))
        else:
            cache = ip.key_value_memory_dict[m.kv_from]          # filled by that layer in this very call
        bstride = cache.shape[1] * cw
        ldo = _round_up(m.heads * m.vdim, 64)
        out = torch.empty(M, ldo, dtype=self.act_dtype, device=dev)
        ap = WindowAttnParams(q=at("q"), q_tok_stride=ldz, k=cache.data_ptr(), v=cache.data_ptr() + kw * esz, k_tok_stride=cw, v_tok_stride=cw,
                              k_batch_stride=bstride, v_batch_stride=bstride, gate=at("g"), gate_tok_stride=ldz, out=out.data_ptr(), ldo=ldo, dtype=self._dt,
                              B=B, Lq=L, H=m.heads, G=m.kv_heads, dk=m.dim, dv=m.vdim, n_maps=1, q_pos0=off, pos_dev=pos_ptr, window=m.window, keep_first=0,
                              scale=m.scale, sink=w[f"l{i}.mix.sink"].data_ptr())
        self._record("window_attn", 2.0 * M * m.heads * self._mean_keys(off, L, m.window) * (m.dim + m.vdim),
                     lambda: check(lib.evo_window_attn_fwd(C.byref(ap), self._stream()), "evo_window_attn_fwd"))
        return self._linear(out, pk["out"], M), pk["out"].Np

    def _latent_attention(self, r, i, m, h, B, L, ip, off, pos_dev):
        pk, w, lib = self._packed["layers"][i], self.weights, _lib.lib()
        M, dev, p = B * L, h.device, f"l{i}.mix."
        z = self._linear(h, pk["in"], M)
        esz, ldz, col = z.element_size(), pk["in"].Np, pk["col"]
        at = lambda n: z.data_ptr() + col[n] * esz
        cq = torch.empty(M, pk["uq"].Kp, dtype=self.act_dtype, device=dev)
        cache = self._latent_rows(r, m, pk["latent"], at("dkv"), ldz, w[p + "dkv.norm"], pk["freq"], m.rot_len, B, L, ip, off, pos_dev,
                                  query=(at("dq"), ldz, w[p + "dq.norm"], m.q_rank, cq))
        q = self._linear(cq, pk["uq"], M)
        self._latent_turn(m, q, pk["uq"].Np, pk["freq"], m.rot_len, B, L, off, pos_dev)
        out = self._latent_attend(m, pk["latent"], q.data_ptr(), pk["uq"].Np, cache, w[p + "uk"], w[p + "uv"], at("g"), ldz, True, B, L, off, pos_dev)
        return self._linear(out, pk["out"], M), pk["out"].Np

    def _lightning(self, r, i, m, h, B, L, rec, fresh):
        """silu of the projections (in the GEMM's epilogue, or in the recurrence), the recurrence, norm over all heads and gate -> output projection."""
        pk, w, lib = self._packed["layers"][i], self.weights, _lib.lib()
        M, dev = B * L, h.device
        col, ldz, vw = pk["col"], pk["in"].Np, m.heads * m.vdim
        z = self._linear(h, pk["in"], M, silu_cols=col["g"] if self._fused else 0)
        esz = z.element_size()
        at = lambda n: z.data_ptr() + col[n] * esz
        state, zero = self._matrix_state(r, rec, B, m.heads, m.dim, m.vdim, fresh)
        y = torch.empty(M, vw, dtype=torch.float32, device=dev)
        sp = DecayScanParams(q=at("q"), k=at("k"), v=at("v"), ld=ldz, decay=pk["decay"].data_ptr(), act=int(not self._fused), q_scale=1.0, state=state.data_ptr(), zero_start=zero,
                             y=y.data_ptr(), dtype=self._dt, B=B, L=L, H=m.heads, dk=m.dim, dv=m.vdim, recurrent=self.decay_recurrent)
        nws = lib.evo_decay_scan_workspace(C.byref(sp))
        ws = torch.empty(nws, dtype=torch.uint8, device=dev) if nws else None
        # roofline bytes: the projections once, the fp32 read-outs once
        self._record("decay_scan", float(M) * m.heads * ((2 * m.dim + m.vdim) * esz + 4 * m.vdim), lambda: check(lib.evo_decay_scan_fwd(C.byref(sp), ptr(ws), nws, self._stream()), "evo_decay_scan_fwd"))
        ldo = _round_up(vw, 64)
        out = torch.empty(M, ldo, dtype=self.act_dtype, device=dev)
        self._record("norm_gate", float(M) * vw * (4.0 + 2.0 * esz), lambda: check(lib.evo_norm_gate(
            ptr(y), C.c_void_p(at("g")), ldz, ptr(w[f"l{i}.mix.norm"]), ptr(out), ldo, M, vw, self.config.eps, self._dt, self._stream()), "evo_norm_gate"))
        return self._linear(out, pk["out"], M), pk["out"].Np

    def _feed_forward(self, i, h, M):
        pk = self._packed["layers"][i]
        return self._linear(self._gelu_gate(h, pk["up"], M), pk["down"], M), pk["down"].Np

    def _body(self, ids, B, L, ipd, off: int, pos_dev=None, rows=None):
        """embed -> every layer -> final norm -> head.  Returns fp32 logits (B*L, V), or (len(rows), V) for the flat row
        indices in `rows` (int64 tensor on the device)."""
        cfg, dev = self.config, ids.device
        lib, w = _lib.lib(), self.weights
        M, D, V = B * L, cfg.width, cfg.vocab_size
        if ipd is None:                              # stateless call: the same path on holders that live for this call only
            ipd = self.initialize_inference_params(max_seqlen=L, max_batch_size=B)
        ip, rec = ipd["mha"], ipd["hyena"]
        fresh = pos_dev is None and off == 0         # a sequence's first tokens: recurrent states start from zero
        Kp = _round_up(D, 64)
        x = torch.empty(M, D, dtype=torch.float32, device=dev)
        check(lib.evo_embed_scaled_f32(ptr(ids), int(ids.dtype == torch.int64), ptr(w["embed"]), ptr(x), M, D, V, cfg.embed_scale, self._stream()), "evo_embed_scaled_f32")
        branches, scale = [], None                   # output of the sublayer that is not in the stream yet

        def open_sublayer(norm):
            h = torch.empty(M, Kp, dtype=self.act_dtype, device=dev)
            self._sum_norm(x, branches, [(h, w[norm])], M, col_scale=scale)
            return h
        for r, run in enumerate(cfg.runs):
            i = run.layer
            layer = cfg.layers[i]
            m = layer.mixer
            h = open_sublayer(f"l{i}.norm1")
            if m.kind == "lightning":
                y, ldy = self._lightning(r, i, m, h, B, L, rec, fresh)
            else:
                mixer = self._latent_attention if m.kind == "latent_attention" else self._window_attention
                y, ldy = mixer(r, i, m, h, B, L, ip, off, pos_dev)
            branches, scale = [(y, ldy, None, 1.0)], w[f"l{i}.ls1"]
            if layer.ff:
                h = open_sublayer(f"l{i}.norm2")
                y, ldy = self._feed_forward(i, h, M)
                branches, scale = [(y, ldy, None, 1.0)], w[f"l{i}.ls2"]
            if self._tap is not None:
                self._sum_norm(x, branches, [], M, col_scale=scale)
                self._tap.append(x.clone())
                branches, scale = [], None
        n_out = M if rows is None else int(rows.numel())
        if n_out == 0:
            return torch.empty(0, V, dtype=torch.float32, device=dev)
        hf = torch.empty(n_out, Kp, dtype=self.act_dtype, device=dev)
        self._sum_norm(x, branches, [(hf, w["final.norm"])], n_out, gather=rows, col_scale=scale)
        raw = self._linear(hf, self._packed["head"], n_out)
        logits = torch.empty(n_out, V, dtype=torch.float32, device=dev)
        check(lib.evo_scale_logits(ptr(raw), self._packed["head"].Np, ptr(logits), n_out, V, 1.0, self._dt, self._stream()), "evo_scale_logits")
        return logits
