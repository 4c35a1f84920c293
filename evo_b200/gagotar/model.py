"""Gagotar: a decoder-only pre-norm model with an fp32 residual stream and per-column layer scales,
x <- x + ls1 * mixer(rms(x) n1), x <- x + ls2 * experts(rms(x) n2).  The mixer runs two mechanisms side by side on the same input and
averages their RMS-normed outputs: attention whose heads exchange scores before the softmax (whole-row query / key norms, rotation with
slowed-down long waves, a chunked causal mask, one sigmoid output gate per head), and gated linear attention with a decay per key channel.
The feed-forward is a mixture of experts with limited activations whose weights are the softmax over the chosen logits.  Executed by
libevo_b200.so.

It follows the object protocol of the framework's other models (see stream_model.StreamDecoder), so the same generation loop, scheduler,
trace replay and command line drive it.  State, keyed by RUN index r:
    d["mha"].key_value_memory_dict[r]   (B, max_seqlen, G*dim + G*vdim): keys (normed, rotated), then values
    d["hyena"].state_dict[r]            (B, heads, dim, vdim) fp32: the gated linear attention's matrix state
The rows of the cache stay where they are; the mask only limits what the kernels read.  Closing one sublayer and opening the next is ONE
row kernel (evo_sum_norm): both sides' norms, their average, the layer scale, the stream and the next sublayer's norm.  All projections
that read the mixer's input are one GEMM.  Linear layers: bf16 activations -> the framework's tcgen05 GEMMs (weights zero-padded once to
their tiles); fp32 activations (dtype=torch.float32) -> evo_gemm_simt, true fp32 multiply-add.
"""
from __future__ import annotations

import ctypes as C
import math
import os

import torch

from .. import _lib
from .._lib import GlaParams, MixedAttnParams, QkPrepParams, check, ptr
from ..stream_model import StreamDecoder, _Packed, _round_up
from .config import GagotarConfig

ACT_LIMITED = 3
GATE_SLOPE = 1.702             # slope of the experts' sigmoid


class Gagotar(StreamDecoder):
    architecture = "Gagotar"
    gemm_env = "EVO_B200_GAGOTAR_GEMM"

    def __init__(self, config: GagotarConfig, dtype: torch.dtype = torch.bfloat16):
        super().__init__(config, dtype)
        # expert mixtures: calls with at least this many rows (outside a captured step) run only the chosen experts, fewer rows run all
        # experts densely with the routing weights multiplied into their columns
        self.moe_sparse_min_rows = int(os.environ.get("EVO_B200_MOE_SPARSE_MIN_ROWS", "1024"))
        self.mixed_attn_cuda_cores = 0             # 1: prompts on the CUDA-core attention kernel as well (comparisons)

    # ---- parameters ----------------------------------------------------------------------------
    def init_random(self, seed: int = 0, device=None) -> "Gagotar":
        """Random weights of a usable scale (benchmarks, tests)."""
        g = torch.Generator().manual_seed(seed)
        for name, t in self.weights.items():
            shape = t.shape
            leaf = name.split(".")[-1]
            if leaf in ("norm1", "norm2", "norm", "out") or name == "final.norm":
                v = 1.0 + torch.randn(shape, generator=g) * 0.1
            elif name.endswith("a2.b"):
                v = torch.randn(shape, generator=g) + 1.0
            elif leaf == "b":
                v = torch.randn(shape, generator=g) * 0.2
            elif leaf in ("ls1", "ls2"):
                v = 0.5 + torch.rand(shape, generator=g)
            elif leaf == "temp":
                v = 0.7 + 0.6 * torch.rand(shape, generator=g)
            elif leaf == "talk":
                v = torch.eye(shape[0]) + torch.randn(shape, generator=g) * 0.3 / math.sqrt(shape[0])
            elif name == "embed":
                v = torch.randn(shape, generator=g)
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
            a, s, f = layer.left, layer.right, layer.mlp
            p = f"l{i}.mix."
            e = {}
            # one projection for everything that reads the mixer's input; the two narrow parts (a gate per head, the decay's low-rank part) come
            # last so that the wide ones start on multiples of the head sizes
            parts = [("left.q", a.heads * a.dim), ("left.k", a.kv_heads * a.dim), ("left.v", a.kv_heads * a.vdim), ("right.q", s.heads * s.dim),
                     ("right.k", s.heads * s.dim), ("right.v", s.heads * s.vdim), ("right.g", s.heads * s.vdim), ("left.g", a.heads), ("right.a1", s.rank)]
            col, e["col"] = 0, {}
            for n, width in parts:
                e["col"][n] = col
                col += width
            e["in"] = _Packed(torch.cat([w[p + n] for n, _ in parts], 0))
            e["left_out"], e["right_out"] = _Packed(w[p + "left.o"]), _Packed(w[p + "right.o"])
            if a.rot_dims > 0:
                e["freq"] = torch.tensor(a.frequencies(), dtype=torch.float64).to(torch.float32).to(dev)
            if f is not None:
                q = f"l{i}.mlp."
                e["up"] = _Packed(torch.cat([w[f"{q}e{k}.gate"] for k in range(f.experts)] + [w[f"{q}e{k}.up"] for k in range(f.experts)], 0))
                e["down"] = _Packed(torch.cat([w[f"{q}e{k}.down"] for k in range(f.experts)], 1))
                e["sparse"] = None                  # per-expert packing, built on the first sparse call
            packed["layers"].append(e)
        self._packed = packed
        return packed

    # ---- kernels ---------------------------------------------------------------------------------
    def _attention(self, r, i, a, z, B, L, ip, off, pos_dev):
        """Biases, norms, rotation and cache rows (evo_qk_prep), then the mixed-score attention over the cache -> left output projection."""
        pk, w, lib = self._packed["layers"][i], self.weights, _lib.lib()
        M, dev, esz, ldz, col = B * L, z.device, z.element_size(), pk["in"].Np, pk["col"]
        p = f"l{i}.mix.left."
        qw, kw, vw = a.heads * a.dim, a.kv_heads * a.dim, a.kv_heads * a.vdim
        cw = kw + vw
        cache = self._kv_rows(ip, r, cw, B, off, L, pos_dev)
        row, bstride = cw, cache.shape[1] * cw
        pos_ptr = pos_dev.data_ptr() if pos_dev is not None else None
        at = lambda n: z.data_ptr() + col[n] * esz
        qp = QkPrepParams(q=at("left.q"), k=at("left.k"), v=at("left.v"), ld=ldz,
                          q_bias=w[p + "q.b"].data_ptr(), k_bias=w[p + "k.b"].data_ptr(), v_bias=w[p + "v.b"].data_ptr(),
                          q_norm_w=w[p + "q.norm"].data_ptr(), k_norm_w=w[p + "k.norm"].data_ptr(), eps=self.config.eps,
                          freq=pk["freq"].data_ptr() if a.rot_dims > 0 else None, rot_dims=a.rot_dims,
                          cache=cache.data_ptr(), cache_row=row, cache_batch_stride=bstride, B=B, L=L, H=a.heads, G=a.kv_heads, dk=a.dim, dv=a.vdim,
                          pos0=off, pos_dev=pos_ptr, dtype=self._dt)
        self._record("qk_prep", 2.0 * esz * M * (qw + cw), lambda: check(lib.evo_qk_prep(C.byref(qp), self._stream()), "evo_qk_prep"))
        ldo = _round_up(a.heads * a.vdim, 64)
        out = torch.empty(M, ldo, dtype=self.act_dtype, device=dev)
        ap = MixedAttnParams(q=at("left.q"), q_tok_stride=ldz, k=cache.data_ptr(), v=cache.data_ptr() + kw * esz, k_tok_stride=row, v_tok_stride=row,
                             k_batch_stride=bstride, v_batch_stride=bstride, gate=at("left.g"), gate_tok_stride=ldz,
                             temp=w[p + "temp"].data_ptr(), talk=w[p + "talk"].data_ptr(), out=out.data_ptr(), ldo=ldo, dtype=self._dt,
                             B=B, Lq=L, H=a.heads, G=a.kv_heads, dk=a.dim, dv=a.vdim, q_pos0=off, pos_dev=pos_ptr, max_keys=cache.shape[1],
                             chunk=a.chunk, scale=a.scale, cuda_cores=self.mixed_attn_cuda_cores)
        nws = lib.evo_mixed_attn_workspace(C.byref(ap))
        ws = torch.empty(nws, dtype=torch.uint8, device=dev) if nws else None
        c = a.chunk if a.chunk > 0 else off + L
        seen = lambda n: n // c * (c * (c + 1) / 2.0) + (n % c) * (n % c + 1) / 2.0          # keys that the first n positions see together
        span = (seen(off + L) - seen(off)) / L
        self._record("mixed_attn", 2.0 * M * a.heads * span * (a.dim + a.vdim),
                     lambda: check(lib.evo_mixed_attn_fwd(C.byref(ap), ptr(ws), nws, self._stream()), "evo_mixed_attn_fwd"))
        return self._linear(out, pk["left_out"], M), pk["left_out"].Np

    def _linear_attention(self, r, i, s, z, B, L, rec, fresh):
        """Decays from their low-rank projection (evo_low_rank_decay), then the recurrence with head norm and gate -> right output projection."""
        pk, w, lib = self._packed["layers"][i], self.weights, _lib.lib()
        M, dev, esz, ldz, col = B * L, z.device, z.element_size(), pk["in"].Np, pk["col"]
        p = f"l{i}.mix.right."
        at = lambda n: z.data_ptr() + col[n] * esz
        C_ = s.heads * s.dim
        alpha = torch.empty(M, C_, dtype=torch.float32, device=dev)
        self._record("low_rank_decay", M * (4.0 * C_ + esz * s.rank), lambda: check(lib.evo_low_rank_decay(
            C.c_void_p(at("right.a1")), ldz, ptr(w[p + "a2"]), ptr(w[p + "a2.b"]), 1.0 / s.tau, ptr(alpha), M, s.rank, C_, self._dt, self._stream()), "evo_low_rank_decay"))
        state, zero = self._matrix_state(r, rec, B, s.heads, s.dim, s.vdim, fresh)
        ldo = _round_up(s.heads * s.vdim, 64)
        out = torch.empty(M, ldo, dtype=self.act_dtype, device=dev)
        gp = GlaParams(q=at("right.q"), k=at("right.k"), v=at("right.v"), ld=ldz, alpha=alpha.data_ptr(), q_scale=s.dim ** -0.5,
                       gate=at("right.g"), ld_gate=ldz, norm_w=w[p + "norm"].data_ptr(), eps=self.config.eps, state=state.data_ptr(), zero_start=zero,
                       out=out.data_ptr(), ldo=ldo, dtype=self._dt, B=B, L=L, H=s.heads, dk=s.dim, dv=s.vdim)
        nws = lib.evo_gla_workspace(C.byref(gp))
        ws = torch.empty(nws, dtype=torch.uint8, device=dev) if nws else None
        self._record("gla", 3.0 * M * s.heads * s.dim * s.vdim, lambda: check(lib.evo_gla_fwd(C.byref(gp), ptr(ws), nws, self._stream()), "evo_gla_fwd"))
        return self._linear(out, pk["right_out"], M), pk["right_out"].Np

    def _mixer(self, r, i, layer, h, B, L, ip, rec, off, pos_dev, fresh):
        pk, w, p = self._packed["layers"][i], self.weights, f"l{i}.mix."
        z = self._linear(h, pk["in"], B * L)
        left, ldl = self._attention(r, i, layer.left, z, B, L, ip, off, pos_dev)
        right, ldr = self._linear_attention(r, i, layer.right, z, B, L, rec, fresh)
        return [(left, ldl, w[p + "left.out"], 0.5), (right, ldr, w[p + "right.out"], 0.5)]

    def _experts(self, i, f, h, M, captured=False):
        pk, lib, q = self._packed["layers"][i], _lib.lib(), f"l{i}.mlp."
        dev, esz, D = h.device, h.element_size(), self.config.width
        act = dict(act=ACT_LIMITED, limit=f.limit, slope=GATE_SLOPE)
        # softmax over the chosen logits = the chosen experts' share of the softmax over all
        route = lambda chosen=None: self._moe_route(h, M, self.weights[q + "router"], f.experts, f.top, chosen=chosen, score_fn=0, normalize=1, scale=1.0)
        if not captured and M >= self.moe_sparse_min_rows and f.top < f.experts:
            if pk["sparse"] is None:
                w = self.weights
                pk["sparse"] = [(_Packed(torch.cat([w[f"{q}e{k}.gate"], w[f"{q}e{k}.up"]], 0)), _Packed(w[f"{q}e{k}.down"])) for k in range(f.experts)]
            chosen = torch.full((M, f.top), -1, dtype=torch.int32, device=dev)
            wts = route(chosen)
            ys, slot_of = self._run_chosen_experts(h, M, chosen, pk["sparse"], f.ff, f.experts, f.top, **act)
            ldo = _round_up(D, 64)
            y = torch.empty(M, ldo, dtype=self.act_dtype, device=dev)
            self._record("moe_combine", float(M) * D * esz * (1.0 + f.top), lambda: check(lib.evo_moe_combine(
                ptr(ys), pk["sparse"][0][1].Np, None, 0, ptr(wts), wts.shape[1], 0, ptr(chosen), ptr(slot_of), ptr(y), ldo, M, D, f.experts, f.top, self._dt,
                self._stream()), "evo_moe_combine"))
            return y, ldo
        # all experts densely: the routing weights (0 for experts that were not chosen) multiply the experts' columns, and the weighted sum over
        # experts is the K-reduction of one down GEMM
        z = self._linear(h, pk["up"], M)
        F = f.experts * f.ff
        a = torch.empty(M, pk["down"].Kp, dtype=self.act_dtype, device=dev)
        self._glu(z.data_ptr(), z.data_ptr() + F * esz, pk["up"].Np, a, pk["down"].Kp, M, F, route=route(), group=f.ff, n_groups=f.experts, **act)
        return self._linear(a, pk["down"], M), pk["down"].Np

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
        check(lib.evo_embed_f32(ptr(ids), int(ids.dtype == torch.int64), ptr(w["embed"]), ptr(x), M, D, V, self._stream()), "evo_embed_f32")
        branches, scale = [], None                   # outputs of the sublayer that is not in the stream yet

        def open_sublayer(norm):
            h = torch.empty(M, Kp, dtype=self.act_dtype, device=dev)
            self._sum_norm(x, branches, [(h, w[norm])], M, col_scale=scale)
            return h
        for r, run in enumerate(cfg.runs):
            i = run.layer
            layer = cfg.layers[i]
            h = open_sublayer(f"l{i}.norm1")
            branches, scale = self._mixer(r, i, layer, h, B, L, ip, rec, off, pos_dev, fresh), w[f"l{i}.ls1"]
            if layer.mlp is not None:
                h = open_sublayer(f"l{i}.norm2")
                y, ldy = self._experts(i, layer.mlp, h, M, captured=pos_dev is not None)
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
