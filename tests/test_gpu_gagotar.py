"""Gagotar on the GPU against the plain oracle (oracle/gagotar_oracle.py): the new kernels alone (mixed-score attention in its three
forms, decays, gated linear attention, limited experts, scaled row sums, softmax over the chosen logits), each side of the mixer alone
over several sizes, then the model -- whole prompts, token-by-token decoding, portions down to two tokens, batches, reused state memory,
far keys, chunk edges, the first tokens of a sequence, long decoding, other sizes -- and greedy generation through the framework's
Generator and command line.  Small configurations, random weights; where random weights would hide a fault the weights are made so that
it shows."""
import ctypes as C
import math

import pytest
import torch

from evo_b200 import _lib
from evo_b200._lib import GlaParams, GluActParams, MixedAttnParams, MoeRouteParams, QkPrepParams, SumNormParams, check, ptr
from oracle import gagotar_oracle as O

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F32, B16, F64 = torch.float32, torch.bfloat16, torch.float64


def _stream():
    return C.c_void_p(torch.cuda.current_stream().cuda_stream)


def _bf(t):
    return t.to(B16)


def _close(got, want, tol, what=""):
    err = (got.double().cpu() - want.double().cpu()).abs().max().item()
    ref = max(want.abs().max().item(), 1e-6)
    assert err <= tol * ref, f"{what}: max err {err:.3e} vs scale {ref:.3e} (tol {tol})"


def _model(cfg, W, dtype=F32):
    from evo_b200.gagotar import Gagotar, GagotarConfig
    m = Gagotar(GagotarConfig.from_dict(cfg, {k: tuple(v.shape) for k, v in W.items()}), dtype=dtype)
    m.load_state_dict(W)
    return m.to(DEV)


def _portions(model, tokens, sizes, max_seqlen=None, state=None):
    state = state or model.initialize_inference_params(max_seqlen=max_seqlen or len(tokens) + 8, max_batch_size=1)
    outs, t = [], 0
    for n in sizes:
        state["mha"].seqlen_offset = state["hyena"].seqlen_offset = t
        lg, _ = model(torch.tensor([tokens[t:t + n]], device=DEV), inference_params_dict=state)
        outs.append(lg[0])
        t += n
    assert t == len(tokens)
    return torch.cat(outs, 0)


def _tokens(cfg, n, seed=1):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


# ------------------------------------------------------------------ kernels alone
def _run_attention(q, k, v, scale, temp, talk, chunk, pos0, gate, dtype, rows, cuda_cores=False, device_pos=False):
    """q (L, H, dk), k / v (T, G, d) through evo_mixed_attn_fwd in calls of `rows` query rows -> (L, H*dv)."""
    L, H, dk = q.shape
    T, G, dv = v.shape
    qd, kd, vd = q.to(DEV, dtype).reshape(L, H * dk), k.to(DEV, dtype).reshape(T, G * dk), v.to(DEV, dtype).reshape(T, G * dv)
    gd = gate.to(DEV, dtype) if gate is not None else None
    tempd = temp.to(DEV) if temp is not None else None
    talkd = talk.to(DEV) if talk is not None else None
    ldo = (H * dv + 63) // 64 * 64
    outs = []
    for lo in range(0, L, rows):
        n = min(rows, L - lo)
        out = torch.full((n, ldo), 5.0, dtype=dtype, device=DEV)
        pd = torch.tensor([pos0 + lo], dtype=torch.int64, device=DEV) if device_pos else None
        p = MixedAttnParams(q=qd[lo:].data_ptr(), q_tok_stride=H * dk, k=kd.data_ptr(), v=vd.data_ptr(), k_tok_stride=G * dk, v_tok_stride=G * dv,
                            k_batch_stride=T * G * dk, v_batch_stride=T * G * dv, gate=gd[lo:].data_ptr() if gd is not None else None, gate_tok_stride=H,
                            temp=tempd.data_ptr() if temp is not None else None, talk=talkd.data_ptr() if talk is not None else None,
                            out=out.data_ptr(), ldo=ldo, dtype=1 if dtype == F32 else 0, B=1, Lq=n, H=H, G=G, dk=dk, dv=dv,
                            q_pos0=0 if device_pos else pos0 + lo, pos_dev=pd.data_ptr() if device_pos else None, max_keys=T, chunk=chunk, scale=scale,
                            cuda_cores=int(cuda_cores))
        lib = _lib.lib()
        nws = lib.evo_mixed_attn_workspace(C.byref(p))
        ws = torch.full((max(nws, 1),), 0xFF, dtype=torch.uint8, device=DEV)          # NaNs where nothing has been written
        check(lib.evo_mixed_attn_fwd(C.byref(p), ptr(ws), nws, _stream()))
        assert (out[:, H * dv:] == 0).all()
        outs.append(out[:, :H * dv])
    return torch.cat(outs, 0)


# heads, key heads, dk, dv, chunk, rows, first position: one head, odd sizes, more than 8 / 16 / 32 heads (one, two, three CTAs per tile), wide heads
ATT_SHAPES = [(4, 2, 16, 12, 24, 100, 0), (1, 1, 8, 8, 0, 50, 7), (3, 1, 10, 9, 17, 90, 37), (12, 4, 32, 48, 50, 120, 11), (16, 16, 24, 16, 64, 70, 0),
              (20, 5, 16, 24, 33, 70, 40), (33, 11, 8, 16, 40, 60, 25), (32, 8, 128, 128, 96, 130, 90), (16, 4, 128, 128, 0, 150, 100), (2, 2, 136, 136, 30, 40, 3),
              (5, 5, 40, 72, 1, 20, 5), (17, 1, 20, 6, 28, 40, 0), (40, 8, 16, 120, 45, 50, 20),
              (24, 6, 64, 64, 70, 80, 30), (3, 1, 192, 64, 37, 90, 13), (16, 16, 128, 128, 61, 50, 9), (6, 3, 72, 24, 100, 60, 150)]


@pytest.mark.parametrize("H,G,dk,dv,chunk,L,pos0", ATT_SHAPES, ids=lambda v: str(v))
def test_mixed_attention_kernels_match_fp64(H, G, dk, dv, chunk, L, pos0):
    """The tensor-core kernel (bf16, 16 rows or more), the CUDA-core kernel in both types, one and several key ranges, host and device positions."""
    g = torch.Generator().manual_seed(H * dk + L)
    T = pos0 + L + 3
    q, k, v = _bf(torch.randn(L, H, dk, generator=g)), _bf(torch.randn(T, G, dk, generator=g)), _bf(torch.randn(T, G, dv, generator=g))
    temp, talk, gate = _bf(0.5 + torch.rand(H, generator=g)), _bf(torch.eye(H) + torch.randn(H, H, generator=g) / math.sqrt(H)), _bf(torch.randn(L, H, generator=g))
    scale = 1.2 / math.sqrt(dk)
    want = O.mixed_head_attention(q.double(), k.double(), v.double(), scale, temp.double(), talk.double(), chunk, pos0)
    want = (want * torch.sigmoid(gate.double())[:, :, None]).reshape(L, H * dv)
    args = (q, k, v, scale, temp, talk, chunk, pos0, gate)
    _close(_run_attention(*args, B16, L), want, 1.2e-2, "prompt rows, bf16")
    _close(_run_attention(*args, B16, 19), want, 1.2e-2, "portions of 19 rows, bf16")
    _close(_run_attention(*args, B16, L, cuda_cores=True), want, 1.2e-2, "prompt rows on the CUDA cores, bf16")
    _close(_run_attention(*args, F32, L), want, 3e-5, "prompt rows, fp32")
    _close(_run_attention(*args, F32, 2), want, 3e-5, "two rows a call, fp32")
    _close(_run_attention(*args, B16, 1, device_pos=True), want, 1.2e-2, "steps with the position in device memory, bf16")


@pytest.mark.parametrize("H,G,dk,dv", [(4, 2, 64, 64), (18, 6, 64, 128), (6, 3, 24, 40)])
def test_mixed_attention_of_several_sequences_in_one_call(H, G, dk, dv):
    """Each sequence has its own cache rows (whole column tiles through tensor maps, padded heads row by row); rows behind the last position hold NaNs."""
    g = torch.Generator().manual_seed(dk)
    B, L, pos0, rows, chunk = 3, 40, 21, 80, 33
    q, kv = _bf(torch.randn(B, L, H * dk, generator=g)), torch.full((B, rows, G * (dk + dv)), float("nan"))
    kv[:, :pos0 + L] = torch.randn(B, pos0 + L, G * (dk + dv), generator=g)
    kv = _bf(kv)
    talk = _bf(torch.eye(H) + torch.randn(H, H, generator=g) / math.sqrt(H))
    qd, kvd, td = q.to(DEV), kv.to(DEV), talk.to(DEV)
    cw, ldo = G * (dk + dv), (H * dv + 63) // 64 * 64
    out = torch.full((B * L, ldo), 5.0, dtype=B16, device=DEV)
    p = MixedAttnParams(q=qd.data_ptr(), q_tok_stride=H * dk, k=kvd.data_ptr(), v=kvd.data_ptr() + 2 * G * dk, k_tok_stride=cw, v_tok_stride=cw, k_batch_stride=rows * cw,
                        v_batch_stride=rows * cw, talk=td.data_ptr(), out=out.data_ptr(), ldo=ldo, dtype=0, B=B, Lq=L, H=H, G=G, dk=dk, dv=dv, q_pos0=pos0, max_keys=rows,
                        chunk=chunk, scale=0.9 / math.sqrt(dk))
    lib = _lib.lib()
    nws = lib.evo_mixed_attn_workspace(C.byref(p))
    ws = torch.empty(max(nws, 1), dtype=torch.uint8, device=DEV)
    check(lib.evo_mixed_attn_fwd(C.byref(p), ptr(ws), nws, _stream()))
    for b in range(B):
        k, v = kv[b, :pos0 + L, :G * dk].double().view(-1, G, dk), kv[b, :pos0 + L, G * dk:].double().view(-1, G, dv)
        want = O.mixed_head_attention(q[b].double().view(L, H, dk), k, v, 0.9 / math.sqrt(dk), torch.ones(H, dtype=F64), talk.double(), chunk, pos0).reshape(L, H * dv)
        _close(out[b * L:(b + 1) * L, :H * dv], want, 1.2e-2, f"sequence {b}")
    lost = C.c_uint(99)
    check(lib.evo_mixed_attn_lost_waits(C.byref(lost)))
    assert lost.value == 0


def test_mixed_attention_without_gate_temperature_and_mixture_is_plain_attention():
    g = torch.Generator().manual_seed(3)
    L, H, G, dk, dv = 70, 4, 2, 16, 16
    q, k, v = _bf(torch.randn(L, H, dk, generator=g)), _bf(torch.randn(L, G, dk, generator=g)), _bf(torch.randn(L, G, dv, generator=g))
    want = O.mixed_head_attention(q.double(), k.double(), v.double(), 0.25, torch.ones(H, dtype=F64), torch.eye(H, dtype=F64), 0).reshape(L, H * dv)
    _close(_run_attention(q, k, v, 0.25, None, None, 0, 0, None, B16, L), want, 1.2e-2, "tensor cores")
    _close(_run_attention(q, k, v, 0.25, None, None, 0, 0, None, F32, L), want, 3e-5, "CUDA cores")


def test_mixed_attention_key_ranges_of_a_long_cache():
    """A step behind 3000 positions spreads its keys over CTAs; positions at and around the ranges' edges, chunk edges and one visible key."""
    g = torch.Generator().manual_seed(5)
    T, H, G, dk, dv = 3100, 6, 3, 16, 8
    k, v = _bf(torch.randn(T, G, dk, generator=g)), _bf(torch.randn(T, G, dv, generator=g))
    temp, talk = _bf(0.5 + torch.rand(H, generator=g)), _bf(torch.eye(H) + 0.4 * torch.randn(H, H, generator=g))
    for chunk in (0, 1000, 64):
        for pos in (0, 1, 62, 63, 64, 65, 127, 128, 999, 1000, 1001, 2047, 3000):
            q = _bf(torch.randn(1, H, dk, generator=g))
            want = O.mixed_head_attention(q.double(), k[:pos + 1].double(), v[:pos + 1].double(), 0.4, temp.double(), talk.double(), chunk, pos).reshape(1, H * dv)
            for dtype, tol in ((F32, 3e-5), (B16, 1.2e-2)):
                _close(_run_attention(q, k, v, 0.4, temp, talk, chunk, pos, None, dtype, 1), want, tol, f"chunk {chunk}, position {pos}")
                _close(_run_attention(q, k, v, 0.4, temp, talk, chunk, pos, None, dtype, 1, device_pos=True), want, tol, f"chunk {chunk}, device position {pos}")


@pytest.mark.parametrize("dtype", [F32, B16])
def test_one_key_decides_just_inside_and_just_outside_a_chunk(dtype):
    """Every score is 0 except at one key, where it is large for every query: rows of the same chunk take that key's value, the others a plain mean."""
    H, G, dk, dv, chunk, T = 3, 1, 16, 8, 40, 130
    talk = _bf(torch.tensor([[1.0, 0.5, 0.25], [0.5, 1.0, 0.5], [2.0, 1.0, 1.0]]))
    temp = _bf(torch.tensor([1.0, 0.75, 1.25]))
    g = torch.Generator().manual_seed(1)
    v = _bf(torch.randn(T, G, dv, generator=g))
    for j in (0, 39, 40, 79, 80, 119):
        k = torch.zeros(T, G, dk)
        k[j, 0, 3] = 8.0
        q = torch.zeros(T, H, dk)
        q[:, :, 3] = 4.0
        want = O.mixed_head_attention(q.double(), k.double(), v.double(), 1.0, temp.double(), talk.double(), chunk).reshape(T, H * dv)
        hit = want.view(T, H, dv)[:, 0]
        for i in range(T):
            sees = j <= i and i // chunk == j // chunk
            if i // chunk * chunk != i:                       # a row that sees several keys
                assert torch.allclose(hit[i], v[j, 0].double(), atol=1e-6) == sees, (i, j)
        for rows in (T, 16, 5, 1):
            _close(_run_attention(_bf(q), _bf(k), v, 1.0, temp, talk, chunk, 0, None, dtype, rows), want, 1e-5 if dtype == F32 else 8e-3, f"key {j}, {rows} rows a call")


@pytest.mark.parametrize("rank,C,M", [(1, 7, 5), (16, 64, 33), (5, 300, 16), (24, 40, 1)])
@pytest.mark.parametrize("dtype", [F32, B16])
def test_low_rank_decays(rank, C, M, dtype):
    g = torch.Generator().manual_seed(rank)
    u, a2, b = _bf(torch.randn(M, rank + 3, generator=g) * 3), _bf(torch.randn(C, rank, generator=g)), _bf(torch.randn(C, generator=g) * 5)
    for tau in (1.0, 16.0):
        alpha = torch.full((M, C), 7.0, device=DEV)
        ud, a2d, bd = u.to(DEV, dtype), a2.to(DEV), b.to(DEV)
        check(_lib.lib().evo_low_rank_decay(ptr(ud), rank + 3, ptr(a2d), ptr(bd), 1.0 / tau, ptr(alpha), M, rank, C, 1 if dtype == F32 else 0, _stream()))
        want = torch.sigmoid(u[:, :rank].double() @ a2.double().T + b.double()) ** (1.0 / tau)
        _close(alpha, want, 5e-6, f"tau {tau}")


@pytest.mark.parametrize("H,dk,dv,L", [(2, 12, 20, 50), (3, 5, 7, 33), (1, 72, 136, 40), (1, 16, 200, 300), (2, 128, 64, 280), (1, 1, 1, 20), (2, 130, 31, 35)])
@pytest.mark.parametrize("dtype", [F32, B16])
def test_gated_linear_attention_kernel(H, dk, dv, L, dtype):
    """Whole, and in two calls through the carried state; heads spread over CTAs, 16 lanes per state column, decays from almost 0 to almost 1."""
    g = torch.Generator().manual_seed(dk + dv)
    qk, vw = H * dk, H * dv
    z = _bf(torch.randn(L, 2 * qk + 2 * vw + 1, generator=g))
    alpha = torch.sigmoid(torch.randn(L, qk, generator=g) * 4 + 2).float()
    nw = _bf(1 + 0.2 * torch.randn(dv, generator=g))
    zz = z.double()
    o = O.decay_scan(zz[:, :qk].view(L, H, dk) * dk ** -0.5, zz[:, qk:2 * qk].view(L, H, dk), zz[:, 2 * qk:2 * qk + vw].view(L, H, dv), alpha.double().view(L, H, dk))
    want = (O.rms(o, 1e-5) * nw.double()).reshape(L, vw) * O.silu(zz[:, 2 * qk + vw:2 * qk + 2 * vw])
    ld, ldo = z.shape[1], (vw + 63) // 64 * 64
    zd, ad, nd = z.to(DEV, dtype), alpha.to(DEV), nw.to(DEV)
    esz = zd.element_size()
    lib = _lib.lib()
    for cuts in ([L], [L - 9, 9], [1, L - 1]):
        state = torch.full((1, H, dk, dv), float("nan"), device=DEV)
        outs, t = [], 0
        for n in cuts:
            out = torch.full((n, ldo), 3.0, dtype=dtype, device=DEV)
            base = zd[t:].data_ptr()
            p = GlaParams(q=base, k=base + qk * esz, v=base + 2 * qk * esz, ld=ld, alpha=ad[t:].data_ptr(), q_scale=dk ** -0.5, gate=base + (2 * qk + vw) * esz, ld_gate=ld,
                          norm_w=nd.data_ptr(), eps=1e-5, state=state.data_ptr(), zero_start=int(t == 0), out=out.data_ptr(), ldo=ldo, dtype=1 if dtype == F32 else 0,
                          B=1, L=n, H=H, dk=dk, dv=dv)
            nws = lib.evo_gla_workspace(C.byref(p))
            ws = torch.empty(max(nws, 1), dtype=torch.uint8, device=DEV)
            check(lib.evo_gla_fwd(C.byref(p), ptr(ws), nws, _stream()))
            assert (out[:, vw:] == 0).all()
            outs.append(out[:, :vw])
            t += n
        _close(torch.cat(outs), want, 5e-5 if dtype == F32 else 1e-2, f"calls of {cuts}")


@pytest.mark.parametrize("D,ldo", [(48, 64), (130, 192), (1032, 1088)])
@pytest.mark.parametrize("dtype", [F32, B16])
def test_row_sum_with_norms_and_a_factor_per_column(D, ldo, dtype):
    M, eps = 6, 1e-5
    g = torch.Generator().manual_seed(D)
    x, ys = torch.randn(M, D, generator=g), [_bf(torch.randn(M, D + 8 * b, generator=g) * 3) for b in range(2)]
    w0, w1, cs, ow = (_bf(torch.randn(D, generator=g)) for _ in range(4))
    want = x.double() + cs.double() * (0.5 * O.rms(ys[0][:, :D].double(), eps) * w0.double() + 0.5 * O.rms(ys[1][:, :D].double(), eps) * w1.double())
    yd = [y.to(DEV, dtype) for y in ys]
    w0d, w1d, csd, owd = (t.to(DEV) for t in (w0, w1, cs, ow))
    xd, out = x.to(DEV), torch.full((M, ldo), 7.0, dtype=dtype, device=DEV)
    p = SumNormParams(x=xd.data_ptr(), n_branches=2, eps=eps, dtype=1 if dtype == F32 else 0, rows=M, D=D, ldo=ldo, col_scale=csd.data_ptr())
    for b, w in enumerate((w0d, w1d)):
        p.y[b], p.ldy[b], p.norm_w[b], p.scale[b] = yd[b].data_ptr(), D + 8 * b, w.data_ptr(), 0.5
    p.out[0], p.w[0] = out.data_ptr(), owd.data_ptr()
    check(_lib.lib().evo_sum_norm(C.byref(p), _stream()))
    _close(xd, want, 3e-6, "stream")
    _close(out[:, :D], O.rms(want, eps) * ow.double(), 5e-6 if dtype == F32 else 6e-3, "normed copy")
    assert (out[:, D:] == 0).all()


@pytest.mark.parametrize("F,grp", [(44, 0), (48, 8), (30, 5)])
@pytest.mark.parametrize("dtype", [F32, B16])
def test_limited_activation_and_expert_weights(F, grp, dtype):
    M, limit = 5, 1.3
    g = torch.Generator().manual_seed(F)
    z = _bf(torch.randn(M, 2 * F + 4, generator=g) * 2)
    assert (z[:, :F] > limit).any() and (z[:, :F] < -limit).any() and (z[:, F:2 * F].abs() > limit).any()
    want = O.limited_glu(z[:, :F].double(), z[:, F:2 * F].double(), limit)
    zd, ldo = z.to(DEV, dtype), (F + 7) // 4 * 4
    out = torch.full((M, ldo), 7.0, dtype=dtype, device=DEV)
    p = GluActParams(gate=zd.data_ptr(), up=zd.data_ptr() + F * zd.element_size(), ld=2 * F + 4, out=out.data_ptr(), ldo=ldo, rows=M, F=F, act=3,
                     dtype=1 if dtype == F32 else 0, limit=limit, slope=O.SLOPE)
    if grp:
        wts = torch.rand(M, F // grp, generator=g)
        wts[:, 1] = 0.0
        wd = wts.to(DEV)
        p.group_w, p.ldw, p.group, p.n_groups = wd.data_ptr(), F // grp, grp, F // grp
        want = want * wts.repeat_interleave(grp, 1).double()
    check(_lib.lib().evo_glu_act_ex(C.byref(p), _stream()))
    _close(out[:, :F], want, 3e-6 if dtype == F32 else 8e-3)
    assert (out[:, F:] == 0).all()


@pytest.mark.parametrize("E,top,M", [(6, 2, 37), (12, 3, 1100), (5, 5, 9), (4, 1, 2), (40, 6, 20)])
def test_router_weights_are_the_softmax_over_the_chosen_logits(E, top, M):
    D = 56
    g = torch.Generator().manual_seed(E)
    h, rw = _bf(torch.randn(M, D, generator=g)), _bf(torch.randn(E, D, generator=g))
    want = O.route(h.double(), rw.double(), top)
    hd, rd = h.to(DEV, F32), rw.to(DEV)
    out, chosen = torch.full((M, E), 9.0, device=DEV), torch.full((M, top), -1, dtype=torch.int32, device=DEV)
    p = MoeRouteParams(h=hd.data_ptr(), ldh=D, router_w=rd.data_ptr(), weights=out.data_ptr(), ldw=E, chosen=chosen.data_ptr(), rows=M, D=D, E=E, top=top,
                       score_fn=0, normalize=1, scale=1.0, dtype=1)
    check(_lib.lib().evo_moe_route_ex(C.byref(p), _stream()))
    _close(out, want, 2e-5)
    assert torch.equal(chosen.cpu().long().sort(-1).values, (want > 0).nonzero()[:, 1].view(M, top))


@pytest.mark.parametrize("scaling", [None, (4.0, 1.0, 4.0, 300), (16.0, 2.0, 3.0, 90)])
@pytest.mark.parametrize("dims", [16, 10])
def test_rotation_with_slowed_waves_biases_and_whole_row_norms(scaling, dims):
    from evo_b200.gagotar import GagotarConfig
    cfg = O.make_config(dim=16, rot_dims=dims, rot_base=400.0, scaling=scaling)
    a = GagotarConfig.from_dict(cfg).layers[0].left
    H, G, dk, dv, L, pos0 = 4, 2, 16, 12, 9, 250
    rot = cfg["layers"][0]["mixer"]["left"]["rot"]
    g = torch.Generator().manual_seed(dims)
    qw, kw, vw = H * dk, G * dk, G * dv
    z = _bf(torch.randn(L, qw + kw + vw, generator=g))
    qb, kb, vb, qn, kn = (_bf(torch.randn(n, generator=g)) for n in (qw, kw, vw, qw, kw))
    pos = torch.arange(pos0, pos0 + L)
    zz = z.double()
    want_q = O.rotate((O.rms(zz[:, :qw] + qb.double(), 1e-5) * qn.double()).view(L, H, dk), pos, rot).reshape(L, qw)
    want_k = O.rotate((O.rms(zz[:, qw:qw + kw] + kb.double(), 1e-5) * kn.double()).view(L, G, dk), pos, rot).reshape(L, kw)
    freq = torch.tensor(a.frequencies(), dtype=F64).to(F32).to(DEV)
    zd, cache = z.to(DEV, F32), torch.zeros(1, pos0 + L, kw + vw, device=DEV)
    keep = [t.to(DEV) for t in (qb, kb, vb, qn, kn)]
    p = QkPrepParams(q=zd.data_ptr(), k=zd.data_ptr() + qw * 4, v=zd.data_ptr() + (qw + kw) * 4, ld=qw + kw + vw, q_bias=keep[0].data_ptr(), k_bias=keep[1].data_ptr(),
                     v_bias=keep[2].data_ptr(), q_norm_w=keep[3].data_ptr(), k_norm_w=keep[4].data_ptr(), eps=1e-5, freq=freq.data_ptr(), rot_dims=dims, cache=cache.data_ptr(),
                     cache_row=kw + vw, cache_batch_stride=cache.shape[1] * (kw + vw), B=1, L=L, H=H, G=G, dk=dk, dv=dv, pos0=pos0, dtype=1)
    check(_lib.lib().evo_qk_prep(C.byref(p), _stream()))
    _close(zd[:, :qw], want_q, 3e-5, "queries")
    _close(cache[0, pos0:, :kw], want_k, 3e-5, "keys")
    _close(cache[0, pos0:, kw:], zz[:, qw + kw:] + vb.double(), 1e-6, "values")


# ------------------------------------------------------------------ each side alone: the other side's output weight is zero, no feed-forward
def _one_side(side, T, seed=0, dtype=F32, rank=5, **sizes):
    cfg = O.make_config(mlps=(None,), **sizes)
    W = O.random_weights(cfg, seed=seed, rank=rank)
    other = "right" if side == "left" else "left"
    W[f"l0.mix.{other}.out"] = torch.zeros_like(W[f"l0.mix.{other}.out"])
    tokens = _tokens(cfg, T, seed=seed + 1)
    return cfg, W, tokens, O.forward(tokens, W, cfg), _model(cfg, W, dtype)


LEFT = [dict(heads=4, kv_heads=2, dim=16, vdim=12, chunk=24), dict(heads=3, kv_heads=1, dim=10, vdim=9, chunk=7, rot_dims=6, width=50),
        dict(heads=2, kv_heads=2, dim=24, vdim=40, chunk=0, rot_dims=24, scaling=None), dict(heads=1, kv_heads=1, dim=8, vdim=140, chunk=1, rot_dims=0, width=40),
        dict(heads=18, kv_heads=6, dim=16, vdim=8, chunk=31, rot_dims=16)]


@pytest.mark.parametrize("sizes", LEFT, ids=lambda s: "h{heads}g{kv_heads}k{dim}v{vdim}c{chunk}".format(**s))
def test_attention_side_matches_the_oracle(sizes):
    cfg, W, tokens, want, model = _one_side("left", 100, seed=sizes["dim"], **sizes)
    got, _ = model(torch.tensor([tokens], device=DEV))
    _close(got[0], want, 3e-5, "whole")
    _close(_portions(model, tokens, [37, 2, 1, 1, 40, 19]), want, 3e-5, "portions and steps")


RIGHT = [dict(lin_heads=2, lin_dim=12, lin_vdim=20, tau=8.0), dict(lin_heads=3, lin_dim=5, lin_vdim=7, tau=1.0, width=50), dict(lin_heads=4, lin_dim=48, lin_vdim=40, tau=16.0, width=96),
         dict(lin_heads=1, lin_dim=72, lin_vdim=136, tau=3.0), dict(lin_heads=1, lin_dim=1, lin_vdim=2, tau=2.0)]


@pytest.mark.parametrize("sizes", RIGHT, ids=lambda s: "h{lin_heads}k{lin_dim}v{lin_vdim}t{tau}".format(**s))
@pytest.mark.parametrize("rank", [1, 20])
def test_linear_attention_side_matches_the_oracle(sizes, rank):
    cfg, W, tokens, want, model = _one_side("right", 70, seed=sizes["lin_dim"], rank=rank, **sizes)
    got, _ = model(torch.tensor([tokens], device=DEV))
    _close(got[0], want, 3e-5, "whole")
    _close(_portions(model, tokens, [1] * 70), want, 3e-5, "token by token")
    _close(_portions(model, tokens, [17, 2, 1, 33, 16, 1]), want, 3e-5, "portions that cut the kernel's rounds of 16 tokens")


def test_linear_attention_remembers_the_first_token():
    """Decays of almost 1: the first token's key and value still shape the answer a hundred tokens later, through portions and steps."""
    cfg = O.make_config(mlps=(None,), vocab=50, chunk=4, tau=16.0)
    W = O.random_weights(cfg, seed=4)
    W["l0.mix.left.out"] = torch.zeros_like(W["l0.mix.left.out"])
    W["l0.mix.right.a2.b"] = _bf(torch.full_like(W["l0.mix.right.a2.b"].float(), 9.0))
    a, b = [7] * 120, [31] + [7] * 119
    wa, wb = O.forward(a, W, cfg), O.forward(b, W, cfg)
    assert (wa[100:] - wb[100:]).abs().max() > 1e-3 * wa.abs().max()
    model = _model(cfg, W)
    for tokens, want in ((a, wa), (b, wb)):
        _close(_portions(model, tokens, [1, 2, 50, 30] + [1] * 37), want, 3e-5)


# ------------------------------------------------------------------ keys far away, chunk edges
@pytest.mark.parametrize("dtype", [F32, B16])
@pytest.mark.parametrize("chunk", [0, 128])
def test_far_key_among_hundreds_and_chunk_edges_through_the_model(chunk, dtype):
    """A prompt of one repeated token with ONE other token, under sharpened queries: rows of its chunk depend on it, rows of the next chunk
    do not see it at all; prompts (whole and cut at, before and behind the edges) and steps follow the oracle."""
    cfg = O.make_config(mlps=(None,), vocab=50, chunk=chunk, rot_dims=0)
    W = O.random_weights(cfg, seed=9)
    W["l0.mix.right.out"] = torch.zeros_like(W["l0.mix.right.out"])
    W["l0.mix.left.q.norm"] = _bf(W["l0.mix.left.q.norm"].float() * 5)
    T = 300
    model = _model(cfg, W, dtype)
    tol = 3e-5 if dtype == F32 else 4e-2
    plain = O.forward([7] * T, W, cfg)
    for j in ((5,) if not chunk else (0, 127, 128, 255)):
        tokens = [7] * T
        tokens[j] = 31
        want = O.forward(tokens, W, cfg)
        moved = (want - plain).abs().amax(-1) > 0.02 * plain.abs().max()
        end = T if not chunk else (j // chunk + 1) * chunk
        assert not moved[:j].any() and not moved[end:].any() and moved[j] and (end - j < 3 or moved[j + 1:end].any())
        got, _ = model(torch.tensor([tokens], device=DEV))
        _close(got[0], want, tol, f"whole, key {j}")
        _close(_portions(model, tokens, [126, 1, 1, 1, 126, 2] + [1] * 43), want, tol, f"cut around the edges, steps, key {j}")
        _close(_portions(model, tokens, [128, 128, 44]), want, tol, f"cut at the edges, key {j}")


# ------------------------------------------------------------------ the model
CONFIGS = {
    "two": dict(),
    "gaps": dict(mlps=("moe", None, "moe", "moe"), width=72, vocab=257, chunk=10, experts=12, top=3, rot_dims=16, dim=16),
    "bare": dict(mlps=(None, "moe"), rot_dims=0, chunk=0, top=1, experts=3),
    "ones": dict(mlps=("moe", "moe"), heads=1, kv_heads=1, lin_heads=1, experts=1, top=1, tau=1.0, scale=1.0, chunk=16),
    "odd": dict(mlps=("moe", "moe", "moe"), width=50, vocab=33, heads=3, kv_heads=1, dim=10, vdim=9, rot_dims=6, chunk=13, lin_heads=3, lin_dim=5, lin_vdim=7, experts=5, top=5, expert_ff=10),
    "wide": dict(mlps=("moe", "moe"), width=200, heads=6, kv_heads=3, dim=72, vdim=40, rot_dims=40, chunk=48, lin_heads=2, lin_dim=70, lin_vdim=136, experts=8, top=4, expert_ff=40, limit=3.0),
    "many": dict(mlps=("moe", "moe"), width=96, heads=24, kv_heads=4, dim=8, vdim=16, rot_dims=8, chunk=20, lin_heads=6, lin_dim=8, lin_vdim=8, scaling=None),
}


def _tolerance(cfg, W, tokens, want):
    """Bound on the 32-bit model's distance from the fp64 oracle: three times what the oracle itself loses when it runs in 32-bit floats, at
    least 3e-5 of the scale."""
    own = ((O.forward(tokens, W, cfg, dtype=F32).double() - want).abs().max() / want.abs().max()).item()
    assert own < 1e-4
    return max(3e-5, 3 * own)


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_model_whole_steps_and_portions_match_the_oracle_in_fp32(name):
    cfg = O.make_config(**CONFIGS[name])
    W = O.random_weights(cfg, seed=len(name), rank=3 + len(name))
    T = 75
    tokens = _tokens(cfg, T)
    streams = []
    want = O.forward(tokens, W, cfg, taps=streams)
    tol = _tolerance(cfg, W, tokens, want)
    model = _model(cfg, W)
    model._tap = []
    got, _ = model(torch.tensor([tokens], device=DEV))
    assert len(model._tap) == len(streams)
    for r, (a, b) in enumerate(zip(model._tap, streams)):
        _close(a, b, tol, f"{name}: stream after layer {r}")
    model._tap = None
    got, _ = model(torch.tensor([tokens], device=DEV))
    _close(got[0], want, tol, f"{name}: whole")
    _close(_portions(model, tokens, [1] * T), want, tol, f"{name}: token by token from the first token")
    _close(_portions(model, tokens, [40] + [1] * 35), want, tol, f"{name}: prompt then steps")
    _close(_portions(model, tokens, [2, 2, 3, 30, 1, 2, 17, 9, 2, 5, 2]), want, tol, f"{name}: portions")
    _close(_portions(model, tokens[:1], [1]), want[:1], tol, f"{name}: a one-token sequence")
    _close(_portions(model, tokens[:2], [2]), want[:2], tol, f"{name}: a two-token sequence")
    model.moe_sparse_min_rows = 1                             # only the chosen experts, row by row, instead of all experts densely
    sparse, _ = model(torch.tensor([tokens], device=DEV))
    _close(sparse[0], want, tol, f"{name}: chosen experts only")


def test_layers_with_their_own_sizes_and_a_cache_that_has_to_grow():
    cfg = O.make_config(mlps=("moe", "moe", None, "moe"), width=104, vocab=211)
    cfg["layers"][1]["type"] = "parallel_2"                   # a numbered type: the same mechanism with sizes of its own
    cfg["layers"][1]["mixer"]["left"] = {"heads": 6, "kv_heads": 3, "dim": 8, "vdim": 40, "scale": 0.2, "mask": {"size": 31}, "rot": {"base": 7.0, "dims": 8}}
    cfg["layers"][2]["mixer"]["right"] = {"heads": 3, "dim": 24, "vdim": 9, "tau": 5.0}
    cfg["layers"][3]["mlp"] = {"kind": "moe", "expert": {"ff": 40, "limit": 0.7}, "router": {"experts": 9, "top": 4}}
    W = O.random_weights(cfg, seed=21)
    extra = O.random_weights(cfg, seed=22, rank=11)           # one layer's decay projection has another rank
    W.update({k: v for k, v in extra.items() if k.startswith("l2.mix.right.a")})
    tokens = _tokens(cfg, 70, seed=8)
    want = O.forward(tokens, W, cfg)
    tol = _tolerance(cfg, W, tokens, want)
    model = _model(cfg, W)
    assert [l.right.rank for l in model.config.layers] == [5, 5, 11, 5]
    got, _ = model(torch.tensor([tokens], device=DEV))
    _close(got[0], want, tol, "whole")
    state = model.initialize_inference_params(max_seqlen=16, max_batch_size=1)
    _close(_portions(model, tokens, [9, 2, 20, 1, 1, 30, 7], state=state), want, tol, "portions through a growing cache")
    assert all(c.shape[1] >= 70 for c in state["mha"].key_value_memory_dict.values())


def test_model_bf16_stays_within_rounding_of_the_oracle_and_of_itself():
    cfg = O.make_config(vdim=16, expert_ff=32)
    W = O.random_weights(cfg, seed=3)
    tokens = _tokens(cfg, 90, seed=2)
    want = O.forward(tokens, W, cfg)
    model = _model(cfg, W, B16)
    whole, _ = model(torch.tensor([tokens], device=DEV))
    cut = _portions(model, tokens, [50, 2, 1, 1, 30, 6])

    def rel(a, b):
        """Median over positions (a close call of the router may move single positions) of the rms difference over the vocabulary."""
        d = (a.double().cpu() - b.double().cpu()).pow(2).mean(-1).sqrt()
        return (d.median() / b.double().pow(2).mean().sqrt()).item()
    assert rel(whole[0], want) < 3e-2
    assert rel(cut, want) < 3e-2
    assert rel(cut, whole[0].cpu()) < 3e-2
    model.gemm_path = "simt"                              # the tensor-core linear layers against the CUDA-core ones
    simt, _ = model(torch.tensor([tokens], device=DEV))
    assert rel(simt[0], whole[0].cpu()) < 2e-2
    model.gemm_path = "tc"
    model.mixed_attn_cuda_cores = 1                       # and the tensor-core attention against the CUDA-core one
    plain, _ = model(torch.tensor([tokens], device=DEV))
    assert rel(plain[0], whole[0].cpu()) < 2e-2


def test_batch_rows_equal_each_sequence_alone_and_wanted_rows_select():
    cfg = O.make_config()
    W = O.random_weights(cfg, seed=5)
    for dtype, tol in ((F32, 2e-6), (B16, 2e-2)):
        model = _model(cfg, W, dtype)
        ids = torch.randint(0, cfg["vocab"], (3, 33), generator=torch.Generator().manual_seed(4)).to(DEV)
        both, _ = model(ids)
        for b in range(3):
            alone, _ = model(ids[b:b + 1])
            _close(both[b], alone[0].double().cpu(), tol, f"row {b}")
        state = model.initialize_inference_params(max_seqlen=64, max_batch_size=3)
        a, _ = model(ids[:, :20], inference_params_dict=state)
        state["mha"].seqlen_offset = state["hyena"].seqlen_offset = 20
        b_, _ = model(ids[:, 20:], inference_params_dict=state)
        if dtype == F32:
            _close(torch.cat([a, b_], 1), both.double().cpu(), 1e-5, "batched portions")
        rows = [0, 7, 32, 40, 98]
        picked, _ = model(ids, logits_rows=rows)
        _close(picked, both.reshape(-1, both.shape[-1])[rows].double().cpu(), tol, "wanted rows")
        none, _ = model(ids, logits_rows=[])
        assert none.shape == (0, cfg["vocab"])


def test_reused_state_memory_and_long_decoding():
    """State holders that still hold another request's rows and matrix states (and NaNs beyond) serve a new request; decoding runs for
    hundreds of steps over many chunks; requests of unequal length interleaved keep their own state."""
    cfg = O.make_config(chunk=50)
    W = O.random_weights(cfg, seed=7)
    model = _model(cfg, W)
    a, b = _tokens(cfg, 260, seed=6), _tokens(cfg, 60, seed=9)
    want_a, want_b = O.forward(a, W, cfg), O.forward(b, W, cfg)
    state = model.initialize_inference_params(max_seqlen=272, max_batch_size=1)
    _close(_portions(model, a, [20] + [1] * 240, state=state), want_a, 3e-5, "long decoding")
    for cache in state["mha"].key_value_memory_dict.values():
        cache[:, 100:, :3] = float("nan")
    _close(_portions(model, b, [7, 2, 51], state=state), want_b, 3e-5, "the same holders, used again from position 0")
    for s in state["hyena"].state_dict.values():
        s.fill_(float("nan"))
    _close(_portions(model, b, [7, 2, 51], state=state), want_b, 3e-5, "stale matrix states do not reach a new request")
    sa = model.initialize_inference_params(max_seqlen=128, max_batch_size=1)
    sb = model.initialize_inference_params(max_seqlen=128, max_batch_size=1)
    outs_a, outs_b, ta, tb = [], [], 0, 0
    for na, nb in ((30, 2), (1, 40), (29, 1), (2, 17)):
        for tokens, st, outs, lo, n in ((a, sa, outs_a, ta, na), (b, sb, outs_b, tb, nb)):
            st["mha"].seqlen_offset = st["hyena"].seqlen_offset = lo
            lg, _ = model(torch.tensor([tokens[lo:lo + n]], device=DEV), inference_params_dict=st)
            outs.append(lg[0])
        ta, tb = ta + na, tb + nb
    _close(torch.cat(outs_a), want_a[:ta], 3e-5, "interleaved a")
    _close(torch.cat(outs_b), want_b[:tb], 3e-5, "interleaved b")


@pytest.mark.parametrize("device_loop", [True, False])
def test_greedy_generation_through_the_generator(device_loop):
    from evo_b200 import CharLevelTokenizer, Generator
    cfg = O.make_config(vocab=512, chunk=32)                  # the new tokens cross a chunk edge
    W = O.random_weights(cfg, seed=11)
    model = _model(cfg, W)
    gen = Generator(model, CharLevelTokenizer(512), top_k=1, top_p=1.0, temperature=1.0)
    gen.device_loop = device_loop
    prompt = torch.randint(0, 512, (2, 21), generator=torch.Generator().manual_seed(8)).to(DEV)
    n_new = 24
    picked, logits, _ = gen.generate(DEV, input_ids=prompt, num_tokens=n_new, cached_generation=True, force_prompt_threshold=64, print_generation=False, stop_at_eos=False)
    assert picked.shape == (2, n_new) and logits.shape == (2, n_new, 512)
    for b in range(2):
        full = prompt[b].tolist() + picked[b].tolist()
        want = O.forward(full, W, cfg)
        for s in range(n_new):                                # each picked token is (within rounding) the oracle's argmax given the same prefix
            row = want[len(full) - n_new - 1 + s]
            assert row[picked[b, s]] >= row.max() - 2e-2, (b, s)
            _close(logits[b, s], row, 3e-5 if not device_loop else 1e-2, f"kept logits {b} {s}")     # the device loop keeps the sampler's bf16 view of the logits


def test_command_line_generates_and_replays_from_a_checkpoint_folder(tmp_path):
    """scripts/generate.py --model-dir and bin/trace_run: config.json picks the model class, the streaming loader fills it."""
    import json
    import os
    import subprocess
    import sys
    import numpy as np
    from tests.test_zaverax_host import ROOT, _write_checkpoint
    from scripts import generate as cli
    cfg = O.make_config(vocab=512)
    W = O.random_weights(cfg, seed=13, rank=7)
    ckpt = str(tmp_path / "ckpt")
    _write_checkpoint(ckpt, cfg, W)
    texts, scores = cli.main(["--model-dir", ckpt, "--prompt", "ACGTTGCA", "--n-samples", "2", "--n-tokens", "9", "--top-k", "1", "--device", DEV, "--verbose", "0"])
    assert len(texts) == 2 and texts[0] == texts[1] and len(scores) == 2
    tokens = _tokens(cfg, 40, seed=5)
    want = O.forward(tokens, W, cfg)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": tokens[:25], "want": [0, 24]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": tokens[25:27], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": tokens[27:28], "want": [0]}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": tokens[28:], "want": [11]}], "end": ["a"]},
             {"step": 4, "entries": [{"id": "b", "tokens": tokens[:3], "want": [2]}], "end": ["b"]}]
    out = str(tmp_path / "out")
    for dtype, tol in (("float32", 3e-5), ("bfloat16", 6e-2)):
        r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", ckpt, "--dtype", dtype, "--out", out, "--max-tokens", "64"],
                           input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
        assert r.returncode == 0, r.stderr
        assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(5)]
        assert not os.path.exists(os.path.join(out, "1.f32"))
        for step, rows in ((0, [0, 24]), (2, [27]), (3, [39]), (4, [2])):
            got = torch.from_numpy(np.fromfile(os.path.join(out, f"{step}.f32"), dtype="<f4").reshape(len(rows), 512).copy())
            _close(got, want[rows], tol, f"replayed step {step} in {dtype}")
