"""Nilatar on the GPU against the plain oracle (oracle/nilatar_oracle.py): the kernels alone (linear attention token by token and block by
block, norm with gate, latent preparation, sink windows), each mixer alone over several sizes, then the model -- whole prompts,
token-by-token decoding, portions down to two tokens, batches, reused state memory, far keys, window edges, the first tokens of a
sequence, long decoding, other sizes -- and greedy generation through the framework's Generator and command line.  Small
configurations, random weights; where random weights would hide a fault the weights are made so that it shows."""
import ctypes as C
import math

import pytest
import torch

from evo_b200 import _lib
from evo_b200._lib import DecayScanParams, LatentPrepParams, WindowAttnParams, check, ptr
from oracle import nilatar_oracle as O

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
    from evo_b200.nilatar import Nilatar, NilatarConfig
    m = Nilatar(NilatarConfig.from_dict(cfg), dtype=dtype)
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


def _whole(model, tokens):
    return model(torch.tensor([tokens], device=DEV))[0][0]


# ------------------------------------------------------------------ kernels alone
def _scan(q, k, v, decay, dtype, cuts, state=None, act=0, q_scale=1.0, pad=0, recurrent=0, part_len=0):
    """q, k (B, T, H, dk), v (B, T, H, dv) through evo_decay_scan_fwd in calls of `cuts` tokens -> (B, T, H, dv), last state."""
    B, T, H, dk = q.shape
    dv = v.shape[-1]
    z = torch.cat([q.reshape(B, T, -1), k.reshape(B, T, -1), v.reshape(B, T, -1), torch.full((B, T, pad), float("nan"))], -1)
    keep = state is not None
    st = (torch.full((B, H, dk, dv), float("nan"), device=DEV) if state == "zero" else state.to(DEV, F32).clone()) if keep else None
    d = decay.to(DEV, F32)
    outs, t = [], 0
    lib = _lib.lib()
    for n in cuts:
        zc = z[:, t:t + n].contiguous().to(DEV, dtype)
        ld, esz = zc.shape[-1], zc.element_size()
        y = torch.full((B, n, H, dv), float("nan"), device=DEV)
        p = DecayScanParams(q=zc.data_ptr(), k=zc.data_ptr() + H * dk * esz, v=zc.data_ptr() + 2 * H * dk * esz, ld=ld, decay=d.data_ptr(), act=act, q_scale=q_scale,
                            state=st.data_ptr() if keep else None, zero_start=int(state is None or (isinstance(state, str) and t == 0)), y=y.data_ptr(),
                            dtype=1 if dtype == F32 else 0, B=B, L=n, H=H, dk=dk, dv=dv, recurrent=recurrent, part_len=part_len)
        nws = lib.evo_decay_scan_workspace(C.byref(p))
        ws = torch.full((max(nws, 1),), 0xFF, dtype=torch.uint8, device=DEV)               # NaNs where nothing has been written
        check(lib.evo_decay_scan_fwd(C.byref(p), ptr(ws), nws, _stream()))
        outs.append(y)
        t += n
    assert t == T
    return torch.cat(outs, 1), st


# heads, dk, dv: one of everything, odd sizes, several 64-channel slices, rows that fill one and two tiles per warp
SCAN_SHAPES = [(2, 16, 24), (1, 1, 1), (3, 5, 7), (2, 32, 64), (2, 64, 130), (1, 72, 136), (2, 128, 128), (1, 120, 66), (1, 100, 33)]


@pytest.mark.parametrize("H,dk,dv", SCAN_SHAPES, ids=lambda v: str(v))
def test_decay_scan_kernels_match_fp64(H, dk, dv):
    """Token by token (fp32 and bf16) and block by block (bf16; one part and several, parts of one and two blocks), a carried state, no state."""
    g = torch.Generator().manual_seed(H * dk + dv)
    B, T = 2, 203
    q, k, v = (_bf(torch.randn(B, T, H, n, generator=g)).float() for n in (dk, dk, dv))
    decay = torch.tensor([0.999, 0.55, 1.0, 0.0][:H])
    start = torch.randn(B, H, dk, dv, generator=g)
    for state in ("zero", start):
        s0 = torch.zeros(B, H, dk, dv) if isinstance(state, str) else state
        want, last = zip(*[O.decay_scan(q[b].double() * 0.5, k[b].double(), v[b].double(), decay.double(), s0[b].double()) for b in range(B)])
        want, last = torch.stack(want), torch.stack(last)
        for what, dtype, tol, kw in (("fp32", F32, 3e-6, {}), ("bf16 tokens", B16, 3e-6, dict(recurrent=1)), ("bf16 blocks", B16, 3e-5, {}),
                                     ("parts of a block", B16, 3e-5, dict(part_len=64)), ("parts of two blocks", B16, 3e-5, dict(part_len=65))):
            for cuts in ([T], [64, 64, 75], [33, 1, 2, 127, 40], [65, 63, 32, 43]):
                y, s = _scan(q, k, v, decay, dtype, cuts, state=state, q_scale=0.5, pad=3, **kw)
                _close(y, want, tol, f"{what}, read-outs, {cuts}")
                _close(s, last, tol, f"{what}, last state, {cuts}")
    want, _ = zip(*[O.decay_scan(q[b].double(), k[b].double(), v[b].double(), decay.double()) for b in range(B)])
    for part_len in (0, 64):
        _close(_scan(q, k, v, decay, B16, [T], part_len=part_len)[0], torch.stack(want), 3e-5, "no state kept")


@pytest.mark.parametrize("dtype,recurrent,tol", [(F32, 0, 3e-6), (B16, 1, 3e-6), (B16, 0, 1.2e-2)])
def test_decay_scan_applies_silu_to_what_it_reads(dtype, recurrent, tol):
    g = torch.Generator().manual_seed(1)
    q, k, v = (_bf(torch.randn(1, 90, 2, n, generator=g) * 2).float() for n in (24, 24, 40))
    decay = torch.tensor([0.9, 0.99])
    want, _ = O.decay_scan(*(O.silu(t[0].double()) for t in (q, k, v)), decay.double())
    _close(_scan(q, k, v, decay, dtype, [90], act=1, recurrent=recurrent)[0][0], want, tol)
    _close(_scan(q, k, v, decay, dtype, [50, 2, 38], act=1, state="zero", recurrent=recurrent)[0][0], want, tol)


@pytest.mark.parametrize("dtype", [F32, B16])
@pytest.mark.parametrize("jump", [0, 1, 62, 63, 64, 65, 127, 128, 190])
def test_decay_scan_one_token_decides(jump, dtype):
    """All keys are zero but one token's: read-outs before it are zero, behind it the decayed value, across every border of the blocks."""
    T, decay = 200, torch.tensor([0.97])
    q, k, v = torch.ones(1, T, 1, 8), torch.zeros(1, T, 1, 8), torch.ones(1, T, 1, 16)
    k[0, jump, 0, 3] = 1.0
    v[0, jump] = torch.arange(16.0)
    want = torch.zeros(T, 1, 16)
    for t in range(jump, T):
        want[t, 0] = 0.97 ** (t - jump) * torch.arange(16.0)
    for cuts in ([T], [64, 136], [63, 65, 72], [100] + [1] * 100):
        for part_len in (0, 64):
            y, _ = _scan(q, k, v, decay, dtype, cuts, state="zero", part_len=part_len)
            assert (y[0, :jump] == 0).all()
            _close(y[0], want, 2e-5, f"{cuts} {part_len}")


@pytest.mark.parametrize("M,width,ld,ldo", [(5, 24, 40, 64), (3, 7, 9, 11), (2, 5000, 5004, 5056), (1, 4096, 4096, 4096), (33, 130, 136, 192)])
@pytest.mark.parametrize("dtype", [F32, B16])
def test_norm_gate(M, width, ld, ldo, dtype):
    g = torch.Generator().manual_seed(width)
    y, gate, w = torch.randn(M, width, generator=g) * 3, _bf(torch.randn(M, ld, generator=g)), _bf(torch.randn(width, generator=g))
    out = torch.full((M, ldo), 5.0, dtype=dtype, device=DEV)
    yd, gd, wd = y.to(DEV), gate.to(DEV, dtype), w.to(DEV)
    check(_lib.lib().evo_norm_gate(ptr(yd), ptr(gd), ld, ptr(wd), ptr(out), ldo, M, width, 1e-3, 1 if dtype == F32 else 0, _stream()))
    want = O.rms(y.double(), w.double(), 1e-3) * torch.sigmoid(gate[:, :width].double())
    _close(out[:, :width], want, 2e-6 if dtype == F32 else 5e-3)
    assert (out[:, width:] == 0).all()


@pytest.mark.parametrize("M,F,K", [(5, 40, 72), (64, 130, 64), (100, 128, 130), (600, 300, 200)])
def test_gelu_gate_and_silu_columns_in_the_gemm_epilogue(M, F, K):
    """Rows for each of the GEMM's tile shapes; the comparator path runs the same weights through a second kernel."""
    from evo_b200.stream_model import _Packed, _PackedGate
    model = _model(O.make_config(), O.make_weights(O.make_config()), B16)
    g = torch.Generator().manual_seed(M)
    gate, up, h = _bf(torch.randn(F, K, generator=g) / math.sqrt(K) * 2), _bf(torch.randn(F, K, generator=g) / math.sqrt(K)), _bf(torch.randn(M, K, generator=g))
    pk, lin = _PackedGate(gate.to(DEV), up.to(DEV)), _Packed(gate.to(DEV))
    hp = torch.zeros(M, pk.Kp, dtype=B16, device=DEV)
    hp[:, :K] = h.to(DEV)
    zg, zu = h.double() @ gate.double().T, h.double() @ up.double().T
    want = O.gelu_tanh(zg) * zu
    for path, tol in (("tc", 5e-3), ("simt", 1.5e-2)):
        model.gemm_path = path
        a = model._gelu_gate(hp, pk, M)
        assert a.shape == (M, (F + 127) // 128 * 128) and (a[:, F:] == 0).all()
        _close(a[:, :F], want, tol, path)
    model.gemm_path = "tc"
    for cols in (F, F - 7, 33, 1):
        z = model._linear(hp, lin, M, silu_cols=cols)
        _close(z[:, :cols], O.silu(zg[:, :cols]), 5e-3, f"{cols} columns through silu")
        if cols < F:
            _close(z[:, cols:F], zg[:, cols:], 5e-3, f"the others of {cols}")
    full = _model(O.make_config(), O.make_weights(O.make_config()), F32)
    a = full._gelu_gate(hp.float(), pk, M)
    _close(a[:, :F], want, 3e-6, "fp32")
    assert (a[:, F:] == 0).all()


def test_scaled_embedding():
    g = torch.Generator().manual_seed(0)
    table = _bf(torch.randn(19, 30, generator=g)).to(DEV)
    for ids in (torch.tensor([0, 18, 7], device=DEV), torch.tensor([3, 3], device=DEV, dtype=torch.int32)):
        out = torch.empty(len(ids), 30, device=DEV)
        check(_lib.lib().evo_embed_scaled_f32(ptr(ids), int(ids.dtype == torch.int64), ptr(table), ptr(out), len(ids), 30, 19, 2.75, _stream()))
        assert torch.equal(out, table.float()[ids.long()] * 2.75)


@pytest.mark.parametrize("dtype", [F32, B16])
@pytest.mark.parametrize("device_pos", [False, True])
def test_latent_preparation_parts(dtype, device_pos):
    """The three parts together and one at a time, partly turned rotated parts, lengths of turned vectors, padded query latents."""
    g = torch.Generator().manual_seed(3)
    B, L, H, dim, rd, dims, rank, q_rank, pos0 = 2, 5, 3, 6, 10, 8, 13, 11, 700
    hd, rank_pad, row, ld_cq, eps, length = dim + rd, 16, 32, 64, 1e-4, 1.3
    z = _bf(torch.randn(B * L, H * hd + rank + rd + q_rank + 2, generator=g))
    nw, qnw = _bf(torch.randn(rank, generator=g)), _bf(torch.randn(q_rank, generator=g))
    rot = {"base": 50.0, "dims": dims}
    freq = torch.tensor(O.turn_frequencies(rot), dtype=F64)
    x = z.double().view(B, L, -1)
    turned = lambda t: torch.stack([O.turn(t[b], rot, pos0) for b in range(B)])
    q, down, dq = x[..., :H * hd].reshape(B, L, H, hd), x[..., H * hd:H * hd + rank + rd], x[..., H * hd + rank + rd:H * hd + rank + rd + q_rank]
    grow = torch.ones(rd, dtype=F64)
    grow[:dims] = length
    want_q = torch.cat([q[..., :dim], turned(q[..., dim:]) * grow], -1).reshape(B * L, H * hd)
    want_c, want_r = O.rms(down[..., :rank], nw.double(), eps), turned(down[..., None, rank:])[..., 0, :] * grow
    want_cq = O.rms(dq, qnw.double(), eps).reshape(B * L, q_rank)
    tol = 1e-5 if dtype == F32 else 8e-3
    fd, nwd, qnwd = freq.to(F32).to(DEV), nw.to(DEV), qnw.to(DEV)
    pd = torch.tensor([pos0], dtype=torch.int64, device=DEV)
    for parts in (("q", "dkv", "dq"), ("q",), ("dkv",), ("dq",), ("dkv", "dq")):
        zd = z.to(DEV, dtype)
        cache = torch.full((B, pos0 + L + 2, row), 7.0, dtype=dtype, device=DEV)
        cq = torch.full((B * L, ld_cq), 7.0, dtype=dtype, device=DEV)
        esz, ld = zd.element_size(), zd.shape[1]
        p = LatentPrepParams(eps=eps, freq=fd.data_ptr(), B=B, L=L, H=H, dim=dim, rot=rd, rank=rank, pos0=0 if device_pos else pos0, pos_dev=pd.data_ptr() if device_pos else None,
                             dtype=1 if dtype == F32 else 0, rot_dims=dims, rot_len=length)
        if "q" in parts:
            p.q, p.ldq = zd.data_ptr(), ld
        if "dkv" in parts:
            p.dkv, p.ld_dkv, p.norm_w = zd.data_ptr() + H * hd * esz, ld, nwd.data_ptr()
            p.cache, p.cache_row, p.cache_batch_stride, p.rank_pad = cache.data_ptr(), row, cache.stride(0), rank_pad
        if "dq" in parts:
            p.dq, p.ld_dq, p.dq_norm_w, p.q_rank, p.cq, p.ld_cq = zd.data_ptr() + (H * hd + rank + rd) * esz, ld, qnwd.data_ptr(), q_rank, cq.data_ptr(), ld_cq
        check(_lib.lib().evo_latent_prep(C.byref(p), _stream()))
        got_q = zd[:, :H * hd]
        if "q" in parts:
            _close(got_q, want_q, tol, "queries")
        else:
            assert torch.equal(got_q, z[:, :H * hd].to(DEV, dtype))
        rows = cache[:, pos0:pos0 + L]
        if "dkv" in parts:
            _close(rows[..., :rank], want_c, tol, "latent")
            assert (rows[..., rank:rank_pad] == 0).all()
            _close(rows[..., rank_pad:rank_pad + rd], want_r, tol, "key part")
        else:
            assert (rows == 7).all()
        assert (cache[:, :pos0] == 7).all() and (cache[:, pos0 + L:] == 7).all()
        if "dq" in parts:
            _close(cq[:, :q_rank], want_cq, tol, "query latent")
            assert (cq[:, q_rank:] == 0).all()
        else:
            assert (cq == 7).all()


# heads, key heads, dk, dv, window: the tensor-core kernel up to 256-wide keys, odd sizes for the CUDA-core kernels
WINDOW_SHAPES = [(4, 2, 16, 16, 24), (2, 1, 192, 128, 70), (2, 2, 256, 64, 0), (3, 3, 200, 24, 33), (1, 1, 5, 7, 1), (6, 3, 40, 48, 64), (2, 2, 136, 8, 65)]


@pytest.mark.parametrize("H,G,dk,dv,window", WINDOW_SHAPES, ids=lambda v: str(v))
def test_sink_windows_with_a_gate_per_channel(H, G, dk, dv, window):
    g = torch.Generator().manual_seed(dk + window)
    L, pos0 = 90, 41
    T = pos0 + L
    q, k, v, gate = (_bf(torch.randn(*s, generator=g)) for s in ((L, H, dk), (T, G, dk), (T, G, dv), (L, H * dv)))
    sink = _bf(torch.randn(H, generator=g) * 2)
    scale = 1.3 / math.sqrt(dk)
    want = O.softmax_attention(q.double(), k.double(), v.double(), scale, window, sink.double(), pos0).reshape(L, H * dv) * torch.sigmoid(gate.double())
    ldo = (H * dv + 63) // 64 * 64
    for dtype, rows, tol in ((B16, L, 1.2e-2), (B16, 17, 1.2e-2), (F32, L, 3e-5), (F32, 1, 3e-5), (B16, 2, 1.2e-2)):
        qd, kd, vd, gd, sd = q.to(DEV, dtype).reshape(L, -1), k.to(DEV, dtype).reshape(T, -1), v.to(DEV, dtype).reshape(T, -1), gate.to(DEV, dtype), sink.to(DEV)
        outs = []
        for lo in range(0, L, rows):
            n = min(rows, L - lo)
            out = torch.full((n, ldo), 5.0, dtype=dtype, device=DEV)
            p = WindowAttnParams(q=qd[lo:].data_ptr(), q_tok_stride=H * dk, k=kd.data_ptr(), v=vd.data_ptr(), k_tok_stride=G * dk, v_tok_stride=G * dv, gate=gd[lo:].data_ptr(),
                                 gate_tok_stride=H * dv, out=out.data_ptr(), ldo=ldo, dtype=1 if dtype == F32 else 0, B=1, Lq=n, H=H, G=G, dk=dk, dv=dv, n_maps=1, q_pos0=pos0 + lo,
                                 window=window, scale=scale, sink=sd.data_ptr())
            check(_lib.lib().evo_window_attn_fwd(C.byref(p), _stream()))
            assert (out[:, H * dv:] == 0).all()
            outs.append(out[:, :H * dv])
        _close(torch.cat(outs, 0), want, tol, f"{dtype}, {rows} rows a call")


# heads, key heads, dk, dv, window, rows, first position: one tile, a tile and a bit, several pairs of tiles; windows of one position, at and
# around a key tile, longer than the sequence; every count of 64-column halves, head sizes that fill none of them
PROMPT_SHAPES = [(2, 1, 64, 64, 0, 128, 0), (2, 2, 128, 128, 0, 300, 77), (1, 1, 192, 128, 0, 257, 3), (3, 1, 192, 40, 200, 400, 130), (4, 2, 48, 48, 136, 310, 0), (2, 1, 128, 128, 1, 260, 5),
                 (2, 2, 64, 128, 128, 520, 64), (2, 1, 72, 72, 129, 385, 1), (1, 1, 136, 8, 127, 300, 900), (2, 2, 8, 16, 40, 140, 0), (2, 1, 128, 64, 5000, 200, 10), (1, 1, 128, 128, 300, 700, 411),
                 (3, 3, 80, 104, 90, 200, 17), (2, 1, 176, 120, 0, 150, 60), (5, 5, 16, 8, 33, 129, 2)]


@pytest.mark.parametrize("H,G,dk,dv,window,L,pos0", PROMPT_SHAPES, ids=lambda v: str(v))
def test_prompt_attention_on_the_tensor_cores(H, G, dk, dv, window, L, pos0):
    """Two sequences in one call, each with cache rows of its own; the rows behind the last position hold NaNs; with and without sink, a
    gate per channel, per head and none."""
    g = torch.Generator().manual_seed(dk + L)
    B, T, lib = 2, pos0 + L, _lib.lib()
    cw, rows = G * (dk + dv), T + 5
    q, kv = _bf(torch.randn(B, L, H, dk, generator=g)), torch.full((B, rows, cw), float("nan"))
    kv[:, :T] = torch.randn(B, T, cw, generator=g)
    kv, gate, sink = _bf(kv), _bf(torch.randn(B * L, H * dv, generator=g)), _bf(torch.randn(H, generator=g) * 2)
    scale, ldo = 1.4 / math.sqrt(dk), (H * dv + 63) // 64 * 64
    qd, kvd, gd, sd = q.to(DEV), kv.to(DEV), gate.to(DEV), sink.to(DEV)
    k, v = kv[:, :T, :G * dk].double().view(B, T, G, dk), kv[:, :T, G * dk:].double().view(B, T, G, dv)
    for with_sink, per_head in ((True, False), (False, True), (False, None)):
        want = torch.stack([O.softmax_attention(q[b].double(), k[b], v[b], scale, window, sink.double() if with_sink else None, pos0) for b in range(B)]).reshape(B * L, H * dv)
        if per_head is not None:
            s = torch.sigmoid(gate.double())
            want = want * (s[:, :H].repeat_interleave(dv, 1) if per_head else s)
        out = torch.full((B * L, ldo), 5.0, dtype=B16, device=DEV)
        p = WindowAttnParams(q=qd.data_ptr(), q_tok_stride=H * dk, k=kvd.data_ptr(), v=kvd.data_ptr() + 2 * G * dk, k_tok_stride=cw, v_tok_stride=cw, k_batch_stride=rows * cw,
                             v_batch_stride=rows * cw, gate=gd.data_ptr() if per_head is not None else None, gate_tok_stride=H * dv, gate_per_head=int(bool(per_head)),
                             out=out.data_ptr(), ldo=ldo, dtype=0, B=B, Lq=L, H=H, G=G, dk=dk, dv=dv, n_maps=1, q_pos0=pos0, window=window, scale=scale,
                             sink=sd.data_ptr() if with_sink else None)
        check(lib.evo_window_attn_fwd(C.byref(p), _stream()))
        _close(out[:, :H * dv], want, 6e-3, f"sink {with_sink}, gate per head {per_head}")
        assert (out[:, H * dv:] == 0).all()


def test_prompt_attention_weights_keep_sixteen_bits():
    """Equal scores over thousands of keys with values of one sign: weights rounded to bf16 would shift every output by up to 2^-9."""
    g = torch.Generator().manual_seed(2)
    T, dk, dv = 2100, 64, 64
    q, k, v = torch.zeros(T, 1, dk), torch.zeros(T, 1, dk), 1.0 + torch.rand(T, 1, dv, generator=g)
    q[..., 0], k[..., 0] = 1.0, torch.randn(T, 1, generator=g) * 0.3
    q, k, v = _bf(q), _bf(k), _bf(v)
    want = O.softmax_attention(q.double(), k.double(), v.double(), 1.0).reshape(T, dv)
    out = torch.empty(T, dv, dtype=B16, device=DEV)
    qd, kd, vd = q.to(DEV), k.to(DEV), v.to(DEV)
    p = WindowAttnParams(q=qd.data_ptr(), q_tok_stride=dk, k=kd.data_ptr(), v=vd.data_ptr(), k_tok_stride=dk, v_tok_stride=dv, k_batch_stride=T * dk, v_batch_stride=T * dv,
                         out=out.data_ptr(), ldo=dv, dtype=0, B=1, Lq=T, H=1, G=1, dk=dk, dv=dv, n_maps=1, scale=1.0)
    check(_lib.lib().evo_window_attn_fwd(C.byref(p), _stream()))
    assert torch.equal(out.cpu(), _bf(want)) or ((out.double().cpu() - want).abs() <= 2.0 ** -8 * 1.02).all()
    assert (out.double().cpu() - _bf(want).double()).ne(0).double().mean() < 0.02      # almost every output is the correctly rounded one


# ------------------------------------------------------------------ each mixer alone
def _one_layer(kind, T, seed, **sizes):
    cfg = O.make_config(kinds=(kind,), ff=(0,), vocab=61, **sizes)
    W = O.make_weights(cfg, seed=seed)
    tokens = _tokens(cfg, T, seed=seed + 1)
    return cfg, W, tokens, O.forward(cfg, W, tokens)[0]


LATENT = [dict(), dict(lat_heads=1, lat_dim=5, rot_dim=2, lat_vdim=7, kv_rank=9, q_rank=6, width=50), dict(lat_heads=16, lat_dim=16, rot_dim=16, lat_vdim=24, kv_rank=64, q_rank=40, width=96),
          dict(lat_heads=13, lat_dim=24, rot_dim=16, lat_vdim=16, kv_rank=128, q_rank=96, scaling=None), dict(lat_heads=2, lat_dim=128, rot_dim=64, lat_vdim=128, kv_rank=72, q_rank=130),
          dict(lat_heads=4, lat_dim=40, rot_dim=24, lat_vdim=136, kv_rank=512, q_rank=1, scaling=(2.0, 9, 3.0, 2.9))]


@pytest.mark.parametrize("sizes", LATENT, ids=lambda s: "-".join(f"{k[-6:]}{v}" for k, v in s.items() if not isinstance(v, tuple)) or "default")
def test_latent_mixer_matches_the_oracle(sizes):
    cfg, W, tokens, want = _one_layer("latent_attention", 90, 3, **sizes)
    cuts = [37, 2, 1, 1, 30, 3, 4, 12]
    for dtype, tol in ((F32, 3e-5), (B16, 5e-2)):
        model = _model(cfg, W, dtype)
        _close(_whole(model, tokens), want, tol, f"{dtype}: whole")
        for path in ("shared", "head"):
            model.latent_decode_path = path
            _close(_portions(model, tokens, cuts), want, tol, f"{dtype}: portions and steps, {path}")
            _close(_portions(model, tokens, [1] * 90), want, tol, f"{dtype}: token by token, {path}")


WINDOW = [dict(), dict(heads=1, kv_heads=1, dim=5, vdim=3, window=1, width=40), dict(heads=6, kv_heads=2, dim=24, vdim=40, window=64), dict(heads=3, kv_heads=3, dim=136, vdim=130, window=17),
          dict(heads=8, kv_heads=1, dim=16, vdim=16, window=1000)]


@pytest.mark.parametrize("sizes", WINDOW, ids=lambda s: "-".join(f"{k}{v}" for k, v in s.items()) or "default")
def test_window_mixer_and_shared_keys_match_the_oracle(sizes):
    """A pair of layers: the second reads the first one's keys and values with queries, sink and gate of its own -- and a window of its own."""
    cfg = O.make_config(kinds=("attention", "shared"), ff=(0, 0), vocab=61, **sizes)
    cfg["layers"][1]["mixer"]["mask"] = {"size": cfg["layers"][0]["mixer"]["mask"]["size"] // 2 + 3}
    cfg["layers"][1]["mixer"]["scale"] = 0.17
    W = O.make_weights(cfg, seed=5)
    tokens = _tokens(cfg, 100)
    want = O.forward(cfg, W, tokens)[0]
    for dtype, tol in ((F32, 3e-5), (B16, 5e-2)):
        model = _model(cfg, W, dtype)
        _close(_whole(model, tokens), want, tol, f"{dtype}: whole")
        state = model.initialize_inference_params(max_seqlen=108, max_batch_size=1)
        _close(_portions(model, tokens, [37, 2, 1, 1, 40, 19], state=state), want, tol, f"{dtype}: portions and steps")
        assert sorted(state["mha"].key_value_memory_dict) == [0]              # the second layer holds no rows
        _close(_portions(model, tokens, [1] * 100), want, tol, f"{dtype}: token by token")


LIGHTNING = [dict(), dict(lin_heads=3, lin_dim=5, lin_vdim=7, width=50), dict(lin_heads=1, lin_dim=72, lin_vdim=136), dict(lin_heads=4, lin_dim=48, lin_vdim=40, decay=[1.0, 0.0, 0.9375, 0.25]),
             dict(lin_heads=2, lin_dim=130, lin_vdim=20), dict(lin_heads=1, lin_dim=1, lin_vdim=2, decay=[0.99])]


@pytest.mark.parametrize("sizes", LIGHTNING, ids=lambda s: "-".join(f"{k}{v}" for k, v in s.items() if k != "decay") or "default")
def test_lightning_mixer_matches_the_oracle(sizes):
    cfg, W, tokens, want = _one_layer("lightning", 150, 7, **sizes)
    for dtype, tol in ((F32, 3e-5), (B16, 5e-2)):
        model = _model(cfg, W, dtype)
        _close(_whole(model, tokens), want, tol, f"{dtype}: whole")
        _close(_portions(model, tokens, [17, 2, 1, 63, 33, 32, 1, 1]), want, tol, f"{dtype}: portions that cut the kernels' rounds and blocks")
        _close(_portions(model, tokens, [1] * 150), want, tol, f"{dtype}: token by token")


@pytest.mark.parametrize("dtype", [F32, B16])
def test_lightning_remembers_the_first_token(dtype):
    """A decay of almost 1: the first token still shapes the answer hundreds of tokens later, through portions and steps."""
    cfg = O.make_config(kinds=("lightning",), ff=(0,), vocab=50, decay=[0.9999, 0.5])
    W = O.make_weights(cfg, seed=4)
    a, b = [7] * 300, [31] + [7] * 299
    # head 0's keys answer to what token 31 has and token 7 has not
    e7, e31 = O.rms(W["embed"][7].double(), 1.0, 0.0), O.rms(W["embed"][31].double(), 1.0, 0.0)
    own = (e31 - e7 * (e31 @ e7) / (e7 @ e7)) / W["l0.norm1"].double()
    W["l0.mix.k"][:12] = _bf(W["l0.mix.k"][:12].double() * 0.5 + 20.0 / 64 * own.expand(12, -1))
    W["l0.mix.norm"][24:] = 0                                 # only head 0 is heard
    wa, wb = O.forward(cfg, W, a)[0], O.forward(cfg, W, b)[0]
    assert (wa[250:] - wb[250:]).abs().max() > 0.1 * wa.abs().max()
    model = _model(cfg, W, dtype)
    tol = 3e-5 if dtype == F32 else 4e-2
    for tokens, want in ((a, wa), (b, wb)):
        _close(_portions(model, tokens, [1, 2, 50, 30, 100] + [1] * 117), want, tol)
        _close(_whole(model, tokens), want, tol)
    if dtype == F32:
        _close(_whole(model, b)[250:] - _whole(model, a)[250:], wb[250:] - wa[250:], 2e-2, "what the first token still does")


# ------------------------------------------------------------------ far keys, window edges, the sink, the first tokens
@pytest.mark.parametrize("dtype", [F32, B16])
@pytest.mark.parametrize("window", [1, 2, 32, 100])
def test_window_edge_with_one_dominant_key(window, dtype):
    """One token's key beats all others by far under every query: the last position that sees it and the first that does not, in a prompt, in
    portions cut at and around the edge, and in steps."""
    cfg = O.make_config(kinds=("attention", "shared"), ff=(0, 0), vocab=50, window=window, heads=2, kv_heads=1, dim=16, vdim=16)
    W = O.make_weights(cfg, seed=9)
    for i in (0, 1):
        W[f"l{i}.mix.q"] = _bf(W[f"l{i}.mix.q"].float() * 3)
    T = 260
    plain = O.forward(cfg, W, [7] * T)[0]
    model = _model(cfg, W, dtype)
    tol = 3e-5 if dtype == F32 else 4e-2
    for j in (0, 63, 130):
        tokens = [7] * T
        tokens[j] = 31
        want, taps = O.forward(cfg, W, tokens)
        moved = (want - plain).abs().amax(-1) > 1e-9
        assert not moved[:j].any() and moved[j:j + window].any() and not moved[j + 2 * window:].any()
        one = O.forward(dict(cfg, layers=cfg["layers"][:1]), W, tokens)[0], O.forward(dict(cfg, layers=cfg["layers"][:1]), W, [7] * T)[0]
        first = (one[0] - one[1]).abs().amax(-1)
        assert first[j + window - 1] > 1e-3 and (first[j + window:] < 1e-12).all()                # layer 0 alone: just inside, just outside
        e = j + window
        _close(_whole(model, tokens), want, tol, f"whole, key {j}")
        for cut in (e - 1, e, e + 1):
            rest = T - cut
            _close(_portions(model, tokens, [cut, 2, rest - 2] if cut else [2, rest - 2]), want, tol, f"cut at {cut}, key {j}")
        _close(_portions(model, tokens, [max(e - 3, 1)] + [1] * 8 + [T - 8 - max(e - 3, 1)]), want, tol, f"steps over the edge, key {j}")


@pytest.mark.parametrize("dtype", [F32, B16])
def test_latent_attention_finds_a_far_key_among_hundreds(dtype):
    cfg = O.make_config(kinds=("latent_attention",), ff=(0,), vocab=50, lat_heads=2)
    W = O.make_weights(cfg, seed=12)
    W["l0.mix.uq"] = _bf(W["l0.mix.uq"].float() * -6)         # token 31's key is the one that token 7's queries look for
    T = 600
    model = _model(cfg, W, dtype)
    tol = 3e-5 if dtype == F32 else 4e-2
    plain = O.forward(cfg, W, [7] * T)[0]
    for j in (0, 5, 64, 300):
        tokens = [7] * T
        tokens[j] = 31
        want = O.forward(cfg, W, tokens)[0]
        assert (want[T - 20:] - plain[T - 20:]).abs().max() > 0.2 * plain.abs().max()
        _close(_whole(model, tokens), want, tol, f"whole, key {j}")
        _close(_portions(model, tokens, [301, 2, 200, 70, 3] + [1] * 24), want, tol, f"portions and steps, key {j}")


@pytest.mark.parametrize("dtype", [F32, B16])
@pytest.mark.parametrize("size", [-30.0, 0.0, 6.0, 40.0])
def test_sink_from_negligible_to_overwhelming(size, dtype):
    cfg = O.make_config(kinds=("attention", "lightning", "shared"), ff=(0, 0, 0), window=9)
    W = O.make_weights(cfg, seed=14)
    W["l0.mix.sink"][:] = size
    W["l2.mix.sink"][0] = size
    tokens = _tokens(cfg, 60)
    want = O.forward(cfg, W, tokens)[0]
    without = O.forward(cfg, dict(W, **{"l0.mix.sink": torch.full_like(W["l0.mix.sink"], -100.0)}), tokens)[0]
    if size >= 0.0:
        assert (want - without).abs().max() > 0.02 * want.abs().max()
    model = _model(cfg, W, dtype)
    tol = 3e-5 if dtype == F32 else 4e-2
    _close(_whole(model, tokens), want, tol, "whole")
    _close(_portions(model, tokens, [1, 2, 20, 1, 1, 35]), want, tol, "portions")


# ------------------------------------------------------------------ the model
CONFIGS = {
    "four": dict(),
    "order": dict(kinds=("lightning", "latent_attention", "attention", "attention", "shared", "lightning", "latent_attention", "shared"), ff=(24, 0, 40, 0, 8, 16, 24, 0), width=72, vocab=257, window=10),
    "bare": dict(kinds=("latent_attention", "lightning"), ff=(0, 0), scaling=None, embed_scale=1.0),
    "ones": dict(heads=1, kv_heads=1, lat_heads=1, lin_heads=1, window=1, scale=1.0, lat_scale=1.0, scaling=(1.0, 64, 8.0, 1.0), decay=[1.0]),
    "odd": dict(width=50, vocab=33, heads=3, kv_heads=1, dim=10, vdim=9, window=13, lat_heads=5, lat_dim=7, rot_dim=6, lat_vdim=11, kv_rank=13, q_rank=17, lin_heads=3, lin_dim=5, lin_vdim=7, ff=(10, 21, 0, 33)),
    "wide": dict(width=200, heads=6, kv_heads=3, dim=72, vdim=40, window=48, lat_heads=4, lat_dim=72, rot_dim=64, lat_vdim=88, kv_rank=136, q_rank=104, lin_heads=2, lin_dim=70, lin_vdim=136, ff=(136, 120, 8, 72)),
    "many": dict(width=96, heads=24, kv_heads=4, dim=8, vdim=16, window=20, lat_heads=20, lat_dim=8, rot_dim=16, lat_vdim=8, kv_rank=64, q_rank=32, lin_heads=6, lin_dim=8, lin_vdim=8),
}


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_model_whole_steps_and_portions_match_the_oracle_in_fp32(name):
    cfg = O.make_config(**CONFIGS[name])
    W = O.make_weights(cfg, seed=len(name))
    T = 75
    tokens = _tokens(cfg, T)
    want, streams = O.forward(cfg, W, tokens)
    tol = 3e-5
    model = _model(cfg, W)
    model._tap = []
    _whole(model, tokens)
    assert len(model._tap) == len(streams)
    for r, (a, b) in enumerate(zip(model._tap, streams)):
        _close(a, b, tol, f"{name}: stream after layer {r}")
    model._tap = None
    _close(_whole(model, tokens), want, tol, f"{name}: whole")
    _close(_portions(model, tokens, [1] * T), want, tol, f"{name}: token by token from the first token")
    _close(_portions(model, tokens, [40] + [1] * 35), want, tol, f"{name}: prompt then steps")
    _close(_portions(model, tokens, [2, 2, 3, 30, 1, 2, 17, 9, 2, 5, 2]), want, tol, f"{name}: portions")
    _close(_portions(model, tokens[:1], [1]), want[:1], tol, f"{name}: a one-token sequence")
    _close(_portions(model, tokens[:2], [2]), want[:2], tol, f"{name}: a two-token sequence")


def _rel(a, b):
    """Root mean square over the vocabulary of the difference, largest over the positions, relative to b's."""
    d = (a.double().cpu() - b.double().cpu()).pow(2).mean(-1).sqrt()
    return (d.max() / b.double().pow(2).mean().sqrt()).item()


@pytest.mark.parametrize("name", ["four", "order", "wide", "many"])
def test_model_bf16_stays_within_rounding_of_the_oracle_and_of_itself(name):
    cfg = O.make_config(**CONFIGS[name])
    W = O.make_weights(cfg, seed=3)
    tokens = _tokens(cfg, 150, seed=2)
    want = O.forward(cfg, W, tokens)[0]
    model = _model(cfg, W, B16)
    whole = _whole(model, tokens)
    cut = _portions(model, tokens, [80, 2, 1, 1, 40, 6, 20])
    assert _rel(whole, want) < 4e-2
    assert _rel(cut, want) < 4e-2
    assert _rel(cut, whole.cpu()) < 5e-2
    model.gemm_path = "simt"                              # the tensor-core linear layers against the CUDA-core ones
    assert _rel(_whole(model, tokens), whole.cpu()) < 5e-2
    model.gemm_path = "tc"
    model.decay_recurrent = 1                             # and the block-wise linear attention against the token-by-token one
    assert _rel(_whole(model, tokens), whole.cpu()) < 5e-2


def test_layers_with_their_own_sizes_and_a_cache_that_has_to_grow():
    cfg = O.make_config(kinds=("attention", "latent_attention", "lightning", "attention", "shared", "latent_attention", "lightning"), ff=(16, 0, 24, 0, 32, 40, 8), width=104, vocab=211)
    cfg["layers"][3]["type"] = "attention_2"                  # a numbered type: the same mechanism with sizes of its own
    for i, win in ((3, 31), (4, 5)):
        cfg["layers"][i]["mixer"].update(heads=6, kv_heads=3, dim=8, vdim=40, scale=0.2, mask={"size": win})
    cfg["layers"][5]["mixer"] = {"heads": 2, "dim": 10, "rot_dim": 4, "vdim": 6, "kv_rank": 40, "q_rank": 8, "scale": 0.3, "rot": {"base": 7.0, "dims": 4}}
    cfg["layers"][6]["mixer"] = {"heads": 5, "dim": 24, "vdim": 9, "decay": [0.1, 0.3, 0.5, 0.7, 0.9]}
    W = O.make_weights(cfg, seed=21)
    tokens = _tokens(cfg, 70, seed=8)
    want = O.forward(cfg, W, tokens)[0]
    model = _model(cfg, W)
    _close(_whole(model, tokens), want, 3e-5, "whole")
    state = model.initialize_inference_params(max_seqlen=16, max_batch_size=1)
    _close(_portions(model, tokens, [9, 2, 20, 1, 1, 30, 7], state=state), want, 3e-5, "portions through a growing cache")
    assert sorted(state["mha"].key_value_memory_dict) == [0, 1, 3, 5] and all(c.shape[1] >= 70 for c in state["mha"].key_value_memory_dict.values())


def test_batch_rows_equal_each_sequence_alone_and_wanted_rows_select():
    cfg = O.make_config()
    W = O.make_weights(cfg, seed=5)
    for dtype, tol in ((F32, 2e-6), (B16, 2e-2)):
        model = _model(cfg, W, dtype)
        ids = torch.randint(0, cfg["vocab"], (3, 83), generator=torch.Generator().manual_seed(4)).to(DEV)
        both, _ = model(ids)
        for b in range(3):
            alone, _ = model(ids[b:b + 1])
            _close(both[b], alone[0].double().cpu(), tol, f"row {b}")
        state = model.initialize_inference_params(max_seqlen=96, max_batch_size=3)
        outs, t = [], 0
        for n in (50, 2, 1, 30):
            state["mha"].seqlen_offset = state["hyena"].seqlen_offset = t
            outs.append(model(ids[:, t:t + n], inference_params_dict=state)[0])
            t += n
        _close(torch.cat(outs, 1), both.double().cpu(), 1e-5 if dtype == F32 else 3e-2, "batched portions and steps")
        rows = [0, 7, 82, 100, 248]
        picked, _ = model(ids, logits_rows=rows)
        _close(picked, both.reshape(-1, both.shape[-1])[rows].double().cpu(), tol, "wanted rows")
        none, _ = model(ids, logits_rows=[])
        assert none.shape == (0, cfg["vocab"])


def test_reused_state_memory_and_long_decoding():
    """State holders that still hold another request's rows and matrix states (and NaNs beyond) serve a new request; decoding runs for
    hundreds of steps past the window; requests of unequal length interleaved keep their own state."""
    cfg = O.make_config(window=50)
    W = O.make_weights(cfg, seed=7)
    model = _model(cfg, W)
    a, b = _tokens(cfg, 260, seed=6), _tokens(cfg, 60, seed=9)
    want_a, want_b = O.forward(cfg, W, a)[0], O.forward(cfg, W, b)[0]
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


@pytest.mark.parametrize("dtype", [F32, B16])
@pytest.mark.parametrize("device_loop", [True, False])
def test_greedy_generation_through_the_generator(device_loop, dtype):
    from evo_b200 import CharLevelTokenizer, Generator
    cfg = O.make_config(vocab=512, window=30, lat_heads=13, kv_rank=64, rot_dim=16)       # the new tokens pass the window
    W = O.make_weights(cfg, seed=11)
    model = _model(cfg, W, dtype)
    gen = Generator(model, CharLevelTokenizer(512), top_k=1, top_p=1.0, temperature=1.0)
    gen.device_loop = device_loop
    prompt = torch.randint(0, 512, (2, 21), generator=torch.Generator().manual_seed(8)).to(DEV)
    n_new = 24
    picked, logits, _ = gen.generate(DEV, input_ids=prompt, num_tokens=n_new, cached_generation=True, force_prompt_threshold=64, print_generation=False, stop_at_eos=False)
    assert picked.shape == (2, n_new) and logits.shape == (2, n_new, 512)
    tol = 6e-2 if dtype == B16 else (1e-2 if device_loop else 3e-5)                         # the device loop keeps the sampler's bf16 view of the logits
    for b in range(2):
        full = prompt[b].tolist() + picked[b].tolist()
        want = O.forward(cfg, W, full)[0]
        for s in range(n_new):                                # each picked token is (within rounding) the oracle's argmax given the same prefix
            row = want[len(full) - n_new - 1 + s]
            assert row[picked[b, s]] >= row.max() - (2e-2 if dtype == F32 else 0.3), (b, s)
            _close(logits[b, s], row, tol, f"kept logits {b} {s}")


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
    W = O.make_weights(cfg, seed=13)
    ckpt = str(tmp_path / "ckpt")
    _write_checkpoint(ckpt, cfg, W)
    texts, scores = cli.main(["--model-dir", ckpt, "--prompt", "ACGTTGCA", "--n-samples", "2", "--n-tokens", "9", "--top-k", "1", "--device", DEV, "--verbose", "0"])
    assert len(texts) == 2 and texts[0] == texts[1] and len(scores) == 2
    tokens = _tokens(cfg, 40, seed=5)
    want = O.forward(cfg, W, tokens)[0]
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
