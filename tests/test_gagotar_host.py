"""Host-side parts of the Gagotar family that need no GPU: configuration reading, the architecture registry, the flat-tensor loader's
strictness (and the size that only a tensor's shape gives), and the oracle's own consistency (mixed scores, chunks, slowed rotations, the
decaying state, the limited experts, the softmax over the chosen logits, causality of the whole model)."""
import math

import pytest
import torch

from evo_b200.gagotar import Gagotar, GagotarConfig
from evo_b200.models import ARCHITECTURES, load_model_dir, read_architecture
from evo_b200.stream_model import StreamDecoder
from oracle import gagotar_oracle as O
from tests.test_zaverax_host import _write_checkpoint

F64 = torch.float64


def test_config_reads_every_size_and_constant():
    d = O.make_config(mlps=("moe", None, "moe"), width=104, vocab=77, eps=3e-6, heads=6, kv_heads=3, dim=10, vdim=14, scale=0.31, chunk=29, rot_dims=6, rot_base=777.0,
                      scaling=(3.0, 1.5, 5.0, 99), lin_heads=5, lin_dim=7, lin_vdim=9, tau=4.5, experts=9, top=4, expert_ff=12, limit=2.25)
    shapes = O.tensor_shapes(d, rank=13)
    c = GagotarConfig.from_dict(d, shapes)
    assert (c.width, c.vocab_size, c.eps, len(c.runs)) == (104, 77, 3e-6, 3)
    a, s, f = c.layers[0].left, c.layers[0].right, c.layers[0].mlp
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.chunk, a.rot_dims, a.rot_base) == (6, 3, 10, 14, 0.31, 29, 6, 777.0)
    assert (a.rot_scaling.factor, a.rot_scaling.low, a.rot_scaling.high, a.rot_scaling.original) == (3.0, 1.5, 5.0, 99)
    assert (s.heads, s.dim, s.vdim, s.tau, s.rank) == (5, 7, 9, 4.5, 13)
    assert (f.ff, f.limit, f.experts, f.top) == (12, 2.25, 9, 4) and c.layers[1].mlp is None
    assert c.tensor_shapes() == shapes
    assert "l1.norm2" not in shapes and c.unused_tensor_names == ("l1.norm2", "l1.ls2")
    # what a configuration does not mention does not exist: no rotation, no slowing, no chunks
    bare = GagotarConfig.from_dict(O.make_config(rot_dims=0, chunk=0)).layers[0].left
    assert (bare.rot_dims, bare.rot_scaling, bare.chunk, bare.frequencies()) == (0, None, 0, [])
    assert GagotarConfig.from_dict(O.make_config(scaling=None)).layers[0].left.rot_scaling is None
    for key, value, err in (("type", "conv", NotImplementedError), ("mlp", {"kind": "dense"}, NotImplementedError)):
        bad = O.make_config()
        bad["layers"][0][key] = value
        with pytest.raises(err):
            GagotarConfig.from_dict(bad)
    for bad in (dict(heads=5, kv_heads=2), dict(rot_dims=18, dim=16), dict(experts=3, top=4), dict(limit=0.0)):
        with pytest.raises(ValueError):
            GagotarConfig.from_dict(O.make_config(**bad))


@pytest.mark.parametrize("dims,base,scaling", [(16, 1000.0, (8.0, 1.0, 4.0, 64)), (6, 50.0, (2.0, 2.0, 2.5, 30)), (64, 1e6, (4.0, 1.0, 8.0, 512)), (8, 10.0, None)])
def test_rotation_frequencies_agree_with_the_oracle(dims, base, scaling):
    d = O.make_config(dim=64, rot_dims=dims, rot_base=base, scaling=scaling)
    want = O.rotation_frequencies(d["layers"][0]["mixer"]["left"]["rot"])
    got = GagotarConfig.from_dict(d).layers[0].left.frequencies()
    assert len(got) == dims // 2 and all(abs(g - w) <= 1e-12 * w for g, w in zip(got, want))
    if scaling:
        factor, low, high, original = scaling
        plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
        for f, p in zip(want, plain):
            wave = 2 * math.pi / p
            assert p / factor * (1 - 1e-12) <= f <= p * (1 + 1e-12)
            if wave < original / high:
                assert f == p
            if wave > original / low:
                assert f == p / factor


def test_registry_picks_the_class_and_the_loader_is_strict(tmp_path):
    cfg = O.make_config()
    W = O.random_weights(cfg, seed=1, rank=9)
    _write_checkpoint(tmp_path / "ok", cfg, W)
    arch, read = read_architecture(str(tmp_path / "ok"))
    assert arch == "Gagotar" and read["width"] == cfg["width"] and torch.float32 in ARCHITECTURES[arch][1]
    model = load_model_dir(str(tmp_path / "ok"))
    assert isinstance(model, Gagotar) and isinstance(model, StreamDecoder) and model.ingest_stats["tensors"] == len(W)
    assert all(torch.equal(model.weights[k], W[k]) for k in W)
    assert model.config.layers[0].right.rank == 9 and GagotarConfig.from_dir(str(tmp_path / "ok")).layers[1].right.rank == 9
    missing = dict(W)
    missing.pop("l0.mix.left.talk")
    _write_checkpoint(tmp_path / "missing", cfg, missing)
    with pytest.raises(RuntimeError, match="Missing"):
        load_model_dir(str(tmp_path / "missing"))
    _write_checkpoint(tmp_path / "rank", cfg, dict(W, **{"l1.mix.right.a2": W["l1.mix.right.a2"][:, :-1].contiguous()}))      # the two halves of the projection disagree
    with pytest.raises(RuntimeError, match="size mismatch"):
        load_model_dir(str(tmp_path / "rank"))
    with pytest.raises(NotImplementedError):
        load_model_dir(str(tmp_path / "ok"), dtype=torch.float16)
    # a layer without feed-forward may still carry its second norm and scale: they are not read
    cfg2 = O.make_config(mlps=(None,))
    W2 = O.random_weights(cfg2, seed=2)
    W2["l0.norm2"] = W2["l0.ls2"] = W2["l0.norm1"].clone()
    _write_checkpoint(tmp_path / "spare", cfg2, W2)
    assert "l0.norm2" not in load_model_dir(str(tmp_path / "spare")).weights


def test_model_refuses_to_run_without_cuda():
    from evo_b200 import _lib
    cfg = O.make_config()
    m = Gagotar(GagotarConfig.from_dict(cfg, O.tensor_shapes(cfg)))
    m.load_state_dict(O.random_weights(cfg))
    with pytest.raises(RuntimeError):
        m.load_state_dict({"embed": torch.zeros(2, 2)})
    with pytest.raises(_lib.EvoError, match="no CPU"):
        m(torch.zeros(1, 4, dtype=torch.long))
    rnd = Gagotar(GagotarConfig.from_dict(cfg)).init_random(seed=3)
    assert set(rnd.weights) == set(O.tensor_shapes(cfg)) and all(torch.isfinite(v.float()).all() for v in rnd.weights.values())


def test_oracle_mixed_scores_and_chunks():
    g = torch.Generator().manual_seed(0)
    T, H, dk, dv = 12, 2, 4, 3
    q, k, v = torch.randn(T, H, dk, generator=g, dtype=F64), torch.randn(T, 1, dk, generator=g, dtype=F64), torch.randn(T, 1, dv, generator=g, dtype=F64)
    temp, swap = torch.tensor([1.0, 2.0], dtype=F64), torch.tensor([[0.0, 1.0], [1.0, 0.0]], dtype=F64)
    out = O.mixed_head_attention(q, k, v, 0.5, temp, swap, 5)
    for i in (0, 4, 5, 9, 11):
        lo = i // 5 * 5
        for h in range(H):                                   # each head reads the other head's scores, with that head's temperature
            s = (k[lo:i + 1, 0] @ q[i, 1 - h]) * 0.5 * temp[1 - h]
            assert torch.allclose(out[i, h], torch.softmax(s, 0) @ v[lo:i + 1, 0])
    assert torch.allclose(out[5], v[5].expand(H, dv)) and torch.allclose(out[10], v[10].expand(H, dv))          # a chunk's first position sees itself alone


def test_oracle_decaying_state_is_the_explicit_sum():
    g = torch.Generator().manual_seed(1)
    T, dk, dv = 9, 3, 4
    q, k, v = (torch.randn(T, 1, n, generator=g, dtype=F64) for n in (dk, dk, dv))
    alpha = torch.rand(T, 1, dk, generator=g, dtype=F64)
    out = O.decay_scan(q, k, v, alpha)
    for t in range(T):
        want = torch.zeros(dv, dtype=F64)
        for s in range(t + 1):
            want = want + (q[t, 0] * alpha[s + 1:t + 1, 0].prod(0) * k[s, 0]).sum() * v[s, 0]
        assert torch.allclose(out[t, 0], want)


def test_oracle_limited_experts_and_router():
    got = O.limited_glu(torch.tensor([5.0, -5.0, 1.0], dtype=F64), torch.tensor([9.0, -9.0, 0.5], dtype=F64), 2.0)
    sig = lambda z: 1 / (1 + math.exp(-z))
    want = [2.0 * sig(O.SLOPE * 2.0) * 3.0, -5.0 * sig(-O.SLOPE * 5.0) * -1.0, sig(O.SLOPE) * 1.5]
    assert torch.allclose(got, torch.tensor(want, dtype=F64))
    w = O.route(torch.eye(4, dtype=F64)[:1], torch.tensor([[1.0], [3.0], [2.0]], dtype=F64) * torch.eye(4, dtype=F64)[:1], 2)[0]
    assert w[0] == 0 and torch.allclose(w[1:], torch.softmax(torch.tensor([3.0, 2.0], dtype=F64), 0))


def test_oracle_model_is_causal_and_layer_scales_switch_sublayers_off():
    cfg = O.make_config()
    W = O.random_weights(cfg, seed=4)
    tokens = torch.randint(0, cfg["vocab"], (30,), generator=torch.Generator().manual_seed(1)).tolist()
    full = O.forward(tokens, W, cfg)
    assert torch.allclose(O.forward(tokens[:9], W, cfg), full[:9], atol=1e-9)
    W2 = {k: torch.zeros_like(v) if k.endswith(("ls1", "ls2")) else v for k, v in W.items()}
    w = {k: v.double() for k, v in W2.items()}
    want = (O.rms(w["embed"][torch.tensor(tokens)], cfg["norm"]["eps"]) * w["final.norm"]) @ w["head"].T
    assert torch.allclose(O.forward(tokens, W2, cfg), want, atol=1e-9)
