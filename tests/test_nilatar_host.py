"""Host-side parts of the Nilatar family that need no GPU: configuration reading, the architecture registry, the flat-tensor loader's
strictness, and the oracle's own consistency (slowed rotations, window and sink, shared keys, the decaying state, causality)."""
import math

import pytest
import torch

from evo_b200.models import ARCHITECTURES, load_model_dir, read_architecture
from evo_b200.nilatar import Nilatar, NilatarConfig
from evo_b200.stream_model import StreamDecoder
from oracle import nilatar_oracle as O
from tests.test_zaverax_host import _write_checkpoint

F64 = torch.float64


def test_config_reads_every_size_and_constant():
    d = O.make_config(kinds=("lightning", "attention", "latent_attention", "shared", "attention", "shared"), ff=(0, 24, 36, 0, 8, 12), width=72, vocab=77, eps=3e-6, embed_scale=2.5,
                      heads=6, kv_heads=3, dim=10, vdim=14, window=29, scale=0.31, lat_heads=5, lat_dim=7, rot_dim=6, lat_vdim=9, kv_rank=11, q_rank=13, lat_scale=0.4,
                      rot_base=777.0, scaling=(3.0, 99, 5.0, 1.5), lin_heads=3, lin_dim=4, lin_vdim=6, decay=[0.5, 1.0, 0.125])
    c = NilatarConfig.from_dict(d)
    assert (c.width, c.vocab_size, c.eps, c.embed_scale, len(c.runs)) == (72, 77, 3e-6, 2.5, 6)
    assert [l.ff for l in c.layers] == [0, 24, 36, 0, 8, 12] and [l.mixer.kind for l in c.layers] == ["lightning", "attention", "latent_attention"] + ["attention"] * 3
    a, lat, lin = c.layers[1].mixer, c.layers[2].mixer, c.layers[0].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.scale, a.kv_from) == (6, 3, 10, 14, 29, 0.31, None)
    assert (c.layers[3].mixer.kv_from, c.layers[5].mixer.kv_from) == (1, 4)
    assert (lat.heads, lat.dim, lat.rot_dim, lat.vdim, lat.kv_rank, lat.q_rank, lat.scale, lat.rot_dims, lat.rot_base) == (5, 7, 6, 9, 11, 13, 0.4, 6, 777.0)
    assert (lat.rot_scaling.factor, lat.rot_scaling.original, lat.rot_scaling.fast, lat.rot_scaling.slow) == (3.0, 99, 5.0, 1.5)
    assert (lin.heads, lin.dim, lin.vdim, lin.decay) == (3, 4, 6, [0.5, 1.0, 0.125])
    assert c.tensor_shapes() == {k: tuple(v.shape) for k, v in O.make_weights(d).items()}
    assert c.unused_tensor_names == ("l0.norm2", "l0.ls2", "l3.norm2", "l3.ls2")
    plain = NilatarConfig.from_dict(O.make_config(scaling=None)).layers[1].mixer
    assert plain.rot_scaling is None and plain.rot_len == 1.0
    numbered = O.make_config()
    numbered["layers"][0]["type"] = "attention_2"             # the same mechanism with sizes of its own
    assert NilatarConfig.from_dict(numbered).layers[0].mixer.kind == "attention"
    for key, value in (("type", "conv"), ("mlp", {"kind": "moe"})):
        bad = O.make_config()
        bad["layers"][0][key] = value
        with pytest.raises(NotImplementedError):
            NilatarConfig.from_dict(bad)
    for where, key, value in ((0, "kv_heads", 3), (1, "rot_dim", 7), (2, "decay", [0.5]), (3, "kv_from", 1), (3, "kv_from", 3), (3, "dim", 8)):
        bad = O.make_config()
        bad["layers"][where]["mixer"][key] = value
        with pytest.raises(ValueError):
            NilatarConfig.from_dict(bad)


@pytest.mark.parametrize("dims,base,scaling", [(16, 1000.0, (8.0, 64, 4.0, 1.0)), (6, 50.0, (2.0, 30, 2.5, 2.0)), (64, 1e6, (4.0, 512, 8.0, 1.0)), (8, 10.0, None), (12, 100.0, (5.0, 7, 2.0, 2.0)),
                                               (10, 30.0, (1.0, 100, 9.0, 3.0))])
def test_rotation_frequencies_agree_with_the_oracle(dims, base, scaling):
    d = O.make_config(rot_dim=dims, rot_base=base, scaling=scaling)
    rot = d["layers"][1]["mixer"]["rot"]
    m = NilatarConfig.from_dict(d).layers[1].mixer
    want, got = O.turn_frequencies(rot), m.frequencies()
    assert len(got) == dims // 2 and all(abs(g - w) <= 1e-12 * w for g, w in zip(got, want))
    assert abs(m.rot_len - O.turn_length(rot)) < 1e-12
    if scaling:
        factor, original, fast, slow = scaling
        turns = lambda f: original * f / (2 * math.pi)
        plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
        for i, (f, p) in enumerate(zip(want, plain)):
            assert p / factor * (1 - 1e-12) <= f <= p * (1 + 1e-12)
            if i and turns(plain[i - 1]) <= slow and slow < fast:                  # a whole pair past the one that makes `slow` turns
                assert abs(f - p / factor) <= 1e-12 * p
            if i + 1 < len(plain) and turns(plain[i + 1]) >= fast:
                assert abs(f - p) <= 1e-12 * p


def test_registry_picks_the_class_and_the_loader_is_strict(tmp_path):
    cfg = O.make_config()
    W = O.make_weights(cfg, seed=1)
    _write_checkpoint(tmp_path / "ok", cfg, W)
    arch, read = read_architecture(str(tmp_path / "ok"))
    assert arch == "Nilatar" and read["width"] == cfg["width"] and torch.float32 in ARCHITECTURES[arch][1]
    model = load_model_dir(str(tmp_path / "ok"))
    assert isinstance(model, Nilatar) and isinstance(model, StreamDecoder) and model.ingest_stats["tensors"] == len(W)
    assert all(torch.equal(model.weights[k], W[k]) for k in W)
    for gone in ("l0.mix.sink", "l1.mix.dq.norm", "l2.ls1"):
        missing = dict(W)
        missing.pop(gone)
        _write_checkpoint(tmp_path / "missing", cfg, missing)
        with pytest.raises(RuntimeError, match="Missing"):
            load_model_dir(str(tmp_path / "missing"))
    _write_checkpoint(tmp_path / "narrow", cfg, dict(W, **{"l1.mix.uq": W["l1.mix.uq"][:, :-1].contiguous()}))
    with pytest.raises(RuntimeError, match="size mismatch"):
        load_model_dir(str(tmp_path / "narrow"))
    _write_checkpoint(tmp_path / "more", cfg, dict(W, **{"l3.mix.k": W["l0.mix.k"]}))          # a layer with shared keys has none of its own
    with pytest.raises(RuntimeError):
        load_model_dir(str(tmp_path / "more"))
    with pytest.raises(NotImplementedError):
        load_model_dir(str(tmp_path / "ok"), dtype=torch.float16)
    _write_checkpoint(tmp_path / "spare", cfg, dict(W, **{"l2.norm2": W["l2.norm1"].clone(), "l2.ls2": W["l2.ls1"].clone()}))   # unread when there is no feed-forward
    assert "l2.norm2" not in load_model_dir(str(tmp_path / "spare")).weights


def test_model_refuses_to_run_without_cuda():
    from evo_b200 import _lib
    cfg = O.make_config()
    m = Nilatar(NilatarConfig.from_dict(cfg))
    m.load_state_dict(O.make_weights(cfg))
    with pytest.raises(RuntimeError):
        m.load_state_dict({"embed": torch.zeros(2, 2)})
    with pytest.raises(_lib.EvoError, match="no CPU"):
        m(torch.zeros(1, 4, dtype=torch.long))
    rnd = Nilatar(NilatarConfig.from_dict(cfg)).init_random(seed=3)
    assert all(torch.isfinite(v.float()).all() for v in rnd.weights.values())


def test_mean_keys_of_a_window():
    for off in (0, 3, 9, 40):
        for L in (1, 2, 17):
            for window in (0, 1, 5, 10, 100):
                want = sum(min(i + 1, window) if window else i + 1 for i in range(off, off + L)) / L
                assert abs(StreamDecoder._mean_keys(off, L, window) - want) < 1e-9, (off, L, window)


def test_oracle_window_and_sink():
    g = torch.Generator().manual_seed(0)
    T, H, dk, dv = 12, 2, 4, 3
    q, k, v = torch.randn(T, H, dk, generator=g, dtype=F64), torch.randn(T, 1, dk, generator=g, dtype=F64), torch.randn(T, 1, dv, generator=g, dtype=F64)
    sink = torch.tensor([0.7, -1.0], dtype=F64)
    out = O.softmax_attention(q, k, v, 0.5, 5, sink)
    for i in (0, 4, 5, 11):
        lo = max(0, i - 4)
        for h in range(H):
            e = torch.exp(0.5 * (k[lo:i + 1, 0] @ q[i, h]))
            assert torch.allclose(out[i, h], (e @ v[lo:i + 1, 0]) / (e.sum() + torch.exp(sink[h])))
    assert torch.allclose(O.softmax_attention(q[7:], k, v, 0.5, 5, sink, pos0=7), out[7:])


def test_oracle_turns_keep_relative_positions_and_scale_lengths():
    rot = {"base": 100.0, "dims": 6, "scaling": {"factor": 4.0, "original": 20, "fast": 3.0, "slow": 1.0}}
    g = torch.Generator().manual_seed(2)
    q, k = torch.randn(1, 1, 8, generator=g, dtype=F64), torch.randn(1, 1, 8, generator=g, dtype=F64)
    a = (O.turn(q, rot, 11) * O.turn(k, rot, 4)).sum()
    assert torch.allclose(a, (O.turn(q, rot, 107) * O.turn(k, rot, 100)).sum())
    assert torch.allclose(O.turn(q, rot, 9)[..., :6].norm(), q[..., :6].norm() * (0.1 * math.log(4.0) + 1.0)) and torch.equal(O.turn(q, rot, 9)[..., 6:], q[..., 6:])


def test_oracle_decaying_state_is_the_explicit_sum():
    g = torch.Generator().manual_seed(1)
    T, dk, dv = 9, 3, 4
    q, k, v = (torch.randn(T, 2, n, generator=g, dtype=F64) for n in (dk, dk, dv))
    decay = torch.tensor([0.5, 0.9], dtype=F64)
    out, last = O.decay_scan(q, k, v, decay)
    for h in range(2):
        for t in range(T):
            want = sum(decay[h] ** (t - s) * (q[t, h] @ k[s, h]) * v[s, h] for s in range(t + 1))
            assert torch.allclose(out[t, h], want)
    first, mid = O.decay_scan(q[:4], k[:4], v[:4], decay)
    rest, end = O.decay_scan(q[4:], k[4:], v[4:], decay, mid)
    assert torch.allclose(torch.cat([first, rest]), out) and torch.allclose(end, last)


def test_oracle_model_is_causal_shares_keys_and_layer_scales_switch_sublayers_off():
    cfg = O.make_config()
    W = O.make_weights(cfg, seed=4)
    tokens = torch.randint(0, cfg["vocab"], (30,), generator=torch.Generator().manual_seed(1)).tolist()
    full, _ = O.forward(cfg, W, tokens)
    assert torch.allclose(O.forward(cfg, W, tokens[:9])[0], full[:9], atol=1e-9)
    other = dict(W, **{"l0.ls1": torch.zeros_like(W["l0.ls1"]), "l0.mix.k": -W["l0.mix.k"]})      # layer 0 adds nothing, its keys still reach layer 3
    base = dict(W, **{"l0.ls1": other["l0.ls1"]})
    a, b = O.forward(cfg, base, tokens)[1], O.forward(cfg, other, tokens)[1]
    assert torch.allclose(a[2], b[2]) and not torch.allclose(a[3], b[3])
    off = {k: torch.zeros_like(v) if k.endswith(("ls1", "ls2")) else v for k, v in W.items()}
    w = {k: v.double() for k, v in off.items()}
    want = O.rms(w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"], w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T
    assert torch.allclose(O.forward(cfg, off, tokens)[0], want, atol=1e-9)
