"""Mixed stacks without a GPU: config and weight readers, the registry, and the reference's own consistency."""
import json

import numpy as np
import pytest

import hybrid_ref as ref
import stack_util as su
from runnburn_b200 import registry
from runnburn_b200.safetensors import SafetensorsFile
from runnburn_b200.stack import StackConfig, dutivik_config, punisun_config


def _mixed(**kw):
    return su.config([su.wkv(), su.retention(), su.latent(scaling=su.YARN), su.wkv(ff=0)], loop={"start": 1, "stop": 3, "times": 3}, **kw)


def test_config_reads_every_size_and_constant():
    cfg = _mixed()
    c = punisun_config(json.loads(json.dumps(cfg)), 123, "float32")
    assert (c.width, c.vocab, c.max_ctx, c.dtype, c.loop) == (72, 97, 123, "float32", (1, 3, 3))
    assert (c.norm_eps, c.residual_mult) == (1e-5, 0.7)
    assert [ly.mixer for ly in c.layers] == ["wkv", "retention", "latent_attention", "wkv"]
    assert [ly.n_ff for ly in c.layers] == [48, 48, 48, 0]
    keep = []
    r, lat = c.layers[1].to_c(keep), c.layers[2].to_c(keep)
    assert [r.decay[i] for i in range(2)] == cfg["layers"][1]["mixer"]["decay"] and r.rot.interleaved == 0 and r.rot.scaled == 0
    assert lat.rot.interleaved == 1 and lat.rot.scaled == 1 and (lat.rot.factor, lat.rot.original, lat.rot.fast, lat.rot.slow) == (4.0, 64.0, 8.0, 1.0)
    assert lat.kv_rank == 56 and lat.rot_dim == 8


def test_config_without_loop_and_bad_configs():
    assert punisun_config(su.config([su.wkv()]), 8, "bfloat16").loop == (0, 0, 1)
    bad = su.config([su.retention(heads=3, decay=[0.9, 0.8])])
    with pytest.raises(ValueError, match="2 decays for 3 heads"):
        punisun_config(bad, 8, "bfloat16").layers[0].to_c([])
    bad = su.config([dict(su.wkv(), type="other")])
    with pytest.raises(ValueError, match="unknown mixer"):
        punisun_config(bad, 8, "bfloat16").layers[0].to_c([])
    bad = su.config([dict(su.wkv(), mlp={"kind": "sparse", "ff": 8})])
    with pytest.raises(ValueError, match="sparse"):
        punisun_config(bad, 8, "bfloat16")
    with pytest.raises(ValueError, match="dtype"):
        StackConfig(8, 8, [], 1e-5, dtype="int8").create(None)


def test_registry_and_safetensors(tmp_path):
    cfg = _mixed()
    w = su.weights(cfg, 3)
    su.save(tmp_path, cfg, w)
    assert registry.read_config(tmp_path, 64).width == 72
    f = SafetensorsFile(tmp_path / "model.safetensors")
    assert set(f.tensors) == set(w)
    for name, (dt, shape, data) in f.items():
        assert dt == "BF16" and shape == np.shape(w[name])
        assert bytes(data) == su.to_bf16_bits(w[name]).tobytes()
    (tmp_path / "config.json").write_text(json.dumps(dict(cfg, architecture="Nothing")))
    with pytest.raises(ValueError, match="not known"):
        registry.read_config(tmp_path, 64)
    (tmp_path / "model.safetensors").write_bytes((1 << 40).to_bytes(8, "little") + b"{}")
    with pytest.raises(ValueError, match="not a safetensors"):
        SafetensorsFile(tmp_path / "model.safetensors")


def test_reference_does_not_depend_on_portions():
    cfg = _mixed()
    w = su.weights(cfg, 1)
    rng = np.random.default_rng(0)
    toks = rng.integers(0, cfg["vocab"], 40)
    whole = ref.Model(cfg, w).forward(toks)
    m = ref.Model(cfg, w)
    parts, at = [], 0
    for n in (1, 2, 13, 1, 23):
        parts.append(m.forward(toks[at:at + n]))
        at += n
    assert np.allclose(np.concatenate(parts), whole, rtol=0, atol=1e-10)


def test_reference_runs_of_a_loop():
    assert ref.runs({"layers": [0] * 4, "loop": {"start": 1, "stop": 3, "times": 2}}) == [(0, False), (1, False), (2, False), (1, True), (2, False), (3, False)]
    assert ref.runs({"layers": [0] * 2, "loop": None}) == [(0, False), (1, False)]


def test_reference_rotation_keeps_relative_positions():
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal((2, 1, 1, 8))
    for inter in (False, True):
        dots = []
        for shift in (0, 57):
            c0, s0 = ref.rotation_tables({"dims": 8, "base": 100.0}, [3 + shift])
            c1, s1 = ref.rotation_tables({"dims": 8, "base": 100.0}, [11 + shift])
            dots.append(float(np.sum(ref.rotate_pairs(q, c0, s0, inter) * ref.rotate_pairs(k, c1, s1, inter))))
        assert abs(dots[0] - dots[1]) < 1e-12


def test_dutivik_config_reads_every_size_and_constant():
    layers = [su.parallel(left=su.window(heads=6, kv_heads=3, dim=10, vdim=12, size=77, dims=4, base=50.0, factor=3.0, scale=0.3), right=su.delta(heads=4, kv_heads=1, dim=20, vdim=28, conv=5),
                          left_scale=0.25, right_scale=2.0, ff=36),
              su.gla(heads=5, dim=14, vdim=18, tau=9.0, ff=0)]
    cfg = su.dutivik(layers + [su.again(layers[1], 1), su.again(layers[0], 0)], eps=1e-4, scale=7.0)
    c = dutivik_config(json.loads(json.dumps(cfg)), 123, "float32")
    assert (c.width, c.vocab, c.max_ctx, c.dtype, c.loop) == (72, 97, 123, "float32", (0, 0, 1))
    assert (c.norm_eps, c.embed_scale, c.residual_mult, c.block, c.norm, c.act) == (1e-4, 7.0, 1.0, "parallel", "layer", "silu")
    assert [(ly.mixer, ly.join, ly.weights_of, ly.n_ff) for ly in c.layers] == [
        ("attention", False, None, 36), ("delta", True, None, 0), ("gla", False, None, 0), ("gla", False, 1, 0), ("attention", False, 0, 36), ("delta", True, 0, 0)]
    a, d, g = (ly.to_c([]) for ly in c.layers[:3])
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.qk_norm, a.head_gate, a.prefix, a.weights_of) == (6, 3, 10, 12, 77, 1, 1, b"mix.left.", -1)
    assert (a.rot.dims, a.rot.base, a.rot.interleaved, a.rot.scaled, a.rot.factor) == (4, 50.0, 1, 2, 3.0)
    assert abs(a.scale - 0.3) < 1e-7 and (a.out_scale, d.out_scale) == (0.25, 2.0)
    assert (d.heads, d.kv_heads, d.dim, d.vdim, d.conv, d.join, d.prefix) == (4, 1, 20, 28, 5, 1, b"mix.right.")
    assert (g.heads, g.dim, g.vdim, g.tau, g.prefix, g.out_scale) == (5, 14, 18, 9.0, b"mix.", 1.0)
    assert c.layers[4].to_c([]).weights_of == 0


def test_dutivik_bad_configs():
    with pytest.raises(ValueError, match="unknown mixer 'other'"):
        dutivik_config(su.dutivik([dict(su.gla(), type="other")]), 8, "bfloat16")
    with pytest.raises(ValueError, match="sparse"):
        dutivik_config(su.dutivik([dict(su.gla(), mlp={"kind": "sparse", "ff": 8})]), 8, "bfloat16")


def test_dutivik_registry(tmp_path):
    cfg = su.dutivik([su.gla(), su.parallel(), su.again(su.gla(), 0)])
    w = su.weights(cfg, 3)
    assert not any(n.startswith("l2.") for n in w)
    su.save(tmp_path, cfg, w)
    assert registry.read_config(tmp_path, 64).embed_scale == 3.0
    assert set(SafetensorsFile(tmp_path / "model.safetensors").tensors) == set(w)


def test_dutivik_reference_does_not_depend_on_portions():
    layers = [su.parallel(), su.gla()]
    cfg = su.dutivik(layers + [su.again(layers[0], 0)])
    w = su.weights(cfg, 1)
    toks = np.random.default_rng(0).integers(0, cfg["vocab"], 40)
    whole = ref.Model(cfg, w).forward(toks)
    m = ref.Model(cfg, w)
    parts, at = [], 0
    for n in (1, 2, 13, 1, 23):
        parts.append(m.forward(toks[at:at + n]))
        at += n
    assert np.allclose(np.concatenate(parts), whole, rtol=0, atol=1e-10)


def test_reference_mechanisms_against_their_definitions():
    rng = np.random.default_rng(0)
    # a window of one token returns the value itself, whatever the scores
    q, k, v = rng.standard_normal((3, 5, 2, 4))
    assert np.allclose(ref.window_softmax(q, k, v, 3.0, 0, 0, 1), v)
    # the delta rule with beta 1 and no decay stores v at a unit key exactly, and a second write replaces it
    e = np.zeros((2, 1, 4))
    e[:, 0, 1] = 1.0
    v = rng.standard_normal((2, 1, 3))
    o, S = ref.delta_recurrence(e, e, v, np.ones((2, 1)), np.ones((2, 1)), np.zeros((1, 4, 3)))
    assert np.allclose(o, v) and np.allclose(S[0, 1], v[1, 0])
    # the last column of the taps belongs to the current input
    x, taps = rng.standard_normal((6, 2)), np.array([[0.0, 0.0, 1.0], [1.0, 0.0, 0.0]])
    y, last = ref.short_convolution(x, np.zeros((2, 2)), taps)
    assert np.allclose(y[:, 0], x[:, 0]) and np.allclose(y[2:, 1], x[:-2, 1]) and np.allclose(y[:2, 1], 0) and np.allclose(last, x[-2:])
    # gated linear attention with decays of one is a running sum
    q, k, v = rng.standard_normal((3, 7, 1, 2))
    o, _ = ref.gla_recurrence(q, k, v, np.ones((7, 1, 2)), np.zeros((1, 2, 2)))
    assert np.allclose(o[-1, 0], sum((k[t, 0] @ q[-1, 0]) * v[t, 0] for t in range(7)))
    assert np.allclose(ref.channel_decay(np.array([0.3]), 4.0), ref.sigmoid(0.3) ** 0.25)
    z = ref.layer_norm(rng.standard_normal((3, 8)) + 5.0, np.ones(8), np.zeros(8), 0.0)
    assert np.allclose(z.mean(-1), 0) and np.allclose((z * z).mean(-1), 1)
