"""Mixed stacks without a GPU: config and weight readers, the registry, and the reference's own consistency."""
import json

import numpy as np
import pytest

import hybrid_ref as ref
import stack_util as su
from runnburn_b200 import registry
from runnburn_b200.safetensors import SafetensorsFile
from runnburn_b200.stack import StackConfig, punisun_config


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
