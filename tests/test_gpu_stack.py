"""Mixed stacks on the GPU against the plain reference (hybrid_ref): mechanisms alone, portions, decoding,
far keys and long memories, loops, sequence reuse, generation and the trace replay."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest

import hybrid_ref as ref
import stack_util as su

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
TOL = su.TOL
DTYPES = ["float32", "bfloat16"]


_bad, _tokens, _feed = su.bad, su.tokens, su.feed

MIXED = [su.wkv(), su.retention(), su.latent(scaling=su.YARN), su.wkv(ff=0), su.retention(heads=1, dim=64, vdim=24, dims=32)]
MECHANISMS = {
    "wkv": (su.wkv(ff=0), 72), "wkv_wide": (su.wkv(heads=2, dim=80, ff=0), 64), "wkv_one": (su.wkv(heads=1, dim=5, ff=0), 40),
    "wkv_64": (su.wkv(heads=3, dim=64, ff=0), 128),
    "retention": (su.retention(ff=0), 72), "retention_partial_rotation": (su.retention(heads=3, dim=32, vdim=8, dims=16, ff=0), 48),
    "retention_wide": (su.retention(heads=2, dim=128, vdim=136, ff=0), 64), "retention_odd": (su.retention(heads=3, dim=6, vdim=7, ff=0), 50),
    "retention_256": (su.retention(heads=1, dim=256, vdim=96, ff=0), 64), "retention_64": (su.retention(heads=2, dim=64, vdim=64, ff=0), 64),
    "latent": (su.latent(ff=0), 72), "latent_yarn": (su.latent(scaling=su.YARN, ff=0), 72),
    "latent_yarn_clamped": (su.latent(rot_dim=16, base=30.0, scaling={"factor": 2.5, "original": 7, "fast": 40.0, "slow": 0.01}, ff=0), 72),
    "latent_odd": (su.latent(heads=1, dim=11, vdim=9, rot_dim=6, kv_rank=21, ff=0), 50), "latent_large": (su.latent(heads=2, dim=128, vdim=128, rot_dim=64, kv_rank=512, ff=0), 64),
    "latent_wide_values": (su.latent(heads=2, dim=16, vdim=264, rot_dim=8, kv_rank=32, ff=0), 64),
    "dense": (su.wkv(heads=1, dim=8, ff=264), 64), "dense_odd": (su.wkv(heads=1, dim=8, ff=37), 51),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(MECHANISMS))
def test_one_layer_residual(name, dtype):
    layer, width = MECHANISMS[name]
    cfg = su.config([layer], width=width)
    w = su.weights(cfg, 7)
    m = ref.Model(cfg, w)
    toks = _tokens(cfg, 150)
    m.trace = []
    m.forward(toks)
    base = w["embed"][toks]
    want = m.trace[0] - base          # what the layer adds
    dec = su.decoder(cfg, w, dtype)
    got = dec.trace_residual(toks)[0] - base
    assert not _bad(got, want, dtype)
    parts = [dec.trace_residual(toks[a:a + n], a)[0] for a, n in ((0, 20), (20, 3), (23, 8), (31, 1), (32, 9), (41, 40), (81, 69))]
    assert not _bad(np.concatenate(parts) - base, want, dtype)
    dec.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("loop", [None, {"start": 0, "stop": 2, "times": 3}, {"start": 1, "stop": 4, "times": 2}, {"start": 2, "stop": 5, "times": 1},
                                  {"start": 3, "stop": 4, "times": 4}])
def test_stack_and_loops(dtype, loop):
    cfg = su.config(MIXED, loop=loop)
    w = su.weights(cfg, 2)
    toks = _tokens(cfg, 90)
    m = ref.Model(cfg, w)
    m.trace = []
    want = m.forward(toks)
    dec = su.decoder(cfg, w, dtype)
    tr = dec.trace_residual(toks)
    assert tr.shape[0] == len(m.trace)
    for got, exp in zip(tr, m.trace):
        assert not _bad(got, exp, dtype)
    assert not _bad(_feed(dec, toks, [90]), want, dtype)
    assert not _bad(_feed(dec, toks, [50] + [1] * 40), want, dtype)
    dec.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_portions_of_every_size(dtype):
    cfg = su.config(MIXED, loop={"start": 0, "stop": 3, "times": 2})
    w = su.weights(cfg, 4)
    toks = _tokens(cfg, 230)
    want = ref.Model(cfg, w).forward(toks)
    dec = su.decoder(cfg, w, dtype)
    for cuts in ([2], [3, 2], [7, 8, 9], [10, 1, 97, 2, 98], [64, 63, 65], [1], [229, 1]):
        assert not _bad(_feed(dec, toks, cuts), want, dtype), cuts
    dec.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_prompt_and_decoding(dtype):
    """Crosses the chunk lengths of the recurrences and several attention tiles and token tiles."""
    cfg = su.config([su.retention(heads=2, dim=16, vdim=16), su.wkv(heads=2, dim=16), su.latent(heads=2)], width=64)
    w = su.weights(cfg, 5)
    toks = _tokens(cfg, 1300)
    want = ref.Model(cfg, w).forward(toks)
    dec = su.decoder(cfg, w, dtype, max_ctx=1300)
    for cuts in ([1300], [1025, 95, 180], [300, 97, 903], [1100] + [1] * 200):
        assert not _bad(_feed(dec, toks, cuts), want, dtype), cuts
    dec.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("place", [0, 1, 63, 64, 127, 128, 191, 199])
def test_far_key_stands_out(dtype, place):
    """One token's key dominates the softmax of every later query: where it sits must not matter, and
    leaving it out would change the result completely."""
    cfg = su.config([su.latent(heads=2, dim=16, vdim=16, rot_dim=4, kv_rank=32, base=1e6, ff=0)], width=64, vocab=32, residual_mult=1.0)
    w = su.weights(cfg, 11)
    D, C = 64, 32
    # the special token's latent points along one axis that every head's query follows strongly
    special = 31
    w["embed"][:, 0] = 0.5
    w["embed"][special, 1] = 16.0
    w["l0.mix.dkv"][0, :] = 0.0
    w["l0.mix.dkv"][0, 1] = 4.0
    w["l0.mix.dkv"][1:C, 1] = 0.0
    w["l0.mix.q"][:, 0] = 3.0
    w["l0.mix.uk"][:, 0] = 2.0
    w = {k: su.bf16_round(v) for k, v in w.items()}
    toks = _tokens(dict(cfg, vocab=31), 230, seed=place)
    toks[place] = special
    without = toks.copy()
    without[place] = 5
    want, other = ref.Model(cfg, w).forward(toks), ref.Model(cfg, w).forward(without)
    assert su.rel(other[205:], want[205:]) > 10 * TOL["bfloat16"]
    dec = su.decoder(cfg, w, dtype)
    for cuts in ([230], [200] + [1] * 30, [70, 5, 125, 2]):
        assert not _bad(_feed(dec, toks, cuts), want, dtype), cuts
    dec.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["wkv", "retention"])
def test_long_memory(dtype, kind):
    """Decays near one: the first token still decides the output a thousand tokens later; and the bonus and
    decay of the newest token show as well."""
    layer = su.wkv(heads=2, dim=16, ff=0) if kind == "wkv" else su.retention(heads=2, dim=16, vdim=16, decay=[0.9999, 0.9995], base=1e6, ff=0)
    cfg = su.config([layer], width=64, vocab=32, residual_mult=1.0)
    w = su.weights(cfg, 13)
    if kind == "wkv":
        w["l0.mix.w0"][:] = -9.0
        w["l0.mix.w2"][:] *= 0.25
    w["embed"][31] *= 1.0
    first = {"wkv": ["l0.mix.k", "l0.mix.v"], "retention": ["l0.mix.k", "l0.mix.v"]}[kind]
    w["embed"][:31, 0] = 0.0
    w["embed"][31, 0] = 12.0
    for n in first:
        w[n][:, 0] *= 8.0
    w = {k: su.bf16_round(v) for k, v in w.items()}
    toks = _tokens(dict(cfg, vocab=31), 1200, seed=1)
    toks[0] = 31
    without = toks.copy()
    without[0] = 3
    want, other = ref.Model(cfg, w).forward(toks), ref.Model(cfg, w).forward(without)
    assert su.rel(other[1100:], want[1100:]) > 3 * TOL["bfloat16"]
    dec = su.decoder(cfg, w, dtype, max_ctx=1200)
    for cuts in ([1200], [1150] + [1] * 50, [100, 3, 97, 200]):
        assert not _bad(_feed(dec, toks, cuts), want, dtype), cuts
    dec.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_extreme_decays(dtype):
    """Channels that forget at once beside channels that never forget: products of decays underflow, nothing overflows."""
    cfg = su.config([su.wkv(heads=2, dim=16, ff=0)], width=64)
    w = su.weights(cfg, 17)
    w["l0.mix.w0"] = su.bf16_round(np.tile([-12.0, 6.0, 0.0, 3.0], 8))
    toks = _tokens(cfg, 400)
    want = ref.Model(cfg, w).forward(toks)
    dec = su.decoder(cfg, w, dtype, max_ctx=400)
    for cuts in ([400], [300] + [1] * 100):
        got = _feed(dec, toks, cuts)
        assert np.isfinite(got).all() and not _bad(got, want, dtype)
    dec.close()


def test_far_positions_rotate_exactly():
    cfg = su.config([su.retention(heads=1, dim=8, vdim=8, base=50.0, decay=[0.99], ff=0), su.latent(heads=1, dim=8, vdim=8, rot_dim=8, kv_rank=16, base=50.0, scaling=su.YARN, ff=0)],
                    width=32, vocab=32)
    w = su.weights(cfg, 19)
    toks = _tokens(cfg, 3000)
    want = ref.Model(cfg, w).forward(toks)[-40:]
    dec = su.decoder(cfg, w, "float32", max_ctx=3000)
    dec.prefill(toks[:2960], 0)
    got = np.concatenate([dec.step(int(toks[p]), p, want_logits=True)[1][None] for p in range(2960, 3000)])
    assert su.rel(got, want) < 1e-4
    dec.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_sequences_one_after_the_other(dtype):
    """A new sequence sees nothing of the one before; the same tokens give the same bits again."""
    cfg = su.config(MIXED, loop={"start": 0, "stop": 3, "times": 2})
    w = su.weights(cfg, 6)
    a, b = _tokens(cfg, 120, 1), _tokens(cfg, 37, 2)
    dec = su.decoder(cfg, w, dtype)
    la = _feed(dec, a, [100, 1, 1, 18])
    lb = _feed(dec, b, [30, 1])
    assert not _bad(lb, ref.Model(cfg, w).forward(b), dtype)
    assert np.array_equal(_feed(dec, a, [100, 1, 1, 18]), la)
    dec.reset()
    assert np.array_equal(_feed(dec, b, [30, 1]), lb)
    dec.close()


def test_positions_are_checked():
    import runnburn_b200 as r
    cfg = su.config([su.wkv(), su.latent()])
    dec = su.decoder(cfg, su.weights(cfg), max_ctx=16)
    dec.prefill([1, 2, 3], 0)
    for bad in (lambda: dec.step(4, 5), lambda: dec.prefill([4, 5], 2), lambda: dec.step_dev(9)):
        with pytest.raises(r.RnbError, match="so far has 3 tokens"):
            bad()
    with pytest.raises(r.RnbError, match="outside the context"):
        dec.prefill(list(range(14)), 3)
    with pytest.raises(r.RnbError, match="outside the vocabulary"):
        dec.prefill([1, cfg["vocab"]], 3)
    with pytest.raises(r.RnbError, match="place"):
        dec.prefill_logits([1, 2], 3, [2])
    dec.step(4, 3)                     # the sequence is still usable
    dec.close()


def test_weights_are_checked():
    import runnburn_b200 as r
    cfg = su.config([su.wkv()])
    w = su.weights(cfg)
    dec = su.decoder(cfg, {k: v for k, v in w.items() if k != "l0.mix.w2"})
    with pytest.raises(r.RnbError, match="'l0.mix.w2' is not set"):
        dec.prefill([1], 0)
    with pytest.raises(r.RnbError, match="no tensor 'l0.mix.q'"):
        dec.set_tensor("l0.mix.q", "BF16", bytes(8), (2, 2))
    with pytest.raises(r.RnbError, match="shape does not match"):
        dec.set_tensor("l0.mix.r", "BF16", bytes(8), (2, 2))
    dec.set_tensor("l0.mix.w2", "BF16", bytes(48 * 13 * 2), (48, 13))
    with pytest.raises(r.RnbError, match="w1 has 12 rows, w2 13"):
        dec.prefill([1], 0)
    dec.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation(dtype, tmp_path):
    """The framework's own loop and the device-chained steps against the reference's argmax, wherever the
    reference is not nearly tied; the command line gives the same ids."""
    cfg = su.config(MIXED[:3], loop={"start": 0, "stop": 2, "times": 2}, vocab=61)
    w = su.weights(cfg, 9)
    prompt = [int(t) for t in _tokens(cfg, 21)]
    dec = su.decoder(cfg, w, dtype)
    ids = dec.generate(prompt, 48)
    m = ref.Model(cfg, w)
    lg = m.forward(prompt)[-1]
    for t in ids:
        assert lg[t] > lg.max() - 4 * TOL[dtype] * np.sqrt(np.mean(lg ** 2))
        lg = m.forward([t])[-1]
    nxt = dec.prefill(prompt, 0)
    assert nxt == ids[0]
    for i in range(1, 48):
        dec.step_dev(-1, True)
        dec.sync()
        assert int(np.argmax(dec.read_logits())) == ids[i]
    dec.close()
    su.save(tmp_path, cfg, w)
    r = subprocess.run([sys.executable, "-m", "runnburn_b200", "generate", "--model", str(tmp_path), "--prompt", ",".join(map(str, prompt)), "-n", "48",
                        "--dtype", dtype, "--max-ctx", "256"], capture_output=True, text=True, cwd=ROOT, timeout=120)
    assert r.returncode == 0, r.stderr
    assert [int(t) for t in r.stdout.split(",")] == ids


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay(dtype, tmp_path):
    cfg = su.config(MIXED, vocab=61)
    w = su.weights(cfg, 10)
    (tmp_path / "m").mkdir()
    (tmp_path / "out").mkdir()
    su.save(tmp_path / "m", cfg, w)
    a, b = [int(t) for t in _tokens(cfg, 60, 1)], [int(t) for t in _tokens(cfg, 30, 2)]
    steps = [("a", a[:40], [0, 39, 7], []), ("a", a[40:42], [], []), ("a", a[42:43], [0], []), ("a", a[43:], [16, 0], ["a"]), ("b", b[:29], [28], []), ("b", b[29:], [0], ["b"])]
    lines = [json.dumps({"step": i, "entries": [{"id": n, "tokens": t, "want": wn}], "end": e}) for i, (n, t, wn, e) in enumerate(steps)]
    r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(tmp_path / "out"), "--max-tokens", "60"],
                       input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=120)
    assert r.returncode == 0, r.stderr
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == [f"done {i}" for i in range(6)]
    la, lb = ref.Model(cfg, w).forward(a), ref.Model(cfg, w).forward(b)
    expect = {0: la[[0, 39, 7]], 2: la[[42]], 3: la[[59, 43]], 4: lb[[28]], 5: lb[[29]]}
    for i in range(6):
        f = tmp_path / "out" / f"{i}.f32"
        assert f.exists() == (i in expect)
        if i in expect:
            assert not _bad(np.fromfile(f, "<f4").reshape(-1, cfg["vocab"]), expect[i], dtype)


def test_many_wanted_places():
    """More rows than one LM-head launch takes, in any order and repeated."""
    cfg = su.config([su.wkv()], vocab=41)
    w = su.weights(cfg, 12)
    toks = _tokens(cfg, 300)
    want = ref.Model(cfg, w).forward(toks)
    for dtype in DTYPES:
        dec = su.decoder(cfg, w, dtype, max_ctx=700)
        places = [5, 5] + list(range(299, -1, -1))
        got, nxt = dec.prefill_logits(toks, 0, places)
        assert not _bad(got, want[places], dtype)
        assert dtype == "bfloat16" or nxt == int(np.argmax(want[299]))
        dec.close()


def test_prompt_longer_than_one_piece():
    """Prompts are cut into internal pieces (512 tokens in f32); the state carries over."""
    cfg = su.config([su.wkv(heads=1, dim=8), su.latent(heads=1)], width=32)
    w = su.weights(cfg, 14)
    toks = _tokens(cfg, 1100)
    want = ref.Model(cfg, w).forward(toks)
    dec = su.decoder(cfg, w, "float32", max_ctx=1100)
    assert su.rel(dec.prefill_logits(toks, 0, [0, 511, 512, 1023, 1024, 1099])[0], want[[0, 511, 512, 1023, 1024, 1099]]) < TOL["float32"]
    dec.close()


def test_quantised_decoder_logits_at_places():
    """prefill_logits on the quantised stack: the logits of a place are those of the prompt that ends there."""
    import runnburn_b200 as r
    from synth import llama_description
    desc = llama_description(seed=3, n_layer=2, hidden=256, n_head=2, n_kv_head=1, n_ff=512, vocab=512)
    dec = r.Decoder(r.ModelConfig(max_ctx=64, **desc["cfg"]))
    dec.load_description(desc)
    toks = np.random.default_rng(0).integers(0, 512, 40)
    got, nxt = dec.prefill_logits(toks, 0, [39, 11])
    assert dec.prefill(toks, 0) == nxt and np.array_equal(dec.read_logits(), got[0])
    dec.prefill(toks[:12], 0)
    assert np.array_equal(dec.read_logits(), got[1])
    dec.close()
