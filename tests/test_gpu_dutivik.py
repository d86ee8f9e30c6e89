"""The Dutivik design on the GPU against the plain reference (hybrid_ref): mechanisms alone, portions, decoding,
window edges, far tokens, convolution and state carried over, rings that wrap, shared weights, generation, trace."""
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
DTYPES = ["float32", "bfloat16"]
PORTIONS = [(0, 20), (20, 3), (23, 8), (31, 1), (32, 9), (41, 40), (81, 2), (83, 67)]


def attention_only(**kw):
    return su.parallel(left=su.window(**kw), left_scale=1.5, right_scale=0.0, ff=0)


def delta_only(**kw):
    return su.parallel(right=su.delta(**kw), left_scale=0.0, right_scale=0.7, ff=0)


MECHANISMS = {
    "gla": (su.gla(ff=0), 72), "gla_tau_1": (su.gla(tau=1.0, ff=0), 72), "gla_odd": (su.gla(heads=1, dim=5, vdim=7, ff=0), 41),
    "gla_64": (su.gla(heads=2, dim=64, vdim=32, ff=0), 64), "gla_wide": (su.gla(heads=2, dim=136, vdim=144, tau=30.0, ff=0), 64),
    "gla_narrow_values": (su.gla(heads=5, dim=40, vdim=8, ff=0), 48),
    "attention": (attention_only(), 72), "attention_one": (attention_only(size=1), 72), "attention_two": (attention_only(size=2, kv_heads=4), 72),
    "attention_all": (attention_only(size=10 ** 6, kv_heads=1), 72), "attention_64": (attention_only(size=64, dim=64, vdim=64, factor=None), 64),
    "attention_65": (attention_only(size=65, heads=6, kv_heads=3, dim=32, vdim=128, dims=8), 64),
    "attention_no_rotation": (attention_only(size=30, dims=0), 48), "attention_odd": (attention_only(heads=3, kv_heads=1, dim=10, vdim=7, size=33, dims=6), 50),
    "attention_many": (attention_only(heads=40, kv_heads=2, dim=32, vdim=16, size=90), 64),
    "attention_wide": (attention_only(heads=2, kv_heads=2, dim=288, vdim=264, size=40), 64), "attention_large": (attention_only(heads=4, kv_heads=1, dim=128, vdim=256, size=100, scale=0.1), 64),
    "delta": (delta_only(), 72), "delta_one_tap": (delta_only(conv=1), 72), "delta_two_taps": (delta_only(conv=2, kv_heads=4), 72), "delta_seven_taps": (delta_only(conv=7, kv_heads=1), 64),
    "delta_odd": (delta_only(heads=3, kv_heads=1, dim=9, vdim=5), 50), "delta_64": (delta_only(heads=2, kv_heads=2, dim=64, vdim=48), 64),
    "delta_wide": (delta_only(heads=2, kv_heads=1, dim=256, vdim=136), 64), "delta_128": (delta_only(heads=2, kv_heads=2, dim=128, vdim=64), 64),
    "delta_very_wide": (delta_only(heads=1, kv_heads=1, dim=320, vdim=40), 64), "delta_48": (delta_only(heads=4, kv_heads=2, dim=48, vdim=16), 64),
    "both": (su.parallel(ff=0), 72), "dense": (su.gla(heads=1, dim=8, vdim=8, ff=264), 64), "dense_odd": (su.gla(heads=1, dim=8, vdim=9, ff=37), 51),
    "everything": (su.parallel(ff=72), 72),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(MECHANISMS))
def test_one_layer_residual(name, dtype):
    """What one layer adds: a whole prompt, portions, and token by token behind a prompt."""
    layer, width = MECHANISMS[name]
    cfg = su.dutivik([layer], width=width)
    w = su.weights(cfg, 7)
    toks = su.tokens(cfg, 150)
    m = ref.Model(cfg, w)
    m.trace = []
    m.forward(toks)
    base = w["embed"][toks] * 3.0
    want = m.trace[0] - base
    dec = su.decoder(cfg, w, dtype)
    assert not su.bad(dec.trace_residual(toks)[0] - base, want, dtype)
    parts = [dec.trace_residual(toks[a:a + n], a)[0] for a, n in PORTIONS]
    assert not su.bad(np.concatenate(parts) - base, want, dtype)
    parts = [dec.trace_residual(toks[:100])[0]] + [dec.trace_residual(toks[a:a + 1], a)[0] for a in range(100, 150)]
    assert not su.bad(np.concatenate(parts) - base, want, dtype)
    dec.close()


MIXED = [su.parallel(), su.gla(), su.parallel(left=su.window(heads=3, kv_heads=3, dim=8, vdim=16, size=40, dims=4), right=su.delta(heads=2, kv_heads=1, dim=32, vdim=8, conv=2), ff=0),
         su.gla(heads=1, dim=32, vdim=40, tau=1.0, ff=0)]
SHARED = MIXED + [su.again(MIXED[0], 0), su.again(MIXED[3], 3), su.again(MIXED[2], 2), su.again(MIXED[0], 0)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rank", [1, 7, 32, 136])
def test_low_rank_decay_of_any_width(rank, dtype):
    cfg = su.dutivik([su.gla(heads=3, dim=24, vdim=16), su.gla(heads=1, dim=96, vdim=8, tau=2.0)], width=64)
    w = su.weights(cfg, 23, rank=rank)
    toks = su.tokens(cfg, 70)
    want = ref.Model(cfg, w).forward(toks)
    dec = su.decoder(cfg, w, dtype)
    for cuts in ([70], [30] + [1] * 40):
        assert not su.bad(su.feed(dec, toks, cuts), want, dtype)
    dec.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("layers", [MIXED, SHARED], ids=["own", "shared"])
def test_stack(dtype, layers):
    cfg = su.dutivik(layers, eps=1e-3, scale=1.0)
    w = su.weights(cfg, 2)
    toks = su.tokens(cfg, 90)
    m = ref.Model(cfg, w)
    m.trace = []
    want = m.forward(toks)
    dec = su.decoder(cfg, w, dtype)
    tr = dec.trace_residual(toks)
    assert tr.shape[0] == len(m.trace) == len(layers)
    for got, exp in zip(tr, m.trace):
        assert not su.bad(got, exp, dtype)
    for cuts in ([90], [50] + [1] * 40, [1]):
        assert not su.bad(su.feed(dec, toks, cuts), want, dtype), cuts
    dec.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_portions_of_every_size(dtype):
    cfg = su.dutivik(SHARED)
    w = su.weights(cfg, 4)
    toks = su.tokens(cfg, 230)
    want = ref.Model(cfg, w).forward(toks)
    dec = su.decoder(cfg, w, dtype)
    for cuts in ([2], [3, 2], [7, 8, 9], [10, 1, 97, 2, 98], [64, 63, 65], [15, 16, 17], [1], [229, 1]):
        assert not su.bad(su.feed(dec, toks, cuts), want, dtype), cuts
    dec.close()


def test_layer_norm_of_rows_far_from_zero():
    """Rows whose mean is large against their spread: the mean comes off before the squares are taken."""
    cfg = su.dutivik([su.gla(heads=1, dim=8, vdim=8)], width=64, scale=1.0)
    w = su.weights(cfg, 3)
    w["embed"] = su.bf16_round(w["embed"] + 60.0)
    toks = su.tokens(cfg, 40)
    want = ref.Model(cfg, w).forward(toks)
    dec = su.decoder(cfg, w, "float32")
    for cuts in ([40], [1]):
        assert su.rel(su.feed(dec, toks, cuts), want) < 1e-4
    dec.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_prompt_and_decoding(dtype):
    """Crosses the chunk lengths of the recurrences, attention tiles, internal pieces (512 tokens in f32) and the
    key ring of a short window."""
    cfg = su.dutivik([su.parallel(left=su.window(size=5, kv_heads=1), right=su.delta(dim=32)), su.gla(heads=2), su.parallel(left=su.window(size=200, heads=2, kv_heads=2))], width=64)
    w = su.weights(cfg, 5)
    toks = su.tokens(cfg, 1300)
    want = ref.Model(cfg, w).forward(toks)
    dec = su.decoder(cfg, w, dtype, max_ctx=1300)
    for cuts in ([1300], [1025, 95, 180], [300, 97, 903], [700] + [1] * 600):
        assert not su.bad(su.feed(dec, toks, cuts), want, dtype), cuts
    dec.close()


def test_ring_of_a_long_sequence_wraps():
    """bf16: 4096-token pieces on a ring of a few rows more; the decode steps behind wrap once more."""
    cfg = su.dutivik([su.parallel(left=su.window(size=3, heads=2, kv_heads=1, dim=8, vdim=8, factor=100.0), right=su.delta(heads=1, kv_heads=1, dim=16, vdim=8), ff=0)], width=32, vocab=31)
    w = su.weights(cfg, 8)
    toks = su.tokens(cfg, 4400)
    want = ref.Model(cfg, w).forward(toks)
    dec = su.decoder(cfg, w, "bfloat16", max_ctx=5000)
    for cuts in ([4400], [4090] + [1] * 30 + [280], [2200, 2200]):
        assert not su.bad(su.feed(dec, toks, cuts), want, "bfloat16"), cuts[:2]
    dec.close()


def _beacon(size, place, n, vocab=32, width=64):
    """One attention layer whose queries all follow one direction; the key of the token at `place` lies along it and every
    other key against it: whether it is seen decides the output."""
    cfg = su.dutivik([attention_only(heads=2, kv_heads=1, dim=16, vdim=16, size=size, dims=2, base=1e8, factor=1e6, scale=1.0)], width=width, vocab=vocab, scale=1.0)
    w = su.weights(cfg, 11)
    special = vocab - 1
    w["l0.norm1"][:], w["l0.norm1.b"][:] = 1.0, 0.0
    w["embed"][:, 0] = 6.0
    w["embed"][:, 1] = -4.0
    w["embed"][special, 1] = 20.0
    w["embed"][special, 2:] *= 3.0
    w["l0.mix.left.q"][:, 0] = 2.0
    w["l0.mix.left.k"][:, 1] = 2.0
    w["l0.mix.left.o"][:] *= 5.0
    w = {k: su.bf16_round(v) for k, v in w.items()}
    toks = su.tokens(dict(cfg, vocab=special), n, seed=place)
    without = toks.copy()
    toks[place] = special
    return cfg, w, toks, without


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size,place", [(1, 9), (2, 9), (16, 0), (63, 5), (64, 5), (65, 63), (65, 64), (100, 27), (128, 0), (128, 1), (129, 127)])
def test_window_edge(dtype, size, place):
    """The last query that sees a token, and the first that does not, in prompts and decoding."""
    n = place + size + 40
    cfg, w, toks, without = _beacon(size, place, n)
    want, other = ref.Model(cfg, w).forward(toks), ref.Model(cfg, w).forward(without)
    last = place + size - 1
    assert np.allclose(other[last + 1:], want[last + 1:])
    if size > 1:
        assert su.rel(other[last:last + 1], want[last:last + 1]) > 10 * su.TOL["bfloat16"]
    dec = su.decoder(cfg, w, dtype, max_ctx=300)
    for cuts in ([n], [max(last - 2, 2)] + [1] * n, [last, n - last], [last + 1, n - last - 1], [place + 1, 2, n], [3]):
        got = su.feed(dec, toks, cuts)
        assert not su.bad(got, want, dtype), cuts[:2]
        for p in (last, last + 1):
            assert not su.bad(got[p:p + 1], want[p:p + 1], dtype), (cuts[:2], p)
    dec.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["gla", "delta"])
def test_long_memory(dtype, kind):
    """Decays near one: the first token still decides the output a thousand tokens later."""
    layer = su.gla(heads=2, dim=32, vdim=16, tau=500.0, ff=0) if kind == "gla" else delta_only(heads=2, kv_heads=2, dim=32, vdim=16, conv=3)
    cfg = su.dutivik([layer], width=64, vocab=32)
    w = su.weights(cfg, 13)
    if kind == "gla":
        w["l0.mix.a2.b"][:] = 6.0
        w["l0.mix.a2"][:] *= 0.25
        w["embed"][:, 1] = 6.0            # every query follows one direction, and the first key lies along it
        w["l0.mix.q"][:, 1] = 1.0
        w["l0.mix.k"][:, 0] = 2.0
        names = ["l0.mix.v"]
    else:
        p = "l0.mix.right."
        w[p + "A_log"][:] = -4.0
        w[p + "dt_bias"][:] = -5.0
        w[p + "a"][:] *= 0.25
        w[p + "b"][:] *= 0.5
        w[p + "b"][:, 1] = -6.0       # only the first token writes much
        w[p + "b"][:, 0] = 6.0
        names = [p + "v"]
        w["embed"][:31, 1] = 6.0
        w["embed"][31, 1] = 0.0
    w["embed"][:31, 0] = 0.0
    w["embed"][31, 0] = 12.0
    for n in names:
        w[n][:, 0] *= 8.0
    w["l0.mix.o" if kind == "gla" else "l0.mix.right.o"][:] *= 6.0
    w = {k: su.bf16_round(v) for k, v in w.items()}
    toks = su.tokens(dict(cfg, vocab=31), 1200, seed=1)
    toks[0] = 31
    without = toks.copy()
    without[0] = 3
    want, other = ref.Model(cfg, w).forward(toks), ref.Model(cfg, w).forward(without)
    assert su.rel(other[1100:], want[1100:]) > 3 * su.TOL["bfloat16"]
    dec = su.decoder(cfg, w, dtype, max_ctx=1200)
    for cuts in ([1200], [1150] + [1] * 50, [100, 3, 97, 200]):
        assert not su.bad(su.feed(dec, toks, cuts), want, dtype), cuts[:2]
    dec.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_extreme_decays(dtype):
    """States that vanish at once beside states that never do: products of decays underflow, nothing overflows; keys
    that repeat (a token many times in a row) keep the delta rule's corrections well behaved."""
    cfg = su.dutivik([su.gla(heads=2, dim=16, vdim=16, tau=1.0, ff=0), delta_only(heads=4, kv_heads=2, dim=16, vdim=16)], width=64)
    w = su.weights(cfg, 17)
    w["l0.mix.a2.b"] = su.bf16_round(np.tile([60.0, -60.0, 0.0, -6.0], 8))
    w["l1.mix.right.A_log"] = su.bf16_round([4.0, -8.0, 0.0, 2.0])
    w["l1.mix.right.dt_bias"] = su.bf16_round([8.0, -8.0, 0.0, 1.0])
    toks = su.tokens(cfg, 400)
    toks[100:160] = 7
    want = ref.Model(cfg, w).forward(toks)
    dec = su.decoder(cfg, w, dtype, max_ctx=400)
    for cuts in ([400], [300] + [1] * 100, [33]):
        got = su.feed(dec, toks, cuts)
        assert np.isfinite(got).all() and not su.bad(got, want, dtype), cuts[:2]
    dec.close()


def test_far_positions_rotate_exactly():
    cfg = su.dutivik([su.parallel(left=su.window(heads=1, kv_heads=1, dim=8, vdim=8, size=50, base=30.0, factor=1.5), right=su.delta(heads=1, kv_heads=1, dim=8, vdim=8))], width=32, vocab=32)
    w = su.weights(cfg, 19)
    toks = su.tokens(cfg, 3000)
    want = ref.Model(cfg, w).forward(toks)[-40:]
    dec = su.decoder(cfg, w, "float32", max_ctx=3000)
    dec.prefill(toks[:2960], 0)
    got = np.concatenate([dec.step(int(toks[p]), p, want_logits=True)[1][None] for p in range(2960, 3000)])
    assert su.rel(got, want) < 1e-4
    dec.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_sequences_one_after_the_other(dtype):
    """A new sequence sees nothing of the one before (states, rings, convolutions); the same tokens give the same bits."""
    cfg = su.dutivik(SHARED)
    w = su.weights(cfg, 6)
    a, b, c = su.tokens(cfg, 120, 1), su.tokens(cfg, 37, 2), su.tokens(cfg, 3, 3)
    dec = su.decoder(cfg, w, dtype)
    la = su.feed(dec, a, [100, 1, 1, 18])
    lb = su.feed(dec, b, [30, 1])
    assert not su.bad(lb, ref.Model(cfg, w).forward(b), dtype)
    assert not su.bad(su.feed(dec, c, [1]), ref.Model(cfg, w).forward(c), dtype)
    assert np.array_equal(su.feed(dec, a, [100, 1, 1, 18]), la)
    dec.reset()
    assert np.array_equal(su.feed(dec, b, [30, 1]), lb)
    dec.close()


def test_weights_and_shapes_are_checked():
    import runnburn_b200 as r
    cfg = su.dutivik([su.gla(), su.parallel(), su.again(su.gla(), 0)])
    w = su.weights(cfg)
    dec = su.decoder(cfg, {k: v for k, v in w.items() if k != "l1.mix.right.q.conv"})
    with pytest.raises(r.RnbError, match="'l1.mix.right.q.conv' is not set"):
        dec.prefill([1], 0)
    with pytest.raises(r.RnbError, match="no tensor 'l2.mix.q'"):
        dec.set_tensor("l2.mix.q", "BF16", bytes(8), (2, 2))
    with pytest.raises(r.RnbError, match="shape does not match"):
        dec.set_tensor("l1.mix.left.k", "BF16", bytes(8), (2, 2))
    dec.close()
    for layers, what in (([su.gla(), su.again(su.gla(dim=24), 0)], "cannot use the weights"), ([su.again(su.gla(), 0)], "cannot use the weights"),
                         ([su.parallel(left=su.window(heads=3, kv_heads=2))], "do not share"), ([su.parallel(right=su.delta(conv=0))], "taps"),
                         ([su.parallel(left=su.window(dims=18))], "rotation"), ([su.gla(tau=0.0)], "tau")):
        with pytest.raises(r.RnbError, match=what):
            su.decoder(su.dutivik(layers), {})


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation(dtype, tmp_path):
    """The framework's own loop and the device-chained steps against the reference's argmax, wherever the
    reference is not nearly tied; the command line gives the same ids."""
    cfg = su.dutivik(SHARED[:6], vocab=61)
    w = su.weights(cfg, 9)
    prompt = [int(t) for t in su.tokens(cfg, 21)]
    dec = su.decoder(cfg, w, dtype)
    ids = dec.generate(prompt, 48)
    m = ref.Model(cfg, w)
    lg = m.forward(prompt)[-1]
    for t in ids:
        assert lg[t] > lg.max() - 4 * su.TOL[dtype] * np.sqrt(np.mean(lg ** 2))
        lg = m.forward([t])[-1]
    assert dec.prefill(prompt, 0) == ids[0]
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
    cfg = su.dutivik(SHARED, vocab=61)
    w = su.weights(cfg, 10)
    (tmp_path / "m").mkdir()
    (tmp_path / "out").mkdir()
    su.save(tmp_path / "m", cfg, w)
    a, b = [int(t) for t in su.tokens(cfg, 60, 1)], [int(t) for t in su.tokens(cfg, 30, 2)]
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
            assert not su.bad(np.fromfile(f, "<f4").reshape(-1, cfg["vocab"]), expect[i], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_new_mixers_in_sandwich_layers(dtype):
    """The mechanisms do not depend on the block around them: gated linear attention between sublayer norms."""
    import runnburn_b200 as r
    from runnburn_b200.stack import MixerLayer, StackConfig
    D, V, eps = 48, 53, 1e-5
    base = su.dutivik([su.gla(heads=2, dim=16, vdim=8, ff=24)], width=D, vocab=V)
    w = su.weights(base, 21)
    rng = np.random.default_rng(5)
    w = {k: v for k, v in w.items() if not k.endswith(".b") or "a2" in k}
    for n in ("l0.norm1", "l0.norm1b", "l0.norm2", "l0.norm2b", "final.norm"):
        w[n] = su.bf16_round(0.2 * rng.standard_normal(D))
    dec = r.Decoder(StackConfig(width=D, vocab=V, layers=[MixerLayer(mixer="gla", heads=2, dim=16, vdim=8, tau=8.0, n_ff=24)], norm_eps=eps, residual_mult=0.5, max_ctx=64, dtype=dtype))
    for name, a in w.items():
        dec.set_tensor(name, "BF16", su.to_bf16_bits(a).tobytes(), np.shape(a))
    toks = su.tokens(base, 50)
    x = w["embed"][toks].astype(np.float64)
    y, _ = ref.mix_gla({"heads": 2, "dim": 16, "vdim": 8, "tau": 8.0}, w, "l0.mix.", ref.norm_about_zero(x, w["l0.norm1"], eps), None, 0, eps)
    x = x + 0.5 * ref.norm_about_zero(y, w["l0.norm1b"], eps)
    y = ref.feed_forward(w, "l0.mlp.", ref.norm_about_zero(x, w["l0.norm2"], eps))
    x = x + 0.5 * ref.norm_about_zero(y, w["l0.norm2b"], eps)
    want = ref.norm_about_zero(x, w["final.norm"], eps) @ w["embed"].T
    for cuts in ([50], [20] + [1] * 30):
        assert not su.bad(su.feed(dec, toks, cuts), want, dtype)
    dec.close()
