"""Small random mixed stacks for the tests: a config.json-shaped dict and its weights (rounded to bf16)."""
from __future__ import annotations

import json

import numpy as np


def to_bf16_bits(a) -> np.ndarray:
    b = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return ((b + 0x7FFF + ((b >> 16) & 1)) >> 16).astype(np.uint16)


def bf16_round(a) -> np.ndarray:
    return (to_bf16_bits(a).astype(np.uint32) << 16).view(np.float32).reshape(np.shape(a))


def wkv(heads=3, dim=16, ff=48):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def retention(heads=2, dim=24, vdim=40, dims=None, base=1e4, decay=None, ff=48):
    decay = decay or [1.0 - 2.0 ** (-3.0 - 2.0 * i) for i in range(heads)]
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay, "rot": {"base": base, "dims": dims or dim}},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def latent(heads=3, dim=24, vdim=40, rot_dim=8, kv_rank=56, base=1e4, scaling=None, scale=None, ff=48):
    rot = {"base": base, "dims": rot_dim}
    if scaling:
        rot["scaling"] = scaling
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "rot_dim": rot_dim, "kv_rank": kv_rank, "rot": rot,
                                                  "scale": scale or (dim + rot_dim) ** -0.5}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def gla(heads=3, dim=16, vdim=24, tau=8.0, ff=40):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def window(heads=4, kv_heads=2, dim=16, vdim=24, size=11, dims=None, base=1e3, factor=2.5, scale=0.4):
    """The attention half of a parallel mixer."""
    rot = {"base": base, "dims": dim if dims is None else dims}
    if factor:
        rot["scaling"] = {"factor": factor}
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size}, "rot": rot, "scale": scale}


def delta(heads=4, kv_heads=2, dim=16, vdim=24, conv=4):
    """The delta-rule half."""
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def parallel(left=None, right=None, left_scale=0.8, right_scale=-1.3, ff=40):
    return {"type": "parallel", "mixer": {"left": left or window(), "right": right or delta(), "left_scale": left_scale, "right_scale": right_scale},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def again(layer, of):
    """The layer once more with the weights of layer `of`."""
    return dict(layer, weights_of=of)


def dutivik(layers, width=72, vocab=97, eps=1e-5, scale=3.0):
    return {"architecture": "Dutivik", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


YARN = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}


def config(layers, width=72, vocab=97, loop=None, eps=1e-5, residual_mult=0.7):
    return {"architecture": "Punisun", "layers": layers, "loop": loop, "norm": {"eps": eps}, "residual_mult": residual_mult, "vocab": vocab, "width": width}


def weights(cfg, seed=0, rank=12) -> dict:
    rng = np.random.default_rng(seed)
    D, out = cfg["width"], {}
    dutivik_design = cfg["architecture"] == "Dutivik"

    def mat(name, rows, cols, gain=1.0):
        out[name] = bf16_round(rng.standard_normal((rows, cols)) * gain / np.sqrt(cols))

    def vec(name, n, mean=0.0, sigma=0.2):
        out[name] = bf16_round(mean + sigma * rng.standard_normal(n))

    out["embed"] = bf16_round(rng.standard_normal((cfg["vocab"], D)))
    for i, ly in enumerate(cfg["layers"]):
        p, m = f"l{i}.", ly["mixer"]
        if dutivik_design:
            if ly.get("weights_of") is None:
                dutivik_layer(ly, p, D, rank, rng, mat, vec, out)
            continue
        x, H, d = p + "mix.", m["heads"], m["dim"]
        V = m.get("vdim", d)
        vec(p + "norm1", D), vec(p + "norm1b", D)
        mat(x + "o", D, H * V)
        if ly["type"] == "wkv":
            for c in "rkvgw":
                out[x + "mu." + c] = bf16_round(rng.uniform(0, 1, D))
            for c in "rkvg":
                mat(x + c, H * d, D)
            mat(x + "w1", rank, D), mat(x + "w2", H * d, rank)
            vec(x + "w0", H * d, -2.0, 1.5)
            out[x + "u"] = bf16_round(rng.standard_normal((H, d)))
            vec(x + "norm", H * d, 1.0)
        elif ly["type"] == "retention":
            mat(x + "q", H * d, D), mat(x + "k", H * d, D), mat(x + "v", H * V, D), mat(x + "g", H * V, D)
        else:
            mat(x + "q", H * (d + m["rot_dim"]), D, 2.0), mat(x + "dkv", m["kv_rank"] + m["rot_dim"], D)
            vec(x + "dkv.norm", m["kv_rank"], 1.0)
            mat(x + "uk", H * d, m["kv_rank"]), mat(x + "uv", H * V, m["kv_rank"])
        if ly["mlp"]:
            ff = ly["mlp"]["ff"]
            vec(p + "norm2", D), vec(p + "norm2b", D)
            mat(p + "mlp.gate", ff, D), mat(p + "mlp.up", ff, D), mat(p + "mlp.down", D, ff)
    vec("final.norm", D, 1.0 if dutivik_design else 0.0)
    if dutivik_design:
        vec("final.norm.b", D)
    return out


def dutivik_layer(ly, p, D, rank, rng, mat, vec, out):
    m, x = ly["mixer"], p + "mix."
    vec(p + "norm1", D, 1.0), vec(p + "norm1.b", D)
    if ly["type"] == "gla":
        H, d, V = m["heads"], m["dim"], m["vdim"]
        mat(x + "q", H * d, D), mat(x + "k", H * d, D), mat(x + "v", H * V, D), mat(x + "g", H * V, D), mat(x + "o", D, H * V)
        mat(x + "a1", rank, D), mat(x + "a2", H * d, rank)
        vec(x + "a2.b", H * d, 1.0, 2.0), vec(x + "norm", V, 1.0)
    else:
        a, b, y, z = m["left"], m["right"], x + "left.", x + "right."
        H, G, d, V = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
        mat(y + "q", H * d, D), mat(y + "k", G * d, D), mat(y + "v", G * V, D), mat(y + "g", H, D, 2.0), mat(y + "o", D, H * V)
        H, G, d, V = b["heads"], b["kv_heads"], b["dim"], b["vdim"]
        for c, n in (("q", G * d), ("k", G * d), ("v", H * V)):
            mat(z + c, n, D, 1.5)
            out[z + c + ".conv"] = bf16_round(rng.standard_normal((n, b["conv"])) * 0.6 + np.eye(1, b["conv"], b["conv"] - 1))
        mat(z + "b", H, D, 2.0), mat(z + "a", H, D, 2.0), mat(z + "g", H * V, D), mat(z + "o", D, H * V)
        vec(z + "A_log", H, -1.0, 1.0), vec(z + "dt_bias", H, -1.0, 1.0), vec(z + "norm", V, 1.0)
    if ly["mlp"]:
        ff = ly["mlp"]["ff"]
        mat(p + "mlp.gate", ff, D), mat(p + "mlp.up", ff, D), mat(p + "mlp.down", D, ff)


def save(folder, cfg, w) -> None:
    """config.json and model.safetensors."""
    header, blobs, at = {"__metadata__": {"format": "pt"}}, [], 0
    for name, a in w.items():
        b = to_bf16_bits(a).tobytes()
        header[name] = {"dtype": "BF16", "shape": list(np.shape(a)), "data_offsets": [at, at + len(b)]}
        at += len(b)
        blobs.append(b)
    h = json.dumps(header).encode()
    h += b" " * (-len(h) % 8)
    (folder / "config.json").write_text(json.dumps(cfg))
    (folder / "model.safetensors").write_bytes(len(h).to_bytes(8, "little") + h + b"".join(blobs))


def decoder(cfg, w, dtype="float32", max_ctx=256):
    import runnburn_b200 as r
    from runnburn_b200.registry import ARCHITECTURES
    dec = r.Decoder(ARCHITECTURES[cfg["architecture"]](cfg, max_ctx, dtype))
    for name, a in w.items():
        dec.set_tensor(name, "BF16", to_bf16_bits(a).tobytes(), np.shape(a))
    return dec


def tokens(cfg, n, seed=0):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n)


def feed(dec, toks, cuts):
    """Logits of all tokens, fed in portions of the sizes `cuts` (repeated until the end)."""
    out, at, i = [], 0, 0
    while at < len(toks):
        n = min(cuts[i % len(cuts)], len(toks) - at)
        i += 1
        if n == 1 and at > 0:
            out.append(dec.step(int(toks[at]), at, want_logits=True)[1][None])
        else:
            out.append(dec.prefill_logits(toks[at:at + n], at, list(range(n)))[0])
        at += n
    return np.concatenate(out)


TOL = {"float32": 2e-5, "bfloat16": 3e-2}


def bad(got, want, dtype) -> str:
    """Empty when the rows agree.  f32: every row.  bf16 rounds the projections, and a head's norm amplifies that
    where its output nearly cancels: the rows together are held to TOL, a single one to four times as much."""
    worst = rel(got, want)
    mean = float(np.sqrt(np.mean((np.asarray(got, np.float64) - want) ** 2) / np.mean(np.asarray(want, np.float64) ** 2)))
    ok = worst < TOL[dtype] if dtype == "float32" else mean < TOL[dtype] and worst < 4 * TOL[dtype]
    return "" if ok else f"worst row {worst:.3g}, together {mean:.3g}"


def rel(got, ref) -> float:
    """Largest root-mean-square row error relative to the reference's overall scale."""
    got, ref = np.asarray(got, np.float64), np.asarray(ref, np.float64)
    return float(np.sqrt(np.max(np.mean((got - ref) ** 2, -1))) / np.sqrt(np.mean(ref ** 2)))
