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


YARN = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}


def config(layers, width=72, vocab=97, loop=None, eps=1e-5, residual_mult=0.7):
    return {"architecture": "Punisun", "layers": layers, "loop": loop, "norm": {"eps": eps}, "residual_mult": residual_mult, "vocab": vocab, "width": width}


def weights(cfg, seed=0, rank=12) -> dict:
    rng = np.random.default_rng(seed)
    D, out = cfg["width"], {}

    def mat(name, rows, cols, gain=1.0):
        out[name] = bf16_round(rng.standard_normal((rows, cols)) * gain / np.sqrt(cols))

    def vec(name, n, mean=0.0, sigma=0.2):
        out[name] = bf16_round(mean + sigma * rng.standard_normal(n))

    out["embed"] = bf16_round(rng.standard_normal((cfg["vocab"], D)))
    for i, ly in enumerate(cfg["layers"]):
        p, m = f"l{i}.", ly["mixer"]
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
    vec("final.norm", D)
    return out


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
    from runnburn_b200.stack import punisun_config
    dec = r.Decoder(punisun_config(cfg, max_ctx, dtype))
    for name, a in w.items():
        dec.set_tensor(name, "BF16", to_bf16_bits(a).tobytes(), np.shape(a))
    return dec


def rel(got, ref) -> float:
    """Largest root-mean-square row error relative to the reference's overall scale."""
    got, ref = np.asarray(got, np.float64), np.asarray(ref, np.float64)
    return float(np.sqrt(np.max(np.mean((got - ref) ** 2, -1))) / np.sqrt(np.mean(ref ** 2)))
