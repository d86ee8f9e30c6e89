"""Configuration of mixed stacks: config.json of a design -> the C ABI's stack and layer records.

A design lists its layers one by one (mixer, sizes, feed-forward) and may loop over a range of them.
Every size and constant comes from the file.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass, field

from . import _lib
from ._lib import check, load

MIXERS = {"wkv": _lib.MIXER_WKV, "retention": _lib.MIXER_RETENTION, "latent_attention": _lib.MIXER_LATENT_ATTENTION, "gla": _lib.MIXER_GLA,
          "attention": _lib.MIXER_ATTENTION, "delta": _lib.MIXER_DELTA}
BLOCKS = {"sandwich": _lib.BLOCK_SANDWICH, "parallel": _lib.BLOCK_PARALLEL}
NORMS = {"rms": _lib.NORM_RMS, "layer": _lib.NORM_LAYER}
ACTS = {"gelu_tanh": _lib.ACT_GELU_TANH, "silu": _lib.ACT_SILU}
# pairs (2i, 2i + 1) rotate together in these mixers, (i, i + dims / 2) in the others
INTERLEAVED = {"latent_attention", "attention"}


@dataclass
class MixerLayer:
    """One layer of the list: the mixer's sizes and constants, and the feed-forward width (0: none).
    `join`: one more mixer of the layer before it in the list, reading the same input."""
    mixer: str
    heads: int
    dim: int
    vdim: int = 0
    rot_dim: int = 0
    kv_rank: int = 0
    decay_rank: int = 0
    scale: float = 1.0
    rot: dict | None = None
    decay: list = field(default_factory=list)
    n_ff: int = 0
    kv_heads: int = 0
    window: int = 0                  # attention: keys that a query sees, its own included (0: all)
    qk_norm: bool = False
    head_gate: bool = False
    conv: int = 0
    tau: float = 1.0
    out_scale: float = 1.0
    join: bool = False
    weights_of: int | None = None    # the layer whose tensors this one uses
    prefix: str = "mix."             # of the tensor names, after the layer's

    def to_c(self, keep: list) -> _lib.MixerCfg:
        if self.mixer not in MIXERS:
            raise ValueError(f"unknown mixer {self.mixer!r} (known: {', '.join(sorted(MIXERS))})")
        c = _lib.MixerCfg()
        c.mixer = MIXERS[self.mixer]
        for k in ("heads", "dim", "vdim", "rot_dim", "kv_rank", "decay_rank", "scale", "n_ff", "kv_heads", "window", "qk_norm", "head_gate", "conv", "tau",
                  "out_scale", "join"):
            setattr(c, k, getattr(self, k))
        c.weights_of = -1 if self.weights_of is None else self.weights_of
        c.prefix = self.prefix.encode()
        if self.rot:
            r = c.rot
            r.dims, r.base, r.interleaved = int(self.rot["dims"]), float(self.rot["base"]), int(self.mixer in INTERLEAVED)
            sc = self.rot.get("scaling")
            if sc and "original" not in sc:
                r.scaled, r.factor = _lib.ROTATION_LINEAR, float(sc["factor"])
            elif sc:
                r.scaled = _lib.ROTATION_YARN
                for k in ("factor", "original", "fast", "slow"):
                    setattr(r, k, float(sc[k]))
        if self.mixer == "retention":
            if len(self.decay) != self.heads:
                raise ValueError(f"retention: {len(self.decay)} decays for {self.heads} heads")
            arr = (C.c_double * len(self.decay))(*self.decay)
            keep.append(arr)
            c.decay = C.cast(arr, C.POINTER(C.c_double))
        return c


@dataclass
class StackConfig:
    width: int
    vocab: int
    layers: list
    norm_eps: float
    residual_mult: float = 1.0
    loop: tuple = (0, 0, 1)          # start, stop, times
    max_ctx: int = 4096
    dtype: str = "bfloat16"          # or "float32": activations and matrix products in 32-bit
    block: str = "sandwich"          # or "parallel": the mixers and the feed-forward read one norm
    norm: str = "rms"                # or "layer"
    act: str = "gelu_tanh"           # or "silu"
    embed_scale: float = 1.0

    def create(self, handle) -> None:
        if self.dtype not in ("bfloat16", "float32"):
            raise ValueError(f"dtype {self.dtype!r} is not supported (bfloat16, float32)")
        keep: list = []
        layers = (_lib.MixerCfg * len(self.layers))(*[ly.to_c(keep) for ly in self.layers])
        c = _lib.StackCfg(n_layer=len(self.layers), width=self.width, vocab=self.vocab, max_ctx=self.max_ctx, loop_start=self.loop[0],
                          loop_stop=self.loop[1], loop_times=self.loop[2], norm_eps=self.norm_eps, residual_mult=self.residual_mult,
                          f32_math=int(self.dtype == "float32"), block=BLOCKS[self.block], norm=NORMS[self.norm], act=ACTS[self.act],
                          embed_scale=self.embed_scale)
        check(load().rnb_b200_decoder_create_stack(C.byref(c), layers, C.byref(handle)))


def punisun_config(cfg: dict, max_ctx: int, dtype: str) -> StackConfig:
    """config.json of the Punisun design."""
    layers = []
    for i, ly in enumerate(cfg["layers"]):
        m, mlp = ly["mixer"], ly.get("mlp")
        if mlp and mlp.get("kind", "dense") != "dense":
            raise ValueError(f"layer {i}: feed-forward {mlp['kind']!r} is not supported")
        if m.get("rot") and ly["type"] == "latent_attention" and int(m["rot"]["dims"]) != int(m["rot_dim"]):
            raise ValueError(f"layer {i}: rot.dims {m['rot']['dims']} must equal rot_dim {m['rot_dim']}")
        layers.append(MixerLayer(mixer=ly["type"], heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m.get("vdim", 0)), rot_dim=int(m.get("rot_dim", 0)),
                                 kv_rank=int(m.get("kv_rank", 0)), scale=float(m.get("scale", 1.0)), rot=m.get("rot"), decay=list(m.get("decay", [])),
                                 n_ff=int(mlp["ff"]) if mlp else 0))
    loop = cfg.get("loop")
    return StackConfig(width=int(cfg["width"]), vocab=int(cfg["vocab"]), layers=layers, norm_eps=float(cfg["norm"]["eps"]),
                       residual_mult=float(cfg.get("residual_mult", 1.0)),
                       loop=(int(loop["start"]), int(loop["stop"]), int(loop["times"])) if loop else (0, 0, 1), max_ctx=max_ctx, dtype=dtype)


def dutivik_config(cfg: dict, max_ctx: int, dtype: str) -> StackConfig:
    """config.json of the Dutivik design: parallel layers under one layer norm; a layer's mixer is gated linear
    attention, or window attention and the gated delta rule side by side."""
    layers = []
    for i, ly in enumerate(cfg["layers"]):
        m, mlp = ly["mixer"], ly.get("mlp")
        if mlp and mlp.get("kind", "dense") != "dense":
            raise ValueError(f"layer {i}: feed-forward {mlp['kind']!r} is not supported")
        of = ly.get("weights_of")
        first = dict(n_ff=int(mlp["ff"]) if mlp else 0, weights_of=None if of is None else int(of))
        if ly["type"] == "gla":
            layers.append(MixerLayer(mixer="gla", heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), tau=float(m["tau"]), **first))
        elif ly["type"] == "parallel":
            a, b = m["left"], m["right"]
            layers.append(MixerLayer(mixer="attention", heads=int(a["heads"]), kv_heads=int(a["kv_heads"]), dim=int(a["dim"]), vdim=int(a["vdim"]),
                                     rot=a.get("rot"), scale=float(a["scale"]), window=int((a.get("mask") or {}).get("size", 0)), qk_norm=True, head_gate=True,
                                     out_scale=float(m["left_scale"]), prefix="mix.left.", **first))
            layers.append(MixerLayer(mixer="delta", heads=int(b["heads"]), kv_heads=int(b["kv_heads"]), dim=int(b["dim"]), vdim=int(b["vdim"]),
                                     conv=int(b["conv"]), out_scale=float(m["right_scale"]), prefix="mix.right.", join=True, weights_of=first["weights_of"]))
        else:
            raise ValueError(f"layer {i}: unknown mixer {ly['type']!r} (known: gla, parallel)")
    return StackConfig(width=int(cfg["width"]), vocab=int(cfg["vocab"]), layers=layers, norm_eps=float(cfg["norm"]["eps"]), max_ctx=max_ctx, dtype=dtype,
                       block="parallel", norm="layer", act="silu", embed_scale=float(cfg["embedding"]["scale"]))
