"""Plain, slow reference of the layered decoders (Punisun, Dutivik): numpy in binary64, one function
per mechanism, token loops where the equations have them.  Shares no code with the package.

A model is (cfg, w): the parsed config.json and a dict name -> float array (weights as stored).
Shapes: x [T, width]; a mixer maps the normed input [T, width] to [T, width].
"""
from __future__ import annotations

import numpy as np

F = np.float64


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm_about_zero(x, w, eps):
    return rms(x, eps) * (1.0 + w)


def layer_norm(x, w, b, eps):
    d = x - np.mean(x, axis=-1, keepdims=True)
    return d / np.sqrt(np.mean(d * d, axis=-1, keepdims=True) + eps) * w + b


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def softplus(z):
    return np.logaddexp(0.0, z)


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


# ---- rotations ---------------------------------------------------------------------------------
def rotation_tables(rot, positions):
    """cos, sin [T, dims/2] (YaRN's factor included) of the angles position * frequency.  A scaling that
    gives nothing but a factor is the linear one: every frequency divided by it."""
    dims, base = int(rot["dims"]), float(rot["base"])
    i = np.arange(dims // 2, dtype=F)
    f = base ** (-2.0 * i / dims)
    mult = 1.0
    sc = rot.get("scaling")
    if sc and "original" not in sc:
        f = f / sc["factor"]
    elif sc:
        def dim_of(turns):
            return dims * np.log(sc["original"] / (2.0 * np.pi * turns)) / (2.0 * np.log(base))
        lo = max(np.floor(dim_of(sc["fast"])), 0.0)
        hi = min(np.ceil(dim_of(sc["slow"])), dims - 1.0)
        ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
        f = f / sc["factor"] * ramp + f * (1.0 - ramp)
        mult = 0.1 * np.log(sc["factor"]) + 1.0
    a = np.asarray(positions, F)[:, None] * f[None, :]
    return np.cos(a) * mult, np.sin(a) * mult


def rotate_pairs(x, cos, sin, interleaved):
    """x [T, heads, d]: the first 2*cos.shape[1] dimensions are rotated, the rest passes."""
    n = cos.shape[1]
    out = x.copy()
    c, s = cos[:, None, :], sin[:, None, :]
    if interleaved:
        u, v = x[..., 0:2 * n:2], x[..., 1:2 * n:2]
        out[..., 0:2 * n:2], out[..., 1:2 * n:2] = u * c - v * s, v * c + u * s
    else:
        u, v = x[..., :n], x[..., n:2 * n]
        out[..., :n], out[..., n:2 * n] = u * c - v * s, v * c + u * s
    return out


# ---- mixers ------------------------------------------------------------------------------------
def token_shift(h, last):
    """The previous token's row for every row; `last` is the row before the first."""
    return np.concatenate([last[None], h[:-1]], axis=0)


def wkv_recurrence(r, k, v, w, u, S):
    """r, k, w [T, H, D], v [T, H, D], u [H, D], S [H, D, D] (key x value) -> o [T, H, D], S."""
    o = np.empty(v.shape, F)
    S = S.copy()
    for t in range(r.shape[0]):
        kv = k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hij,hi->hj", S + u[:, :, None] * kv, r[t])
        S = w[t][:, :, None] * S + kv
    return o, S


def mix_wkv(m, w, p, h, state, pos0, eps):
    H, D = m["heads"], m["dim"]
    T = h.shape[0]
    if state is None:
        state = {"h": np.zeros(h.shape[1]), "S": np.zeros((H, D, D))}
    hp = token_shift(h, state["h"])
    mix = {c: h + (hp - h) * w[p + "mu." + c] for c in "rkvgw"}
    r, k, v = ((mix[c] @ w[p + c].T).reshape(T, H, D) for c in "rkv")
    gate = silu(mix["g"] @ w[p + "g"].T)
    decay = np.exp(-np.exp(np.tanh(mix["w"] @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"])).reshape(T, H, D)
    o, S = wkv_recurrence(r, k, v, decay, w[p + "u"].reshape(H, D), state["S"])
    o = rms(o, eps).reshape(T, H * D) * w[p + "norm"] * gate
    return o @ w[p + "o"].T, {"h": h[-1].copy(), "S": S}


def retention_recurrence(q, k, v, decay, S):
    o = np.empty(v.shape, F)
    S = S.copy()
    for t in range(q.shape[0]):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hij,hi->hj", S, q[t])
    return o, S


def mix_retention(m, w, p, h, state, pos0, eps):
    H, D, V = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    if state is None:
        state = {"S": np.zeros((H, D, V))}
    cos, sin = rotation_tables(m["rot"], np.arange(pos0, pos0 + T))
    q = rotate_pairs((h @ w[p + "q"].T).reshape(T, H, D), cos, sin, False)
    k = rotate_pairs((h @ w[p + "k"].T).reshape(T, H, D), cos, sin, False) * D ** -0.5
    v = (h @ w[p + "v"].T).reshape(T, H, V)
    o, S = retention_recurrence(q, k, v, np.asarray(m["decay"], F), state["S"])
    o = rms(o, eps).reshape(T, H * V) * silu(h @ w[p + "g"].T)
    return o @ w[p + "o"].T, {"S": S}


def latent_scores_softmax(qn, qr, kn, kr, v, scale, pos0):
    """qn [T,H,D], qr [T,H,R], kn [S,H,D], kr [S,R], v [S,H,V]; query t sees keys 0..pos0+t."""
    s = (np.einsum("thd,shd->hts", qn, kn) + np.einsum("thr,sr->hts", qr, kr)) * scale
    T, S = s.shape[1:]
    s = np.where(np.arange(S)[None, None, :] <= pos0 + np.arange(T)[None, :, None], s, -np.inf)
    p = np.exp(s - s.max(-1, keepdims=True))
    p /= p.sum(-1, keepdims=True)
    return np.einsum("hts,shv->thv", p, v)


def mix_latent_attention(m, w, p, h, state, pos0, eps):
    H, D, R, V, C = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    T = h.shape[0]
    if state is None:
        state = {"c": np.zeros((0, C)), "kr": np.zeros((0, R))}
    cos, sin = rotation_tables(m["rot"], np.arange(pos0, pos0 + T))
    q = (h @ w[p + "q"].T).reshape(T, H, D + R)
    qn, qr = q[..., :D], rotate_pairs(q[..., D:], cos, sin, True)
    y = h @ w[p + "dkv"].T
    c = np.concatenate([state["c"], rms(y[:, :C], eps) * w[p + "dkv.norm"]])
    kr = np.concatenate([state["kr"], rotate_pairs(y[:, None, C:], cos, sin, True)[:, 0]])
    S = c.shape[0]
    kn, v = (c @ w[p + "uk"].T).reshape(S, H, D), (c @ w[p + "uv"].T).reshape(S, H, V)
    o = latent_scores_softmax(qn, qr, kn, kr, v, m["scale"], pos0)
    return o.reshape(T, H * V) @ w[p + "o"].T, {"c": c, "kr": kr}


def channel_decay(z, tau):
    """sigmoid(z)^(1 / tau)"""
    return np.exp(-softplus(-z) / tau)


def gla_recurrence(q, k, v, alpha, S):
    """q, k, alpha [T, H, D], v [T, H, V], S [H, D, V]: every key channel decays by its own factor, then the
    token is written, then the state is read."""
    o = np.empty(v.shape, F)
    S = S.copy()
    for t in range(q.shape[0]):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hij,hi->hj", S, q[t])
    return o, S


def mix_gla(m, w, p, h, state, pos0, eps):
    H, D, V = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    if state is None:
        state = {"S": np.zeros((H, D, V))}
    q = (h @ w[p + "q"].T).reshape(T, H, D) * D ** -0.5
    k, v = (h @ w[p + "k"].T).reshape(T, H, D), (h @ w[p + "v"].T).reshape(T, H, V)
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
    o, S = gla_recurrence(q, k, v, channel_decay(z, m["tau"]).reshape(T, H, D), state["S"])
    o = (rms(o, eps) * w[p + "norm"]).reshape(T, H * V) * silu(h @ w[p + "g"].T)
    return o @ w[p + "o"].T, {"S": S}


def window_softmax(q, k, v, scale, pos0, first, window):
    """q [T,H,D] at positions pos0.., k [S,G,D], v [S,G,V] at positions first..; query i sees key j when
    0 <= i - j < window (None: every j <= i)."""
    T, H, _ = q.shape
    S, G, V = v.shape
    rep = H // G
    back = (pos0 + np.arange(T))[:, None] - (first + np.arange(S))[None, :]
    seen = (back >= 0) & (back < (window if window else np.inf))
    o = np.empty((T, H, V), F)
    for h in range(H):
        s = np.where(seen, q[:, h] @ k[:, h // rep].T * scale, -np.inf)
        e = np.exp(s - s.max(-1, keepdims=True))
        o[:, h] = (e / e.sum(-1, keepdims=True)) @ v[:, h // rep]
    return o


def mix_window_attention(m, w, p, h, state, pos0, eps):
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    if state is None:
        state = {"k": np.zeros((0, G, D)), "v": np.zeros((0, G, V)), "first": 0}
    cos, sin = rotation_tables(m["rot"], np.arange(pos0, pos0 + T))
    q = rms(rotate_pairs((h @ w[p + "q"].T).reshape(T, H, D), cos, sin, True), eps)
    k = rms(rotate_pairs((h @ w[p + "k"].T).reshape(T, G, D), cos, sin, True), eps)
    k, v = np.concatenate([state["k"], k]), np.concatenate([state["v"], (h @ w[p + "v"].T).reshape(T, G, V)])
    o = window_softmax(q, k, v, m["scale"], pos0, state["first"], (m.get("mask") or {}).get("size"))
    o = o * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, H * V) @ w[p + "o"].T, {"k": k, "v": v, "first": state["first"]}


def short_convolution(x, last, taps):
    """x [T, C], last [n - 1, C] the inputs before them, taps [C, n] (last column: the current input)."""
    n = taps.shape[1]
    z = np.concatenate([last, x])
    y = np.zeros(x.shape, F)
    for t in range(x.shape[0]):
        for j in range(n):
            y[t] += taps[:, j] * z[t + j]
    return y, z[len(z) - (n - 1):].copy()


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def delta_recurrence(q, k, v, g, beta, S):
    """q, k [T, H, D], v [T, H, V], g, beta [T, H], S [H, D, V]: decay, write what the state does not yet
    answer to k, read."""
    o = np.empty(v.shape, F)
    S = S.copy()
    for t in range(q.shape[0]):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - np.einsum("hij,hi->hj", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = np.einsum("hij,hi->hj", S, q[t])
    return o, S


def mix_delta(m, w, p, h, state, pos0, eps):
    H, G, D, V, n = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
    T = h.shape[0]
    if state is None:
        state = {"S": np.zeros((H, D, V)), **{c: np.zeros((n - 1, G * D if c in "qk" else H * V)) for c in "qkv"}}
    new, x = {}, {}
    for c in "qkv":
        y, new[c] = short_convolution(h @ w[p + c].T, state[c], w[p + c + ".conv"])
        x[c] = silu(y)
    rep = np.arange(H) // (H // G)
    q = (unit(x["q"].reshape(T, G, D)) * D ** -0.5)[:, rep]
    k = unit(x["k"].reshape(T, G, D))[:, rep]
    beta = sigmoid(h @ w[p + "b"].T)
    g = np.exp(-np.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    o, new["S"] = delta_recurrence(q, k, x["v"].reshape(T, H, V), g, beta, state["S"])
    o = rms(o, eps) * w[p + "norm"] * silu(h @ w[p + "g"].T).reshape(T, H, V)
    return o.reshape(T, H * V) @ w[p + "o"].T, new


def mix_parallel(m, w, p, h, state, pos0, eps):
    a, b = state or (None, None)
    left, a = mix_window_attention(m["left"], w, p + "left.", h, a, pos0, eps)
    right, b = mix_delta(m["right"], w, p + "right.", h, b, pos0, eps)
    return m["left_scale"] * left + m["right_scale"] * right, (a, b)


MIXERS = {"wkv": mix_wkv, "retention": mix_retention, "latent_attention": mix_latent_attention, "gla": mix_gla, "parallel": mix_parallel}


def feed_forward(w, p, h, act=gelu_tanh):
    return (act(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


# ---- the stack ---------------------------------------------------------------------------------
def runs(cfg):
    """(layer, adds_embedding) of every layer run in order."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b, times = loop["start"], loop["stop"], loop["times"]
    out = [(i, False) for i in range(a)]
    for t in range(times):
        out += [(i, t > 0 and i == a) for i in range(a, b)]
    return out + [(i, False) for i in range(b, n)]


class Model:
    """`forward(tokens)` continues the sequence and returns the logits of the new tokens; the states
    of every layer run are kept.  `trace` collects the residual stream after every run when set."""

    def __init__(self, cfg, weights):
        self.cfg = cfg
        self.w = {k: np.asarray(v, F) for k, v in weights.items()}
        self.reset()

    def reset(self):
        self.pos, self.states, self.trace = 0, {}, None

    def forward(self, tokens):
        if self.cfg["architecture"] == "Dutivik":
            return self.forward_parallel(tokens)
        cfg, w = self.cfg, self.w
        eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
        e = w["embed"][np.asarray(tokens, int)]
        x = e.copy()
        for j, (i, again) in enumerate(runs(cfg)):
            ly, p = cfg["layers"][i], f"l{i}."
            if again:
                x = x + e
            y, self.states[j] = MIXERS[ly["type"]](ly["mixer"], w, p + "mix.", norm_about_zero(x, w[p + "norm1"], eps), self.states.get(j), self.pos, eps)
            x = x + m * norm_about_zero(y, w[p + "norm1b"], eps)
            if ly.get("mlp"):
                y = feed_forward(w, p + "mlp.", norm_about_zero(x, w[p + "norm2"], eps))
                x = x + m * norm_about_zero(y, w[p + "norm2b"], eps)
            if self.trace is not None:
                self.trace.append(x.copy())
        self.pos += len(tokens)
        self.hidden = x
        return norm_about_zero(x, w["final.norm"], eps) @ w["embed"].T

    def forward_parallel(self, tokens):
        """One norm per layer; the mixer and the feed-forward both read it.  A layer may use another one's weights."""
        cfg, w = self.cfg, self.w
        eps = cfg["norm"]["eps"]
        x = w["embed"][np.asarray(tokens, int)] * cfg["embedding"]["scale"]
        for i, ly in enumerate(cfg["layers"]):
            p = f"l{ly.get('weights_of', i)}."
            h = layer_norm(x, w[p + "norm1"], w[p + "norm1.b"], eps)
            y, self.states[i] = MIXERS[ly["type"]](ly["mixer"], w, p + "mix.", h, self.states.get(i), self.pos, eps)
            if ly.get("mlp"):
                y = y + feed_forward(w, p + "mlp.", h, silu)
            x = x + y
            if self.trace is not None:
                self.trace.append(x.copy())
        self.pos += len(tokens)
        self.hidden = x
        return layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["embed"].T
