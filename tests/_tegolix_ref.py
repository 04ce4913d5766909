"""Plain numpy statement of the Tegolix design, one function per mechanism, float64 throughout.

It keeps no cache and no state: every function sees the whole sequence.  It shares no code with the product path; the tests
compare the CUDA executor with it.

A model is (cfg, W): cfg the dictionary of config.json, W a dictionary name -> float array (bfloat16 values widened).
"""
from __future__ import annotations

import numpy as np


# ------------------------------------------------------------------------------------------------------------ small pieces
def bf16_round(a):
    """round to the nearest bfloat16 value (ties to even), returned as float32"""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32).astype(np.uint64)
    u = (u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000
    return u.astype(np.uint32).view(np.float32).reshape(np.shape(a))


def unit_rms(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def offset_norm(x, w, eps):
    """the weight is stored around zero"""
    return unit_rms(x, eps) * (1.0 + w)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.log1p(np.exp(-np.abs(z))) + np.maximum(z, 0.0)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def heads_of(x, n, d):
    """[T, n * d] -> [n, T, d]"""
    return x.reshape(x.shape[0], n, d).transpose(1, 0, 2)


def flat(x):
    """[n, T, d] -> [T, n * d]"""
    return x.transpose(1, 0, 2).reshape(x.shape[1], -1)


# ------------------------------------------------------------------------------------------------------------ rotation
def yarn(dims, base, scaling):
    """frequencies [dims / 2] and the factor on cos and sin"""
    f = float(base) ** (-2.0 * np.arange(dims // 2) / dims)
    if not scaling:
        return f, 1.0

    def at(turns):
        return dims * np.log(scaling["original"] / (2.0 * np.pi * turns)) / (2.0 * np.log(base))

    lo, hi = max(np.floor(at(scaling["fast"])), 0.0), min(np.ceil(at(scaling["slow"])), dims - 1.0)
    ramp = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / scaling["factor"] * ramp + f * (1.0 - ramp), 0.1 * np.log(scaling["factor"]) + 1.0


def rotate_halves(v, angles, factor=1.0):
    """v [..., T, n]: entry i of the first 2 * angles.shape[1] is paired with the entry half of them further on; angles [T, pairs]"""
    out = np.array(v, dtype=np.float64, copy=True)
    n = angles.shape[1]
    c, s = np.cos(angles) * factor, np.sin(angles) * factor
    a, b = v[..., :n], v[..., n:2 * n]
    out[..., :n] = a * c - b * s
    out[..., n:2 * n] = b * c + a * s
    return out


# ------------------------------------------------------------------------------------------------------------ attention
def window_mask(T, size):
    d = np.arange(T)[:, None] - np.arange(T)[None, :]
    return (d >= 0) & (d < size)


def masked_softmax(s, m):
    s = np.where(m, s, -np.inf)
    e = np.exp(s - s.max(-1, keepdims=True))
    return e / e.sum(-1, keepdims=True)


def softcapped(s, cap):
    return cap * np.tanh(s / cap) if cap else s


def attention(h, m, W, p, eps):
    """windowed, soft-capped, q / k normed per head then rotated, values rotated by their own position and turned back by the query's, gated"""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rot, pos = m["rot"], np.arange(T, dtype=np.float64)[:, None]
    q = unit_rms(heads_of(h @ W[p + "q"].T, H, d), eps) * W[p + "q.norm"]
    k = unit_rms(heads_of(h @ W[p + "k"].T, G, d), eps) * W[p + "k.norm"]
    v = heads_of(h @ W[p + "v"].T, G, dv)
    f, factor = yarn(rot["dims"], rot["base"], rot.get("scaling"))
    q, k = rotate_halves(q, pos * f, factor), rotate_halves(k, pos * f, factor)
    fv, _ = yarn(dv, rot["base"], None)
    v = rotate_halves(v, pos * fv)
    gate = sigmoid(h @ W[p + "g"].T)
    mask = window_mask(T, m["mask"]["size"])
    out = []
    for hh in range(H):
        g = hh // (H // G)
        w = masked_softmax(softcapped(q[hh] @ k[g].T * m["scale"], m.get("softcap")), mask)
        out.append(rotate_halves(w @ v[g], -pos * fv) * gate[:, hh:hh + 1])
    return np.concatenate(out, -1) @ W[p + "o"].T


# ------------------------------------------------------------------------------------------------------------ recurrences
def time_mix_recurrence(r, k, v, w, u):
    """one head, [T, d] each: the current token counts with the bonus u, the past through the state"""
    S, out = np.zeros((k.shape[1], v.shape[1])), np.empty_like(v)
    for t in range(k.shape[0]):
        kv = np.outer(k[t], v[t])
        out[t] = (S + u[:, None] * kv).T @ r[t]
        S = w[t][:, None] * S + kv
    return out


def time_mix(h, m, W, p, eps):
    H, d = m["heads"], m["dim"]
    before = np.concatenate([np.zeros_like(h[:1]), h[:-1]])

    def mixed(s):
        return h + (before - h) * W[p + "mu." + s]

    r, k, v = (heads_of(mixed(s) @ W[p + s].T, H, d) for s in "rkv")
    gate = silu(mixed("g") @ W[p + "g"].T)
    w = heads_of(np.exp(-np.exp(np.tanh(mixed("w") @ W[p + "w1"].T) @ W[p + "w2"].T + W[p + "w0"])), H, d)
    o = np.stack([time_mix_recurrence(r[i], k[i], v[i], w[i], W[p + "u"][i]) for i in range(H)])
    return (flat(unit_rms(o, eps)) * W[p + "norm"] * gate) @ W[p + "o"].T


def gated_recurrence(q, k, v, alpha):
    """one head, [T, d] each: every key channel of the state decays by its own factor"""
    S, out = np.zeros((k.shape[1], v.shape[1])), np.empty_like(v)
    for t in range(k.shape[0]):
        S = alpha[t][:, None] * S + np.outer(k[t], v[t])
        out[t] = S.T @ q[t]
    return out


def gla(h, m, W, p, eps):
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q, k = heads_of(h @ W[p + "q"].T * d ** -0.5, H, d), heads_of(h @ W[p + "k"].T, H, d)
    v = heads_of(h @ W[p + "v"].T, H, dv)
    z = (h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "a2.b"]
    alpha = heads_of(np.exp(-softplus(-z) / m["tau"]), H, d)
    o = np.stack([gated_recurrence(q[i], k[i], v[i], alpha[i]) for i in range(H)])
    return (flat(unit_rms(o, eps) * W[p + "norm"]) * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


# ------------------------------------------------------------------------------------------------------------ feed-forwards
def unit(h, W, p, act):
    return (act(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def route(z, correction, top):
    """[T, E] logits -> [T, E] weights: soft-max scores of the `top` experts with the largest corrected scores, zero elsewhere"""
    e = np.exp(z - z.max(-1, keepdims=True))
    s = e / e.sum(-1, keepdims=True)
    out = np.zeros_like(s)
    for t in range(z.shape[0]):
        best = np.argsort(-(s[t] + correction), kind="stable")[:top]
        out[t, best] = s[t, best]
    return out


def mixture(h, f, W, p):
    E, I = f["router"]["experts"], f["router"].get("identity", 0)
    w = route(h @ W[p + "router"].T, W[p + "correction"], f["router"]["top"])
    y = sum(w[:, e:e + 1] * unit(h, W, p + f"e{e}.", silu) for e in range(E)) + w[:, E:E + I].sum(-1, keepdims=True) * h
    if f.get("shared"):
        y = y + sigmoid(h @ W[p + "shared.sg"].T) * unit(h, W, p + "shared.", silu)
    return y


# ------------------------------------------------------------------------------------------------------------ the model
def token_input(x, e, W, p, eps):
    g = gelu_tanh(x @ W[p + "gate"].T) * e
    return unit_rms(g @ W[p + "proj"].T, eps) * W[p + "norm"]


def mixer(h, l, W, p, eps):
    m = l["mixer"]
    if l["type"] == "gla":
        return gla(h, m, W, p, eps)
    if l["type"] == "parallel":
        return m["left_scale"] * attention(h, m["left"], W, p + "left.", eps) + m["right_scale"] * time_mix(h, m["right"], W, p + "right.", eps)
    raise ValueError(l["type"])


def layer(x, tokens, l, W, i, eps, side_dim):
    p = f"l{i}."
    x = x + W[p + "ls1"] * offset_norm(mixer(offset_norm(x, W[p + "norm1"], eps), l, W, p + "mix.", eps), W[p + "norm1b"], eps)
    f = l.get("mlp")
    if f is not None:
        h = offset_norm(x, W[p + "norm2"], eps)
        y = unit(h, W, p + "mlp.", lambda z: np.maximum(z, 0.0)) if f["kind"] == "dense" else mixture(h, f, W, p + "mlp.")
        x = x + W[p + "ls2"] * offset_norm(y, W[p + "norm2b"], eps)
    return x + token_input(x, W["side.embed"][tokens, i * side_dim:(i + 1) * side_dim], W, p + "side.", eps)


def forward(cfg, W, tokens, taps=None):
    """tokens [T] -> logits [T, vocab]; taps (a list) receives the residual stream after every layer"""
    eps, tokens = cfg["norm"]["eps"], np.asarray(tokens)
    W = {k: np.asarray(v, np.float64) for k, v in W.items()}
    x = W["embed"][tokens]
    for i, l in enumerate(cfg["layers"]):
        x = layer(x, tokens, l, W, i, eps, cfg["token_side"]["dim"])
        if taps is not None:
            taps.append(x)
    return offset_norm(x, W["final.norm"], eps) @ W["head"].T
