"""Plain numpy statement of the Momedra design, one function per mechanism, float64 throughout.

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


def layer_norm(x, w, eps):
    d = x - x.mean(-1, keepdims=True)
    return d / np.sqrt((d * d).mean(-1, keepdims=True) + eps) * w


def rms_norm(x, w, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def softplus(z):
    return np.log1p(np.exp(-np.abs(z))) + np.maximum(z, 0.0)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def relu_squared(z):
    return np.maximum(z, 0.0) ** 2


def heads_of(x, n, d):
    """[T, n * d] -> [n, T, d]"""
    return x.reshape(x.shape[0], n, d).transpose(1, 0, 2)


def rotate_pairs(v, pos, dims, base):
    """v [..., T, n]: the first `dims` entries in neighbouring pairs, pair i turned by pos * base^(-2i / dims)"""
    out = np.array(v, dtype=np.float64, copy=True)
    a = np.asarray(pos, np.float64)[:, None] * (float(base) ** (-2.0 * np.arange(dims // 2) / dims))[None, :]
    u, w = v[..., 0:dims:2], v[..., 1:dims:2]
    out[..., 0:dims:2] = u * np.cos(a) - w * np.sin(a)
    out[..., 1:dims:2] = w * np.cos(a) + u * np.sin(a)
    return out


def causal_softmax(s, sink=None):
    """[T, T] scores -> weights over the keys j <= i; a sink adds exp(sink) to every denominator"""
    T = s.shape[0]
    m = np.tril(np.ones((T, T), bool))
    s = np.where(m, s, -np.inf)
    top = s.max(-1, keepdims=True)
    if sink is not None:
        top = np.maximum(top, sink)
    e = np.where(m, np.exp(s - top), 0.0)
    den = e.sum(-1, keepdims=True)
    if sink is not None:
        den = den + np.exp(sink - top)
    return e / den


def query_temperature(pos, t):
    """1 + coef ln(floor((p + 1) / every) + 1)"""
    if not t:
        return np.ones(len(pos))
    return 1.0 + t["coef"] * np.log(np.floor((np.asarray(pos, np.float64) + 1.0) / t["every"]) + 1.0)


# ------------------------------------------------------------------------------------------------------------ mixers
def attention(h, m, W, p, eps):
    """grouped-query; biased q / k / v; per-head norms of q and k; a temperature on q that grows with the position; one gate number a head"""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(heads_of(h @ W[p + "q"].T + W[p + "q.b"], H, d), W[p + "q.norm"], eps)
    k = rms_norm(heads_of(h @ W[p + "k"].T + W[p + "k.b"], G, d), W[p + "k.norm"], eps)
    v = heads_of(h @ W[p + "v"].T + W[p + "v.b"], G, dv)
    q = q * query_temperature(np.arange(T), m.get("q_temp"))[None, :, None]
    gate = sigmoid(h @ W[p + "g"].T)
    out = []
    for hh in range(H):
        g = hh // (H // G)
        out.append(causal_softmax(q[hh] @ k[g].T * m["scale"]) @ v[g] * gate[:, hh:hh + 1])
    return np.concatenate(out, -1) @ W[p + "o"].T


def latent_attention(h, m, W, p, eps):
    """keys and values from a normed latent, one rotated key part for all heads, queries straight from h, a sink per head"""
    T = h.shape[0]
    H, dn, dr, dv, rk = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(T)
    q = heads_of(h @ W[p + "q"].T, H, dn + dr)
    t = h @ W[p + "dkv"].T
    c = rms_norm(t[:, :rk], W[p + "dkv.norm"], eps)
    kr = rotate_pairs(t[:, rk:], pos, m["rot"]["dims"], m["rot"]["base"])
    qr = rotate_pairs(q[..., dn:], pos, m["rot"]["dims"], m["rot"]["base"])
    kn, v = heads_of(c @ W[p + "uk"].T, H, dn), heads_of(c @ W[p + "uv"].T, H, dv)
    out = [causal_softmax((q[hh, :, :dn] @ kn[hh].T + qr[hh] @ kr.T) * m["scale"], W[p + "sink"][hh]) @ v[hh] for hh in range(H)]
    return np.concatenate(out, -1) @ W[p + "o"].T


def causal_conv(u, w, b):
    """[T, C], w [C, taps] (last tap = the current token), zeros before the start"""
    T, taps = u.shape[0], w.shape[1]
    out = np.tile(np.asarray(b, np.float64), (T, 1))
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            out[back:] += u[:T - back] * w[:, j]
    return out


def gated_linear_recurrence(u, r, i, lam):
    """S_t = a S_(t-1) + sqrt(1 - a^2) i u from zero, log a = -8 r softplus(lam)"""
    la = -8.0 * r * softplus(lam)
    a, b = np.exp(la), np.sqrt(-np.expm1(2.0 * la)) * i * u
    S, out = np.zeros(u.shape[1]), np.empty_like(u)
    for t in range(u.shape[0]):
        S = a[t] * S + b[t]
        out[t] = S
    return out


def block_diagonal(u, M, b):
    """u [T, n * s], M [n, s, s] as [out, in], b [n, s]"""
    n, s = M.shape[0], M.shape[1]
    return np.concatenate([u[:, k * s:(k + 1) * s] @ M[k].T + b[k] for k in range(n)], -1)


def rglru(h, m, W, p):
    y = gelu_tanh(h @ W[p + "y"].T + W[p + "y.b"])
    u = causal_conv(h @ W[p + "x"].T + W[p + "x.b"], W[p + "conv"], W[p + "conv.b"])
    r = sigmoid(block_diagonal(u, W[p + "ra"], W[p + "ra.b"]))
    i = sigmoid(block_diagonal(u, W[p + "ri"], W[p + "ri.b"]))
    return (gated_linear_recurrence(u, r, i, W[p + "lam"]) * y) @ W[p + "o"].T


# ------------------------------------------------------------------------------------------------------------ feed-forwards
def unit(h, W, p):
    return relu_squared(h @ W[p + "up"].T) @ W[p + "down"].T


def route(z, top):
    """[T, E] logits -> [T, E] weights: soft-max over the `top` largest logits, zero elsewhere"""
    out = np.zeros_like(z)
    for t in range(z.shape[0]):
        best = np.argsort(-z[t], kind="stable")[:top]
        e = np.exp(z[t, best] - z[t, best].max())
        out[t, best] = e / e.sum()
    return out


def mixture(h, f, W, p):
    w = route(h @ W[p + "router"].T + W[p + "router.b"], f["router"]["top"])
    y = sum(w[:, e:e + 1] * unit(h, W, p + f"e{e}.") for e in range(f["router"]["experts"]))
    return y + unit(h, W, p + "shared.") if f.get("shared") else y


# ------------------------------------------------------------------------------------------------------------ the model
def layer_runs(cfg):
    """[(layer, does this run open a pass)]"""
    n = len(cfg["layers"])
    lp = cfg.get("loop") or {"start": 0, "stop": 0, "times": 1}
    a, b = lp["start"], lp["stop"]
    return [(i, False) for i in range(a)] + [(i, i == a) for _ in range(lp["times"] if b > a else 0) for i in range(a, b)] + [(i, False) for i in range(b, n)]


def layer(x, l, W, i, eps, mult):
    p = f"l{i}."
    h = layer_norm(x, W[p + "norm1"], eps)
    kind = l["type"]
    if kind == "attention":
        y = attention(h, l["mixer"], W, p + "mix.", eps)
    elif kind == "latent_attention":
        y = latent_attention(h, l["mixer"], W, p + "mix.", eps)
    elif kind == "rglru":
        y = rglru(h, l["mixer"], W, p + "mix.")
    else:
        raise ValueError(kind)
    f = l.get("mlp")
    if f is not None:
        y = y + (unit(h, W, p + "mlp.") if f["kind"] == "dense" else mixture(h, f, W, p + "mlp."))
    return x + mult * y


def forward(cfg, W, tokens, taps=None):
    """tokens [T] -> logits [T, vocab]; taps (a list) receives the residual stream after every layer run"""
    eps = cfg["norm"]["eps"]
    W = {k: np.asarray(v, np.float64) for k, v in W.items()}
    x0 = W["embed"][np.asarray(tokens)]
    x = x0
    for i, opens in layer_runs(cfg):
        if opens:
            x = np.concatenate([x, x0], -1) @ W["loop.in"].T
        x = layer(x, cfg["layers"][i], W, i, eps, cfg["residual_mult"])
        if taps is not None:
            taps.append(x)
    return layer_norm(x, W["final.norm"], eps) @ W["head"].T
