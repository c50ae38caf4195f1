"""A plain, slow restatement of the Leduvik design in numpy (float64), one function per mechanism.

It keeps no cache: every function sees whole sequences, and a sequence is computed from its first token on. Weights are a
dict name -> float array, the configuration is the dict config.json holds. Nothing here is shared with the product.
"""
from __future__ import annotations

import numpy as np


def unit_rms(x, eps):
    """x over the root of (mean of squares + eps), along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def temperature(pos, coef, every):
    """How much longer the query of position `pos` gets: 1 + coef ln(floor((pos + 1) / every) + 1)."""
    return 1.0 + coef * np.log(np.floor((pos + 1) / every) + 1.0)


def attend(q, k, v, scale, window=None):
    """q [time, H, dim], k [time, G, dim], v [time, G, vdim]: softmax over the visible past -- all of it, or the last `window`
    positions with one's own; -> [time, H, vdim]."""
    time, heads, _ = q.shape
    per = heads // k.shape[1]
    out = np.zeros((time, heads, v.shape[2]))
    for t in range(time):
        lo = 0 if window is None else max(0, t - window + 1)
        for h in range(heads):
            s = (k[lo:t + 1, h // per] @ q[t, h]) * scale
            p = np.exp(s - s.max())
            out[t, h] = (p / p.sum()) @ v[lo:t + 1, h // per]
    return out


def projected_heads(h, w, pre, m):
    n = h.shape[0]
    return ((h @ w[pre + "q"].T).reshape(n, m["heads"], m["dim"]), (h @ w[pre + "k"].T).reshape(n, m["kv_heads"], m["dim"]),
            (h @ w[pre + "v"].T).reshape(n, m["kv_heads"], m["vdim"]))


def window_attention(h, w, pre, m, eps):
    """Heads of unit length, no positions in the scores, the last mask.size positions."""
    q, k, v = projected_heads(h, w, pre, m)
    o = attend(unit_rms(q, eps), unit_rms(k, eps), v, m["scale"], m["mask"]["size"])
    return o.reshape(len(h), -1) @ w[pre + "o"].T


def tempered_attention(h, w, pre, m):
    """All positions, queries longer with the position."""
    q, k, v = projected_heads(h, w, pre, m)
    t = temperature(np.arange(len(h)), m["q_temp"]["coef"], m["q_temp"]["every"])
    o = attend(q * t[:, None, None], k, v, m["scale"])
    return o.reshape(len(h), -1) @ w[pre + "o"].T


def time_mix_core(r, k, v, w, u):
    """r, k, w [time, H, n], v [time, H, n], u [H, n]: the recurrence, read before the token is added, with a bonus for it."""
    time, heads, n = r.shape
    out = np.zeros((time, heads, v.shape[2]))
    for h in range(heads):
        S = np.zeros((n, v.shape[2]))
        for t in range(time):
            kv = np.outer(k[t, h], v[t, h])
            out[t, h] = (S + u[h][:, None] * kv).T @ r[t, h]
            S = w[t, h][:, None] * S + kv
    return out


def token_shift(h, mu):
    """Each row moved towards the row before it (zeros before the first)."""
    before = np.concatenate([np.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mu


def time_mixing(h, w, pre, m, eps):
    n, shape = len(h), (len(h), m["heads"], m["dim"])
    mix = {c: token_shift(h, w[pre + "mu." + c]) for c in "rkvgw"}
    r, k, v = ((mix[c] @ w[pre + c].T).reshape(shape) for c in "rkv")
    gate = silu(mix["g"] @ w[pre + "g"].T)
    decay = np.exp(-np.exp(np.tanh(mix["w"] @ w[pre + "w1"].T) @ w[pre + "w2"].T + w[pre + "w0"])).reshape(shape)
    o = unit_rms(time_mix_core(r, k, v, decay, w[pre + "u"]), eps)
    return (o.reshape(n, -1) * w[pre + "norm"] * gate) @ w[pre + "o"].T


def parallel(h, w, pre, m, eps):
    left = unit_rms(tempered_attention(h, w, pre + "left.", m["left"]), eps) * w[pre + "left.out"]
    right = unit_rms(time_mixing(h, w, pre + "right.", m["right"], eps), eps) * w[pre + "right.out"]
    return 0.5 * (left + right)


def causal_conv(u, taps, bias):
    """u [time, channels], taps [channels, n], the last tap on the row itself, zeros before the start."""
    n = taps.shape[1]
    y = np.zeros_like(u) + bias
    for t in range(u.shape[0]):
        for j in range(n):
            if t - n + 1 + j >= 0:
                y[t] += taps[:, j] * u[t - n + 1 + j]
    return y


def state_space_core(x, B, C, dt, a_log, D):
    """x [time, H, vdim], B, C [time, G, N], dt [time, H]: S = exp(-exp(a_log) dt) S + dt B x^T; y = S^T C + D x."""
    time, heads, vdim = x.shape
    per = heads // B.shape[1]
    y = np.zeros_like(x)
    for h in range(heads):
        S = np.zeros((B.shape[2], vdim))
        for t in range(time):
            S = np.exp(-np.exp(a_log[h]) * dt[t, h]) * S + dt[t, h] * np.outer(B[t, h // per], x[t, h])
            y[t, h] = S.T @ C[t, h // per] + D[h] * x[t, h]
    return y


def state_space(h, w, pre, m, eps):
    n, inner, N, G = len(h), m["heads"] * m["vdim"], m["state"], m["groups"]
    z, xbc, dt = np.split(h @ w[pre + "in"].T, [inner, 2 * inner + 2 * G * N], axis=1)
    x, B, C = np.split(silu(causal_conv(xbc, w[pre + "conv"], w[pre + "conv.b"])), [inner, inner + G * N], axis=1)
    y = state_space_core(x.reshape(n, m["heads"], m["vdim"]), B.reshape(n, G, N), C.reshape(n, G, N), softplus(dt + w[pre + "dt_bias"]), w[pre + "A_log"], w[pre + "D"])
    y = unit_rms((y.reshape(n, inner) * silu(z)).reshape(n, m["norm_groups"], -1), eps).reshape(n, inner)
    return (y * w[pre + "norm"]) @ w[pre + "o"].T


def feed_forward(h, w, pre):
    return np.square(np.maximum(h @ w[pre + "up"].T, 0.0)) @ w[pre + "down"].T


def mixer(h, w, i, lc, eps):
    pre, m = f"l{i}.mix.", lc["mixer"]
    if lc["type"] == "attention":
        return window_attention(h, w, pre, m, eps)
    if lc["type"] == "mamba2":
        return state_space(h, w, pre, m, eps)
    return parallel(h, w, pre, m, eps)


def layer(x, w, i, lc, eps):
    x = x + mixer(unit_rms(x, eps) * w[f"l{i}.norm1"], w, i, lc, eps)
    if lc.get("mlp"):
        x = x + feed_forward(unit_rms(x, eps) * w[f"l{i}.norm2"], w, f"l{i}.mlp.")
    return x


def layer_order(cfg):
    """(layer, whether the embedding output is added first) in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return ([(i, False) for i in range(a)] + [(i, i == a and t > 0) for t in range(loop["times"]) for i in range(a, b)] + [(i, False) for i in range(b, n)])


def embedding(w, tokens):
    return w["embed"][np.asarray(tokens)] + w["pos"][:len(tokens)]


def forward(cfg, w, tokens):
    """-> logits [time, vocab] and the residual stream after every layer run."""
    eps = cfg["norm"]["eps"]
    x0 = embedding(w, tokens)
    x, runs = x0, []
    for i, again in layer_order(cfg):
        x = layer(x + x0 if again else x, w, i, cfg["layers"][i], eps)
        runs.append(x)
    return (unit_rms(x, eps) * w["final.norm"]) @ w["head"].T * cfg["logit_scale"], runs
