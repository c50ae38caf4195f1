"""A plain, slow restatement of the Lonasun design in numpy (float64), one function per mechanism.

It keeps no cache: every function sees whole sequences, and a sequence is computed from its first token on. Weights are a
dict name -> float array, the configuration is the dict config.json holds. Nothing here is shared with the product.
"""
from __future__ import annotations

import numpy as np


def rms_norm(x, w, eps):
    """x over its root mean square (eps under the root), times 1 + w."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * (1.0 + w)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def short_conv(u, taps):
    """u [time, channels], taps [channels, n]: y[t, c] = sum_j taps[c, j] u[t - n + 1 + j, c], zeros before the start."""
    n = taps.shape[1]
    y = np.zeros_like(u)
    for t in range(u.shape[0]):
        for j in range(n):
            s = t - n + 1 + j
            if s >= 0:
                y[t] += taps[:, j] * u[s]
    return y


def rotate(x, positions, base, dims):
    """x [time, heads, dim]: dimensions i and i + dims / 2 of the first `dims` turn by position * base^(-2 i / dims)."""
    half = dims // 2
    out = x.copy()
    for i in range(half):
        a = positions * float(base) ** (-2.0 * i / dims)
        c, s = np.cos(a)[:, None], np.sin(a)[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        out[:, :, i] = u * c - v * s
        out[:, :, i + half] = v * c + u * s
    return out


def chunked_attention(q, k, v, scale, size):
    """q [time, H, dim], k [time, G, dim], v [time, G, vdim]: causal, within position blocks of `size`; -> [time, H, vdim]."""
    time, heads, _ = q.shape
    per = heads // k.shape[1]
    out = np.zeros((time, heads, v.shape[2]))
    for t in range(time):
        lo = t // size * size
        for h in range(heads):
            g = h // per
            s = (k[lo:t + 1, g] @ q[t, h]) * scale
            p = np.exp(s - s.max())
            out[t, h] = (p / p.sum()) @ v[lo:t + 1, g]
    return out


def attention_mixer(h, w, pre, m, first=0):
    """The mixer on its normed input h [time, width]; `pre` is the tensors' prefix, `m` the layer's sizes."""
    time = h.shape[0]
    n_q, n_kv, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    proj = {c: short_conv(h @ w[pre + c].T, w[pre + c + ".conv"]) for c in "qkv"}
    pos = np.arange(first, first + time, dtype=np.float64)
    q = rotate(proj["q"].reshape(time, n_q, dim), pos, m["rot"]["base"], m["rot"]["dims"])
    k = rotate(proj["k"].reshape(time, n_kv, dim), pos, m["rot"]["base"], m["rot"]["dims"])
    o = chunked_attention(q, k, proj["v"].reshape(time, n_kv, vdim), m["scale"], m["mask"]["size"])
    return (o.reshape(time, n_q * vdim) * sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T


def expert(h, up, down):
    return np.square(np.maximum(h @ up.T, 0.0)) @ down.T


def route(h, router, correction, top):
    """-> chosen experts and their weights, [time, top] each: chosen by score + correction, weighted by the scores alone."""
    z = h @ router.T
    e = np.exp(z - z.max(axis=1, keepdims=True))
    s = e / e.sum(axis=1, keepdims=True)
    ids = np.argsort(-(s + correction), axis=1, kind="stable")[:, :top]
    wt = np.take_along_axis(s, ids, axis=1)
    return ids, wt / (wt.sum(axis=1, keepdims=True) + 1e-20)


def moe(h, w, pre, m):
    n_exp = m["router"]["experts"]
    ids, wt = route(h, w[pre + "router"], w[pre + "correction"], m["router"]["top"])
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for i, g in zip(ids[t], wt[t]):
            out[t] += g * (h[t] if i >= n_exp else expert(h[t:t + 1], w[f"{pre}e{i}.up"], w[f"{pre}e{i}.down"])[0])
    if m.get("shared"):
        out += expert(h, w[pre + "shared.up"], w[pre + "shared.down"])
    return out


def layer(x, w, i, lc, eps):
    x = x + attention_mixer(rms_norm(x, w[f"l{i}.norm1"], eps), w, f"l{i}.mix.", lc["mixer"])
    if lc.get("mlp"):
        x = x + moe(rms_norm(x, w[f"l{i}.norm2"], eps), w, f"l{i}.mlp.", lc["mlp"])
    return x


def layer_order(cfg):
    """(layer, whether a loop pass begins with it) in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return ([(i, False) for i in range(a)] + [(i, i == a) for _ in range(loop["times"]) for i in range(a, b)] + [(i, False) for i in range(b, n)])


def forward(cfg, w, tokens):
    """-> logits [time, vocab] and the residual stream after every layer run."""
    eps = cfg["norm"]["eps"]
    x0 = w["embed"][np.asarray(tokens)]
    x, runs = x0, []
    for i, begins in layer_order(cfg):
        if begins:
            x = np.concatenate([x, x0], axis=1) @ w["loop.in"].T
        x = layer(x, w, i, cfg["layers"][i], eps)
        runs.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T, runs
