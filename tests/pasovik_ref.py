"""A plain, slow restatement of the Pasovik design in numpy (float64), one function per mechanism.

It keeps no cache: every function sees whole sequences, and a sequence is computed from its first token on. Weights are a
dict name -> float array, the configuration is the dict config.json holds. Nothing here is shared with the product.
"""
from __future__ import annotations

import numpy as np


def rms_norm(x, w, eps):
    """Along the last axis: x over the root of (mean of squares + eps), times w."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def rotate(x, rot):
    """x [time, ..., size]: neighbours (2 i, 2 i + 1) of the first rot.dims entries turn by the position times the pair's frequency."""
    out = np.array(x, float)
    scaling = rot.get("scaling")
    pos = np.arange(x.shape[0]).reshape((-1,) + (1,) * (x.ndim - 2))
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        if scaling:
            f = f / scaling["factor"]
        c, s = np.cos(pos * f), np.sin(pos * f)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def soften(score, cap):
    return cap * np.tanh(score / cap)


def causal(q, k, v, scale, cap=None):
    """q [time, H, dim], k [time, G, dim], v [time, G, vdim] -> [time, H, vdim]: every position over itself and all before it."""
    time, heads, _ = q.shape
    per = heads // k.shape[1]
    out = np.zeros((time, heads, v.shape[2]))
    for h in range(heads):
        s = q[:, h] @ k[:, h // per].T * scale
        if cap:
            s = soften(s, cap)
        s = np.where(np.tri(time, dtype=bool), s, -np.inf)
        p = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = p / p.sum(axis=1, keepdims=True) @ v[:, h // per]
    return out


def attention_heads(x, w, pre, m, eps):
    n = len(x)
    q = rotate(rms_norm((x @ w[pre + "q"].T).reshape(n, m["heads"], m["dim"]), w[pre + "q.norm"], eps), m["rot"])
    k = rotate(rms_norm((x @ w[pre + "k"].T).reshape(n, m["kv_heads"], m["dim"]), w[pre + "k.norm"], eps), m["rot"])
    v = (x @ w[pre + "v"].T).reshape(n, m["kv_heads"], m["vdim"])
    return causal(q, k, v, m["scale"], m["softcap"]).reshape(n, -1)


def attention(x, w, pre, m, eps):
    return attention_heads(x, w, pre, m, eps) @ w[pre + "o"].T


def latent_rows(x, w, pre, m, eps):
    """What a latent layer keeps of every position: the normed latent and the rotated part of its key."""
    c, r = np.split(x @ w[pre + "dkv"].T, [m["kv_rank"]], axis=1)
    return rms_norm(c, w[pre + "dkv.norm"], eps), rotate(r, m["rot"])


def latent_heads(x, w, pre, m, eps, kept):
    n, H = len(x), m["heads"]
    c, r = kept
    q = (rms_norm(x @ w[pre + "dq"].T, w[pre + "dq.norm"], eps) @ w[pre + "uq"].T).reshape(n, H, m["dim"] + m["rot_dim"])
    q = np.concatenate([q[..., :m["dim"]], rotate(q[..., m["dim"]:], m["rot"])], axis=-1)
    k = np.concatenate([(c @ w[pre + "uk"].T).reshape(n, H, m["dim"]), np.repeat(r[:, None], H, axis=1)], axis=-1)
    v = (c @ w[pre + "uv"].T).reshape(n, H, m["vdim"])
    return causal(q, k, v, m["scale"]).reshape(n, -1) * sigmoid(x @ w[pre + "g"].T)


def latent_attention(x, w, pre, m, eps, kept):
    return latent_heads(x, w, pre, m, eps, kept) @ w[pre + "o"].T


def lightning_core(q, k, v, decay):
    """q, k [time, H, dim], v [time, H, vdim]: the state fades, takes the token in, and is read."""
    S, out = np.zeros((q.shape[1], q.shape[2], v.shape[2])), np.zeros_like(v)
    for t in range(len(q)):
        S = np.asarray(decay)[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hkv,hk->hv", S, q[t])
    return out


def lightning(x, w, pre, m, eps):
    n, H = len(x), m["heads"]
    q, k, v = (silu(x @ w[pre + c].T).reshape(n, H, -1) for c in "qkv")
    o = rms_norm(lightning_core(q, k, v, m["decay"]).reshape(n, -1), w[pre + "norm"], eps)
    return (o * sigmoid(x @ w[pre + "g"].T)) @ w[pre + "o"].T


def dense(x, w, pre):
    return (silu(x @ w[pre + "gate"].T) * (x @ w[pre + "up"].T)) @ w[pre + "down"].T


def expert(x, w, pre, limit):
    g, u = np.minimum(x @ w[pre + "gate"].T, limit), np.clip(x @ w[pre + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[pre + "down"].T


def chosen(x, w, pre, m):
    """Per token: the experts with the largest scores, and those scores."""
    s = sigmoid(x @ w[pre + "router"].T)
    ids = np.argsort(-s, axis=1, kind="stable")[:, :m["router"]["top"]]
    return ids, np.take_along_axis(s, ids, axis=1)


def experts(x, w, pre, m):
    ids, s = chosen(x, w, pre, m)
    y = np.zeros_like(x)
    for t in range(len(x)):
        for e, weight in zip(ids[t], s[t]):
            y[t] += expert(weight * x[t:t + 1], w, f"{pre}e{e}.", m["expert"]["limit"])[0]
    return y


def side_input(x, w, i, tokens, dim, eps):
    """What a layer adds that comes from its own part of the tokens' side embedding."""
    e = w["side.embed"][np.asarray(tokens)][:, i * dim:(i + 1) * dim]
    g = gelu_tanh(x @ w[f"l{i}.side.gate"].T) * e
    return rms_norm(g @ w[f"l{i}.side.proj"].T, w[f"l{i}.side.norm"], eps)


def mixer(x, w, i, cfg, kept):
    lc, eps, pre = cfg["layers"][i], cfg["norm"]["eps"], f"l{i}.mix."
    m = lc["mixer"]
    if lc["type"] == "attention":
        return attention(x, w, pre, m, eps)
    if lc["type"] == "lightning":
        return lightning(x, w, pre, m, eps)
    if m.get("kv_from") is None:
        kept[i] = latent_rows(x, w, pre, m, eps)
    return latent_attention(x, w, pre, m, eps, kept[i if m.get("kv_from") is None else m["kv_from"]])


def layer(x, w, i, cfg, tokens, kept):
    """kept: layer -> what latent layers have kept, filled here."""
    eps, mlp = cfg["norm"]["eps"], cfg["layers"][i].get("mlp")
    x = x + rms_norm(mixer(x, w, i, cfg, kept), w[f"l{i}.norm1"], eps)
    if mlp:
        f = dense(x, w, f"l{i}.mlp.") if mlp["kind"] == "dense" else experts(x, w, f"l{i}.mlp.", mlp)
        x = x + rms_norm(f, w[f"l{i}.norm2"], eps)
    return x + side_input(x, w, i, tokens, cfg["token_side"]["dim"], eps)


def forward(cfg, w, tokens):
    """-> logits [time, vocab] and the residual stream after every layer."""
    x, runs, kept = w["embed"][np.asarray(tokens)], [], {}
    for i in range(len(cfg["layers"])):
        x = layer(x, w, i, cfg, tokens, kept)
        runs.append(x)
    return rms_norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T, runs
