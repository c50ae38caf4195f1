"""A plain, slow restatement of the Sopetar design in numpy (float64), one function per mechanism.

It keeps no cache: every function sees whole sequences, and a sequence is computed from its first token on. Weights are a
dict name -> float array, the configuration is the dict config.json holds. Nothing here is shared with the product.
"""
from __future__ import annotations

import numpy as np


def over_rms(x, eps):
    """Along the last axis: x over the root of (mean of squares + eps)."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def layer_norm(x, w, b, eps):
    d = x - x.mean(axis=-1, keepdims=True)
    return d / np.sqrt(np.mean(d * d, axis=-1, keepdims=True) + eps) * w + b


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def rotate(x, rot):
    """x [time, ..., size]: neighbours (2 i, 2 i + 1) of the first rot.dims entries turn by the position times the pair's frequency."""
    out = np.array(x, float)
    pos = np.arange(x.shape[0]).reshape((-1,) + (1,) * (x.ndim - 2))
    for i in range(rot["dims"] // 2):
        a = pos * rot["base"] ** (-2.0 * i / rot["dims"])
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a)
    return out


def visible(time, mask):
    """[query, key]: the last mask.size positions, and the first mask.keep_first of the sequence."""
    i, j = np.arange(time)[:, None], np.arange(time)[None, :]
    return (j <= i) & ((i - j < mask["size"]) | (j < mask.get("keep_first", 0)))


def soften(score, cap):
    return cap * np.tanh(score / cap)


def slopes(heads):
    return 2.0 ** (-8.0 * np.arange(1, heads + 1) / heads)


def farther(score, slope):
    """What distance costs: slope times (query's position - key's)."""
    i, j = np.indices(score.shape)
    return score - slope * (i - j)


def weights(score, seen, sink=None):
    """Softmax over the keys seen; sink: a logit that takes its share and has no value."""
    s = np.where(seen, score, -np.inf)
    top = s.max(axis=1, keepdims=True) if sink is None else np.maximum(s.max(axis=1, keepdims=True), sink)
    p = np.exp(s - top)
    return p / (p.sum(axis=1, keepdims=True) + (0.0 if sink is None else np.exp(sink - top)))


def attention_parts(x, w, pre, m, eps):
    """q, k, v [time, heads, size] before values are mixed."""
    n = len(x)
    q, k, v = (x @ w[pre + c].T + w[pre + c + ".b"] for c in "qkv")
    q = over_rms(q.reshape(n, m["heads"], m["dim"]), eps)
    k = over_rms(k.reshape(n, m["kv_heads"], m["dim"]), eps)
    return q, k, over_rms(v.reshape(n, m["kv_heads"], m["vdim"]), eps)


def mix_values(v, first, share):
    return (1.0 - share) * v + share * first


def attention_core(q, k, v, m):
    """-> [time, H, vdim]."""
    n, H, _ = q.shape
    per, seen, slope = H // k.shape[1], visible(n, m["mask"]), slopes(H)
    out = np.zeros((n, H, v.shape[2]))
    for h in range(H):
        s = farther(soften(q[:, h] @ k[:, h // per].T * m["scale"], m["softcap"]), slope[h])
        out[:, h] = weights(s, seen) @ v[:, h // per]
    return out


def attention_heads(x, w, pre, m, eps, kept):
    """kept['v']: the values of the first layer that mixes them, written there by that layer."""
    q, k, v = attention_parts(x, w, pre, m, eps)
    if m.get("v_mix"):
        if "v" in kept:
            v = mix_values(v, kept["v"], w[pre + "vmix"])
        else:
            kept["v"] = v
    return attention_core(q, k, v, m).reshape(len(x), -1)


def latent_rows(x, w, pre, m, eps):
    """What a latent layer keeps of every position: the normed latent and the rotated part of its key."""
    c, r = np.split(x @ w[pre + "dkv"].T, [m["kv_rank"]], axis=1)
    return over_rms(c, eps) * w[pre + "dkv.norm"], rotate(r, m["rot"])


def latent_heads(x, w, pre, m, eps):
    n, H = len(x), m["heads"]
    c, r = latent_rows(x, w, pre, m, eps)
    q = (x @ w[pre + "q"].T).reshape(n, H, m["dim"] + m["rot_dim"])
    turned = rotate(q[..., m["dim"]:], m["rot"])
    k = (c @ w[pre + "uk"].T).reshape(n, H, m["dim"])
    v = (c @ w[pre + "uv"].T).reshape(n, H, m["vdim"])
    seen, gate = visible(n, {"size": m["mask"]["size"]}), sigmoid(x @ w[pre + "g"].T)
    out = np.zeros((n, H, m["vdim"]))
    for h in range(H):
        s = (q[:, h, :m["dim"]] @ k[:, h].T + turned[:, h] @ r.T) * m["scale"]
        out[:, h] = weights(s, seen, w[pre + "sink"][h]) @ v[:, h] * gate[:, h:h + 1]
    return out.reshape(n, -1)


def heads(x, w, i, cfg, kept):
    """A mixer's heads side by side, before its output matrix."""
    lc, eps, pre = cfg["layers"][i], cfg["norm"]["eps"], f"l{i}.mix."
    if lc["type"] == "attention":
        return attention_heads(x, w, pre, lc["mixer"], eps, kept)
    return latent_heads(x, w, pre, lc["mixer"], eps)


def feed_forward(x, w, pre, limit):
    g = np.minimum(x @ w[pre + "gate"].T + w[pre + "gate.b"], limit)
    u = np.clip(x @ w[pre + "up"].T + w[pre + "up.b"], -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[pre + "down"].T + w[pre + "down.b"]


def layer(x, w, i, cfg, kept):
    """Both sublayers side by side on the same normed rows."""
    L, mlp = f"l{i}.", cfg["layers"][i].get("mlp")
    h = layer_norm(x, w[L + "norm1"], w[L + "norm1.b"], cfg["norm"]["eps"])
    y = heads(h, w, i, cfg, kept) @ w[L + "mix.o"].T
    if mlp:
        y = y + feed_forward(h, w, L + "mlp.", mlp["limit"])
    return x + y


def depth_average(results, share):
    return sum(s * x for s, x in zip(share, results))


def forward(cfg, w, tokens):
    """-> logits [time, vocab] and what goes on from every layer."""
    results, runs, kept = [w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]], [], {}
    x = results[0]
    for i in range(len(cfg["layers"])):
        results.append(layer(x, w, i, cfg, kept))
        x = depth_average(results, w[f"l{i}.dwa"])
        runs.append(x)
    return layer_norm(x, w["final.norm"], w["final.norm.b"], cfg["norm"]["eps"]) @ w["head"].T, runs
