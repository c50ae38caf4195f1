"""Leduvik model folders (config.json, model.safetensors): tensor shapes and random-init weights, for tests and benchmarks. The
engine reads the folders itself (csrc/leduvik.h)."""
from __future__ import annotations

import numpy as np

from .folders import Pool, from_bf16, to_bf16, write_model  # noqa: F401  (callers take them from here)


def dense(ff):
    return {"kind": "dense", "ff": ff} if ff else None


def window(heads, kv_heads, dim, vdim, size, scale, ff=0) -> dict:
    """A layer of sliding-window attention; the layers are entries of config['layers']. ff 0: no feed-forward."""
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size}, "scale": scale}, "mlp": dense(ff)}


def state_space(heads, vdim, state, groups=1, norm_groups=1, conv=4, ff=0) -> dict:
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}, "mlp": dense(ff)}


def parallel(heads, kv_heads, dim, vdim, right_heads, right_dim, coef=0.2, every=100, scale=None, ff=0) -> dict:
    """Attention over all positions beside time mixing."""
    return {"type": "parallel", "mlp": dense(ff), "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "q_temp": {"coef": coef, "every": every}, "scale": dim ** -0.5 if scale is None else scale},
        "right": {"heads": right_heads, "dim": right_dim}}}


def config(width, vocab, layers, loop=None, eps=1e-5, max_positions=1024, logit_scale=1.0) -> dict:
    """loop: (start, stop, times) or None."""
    return {"architecture": "Leduvik", "width": width, "vocab": vocab, "layers": layers, "norm": {"eps": eps}, "max_positions": max_positions,
            "logit_scale": logit_scale, "loop": dict(zip(("start", "stop", "times"), loop)) if loop else None}


def shapes(cfg: dict, rank: int = 16) -> dict:
    """rank: of the decays' inner matrices, which the configuration does not name."""
    d = cfg["width"]
    out = {"embed": (cfg["vocab"], d), "pos": (cfg["max_positions"], d)}

    def attention(pre, m):
        out[pre + "q"] = (m["heads"] * m["dim"], d)
        out[pre + "k"] = (m["kv_heads"] * m["dim"], d)
        out[pre + "v"] = (m["kv_heads"] * m["vdim"], d)
        out[pre + "o"] = (d, m["heads"] * m["vdim"])

    for i, lc in enumerate(cfg["layers"]):
        L, m = f"l{i}.", lc["mixer"]
        mx = L + "mix."
        out[L + "norm1"] = (d,)
        if lc["type"] == "attention":
            attention(mx, m)
        elif lc["type"] == "mamba2":
            inner = m["heads"] * m["vdim"]
            ch = inner + 2 * m["groups"] * m["state"]
            out.update({mx + "in": (inner + ch + m["heads"], d), mx + "conv": (ch, m["conv"]), mx + "conv.b": (ch,), mx + "dt_bias": (m["heads"],), mx + "A_log": (m["heads"],),
                        mx + "D": (m["heads"],), mx + "norm": (inner,), mx + "o": (d, inner)})
        else:
            r, R = m["right"], mx + "right."
            K = r["heads"] * r["dim"]
            attention(mx + "left.", m["left"])
            out.update({R + "mu." + c: (d,) for c in "rkvgw"})
            out.update({R + c: (K, d) for c in "rkvg"})
            out.update({R + "w1": (rank, d), R + "w2": (K, rank), R + "w0": (K,), R + "u": (r["heads"], r["dim"]), R + "norm": (K,), R + "o": (d, K),
                        mx + "left.out": (d,), mx + "right.out": (d,)})
        if lc.get("mlp"):
            out.update({L + "norm2": (d,), L + "mlp.up": (lc["mlp"]["ff"], d), L + "mlp.down": (d, lc["mlp"]["ff"])})
    out["final.norm"] = (d,)
    out["head"] = (cfg["vocab"], d)
    return out


def random_weights(cfg: dict, seed: int = 0, pool: int = 1 << 22, rank: int = 16) -> dict:
    """name -> bf16 bits. Matrices N(0, 1 / fan-in); norms around 1; convolutions with the newest tap raised; decays that keep from
    a few tokens to a few hundred."""
    values, out = Pool(seed, pool), {}
    for name, shape in shapes(cfg, rank).items():
        v, leaf = values.take(shape), name.rsplit(".", 1)[-1]
        if leaf in ("norm", "norm1", "norm2", "out"):
            v = 1.0 + 0.1 * v
        elif ".mu." in name:
            v = 0.5 + 0.2 * v
        elif leaf == "conv":
            v = v * 0.3
            v[:, -1] += 0.8
        elif leaf in ("b", "D"):
            v = v * 0.3 + (leaf == "D")
        elif leaf == "dt_bias":
            v = v * 0.7 - 3.0
        elif leaf == "A_log":
            v = v * 0.5
        elif leaf == "w0":
            v = v * 1.2 - 3.0
        elif leaf == "u":
            v = v * 0.5
        elif name == "pos":
            v = v * 0.3
        elif name != "embed":
            v = v * (shape[-1] ** -0.5)
        out[name] = to_bf16(np.ascontiguousarray(v))
    return out
