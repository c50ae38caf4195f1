"""Sopetar model folders (config.json, model.safetensors): tensor shapes and random-init weights, for tests and benchmarks. The
engine reads the folders itself (csrc/sopetar.h)."""
from __future__ import annotations

import numpy as np

from .folders import Pool, from_bf16, to_bf16, write_model  # noqa: F401  (callers take them from here)


def dense(ff, limit=7.0) -> dict:
    return {"kind": "dense", "ff": ff, "limit": limit}


def attention(heads, kv_heads, dim, vdim, window, keep=0, scale=None, softcap=50.0, v_mix=True, mlp=None) -> dict:
    """A layer of soft-capped attention over a window and the first `keep` positions; the layers are entries of config['layers'].
    v_mix: its values take part in the mix with the first such layer's. mlp: dense() or None."""
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale, "softcap": softcap,
                                                       "mask": {"size": window, "keep_first": keep}, "v_mix": v_mix}}


def latent(heads, dim, rot_dim, vdim, kv_rank, window, scale=None, base=10000.0, mlp=None) -> dict:
    return {"type": "latent_attention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": (dim + rot_dim) ** -0.5 if scale is None else scale,
                                                              "rot": {"base": base, "dims": rot_dim}, "mask": {"size": window}}}


def config(width, vocab, layers, embed_scale=1.0, eps=1e-5) -> dict:
    return {"architecture": "Sopetar", "width": width, "vocab": vocab, "embedding": {"scale": embed_scale}, "layers": layers, "norm": {"eps": eps}}


def shapes(cfg: dict) -> dict:
    d = cfg["width"]
    out = {"embed": (cfg["vocab"], d)}
    for i, lc in enumerate(cfg["layers"]):
        L, m, f = f"l{i}.", lc["mixer"], lc.get("mlp")
        mx, ml, inner = L + "mix.", L + "mlp.", m["heads"] * m["vdim"]
        out.update({L + "norm1": (d,), L + "norm1.b": (d,)})
        if lc["type"] == "attention":
            for c, rows in (("q", m["heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
                out.update({mx + c: (rows, d), mx + c + ".b": (rows,)})
            if m["v_mix"]:
                out[mx + "vmix"] = ()
        else:
            out.update({mx + "q": (m["heads"] * (m["dim"] + m["rot_dim"]), d), mx + "dkv": (m["kv_rank"] + m["rot_dim"], d), mx + "dkv.norm": (m["kv_rank"],),
                        mx + "uk": (m["heads"] * m["dim"], m["kv_rank"]), mx + "uv": (inner, m["kv_rank"]), mx + "sink": (m["heads"],), mx + "g": (m["heads"], d)})
        out[mx + "o"] = (d, inner)
        if f:
            for c, rows, cols in (("gate", f["ff"], d), ("up", f["ff"], d), ("down", d, f["ff"])):
                out.update({ml + c: (rows, cols), ml + c + ".b": (rows,)})
        out[L + "dwa"] = (i + 2,)
    out.update({"final.norm": (d,), "final.norm.b": (d,), "head": (cfg["vocab"], d)})
    return out


def random_weights(cfg: dict, seed: int = 0, pool: int = 1 << 22) -> dict:
    """name -> bf16 bits. Matrices N(0, 1 / fan-in), norms around 1, biases and sinks of a size that shows, averages that keep most of
    the last result."""
    values, out = Pool(seed, pool), {}
    for name, shape in shapes(cfg).items():
        v, leaf = np.array(values.take(shape), np.float32), name.rsplit(".", 1)[-1]
        if leaf in ("norm", "norm1"):
            v = 1.0 + 0.1 * v
        elif leaf == "b":
            v = 0.2 * v
        elif leaf == "dwa":
            v = 0.2 * v
            v[-1] += 1.0
        elif leaf == "vmix":
            v = 0.4 + 0.1 * v
        elif leaf == "sink":
            v = 2.0 + v
        elif name != "embed":
            v = v * (shape[-1] ** -0.5)
        out[name] = to_bf16(v).reshape(shape)
    return out
