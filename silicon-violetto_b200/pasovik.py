"""Pasovik model folders (config.json, model.safetensors): tensor shapes and random-init weights, for tests and benchmarks. The
engine reads the folders itself (csrc/pasovik.h)."""
from __future__ import annotations

import numpy as np

from .folders import Pool, from_bf16, to_bf16, write_model  # noqa: F401  (callers take them from here)


def dense(ff) -> dict:
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit=7.0) -> dict:
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}


def attention(heads, kv_heads, dim, vdim, scale=None, softcap=50.0, rot_dims=None, base=10000.0, factor=1.0, mlp=None) -> dict:
    """A layer of soft-capped attention; the layers are entries of config['layers']. mlp: dense(), moe() or None."""
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale, "softcap": softcap,
                                                       "rot": {"base": base, "dims": dim if rot_dims is None else rot_dims, "scaling": {"factor": factor}}}}


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale=None, base=10000.0, kv_from=None, mlp=None) -> dict:
    """kv_from: the layer whose latents this one reads (None: its own)."""
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": (dim + rot_dim) ** -0.5 if scale is None else scale,
         "rot": {"base": base, "dims": rot_dim}}
    return {"type": "latent_attention", "mlp": mlp, "mixer": m if kv_from is None else {**m, "kv_from": kv_from}}


def lightning(dim, vdim, decay, mlp=None) -> dict:
    """decay: one a head."""
    return {"type": "lightning", "mlp": mlp, "mixer": {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}}


def config(width, vocab, layers, side=32, eps=1e-5) -> dict:
    """side: each layer's span of the tokens' side embedding (None: there is none)."""
    return {"architecture": "Pasovik", "width": width, "vocab": vocab, "layers": layers, "norm": {"eps": eps}, "token_side": side and {"dim": side}}


def shapes(cfg: dict) -> dict:
    d, side = cfg["width"], (cfg["token_side"] or {"dim": 0})["dim"]
    out = {"embed": (cfg["vocab"], d)}
    if side:
        out["side.embed"] = (cfg["vocab"], side * len(cfg["layers"]))
    for i, lc in enumerate(cfg["layers"]):
        L, m, f = f"l{i}.", lc["mixer"], lc.get("mlp")
        mx, ml = L + "mix.", L + "mlp."
        out[L + "norm1"] = (d,)
        inner = m["heads"] * m["vdim"]
        if lc["type"] == "attention":
            out.update({mx + "q": (m["heads"] * m["dim"], d), mx + "k": (m["kv_heads"] * m["dim"], d), mx + "v": (m["kv_heads"] * m["vdim"], d), mx + "q.norm": (m["dim"],),
                        mx + "k.norm": (m["dim"],)})
        elif lc["type"] == "lightning":
            out.update({mx + "q": (m["heads"] * m["dim"], d), mx + "k": (m["heads"] * m["dim"], d), mx + "v": (inner, d), mx + "g": (inner, d), mx + "norm": (inner,)})
        else:
            out.update({mx + "dq": (m["q_rank"], d), mx + "dq.norm": (m["q_rank"],), mx + "uq": (m["heads"] * (m["dim"] + m["rot_dim"]), m["q_rank"])})
            if m.get("kv_from") is None:
                out.update({mx + "dkv": (m["kv_rank"] + m["rot_dim"], d), mx + "dkv.norm": (m["kv_rank"],)})
            out.update({mx + "uk": (m["heads"] * m["dim"], m["kv_rank"]), mx + "uv": (inner, m["kv_rank"]), mx + "g": (inner, d)})
        out[mx + "o"] = (d, inner)
        if f:
            out[L + "norm2"] = (d,)
            parts, ff = ([""], f["ff"]) if f["kind"] == "dense" else ([f"e{e}." for e in range(f["router"]["experts"])], f["expert"]["ff"])
            for p in parts:
                out.update({ml + p + "gate": (ff, d), ml + p + "up": (ff, d), ml + p + "down": (d, ff)})
            if f["kind"] == "moe":
                out[ml + "router"] = (f["router"]["experts"], d)
        if side:
            out.update({L + "side.gate": (side, d), L + "side.proj": (d, side), L + "side.norm": (d,)})
    out["final.norm"] = (d,)
    out["head"] = (cfg["vocab"], d)
    return out


def random_weights(cfg: dict, seed: int = 0, pool: int = 1 << 22) -> dict:
    """name -> bf16 bits. Matrices N(0, 1 / fan-in), norms around 1."""
    values, out = Pool(seed, pool), {}
    for name, shape in shapes(cfg).items():
        v, leaf = values.take(shape), name.rsplit(".", 1)[-1]
        if leaf in ("norm", "norm1", "norm2"):
            v = 1.0 + 0.1 * v
        elif name not in ("embed", "side.embed"):
            v = v * (shape[-1] ** -0.5)
        out[name] = to_bf16(np.ascontiguousarray(v))
    return out
