"""Lonasun model folders (config.json, model.safetensors): tensor shapes, random-init weights and the writer, for tests and
benchmarks. The engine reads the folders itself (csrc/lonasun.h)."""
from __future__ import annotations

from .folders import Pool, from_bf16, to_bf16, write_model  # noqa: F401  (callers take them from here)


def layer(heads, kv_heads, dim, vdim, chunk, conv=4, rot_dims=None, base=10000.0, scale=None, moe=None) -> dict:
    """One entry of config['layers']; moe: dict(experts, top, ff, identity=0, shared=0) or None."""
    out = {"type": "attention",
           "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "mask": {"size": chunk},
                     "rot": {"base": base, "dims": dim if rot_dims is None else rot_dims}, "scale": dim ** -0.5 if scale is None else scale},
           "mlp": None}
    if moe:
        out["mlp"] = {"kind": "moe", "expert": {"ff": moe["ff"]}, "router": {"experts": moe["experts"], "identity": moe.get("identity", 0), "top": moe["top"]},
                      "shared": {"ff": moe["shared"]} if moe.get("shared") else None}
    return out


def config(width, vocab, layers, loop=None, eps=1e-5) -> dict:
    """loop: (start, stop, times) or None."""
    return {"architecture": "Lonasun", "width": width, "vocab": vocab, "layers": layers, "norm": {"eps": eps},
            "loop": dict(zip(("start", "stop", "times"), loop)) if loop else None}


def shapes(cfg: dict) -> dict:
    d, out = cfg["width"], {"embed": (cfg["vocab"], cfg["width"])}
    if cfg.get("loop"):
        out["loop.in"] = (d, 2 * d)
    for i, lc in enumerate(cfg["layers"]):
        m, L = lc["mixer"], f"l{i}."
        out[L + "norm1"] = (d,)
        rows = {"q": m["heads"] * m["dim"], "k": m["kv_heads"] * m["dim"], "v": m["kv_heads"] * m["vdim"]}
        for k, r in rows.items():
            out[L + "mix." + k] = (r, d)
            out[L + f"mix.{k}.conv"] = (r, m["conv"])
        out[L + "mix.g"] = (m["heads"] * m["vdim"], d)
        out[L + "mix.o"] = (d, m["heads"] * m["vdim"])
        f = lc.get("mlp")
        if not f:
            continue
        out[L + "norm2"] = (d,)
        r = f["router"]
        for e in range(r["experts"]):
            out[L + f"mlp.e{e}.up"] = (f["expert"]["ff"], d)
            out[L + f"mlp.e{e}.down"] = (d, f["expert"]["ff"])
        out[L + "mlp.router"] = (r["experts"] + r.get("identity", 0), d)
        out[L + "mlp.correction"] = (r["experts"] + r.get("identity", 0),)
        if f.get("shared"):
            out[L + "mlp.shared.up"] = (f["shared"]["ff"], d)
            out[L + "mlp.shared.down"] = (d, f["shared"]["ff"])
    out["final.norm"] = (d,)
    out["head"] = (cfg["vocab"], d)
    return out


def random_weights(cfg: dict, seed: int = 0, pool: int = 1 << 22) -> dict:
    """name -> bf16 bits. Matrices N(0, 1 / fan-in), convolutions N(0, 1 / taps) with the newest tap raised, norms and
    corrections small."""
    values, out = Pool(seed, pool), {}
    for name, shape in shapes(cfg).items():
        v = values.take(shape)
        if name.endswith("norm1") or name.endswith("norm2") or name == "final.norm":
            v = v * 0.1
        elif name.endswith("correction"):
            v = v * 0.02
        elif name.endswith(".conv"):
            v = v * 0.3
            v[:, -1] += 0.8
        elif name != "embed":
            v = v * (shape[-1] ** -0.5)
        out[name] = to_bf16(v)
    return out
