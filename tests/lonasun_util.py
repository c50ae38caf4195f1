"""Small Lonasun models for the tests: configurations, weights that make an attended key stand out, engines, schedules."""
from __future__ import annotations

import tempfile
from pathlib import Path

import numpy as np

from silicon_violetto_b200 import lonasun
from tests.folder_util import LIMIT, engine, error, portions, prompt, replay  # noqa: F401  (the tests take them from here)

_TMP = Path(tempfile.mkdtemp(prefix="vlt_lonasun_"))


def moe(experts, top, ff, identity=0, shared=0):
    return dict(experts=experts, top=top, ff=ff, identity=identity, shared=shared)


CONFIGS = {
    # Sizes no tensor-core kernel takes: odd head and expert sizes, dim != vdim, different layers, a loop in the middle.
    "odd": lonasun.config(88, 301, [
        lonasun.layer(6, 2, 20, 28, 24, conv=3, rot_dims=12, base=1000.0, scale=0.31, moe=moe(5, 2, 24, identity=3, shared=40)),
        lonasun.layer(5, 5, 36, 16, 41, conv=1, rot_dims=36, base=77.0, moe=None),
        lonasun.layer(9, 1, 32, 44, 70, conv=6, rot_dims=2, base=2e5, moe=moe(7, 1, 30)),
        lonasun.layer(2, 1, 24, 24, 16, conv=2, rot_dims=8, base=1e4, moe=moe(3, 3, 16, identity=1))], loop=(1, 3, 2), eps=3e-4),
    # Sizes the tensor-core kernels take: attention of 64 and 128 (also unequal), more than 8 query heads a kv head, experts
    # of 128-row tiles with and without identity experts and a shared one, a loop over the first layers.
    "fast": lonasun.config(256, 512, [
        lonasun.layer(4, 2, 128, 128, 100, conv=4, rot_dims=64, base=1e5, moe=moe(6, 2, 128, identity=2, shared=128)),
        lonasun.layer(20, 2, 64, 64, 70, conv=2, rot_dims=64, base=1e4, moe=moe(16, 4, 192)),
        lonasun.layer(3, 1, 128, 64, 130, conv=3, rot_dims=20, base=5e5, moe=None),
        lonasun.layer(8, 4, 64, 128, 33, conv=4, rot_dims=32, base=1e4, moe=moe(4, 1, 64, identity=1, shared=64))], loop=(0, 2, 2)),
    # One layer of each kind, no loop: for faults that must not hide behind others.
    "one": lonasun.config(128, 200, [lonasun.layer(4, 2, 64, 64, 150, conv=4, rot_dims=16, base=1e4, scale=0.25, moe=None)]),
    "one_odd": lonasun.config(96, 200, [lonasun.layer(3, 3, 40, 24, 90, conv=5, rot_dims=10, base=1e4, scale=0.3, moe=None)]),
    "experts": lonasun.config(128, 200, [lonasun.layer(2, 1, 64, 64, 64, conv=2, rot_dims=64, moe=moe(8, 3, 128, identity=4, shared=256))]),
}
_made: dict = {}


def model(name: str, seed: int = 0, change=None, tag: str = ""):
    """(folder, config, weights as float64) of a configuration; `change(cfg, weights)` edits the bf16 bits in place."""
    key = (name, seed, tag)
    if key not in _made:
        cfg = CONFIGS[name]
        bits = lonasun.random_weights(cfg, seed, pool=1 << 20)
        if change:
            change(cfg, bits)
        folder = lonasun.write_model(_TMP / f"{name}_{seed}_{tag}", cfg, bits)
        _made[key] = (folder, cfg, {k: lonasun.from_bf16(v).astype(np.float64) for k, v in bits.items()})
    return _made[key]


def standing_keys(special):
    """An edit after which the keys of the tokens `special` score far above all others for every query, wherever they stand:
    all embeddings share a direction the queries answer with, the special ones have one of their own their keys answer with,
    both on head dimensions that do not turn."""
    def change(cfg, bits):
        d, rng = cfg["width"], np.random.default_rng(5)
        common, mark = rng.standard_normal((2, d)).astype(np.float32)
        common /= np.linalg.norm(common)
        mark -= (mark @ common) * common
        mark /= np.linalg.norm(mark)
        e = lonasun.from_bf16(bits["embed"]).reshape(cfg["vocab"], d) * 0.5
        e -= np.outer(e @ mark, mark)
        e += 0.35 * np.sqrt(d) * common
        for s in special:
            e[s] += 0.7 * np.sqrt(d) * mark
        bits["embed"] = lonasun.to_bf16(e).reshape(cfg["vocab"], d)
        for i, lc in enumerate(cfg["layers"]):
            m = lc["mixer"]
            for c, heads, direction in (("q", m["heads"], common), ("k", m["kv_heads"], mark)):
                name = f"l{i}.mix.{c}"
                w = lonasun.from_bf16(bits[name]).reshape(heads, m["dim"], d) * 0.5
                w[:, m["dim"] - 1] += 1.2 * direction * (0.35 * d) ** 0.25
                bits[name] = lonasun.to_bf16(w).reshape(-1, d)
    return change


def decided_routing(cfg, bits):
    """An edit after which no choice of experts is a close one, so that bf16 and 32-bit choose alike: the routers read
    directions that nothing but the embeddings writes, and every token has its own order of them with even steps."""
    d, rng = cfg["width"], np.random.default_rng(11)
    most = max(lc["mlp"]["router"]["experts"] + lc["mlp"]["router"]["identity"] for lc in cfg["layers"] if lc.get("mlp"))
    R = np.linalg.qr(rng.standard_normal((d, most)))[0].T  # [directions][d]
    off = lambda w: w - R.T @ (R @ w)  # a matrix that writes the stream, without the directions
    get = lambda n: lonasun.from_bf16(bits[n]).reshape(bits[n].shape).astype(np.float64)
    put = lambda n, w: bits.__setitem__(n, lonasun.to_bf16(w.astype(np.float32)).reshape(w.shape))
    order = np.stack([rng.permutation(most) for _ in range(cfg["vocab"])]) - (most - 1) / 2
    put("embed", off(get("embed").T).T + 24.0 / most * order @ R)
    if cfg.get("loop"):
        a, b = get("loop.in")[:, :d], get("loop.in")[:, d:]
        put("loop.in", np.concatenate([0.6 * np.eye(d) + off(off(a).T).T * 0.5, 0.4 * np.eye(d) + off(off(b).T).T * 0.5], axis=1))
    for name in list(bits):
        if name.endswith(".mix.o") or name.endswith(".down"):
            put(name, off(get(name)))
        elif name.endswith("norm2"):
            put(name, np.zeros(d))
        elif name.endswith(".router"):
            put(name, 0.4 * R[:bits[name].shape[0]])
        elif name.endswith(".correction"):
            put(name, get(name) * 0.01)
