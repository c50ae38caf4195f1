"""Small Leduvik models for the tests: configurations, and weights that make one key, or what a state remembers, stand out."""
from __future__ import annotations

import tempfile
from pathlib import Path

import numpy as np

from silicon_violetto_b200 import leduvik as lv
from tests.folder_util import LIMIT, engine, error, portions, prompt, replay  # noqa: F401  (the tests take them from here)

_TMP = Path(tempfile.mkdtemp(prefix="vlt_leduvik_"))

CONFIGS = {
    # Sizes no tensor-core kernel takes, none like another: value and key sizes differ, states and heads of sizes that are no
    # multiple of four, several groups, layers with and without a feed-forward, a loop in the middle.
    "odd": lv.config(88, 301, [
        lv.window(6, 2, 20, 28, 37, 0.31, ff=100),
        lv.state_space(6, 7, 10, groups=3, norm_groups=2, conv=5, ff=72),
        lv.parallel(5, 5, 36, 18, 3, 9, coef=0.4, every=7, scale=0.2, ff=0),
        lv.state_space(4, 22, 33, groups=1, norm_groups=11, conv=1),
        lv.parallel(9, 3, 12, 40, 2, 44, coef=0.15, every=50, ff=56),
        lv.window(4, 1, 32, 12, 3, 0.25, ff=0)], loop=(1, 4, 3), eps=3e-4, max_positions=700, logit_scale=0.7),
    # Sizes the tensor-core kernels take, more than 8 query heads a kv head, a grouped projection, a loop over the first layers.
    "fast": lv.config(384, 512, [
        lv.parallel(20, 2, 64, 128, 4, 64, coef=0.25, every=32, ff=512),
        lv.window(4, 2, 128, 128, 100, 0.15, ff=256),
        lv.state_space(10, 64, 128, groups=2, norm_groups=5, conv=4, ff=640),
        lv.window(8, 4, 64, 64, 70, 0.2)], loop=(0, 2, 2), logit_scale=1.5),
    # One layer of each kind, no loop: for faults that must not hide behind others.
    "window": lv.config(128, 200, [lv.window(4, 2, 64, 64, 150, 0.3, ff=192)]),
    "window_odd": lv.config(96, 200, [lv.window(3, 3, 40, 24, 90, 0.3)]),
    "window_few": lv.config(96, 200, [lv.window(2, 1, 64, 64, 5, 0.3)]),
    "state": lv.config(128, 200, [lv.state_space(6, 32, 64, groups=2, norm_groups=3, conv=4, ff=128)]),
    "state_odd": lv.config(96, 200, [lv.state_space(3, 10, 150, groups=3, norm_groups=1, conv=2)]),
    "beside": lv.config(128, 200, [lv.parallel(4, 2, 64, 64, 2, 64, coef=0.5, every=20, ff=128)]),
    "beside_odd": lv.config(96, 200, [lv.parallel(3, 1, 24, 40, 3, 130, coef=0.3, every=1)]),
}
# Key channels up to the largest kernel's.
for n, N in enumerate((5, 40, 70, 100, 170, 230, 300, 512)):
    CONFIGS[f"wide{N}"] = lv.config(64, 96, [lv.state_space(2, 20 - n, N, conv=3), lv.parallel(2, 1, 16, 16, 1, N)])
_made: dict = {}


def model(name: str, seed: int = 0, change=None, tag: str = ""):
    """(folder, config, weights as float64) of a configuration; `change(cfg, weights)` edits the bf16 bits in place."""
    key = (name, seed, tag)
    if key not in _made:
        cfg = CONFIGS[name]
        bits = lv.random_weights(cfg, seed, pool=1 << 20, rank=12 if "odd" in name else 32)
        if change:
            change(cfg, bits)
        folder = lv.write_model(_TMP / f"{name}_{seed}_{tag}", cfg, bits)
        _made[key] = (folder, cfg, {k: lv.from_bf16(v).astype(np.float64) for k, v in bits.items()})
    return _made[key]


def standing_keys(special):
    """An edit after which the keys of the tokens `special` score far above all others for every query of every attention: all
    embeddings share a direction the queries answer with, the special ones have one of their own their keys answer with."""
    def change(cfg, bits):
        d, rng = cfg["width"], np.random.default_rng(5)
        common, mark = rng.standard_normal((2, d)).astype(np.float32)
        common /= np.linalg.norm(common)
        mark -= (mark @ common) * common
        mark /= np.linalg.norm(mark)
        e = lv.from_bf16(bits["embed"]).reshape(cfg["vocab"], d) * 0.5
        e -= np.outer(e @ mark, mark)
        e += 0.35 * np.sqrt(d) * common
        for s in special:
            e[s] += 0.7 * np.sqrt(d) * mark
        bits["embed"] = lv.to_bf16(e).reshape(cfg["vocab"], d)
        bits["pos"] = lv.to_bf16(lv.from_bf16(bits["pos"]) * 0.2).reshape(bits["pos"].shape)
        for i, lc in enumerate(cfg["layers"]):
            if lc["type"] == "mamba2":
                continue
            both = lc["type"] == "parallel"
            m, pre = (lc["mixer"]["left"], f"l{i}.mix.left.") if both else (lc["mixer"], f"l{i}.mix.")
            for c, heads, direction in (("q", m["heads"], common), ("k", m["kv_heads"], mark)):
                w = lv.from_bf16(bits[pre + c]).reshape(heads, m["dim"], d) * 0.5
                w[:, m["dim"] - 1] += (2.0 if both else 1.5) * direction * (0.35 * d) ** 0.25
                bits[pre + c] = lv.to_bf16(w).reshape(-1, d)
    return change


def long_memory(cfg, bits):
    """An edit after which the recurrences hardly forget: what a state lost at any place shows at every later one."""
    for name in list(bits):
        leaf = name.rsplit(".", 1)[-1]
        if leaf == "w0":
            bits[name] = lv.to_bf16(np.full(bits[name].shape, -6.0, np.float32))
        elif leaf == "dt_bias":
            bits[name] = lv.to_bf16(np.full(bits[name].shape, -3.5, np.float32))
        elif leaf == "A_log":
            bits[name] = lv.to_bf16(np.full(bits[name].shape, -2.5, np.float32))
