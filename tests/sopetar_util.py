"""Small Sopetar models for the tests: configurations, and weights that make one key, or a sink, stand out."""
from __future__ import annotations

import tempfile
from pathlib import Path

import numpy as np

from silicon_violetto_b200 import sopetar as sv
from tests.folder_util import LIMIT, engine, error, portions, prompt, replay  # noqa: F401  (the tests take them from here)

_TMP = Path(tempfile.mkdtemp(prefix="vlt_sopetar_"))

CONFIGS = {
    # Sizes no tensor-core kernel takes, none like another: value and key sizes differ, ranks that are no multiple of four, heads in
    # numbers that are no power of two, layers with and without a feed-forward, values mixed in some layers and not in others.
    "odd": sv.config(88, 301, [
        sv.attention(5, 5, 36, 16, window=41, keep=3, scale=0.2, softcap=8.0, v_mix=False, mlp=sv.dense(50, 1.1)),
        sv.latent(5, 22, 6, 14, 35, window=29, scale=0.2, base=500.0, mlp=sv.dense(72, 0.6)),
        sv.attention(6, 2, 20, 28, window=17, keep=9, scale=0.31, softcap=3.0, mlp=None),
        sv.latent(3, 10, 8, 30, 20, window=70, scale=0.3, base=77.0),
        sv.attention(4, 2, 13, 28, window=90, keep=0, scale=0.5, softcap=5.0, mlp=sv.dense(33, 2.0)),
        sv.latent(7, 9, 2, 5, 43, window=3, mlp=sv.dense(21, 0.3)),
        sv.attention(10, 2, 7, 28, window=1, keep=66, scale=0.4, softcap=2.0)], embed_scale=1.7, eps=3e-4),
    # Sizes the tensor-core kernels take, more than 8 query heads a kv head, more heads than a block has rows.
    "fast": sv.config(384, 512, [
        sv.latent(12, 64, 32, 128, 128, window=75, base=2e4, mlp=sv.dense(512, 1.0)),
        sv.attention(20, 2, 64, 128, window=50, keep=21, scale=0.25, softcap=6.0, mlp=sv.dense(256, 0.5)),
        sv.latent(34, 24, 16, 20, 64, window=130, base=3e3),
        sv.attention(6, 2, 128, 128, window=100, keep=2, softcap=20.0, mlp=sv.dense(128, 1.5)),
        sv.attention(8, 2, 64, 64, window=33, keep=70, softcap=9.0, v_mix=False),
        sv.latent(20, 128, 64, 64, 192, window=40, mlp=sv.dense(192, 0.8))], embed_scale=0.6),
    # One mechanism each: for faults that must not hide behind others.
    "kept": sv.config(128, 200, [sv.attention(4, 2, 64, 64, window=45, keep=11, scale=0.3, softcap=13.0)], embed_scale=0.3),
    "kept_odd": sv.config(96, 200, [sv.attention(3, 3, 40, 24, window=45, keep=11, scale=0.4, softcap=13.0)], embed_scale=0.3),
    "latent": sv.config(128, 200, [sv.latent(6, 64, 16, 64, 64, window=45, scale=0.3)], embed_scale=0.3),
    "latent_odd": sv.config(96, 200, [sv.latent(3, 20, 6, 13, 30, window=45, scale=0.5)], embed_scale=0.3),
    "mixed": sv.config(128, 200, [sv.attention(4, 2, 64, 64, window=60, v_mix=v) for v in (False, True, True, True)], embed_scale=0.4),
    "mixed_odd": sv.config(96, 200, [sv.attention(3, 1, 20, 12, window=60, keep=4) for _ in range(3)], embed_scale=0.4),
    "dense": sv.config(128, 200, [sv.latent(2, 64, 16, 64, 64, window=9, mlp=sv.dense(192, 0.7)) for _ in range(2)], embed_scale=0.4),
    "dense_odd": sv.config(90, 200, [sv.latent(2, 16, 4, 8, 24, window=9, mlp=sv.dense(75, 0.4)) for _ in range(2)], embed_scale=0.4),
}
WINDOWS = [(1, 0), (2, 1), (7, 8), (8, 0), (9, 16), (16, 17), (63, 1), (64, 64), (65, 65), (30, 130), (128, 5), (129, 80)]
# A window and the first positions kept, for both kinds of attention, on the tensor cores and beside them: both in one model.
for size, keep in WINDOWS:
    CONFIGS[f"window{size}_{keep}"] = sv.config(128, 96, [sv.attention(4, 2, 64, 64, window=size, keep=keep, scale=0.3, softcap=13.0), sv.latent(4, 64, 16, 32, 64, window=size, scale=0.3)])
    CONFIGS[f"window{size}_{keep}_odd"] = sv.config(72, 96, [sv.attention(3, 1, 24, 20, window=size, keep=keep, scale=0.5, softcap=13.0), sv.latent(3, 20, 6, 13, 30, window=size, scale=0.5)])
# Latents up to the largest kernel's, in every number of rows a block may have, and in ranks between those a kernel is laid out for.
for rank, rot, heads in ((512, 64, 16), (512, 64, 24), (512, 64, 40), (384, 32, 70), (256, 128, 4), (136, 8, 5), (40, 88, 33), (24, 8, 3)):
    CONFIGS[f"rank{rank}_{rot}_{heads}"] = sv.config(128, 96, [sv.latent(heads, 64, rot, 16, rank, window=100, scale=0.12)])
_made: dict = {}


def model(name: str, seed: int = 0, change=None, tag: str = ""):
    """(folder, config, weights as float64) of a configuration; `change(cfg, weights)` edits the bf16 bits in place."""
    key = (name, seed, tag)
    if key not in _made:
        cfg = CONFIGS[name]
        bits = sv.random_weights(cfg, seed, pool=1 << 20)
        if change:
            change(cfg, bits)
        folder = sv.write_model(_TMP / f"{name}_{seed}_{tag}", cfg, bits)
        _made[key] = (folder, cfg, {k: sv.from_bf16(v).reshape(v.shape).astype(np.float64) for k, v in bits.items()})
    return _made[key]


def standing_keys(special, share=1.0):
    """An edit after which the keys of the tokens `special` score far above all others for every query of every attention, wherever
    they stand: all embeddings share a direction the queries answer with, the special ones have one of their own their keys answer
    with, both on a head's last dimension that does not turn."""
    def change(cfg, bits):
        d, rng = cfg["width"], np.random.default_rng(5)
        common, mark = rng.standard_normal((2, d)).astype(np.float32)
        common -= common.mean()
        common /= np.linalg.norm(common)
        mark -= mark.mean()
        mark -= (mark @ common) * common
        mark /= np.linalg.norm(mark)
        get = lambda n: sv.from_bf16(bits[n]).reshape(bits[n].shape)
        put = lambda n, w: bits.__setitem__(n, sv.to_bf16(w).reshape(w.shape))
        e = get("embed") * 0.5
        e -= np.outer(e @ mark, mark)
        e += 0.35 * np.sqrt(d) * common
        for s in special:
            e[s] += 0.7 * share * np.sqrt(d) * mark
        put("embed", e)
        for i, lc in enumerate(cfg["layers"]):
            m, pre = lc["mixer"], f"l{i}.mix."
            if lc["type"] == "attention":
                for c, heads, direction in (("q", m["heads"], common), ("k", m["kv_heads"], mark)):
                    w = get(pre + c).reshape(heads, m["dim"], d) * 0.5
                    w[:, m["dim"] - 1] += 1.5 * direction
                    put(pre + c, w.reshape(-1, d))
            else:
                w = get(pre + "q").reshape(m["heads"], -1, d) * 0.5
                w[:, m["dim"] - 1] += 1.5 * common
                put(pre + "q", w.reshape(-1, d))
                w = get(pre + "dkv")
                w[0] += 2.0 * mark
                put(pre + "dkv", w)
                w = get(pre + "uk").reshape(m["heads"], m["dim"], m["kv_rank"]) * 0.5
                w[:, m["dim"] - 1, 0] += 2.0
                put(pre + "uk", w.reshape(-1, m["kv_rank"]))
    return change


def standing_sinks(cfg, bits):
    """An edit after which the sinks' share is most of every softmax, and the heads weigh more."""
    for name in bits:
        if name.endswith(".sink"):
            bits[name] = sv.to_bf16(np.full(bits[name].shape, 6.0, np.float32) + np.arange(len(bits[name]), dtype=np.float32) % 3)
        elif name.endswith(".o"):
            bits[name] = sv.to_bf16(3.0 * sv.from_bf16(bits[name])).reshape(bits[name].shape)
