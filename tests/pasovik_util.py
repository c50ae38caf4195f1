"""Small Pasovik models for the tests: configurations, and weights that make one key, or what a state remembers, stand out, or that
leave no choice of experts a close one."""
from __future__ import annotations

import tempfile
from pathlib import Path

import numpy as np

from silicon_violetto_b200 import pasovik as pv
from tests.folder_util import LIMIT, engine, error, portions, prompt, replay  # noqa: F401  (the tests take them from here)

_TMP = Path(tempfile.mkdtemp(prefix="vlt_pasovik_"))

CONFIGS = {
    # Sizes no tensor-core kernel takes, none like another: value and key sizes differ, states and ranks that are no multiple of
    # four, layers with each kind of feed-forward and with none, latents read by two later layers.
    "odd": pv.config(88, 301, [
        pv.attention(6, 2, 20, 28, 0.31, softcap=3.0, rot_dims=12, base=1000.0, factor=3.0, mlp=pv.moe(5, 2, 24, limit=0.8)),
        pv.latent(5, 22, 6, 14, 35, 27, scale=0.2, base=500.0, mlp=pv.dense(72)),
        pv.lightning(10, 7, [0.9, 0.35, 0.995], mlp=None),
        pv.latent(3, 10, 6, 30, 35, 44, scale=0.3, base=500.0, kv_from=1, mlp=pv.moe(7, 1, 30, limit=0.5)),
        pv.latent(4, 13, 2, 9, 18, 20, base=77.0, mlp=None),
        pv.lightning(33, 22, [0.97, 0.6], mlp=pv.moe(3, 3, 16, limit=2.0)),
        pv.latent(7, 9, 6, 5, 35, 12, base=500.0, kv_from=1, mlp=pv.dense(50)),
        pv.attention(5, 5, 36, 16, 0.25, softcap=8.0, rot_dims=36, base=77.0, factor=1.5)], side=13, eps=3e-4),
    # Sizes the tensor-core kernels take, more than 8 query heads a kv head, experts of whole tiles, latents of two sizes.
    "fast": pv.config(384, 512, [
        pv.lightning(64, 128, [0.99, 0.8, 0.5, 0.999], mlp=pv.dense(512)),
        pv.attention(20, 2, 64, 128, softcap=6.0, rot_dims=32, base=5e4, factor=4.0, mlp=pv.moe(6, 2, 128, limit=1.0)),
        pv.latent(12, 64, 32, 128, 128, 192, base=2e4, mlp=pv.dense(256)),
        pv.latent(20, 128, 32, 64, 128, 128, base=2e4, kv_from=2, mlp=pv.moe(16, 1, 64, limit=1.5)),
        pv.lightning(128, 64, [0.95, 0.9995]),
        pv.latent(34, 24, 16, 20, 64, 64, base=3e3),
        pv.attention(4, 4, 128, 64, softcap=20.0, mlp=pv.dense(128))], side=64),
    # One mechanism each: for faults that must not hide behind others.
    "capped": pv.config(128, 200, [pv.attention(4, 2, 64, 64, 0.35, softcap=12.0, rot_dims=32, factor=2.0)]),
    "capped_odd": pv.config(96, 200, [pv.attention(3, 3, 40, 24, 0.45, softcap=13.0, rot_dims=10, factor=5.0)], side=5),
    "latent": pv.config(128, 200, [pv.latent(6, 64, 16, 64, 64, 128, scale=0.3)]),
    "latent_odd": pv.config(96, 200, [pv.latent(3, 20, 6, 13, 30, 21, scale=0.5)], side=5),
    "latent_pair": pv.config(128, 200, [pv.latent(4, 64, 64, 128, 200, 64, scale=0.25), pv.latent(18, 64, 64, 64, 200, 64, scale=0.25, kv_from=0)]),
    "fade": pv.config(128, 200, [pv.lightning(64, 64, [0.999, 0.99, 0.7])]),
    "fade_odd": pv.config(96, 200, [pv.lightning(22, 9, [0.998, 0.93, 0.99, 0.5])], side=5),
    "experts": pv.config(128, 200, [pv.lightning(64, 64, [0.9, 0.8], mlp=pv.moe(8, 3, 128, limit=0.7))]),
    "experts_odd": pv.config(96, 200, [pv.lightning(16, 16, [0.9], mlp=pv.moe(5, 1, 22, limit=0.4))], side=5),
    "dense": pv.config(128, 200, [pv.lightning(64, 64, [0.9, 0.8], mlp=pv.dense(192))]),
}
# Latents up to the largest kernel's, in every number of rows a block may have, and in ranks between those a kernel is laid out for.
for rank, rot, heads in ((512, 64, 16), (512, 64, 24), (512, 64, 40), (384, 32, 70), (256, 64, 8), (256, 128, 4), (136, 8, 5), (40, 88, 33), (24, 8, 3), (512, 128, 2)):
    CONFIGS[f"rank{rank}_{rot}_{heads}"] = pv.config(128, 96, [pv.latent(heads, 64, rot, 16, rank, 64, scale=0.12)], side=64)
# Key channels up to the largest kernel's.
for n, N in enumerate((5, 40, 70, 100, 170, 230, 300, 512)):
    CONFIGS[f"wide{N}"] = pv.config(64, 96, [pv.lightning(N, 20 - n, [0.99, 0.6])], side=9)
_made: dict = {}


def model(name: str, seed: int = 0, change=None, tag: str = ""):
    """(folder, config, weights as float64) of a configuration, its choices of experts decided; `change(cfg, weights)` edits the bf16
    bits in place."""
    key = (name, seed, tag)
    if key not in _made:
        cfg = CONFIGS[name]
        bits = pv.random_weights(cfg, seed, pool=1 << 20)
        decided_routing(cfg, bits)
        if change:
            change(cfg, bits)
        folder = pv.write_model(_TMP / f"{name}_{seed}_{tag}", cfg, bits)
        _made[key] = (folder, cfg, {k: pv.from_bf16(v).astype(np.float64) for k, v in bits.items()})
    return _made[key]


def decided_routing(cfg, bits):
    """After this no choice of experts is a close one, so that bf16 and 32-bit choose alike: the routers read coordinates that nothing
    but the embedding writes, and every token has its own order of them with even steps."""
    most = max([lc["mlp"]["router"]["experts"] for lc in cfg["layers"] if lc.get("mlp") and lc["mlp"]["kind"] == "moe"], default=0)
    if not most:
        return
    rng = np.random.default_rng(11)
    order = np.stack([rng.permutation(most) for _ in range(cfg["vocab"])]) - (most - 1) / 2
    bits["embed"][:, :most] = pv.to_bf16((3.0 / most * order).astype(np.float32))
    for name in list(bits):
        if name.endswith((".norm1", ".norm2", ".side.norm")):
            bits[name][:most] = 0
        elif name.endswith(".router"):
            bits[name][:] = 0
            for e in range(len(bits[name])):
                bits[name][e, (e * 5 + 1) % most if most % 5 else e] = pv.to_bf16(np.array([0.8], np.float32))[0]


def standing_keys(special):
    """An edit after which the keys of the tokens `special` score far above all others for every query of every attention, wherever
    they stand: all embeddings share a direction the queries answer with, the special ones have one of their own their keys answer
    with, both on a head's last dimension that does not turn."""
    def change(cfg, bits):
        d, rng = cfg["width"], np.random.default_rng(5)
        common, mark = rng.standard_normal((2, d)).astype(np.float32)
        common /= np.linalg.norm(common)
        mark -= (mark @ common) * common
        mark /= np.linalg.norm(mark)
        get = lambda n: pv.from_bf16(bits[n]).reshape(bits[n].shape)
        put = lambda n, w: bits.__setitem__(n, pv.to_bf16(w).reshape(w.shape))
        e = get("embed") * 0.5
        e -= np.outer(e @ mark, mark)
        e += 0.35 * np.sqrt(d) * common
        for s in special:
            e[s] += 0.7 * np.sqrt(d) * mark
        put("embed", e)
        for i, lc in enumerate(cfg["layers"]):
            m, pre = lc["mixer"], f"l{i}.mix."
            if lc["type"] == "attention":
                for c, heads, direction in (("q", m["heads"], common), ("k", m["kv_heads"], mark)):
                    w = get(pre + c).reshape(heads, m["dim"], d) * 0.5
                    w[:, m["dim"] - 1] += 1.5 * direction
                    put(pre + c, w.reshape(-1, d))
            elif lc["type"] == "latent_attention":
                w = get(pre + "dq")
                w[0] += 1.5 * common
                put(pre + "dq", w)
                w = get(pre + "uq").reshape(m["heads"], -1, m["q_rank"]) * 0.5
                w[:, m["dim"] - 1, 0] += 1.0
                put(pre + "uq", w.reshape(-1, m["q_rank"]))
                if m.get("kv_from") is None:
                    w = get(pre + "dkv")
                    w[0] += 2.0 * mark
                    put(pre + "dkv", w)
                w = get(pre + "uk").reshape(m["heads"], m["dim"], m["kv_rank"]) * 0.5
                w[:, m["dim"] - 1, 0] += 2.0
                put(pre + "uk", w.reshape(-1, m["kv_rank"]))
    return change
