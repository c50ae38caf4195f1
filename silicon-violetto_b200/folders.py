"""Model folders (config.json, model.safetensors): bf16 bits and the writer, for tests and benchmarks. The engine reads the
folders itself (csrc/layered.h)."""
from __future__ import annotations

import json
import struct
from pathlib import Path

import numpy as np


def to_bf16(a: np.ndarray) -> np.ndarray:
    """fp32 -> bf16 bit patterns, round to nearest even."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def from_bf16(bits: np.ndarray) -> np.ndarray:
    return (bits.astype(np.uint32) << 16).view(np.float32)


class Pool:
    """Standard normal values for random weights. Large models repeat a pool of them (their speed does not depend on it)."""

    def __init__(self, seed: int, size: int):
        self.rng = np.random.default_rng(seed)
        self.base, self.at = self.rng.standard_normal(size, dtype=np.float32), 0

    def take(self, shape) -> np.ndarray:
        n, size = int(np.prod(shape)), len(self.base)
        if n <= size - self.at:
            v = self.base[self.at:self.at + n]
            self.at += n
        else:
            self.at = int(self.rng.integers(0, size // 2)) | 1
            v = np.resize(np.roll(self.base, -self.at), n)
        return v.reshape(shape)


def write_model(folder, cfg: dict, weights: dict) -> Path:
    """weights: name -> bf16 bits (uint16)."""
    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg, indent=1))
    head, at = {}, 0
    for name, w in weights.items():
        head[name] = {"dtype": "BF16", "shape": list(w.shape), "data_offsets": [at, at + w.nbytes]}
        at += w.nbytes
    text = json.dumps(head).encode()
    text += b" " * (-len(text) % 8)
    with open(folder / "model.safetensors", "wb") as f:
        f.write(struct.pack("<Q", len(text)) + text)
        for w in weights.values():
            f.write(np.ascontiguousarray(w).tobytes())
    return folder
