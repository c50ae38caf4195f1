"""What the tests of the model folders' designs share: engines, schedules of steps, errors."""
from __future__ import annotations

import numpy as np

from silicon_violetto_b200 import engine as E


def prompt(cfg, n, seed):
    return [int(t) for t in np.random.default_rng(seed).integers(0, cfg["vocab"], n)]


def engine(folder, fp32: bool, tokens: int = 512, seqs: int = 4, head_rows: int | None = None, kv_tokens: int | None = None, tuning=None) -> E.Engine:
    return E.Engine(folder, E.EngineConfig(max_seqs=seqs, max_step_tokens=tokens, max_chunk=tokens, global_kv_tokens=kv_tokens or tokens * 2, max_seq_len=max(tokens, 1024),
                                           max_head_rows=head_rows or tokens, fp32=fp32), tuning)


def replay(eng, prompts: dict, steps, rows: dict | None = None) -> dict:
    """Runs the steps -- lists of (name, count) -- every token's logits kept; a request that is through gives back its slot.
    Returns name -> logits [tokens, vocab]."""
    at, seq = {n: 0 for n in prompts}, {}
    out = {n: [] for n in prompts}
    for step in steps:
        runs = []
        for n, count in step:
            if n not in seq:
                seq[n] = eng.new_seq()
            runs.append(E.Run(seq[n], prompts[n][at[n]:at[n] + count]))
        got = eng.step_rows(runs, [list(range(c)) for _, c in step], E.StepOptions(read_logits=True)).logits
        lo = 0
        for n, count in step:
            out[n].append(got[lo:lo + count])
            lo += count
            at[n] += count
            if at[n] == len(prompts[n]):
                eng.free_seq(seq.pop(n))
    for s in seq.values():
        eng.free_seq(s)
    return {n: np.concatenate(v) if v else None for n, v in out.items()}


def portions(n: int, sizes) -> list:
    out, i = [], 0
    while sum(out) < n:
        out.append(min(sizes[i % len(sizes)], n - sum(out)))
        i += 1
    return out


def error(got, want) -> np.ndarray:
    """Per position: the rms of the difference over the vocabulary, the mean taken off, relative to the logits' own spread."""
    d = got - want
    d = d - d.mean(axis=1, keepdims=True)
    return np.sqrt((d * d).mean(axis=1)) / want.std()


LIMIT = {True: 2e-5, False: 0.05}  # fp32 engine, bf16 engine
