"""The Lonasun design on the GPU against the slow restatement (lonasun_ref.py): its mechanisms, prompts, decoding, portions,
batches, edges, reused pages and slots, verified drafts, generation, and the trace replay program; in 32-bit and in bf16."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest

from silicon_violetto_b200 import engine as E, files, lonasun
from tests import lonasun_ref as ref, lonasun_util as lu

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parents[1]
BOTH = pytest.mark.parametrize("fp32", [True, False], ids=["fp32", "bf16"])
NAMES = ["odd", "fast", "one", "one_odd", "experts"]


prompt = lu.prompt


def close(got, want, fp32, factor=1.0):
    e = lu.error(got, want)
    assert e.max() < factor * lu.LIMIT[fp32], (int(e.argmax()), float(e.max()))


def routed(name, seed):
    """A configuration's model whose choices of experts are no close calls (so that bf16 and 32-bit choose alike)."""
    if any(lc.get("mlp") for lc in lu.CONFIGS[name]["layers"]):
        return lu.model(name, seed, lu.decided_routing, "decided")
    return lu.model(name, seed)


# ---- mechanisms, through the layer captures of one-layer models
@BOTH
@pytest.mark.parametrize("name", ["one", "one_odd", "experts"])
def test_one_layer(name, fp32):
    """The gated attention's output and the stream after the layer, of a prompt over several pages and chunks."""
    folder, cfg, w = routed(name, 3)
    toks, lc, eps = prompt(cfg, 210, 1), cfg["layers"][0], cfg["norm"]["eps"]
    eng = lu.engine(folder, fp32)
    out, caps = eng.step_capture([E.Run(eng.new_seq(), toks)], E.StepOptions(head=E.Rows.ALL, read_logits=True))
    eng.close()
    x0 = w["embed"][toks]
    assert np.array_equal(caps[0]["resid_in"], x0.astype(np.float32))
    h = ref.rms_norm(x0, w["l0.norm1"], eps)
    wo, tol = w["l0.mix.o"], 2e-5 if fp32 else 2e-2
    ident = dict(w, **{"l0.mix.o": np.eye(wo.shape[1])})  # the mixer up to its output projection
    want = ref.attention_mixer(h, ident, "l0.mix.", lc["mixer"])
    assert np.abs(caps[0]["sdpa_out"] - want).max() < tol * np.abs(want).max()
    mid = x0 + want @ wo.T
    after = mid
    if lc["mlp"]:
        after = mid + ref.moe(ref.rms_norm(mid, w["l0.norm2"], eps), w, "l0.mlp.", lc["mlp"])
    d = np.abs(caps[0]["resid_out"] - after).max(axis=1) / np.abs(after).max()
    assert d.max() < tol
    close(out.logits, ref.forward(cfg, w, toks)[0], fp32)


@BOTH
def test_router_correction_identity_and_shared(fp32):
    """Corrections large enough to decide the choice alone: fixed experts, the identity ones among them, weights by the scores."""
    def change(cfg, bits):
        c = np.full(12, -3.0, np.float32)
        c[[2, 9, 11]] = [3.0, 2.5, 2.0]
        bits["l0.mlp.correction"] = lonasun.to_bf16(c)
    folder, cfg, w = lu.model("experts", 4, change, "corr")
    ids, wt = ref.route(np.random.default_rng(0).standard_normal((4, cfg["width"])), w["l0.mlp.router"], w["l0.mlp.correction"], 3)
    assert all(sorted(r) == [2, 9, 11] for r in ids.tolist()) and np.allclose(wt.sum(1), 1)
    for n in (1, 7, 40, 300):  # row counts that take different kernels
        toks = prompt(cfg, n, n)
        eng = lu.engine(folder, fp32)
        got = lu.replay(eng, {"a": toks}, [[("a", n)]])["a"]
        eng.close()
        close(got, ref.forward(cfg, w, toks)[0], fp32)


# ---- whole prompts, decoding, portions, batches
@BOTH
@pytest.mark.parametrize("name", NAMES)
def test_prompt_decode_and_portions(name, fp32):
    folder, cfg, w = routed(name, 1)
    toks = prompt(cfg, 230, 2)
    want, _ = ref.forward(cfg, w, toks)
    eng = lu.engine(folder, fp32, tokens=256)
    whole = lu.replay(eng, {"a": toks}, [[("a", 230)]])["a"]
    close(whole, want, fp32)
    for sizes in ([2], [150] + [1] * 80, [3, 2, 17, 64, 9, 1, 1, 5], [63, 2, 65]):
        got = lu.replay(eng, {"a": toks}, [[("a", c)] for c in lu.portions(230, sizes)])["a"]
        close(got, want, fp32)
        if fp32:
            close(got, whole, fp32)
    eng.close()


@BOTH
@pytest.mark.parametrize("name", ["odd", "fast"])
def test_unequal_batches_and_reused_pages_and_slots(name, fp32):
    """Portions of prompts beside single tokens of others, requests left out of steps, ended and replaced in a pool that holds
    only the live ones: every request as if it were alone."""
    folder, cfg, w = routed(name, 1)
    lens = {"a": 140, "b": 9, "c": 65, "d": 100, "e": 130, "f": 3, "g": 64}
    prompts = {n: prompt(cfg, k, 10 + i) for i, (n, k) in enumerate(lens.items())}
    steps = [[("a", 50), ("b", 1), ("c", 2)], [("b", 2), ("c", 3), ("d", 20)], [("a", 1), ("c", 1), ("b", 6)], [("a", 1), ("c", 59), ("d", 1)],
             [("d", 2), ("e", 90), ("a", 70)], [("a", 1), ("d", 1), ("e", 1), ("f", 3)], [("a", 17), ("e", 2), ("d", 76), ("g", 40)], [("e", 37), ("g", 24)]]
    eng = lu.engine(folder, fp32, tokens=256, kv_tokens=9 * 64)
    for _ in range(2):  # the second time on pages and slots the first has used
        got = lu.replay(eng, prompts, steps)
        for n, toks in prompts.items():
            close(got[n], ref.forward(cfg, w, toks)[0], fp32)
    assert len(eng.debug_read("free_pages")) == 9
    eng.close()


@BOTH
@pytest.mark.parametrize("name", ["one", "one_odd"])
def test_keys_at_every_edge(name, fp32):
    """A key that outshines all others at the chunk's first and last positions, at page borders, far back, and in the first
    tokens; asked for from prompts, portions and decoding on both sides of the edge (test_lonasun_host.py shows that this
    model tells a chunk that is one position off)."""
    folder, cfg, w = lu.model(name, change=lu.standing_keys([7]), tag="standing")
    size = cfg["layers"][0]["mixer"]["mask"]["size"]
    n = 2 * size + 20
    eng = lu.engine(folder, fp32, tokens=512)
    for places in ([size - 1], [size], [0], [1, size + 1], [63], [64], [127, 128], [2 * size - 1], [2 * size]):
        toks = prompt(cfg, n, 3)
        toks = [t if t != 7 else 8 for t in toks]
        for p in places:
            toks[p] = 7
        want, _ = ref.forward(cfg, w, toks)
        for steps in ([n], [size - 2] + [1] * 6 + [n], [size] + [1] * 3 + [n], [size + 1, 2, 60, 1, 2 * size - size - 66] + [1] * 30, [2 * size - 3] + [1] * 23):
            got = lu.replay(eng, {"a": toks}, [[("a", c)] for c in lu.portions(n, steps)])["a"]
            close(got, want, fp32)
    eng.close()


@BOTH
def test_long_decoding(fp32):
    """400 tokens one by one from the second on: the convolution's ring and the chunks wrap many times."""
    folder, cfg, w = lu.model("one", 6)
    toks = prompt(cfg, 400, 5)
    eng = lu.engine(folder, fp32, tokens=512)
    got = lu.replay(eng, {"a": toks}, [[("a", 1)]] * 400)["a"]
    eng.close()
    close(got, ref.forward(cfg, w, toks)[0], fp32)


@pytest.mark.parametrize("keys", [64, 128, 0])
def test_key_splits_of_the_decode_kernel(keys):
    """The decode kernel's clusters: a row's keys over one to sixteen blocks."""
    cfg = lonasun.config(128, 128, [lonasun.layer(10, 1, 128, 64, 900, conv=2, rot_dims=32)])
    bits = lonasun.random_weights(cfg, 9)
    folder = lonasun.write_model(lu._TMP / f"splits", cfg, bits)
    w = {k: lonasun.from_bf16(v).astype(np.float64) for k, v in bits.items()}
    toks = prompt(cfg, 915, 4)
    want, _ = ref.forward(cfg, w, toks)
    eng = lu.engine(folder, False, tokens=1024, tuning=E.Tuning(attn_keys_per_cta=keys))
    got = lu.replay(eng, {"a": toks, "b": toks[:40]}, [[("a", 880), ("b", 39)], [("a", 1), ("b", 1)]] + [[("a", 1)]] * 12 + [[("a", 3)], [("a", 1)], [("a", 18)]])
    eng.close()
    close(got["a"], want, False)
    close(got["b"], want[:40], False)


@BOTH
def test_rows_do_not_depend_on_the_batch(fp32):
    """A row's logits with 1 to 40 other requests in the step stay within rounding of its own alone."""
    folder, cfg, w = routed("fast", 1)
    toks = prompt(cfg, 90, 8)
    want, _ = ref.forward(cfg, w, toks)
    eng = lu.engine(folder, fp32, tokens=256, seqs=41, kv_tokens=64 * 60)
    for others in (0, 3, 8, 40):
        prompts = {"a": toks, **{f"o{i}": prompt(cfg, 6 + i, 50 + i) for i in range(others)}}
        first = [("a", 80)] + [(n, 3) for n in prompts if n != "a"]
        steps = [first] + [[("a", 1)] + [(n, 1) for n in prompts if n != "a"] for _ in range(3)] + [[("a", 1)]] * 7
        got = lu.replay(eng, prompts, steps)["a"]
        close(got, want, fp32)
    eng.close()


# ---- verified drafts
@BOTH
@pytest.mark.parametrize("name", ["odd", "fast", "one"])
def test_draft_tree_rows_and_compaction(name, fp32):
    """A draft tree: each row's logits are those of its own path; the accepted path, which is not a prefix of the rows, is
    moved into place (keys, values and the convolutions' rows) and decoding goes on from it."""
    folder, cfg, w = routed(name, 1)
    chunk = cfg["layers"][0]["mixer"]["mask"]["size"]
    node = lambda depth, parent, sees: depth | parent << 8 | sees << 16
    for start in (19, chunk - 2, 64 - 1):  # within a page and chunk, across the chunk's edge, across a page's
        eng = lu.engine(folder, fp32, tokens=256, head_rows=256)
        s, toks = eng.new_seq(), prompt(cfg, start, 20 + start)
        eng.step([E.Run(s, toks)])
        draws, path = [], list(toks)
        for _ in range(4):
            draws.append(int(ref.forward(cfg, w, path)[0][-1].argmax()))
            path.append(draws[-1])
        v, g = cfg["vocab"], draws
        if int(eng.debug_read("feed")[s * 16]) != g[0]:
            eng.close()
            continue  # (bf16: the greedy token is a near tie)
        feed = [g[0], (g[1] + 1) % v, g[1], g[2], g[2], (g[3] + 5) % v]
        tree = [node(0, 255, 1), node(1, 0, 0b000011), node(1, 0, 0b000101), node(2, 1, 0b001011), node(2, 2, 0b010101), node(3, 4, 0b110101)]
        eng.debug_write("feed", s * 16, feed)
        eng.debug_write("tree", s * 16, tree)
        out = eng.debug_step([(s, [E.FEED_ROW + i for i in range(6)], E.Rows.LAST, True)], E.StepOptions(read_logits=True))
        rows = [[0], [0, 1], [0, 2], [0, 1, 3], [0, 2, 4], [0, 2, 4, 5]]
        want = np.stack([ref.forward(cfg, w, toks + [feed[i] for i in r])[0][-1] for r in rows])
        close(out.logits, want, fp32)
        n = int(eng.debug_read("path_len")[0])
        if fp32:
            assert n == 3 and eng.debug_read("path")[:3].tolist() == [0, 2, 4]
        if n == 3:
            eng.settle(s, 6 - 3)
            seq = toks + [feed[i] for i in (0, 2, 4)]
            more = prompt(cfg, 9, 99)
            got = [eng.step_rows([E.Run(s, [t])], [[0]], E.StepOptions(read_logits=True)).logits[0] for t in more[:5]]
            got += list(eng.step_rows([E.Run(s, more[5:])], [[0, 1, 2, 3]], E.StepOptions(read_logits=True)).logits)
            close(np.stack(got), ref.forward(cfg, w, seq + more)[0][len(seq):], fp32)
        eng.close()


# ---- generation
def greedy(cfg, w, toks, n):
    out = list(toks)
    for _ in range(n):
        out.append(int(ref.forward(cfg, w, out)[0][-1].argmax()))
    return out[len(toks):]


@pytest.mark.parametrize("name", ["odd", "fast"])
def test_greedy_generation_through_the_scheduler(name):
    """More requests than slots through Generator: prompts in chunks beside decoding, plain and with replayed drafts."""
    folder, cfg, w = lu.model(name, 2)
    prompts = [prompt(cfg, k, 30 + k) for k in (37, 5, 70, 1, 20)]
    want = [greedy(cfg, w, p, 12) for p in prompts]
    eng = lu.engine(folder, True, tokens=32, seqs=3, head_rows=32, kv_tokens=64 * 6)
    for draft, rate in ((E.Draft.NONE, 0.0), (E.Draft.REPLAY, 0.0), (E.Draft.REPLAY, 0.4)):
        with eng.generator() as g:
            g.set_replay_mistakes(rate, 3)
            ids = [g.submit(E.Request(p, 12, draft=draft, rows=5 if draft else 1, trace=p + o if draft else [])) for p, o in zip(prompts, want)]
            got = {i: [] for i in ids}
            while not g.is_idle():
                for ev in g.step():
                    if ev.kind == "token":
                        got[ev.req].append(ev.value)
        assert [got[i] for i in ids] == want, (draft, rate)
    assert len(eng.debug_read("free_pages")) == 6
    eng.close()


def test_generate_from_a_request_file(tmp_path):
    """The batch driver and its command line take a model folder like any weight file."""
    folder, cfg, w = lu.model("odd", 2)
    prompts = {"x": prompt(cfg, 12, 1), "y": prompt(cfg, 33, 2)}
    files.write_requests(tmp_path / "reqs.txt", [files.RequestLine(n, "max_tokens=6,temperature=0", p) for n, p in prompts.items()])
    r = subprocess.run([sys.executable, str(ROOT / "bin" / "generate"), str(folder), str(tmp_path / "reqs.txt"), str(tmp_path / "out.jsonl"), "--dtype", "float32", "--chunk", "16"],
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    got = files.read_outputs(tmp_path / "out.jsonl")
    assert got == {n: greedy(cfg, w, p, 6) for n, p in prompts.items()}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay(tmp_path, dtype):
    folder, cfg, w = routed("fast", 1)
    a, b = prompt(cfg, 40, 1), prompt(cfg, 30, 2)
    steps = [dict(step=0, entries=[dict(id="a", tokens=a[:30], want=[0, 29]), dict(id="b", tokens=b[:2], want=[])], end=[]),
             dict(step=1, entries=[dict(id="b", tokens=b[2:30], want=[27, 3])], end=["b"]),
             dict(step=2, entries=[dict(id="a", tokens=a[30:], want=[])], end=["a"]),
             dict(step=3, entries=[dict(id="c", tokens=a, want=[39])], end=["c"])]
    r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "128"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    wa, wb = ref.forward(cfg, w, a)[0], ref.forward(cfg, w, b)[0]
    read = lambda i: np.fromfile(tmp_path / f"{i}.f32", "<f4").reshape(-1, cfg["vocab"])
    fp32 = dtype == "float32"
    close(np.concatenate([read(0), read(1), read(3)]), np.concatenate([wa[[0, 29]], wb[[29, 5]], wa[[39]]]), fp32)
    assert not (tmp_path / "2.f32").exists()
