"""The Sopetar design on the GPU against the slow restatement (sopetar_ref.py): its mechanisms, prompts, decoding, portions, batches,
windows and first positions, far keys, sinks, reused pages and slots, verified drafts, generation, and the trace replay program; in
32-bit and in bf16."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest

from silicon_violetto_b200 import engine as E, files, sopetar as sv
from tests import sopetar_ref as ref, sopetar_util as su

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parents[1]
BOTH = pytest.mark.parametrize("fp32", [True, False], ids=["fp32", "bf16"])
SINGLE = ["kept", "kept_odd", "latent", "latent_odd", "mixed", "mixed_odd", "dense", "dense_odd"]
ATTENDING = ["kept", "kept_odd", "latent", "latent_odd"]
prompt = su.prompt


def close(got, want, fp32, factor=1.0):
    """In bf16 a few positions feel the rounding more than others. (Mistakes cost more: test_sopetar_host.py.)"""
    e = su.error(got, want)
    assert e.max() < (1 if fp32 else 2) * factor * su.LIMIT[fp32], (int(e.argmax()), float(e.max()))
    assert np.median(e) < 0.5 * factor * su.LIMIT[fp32], float(np.median(e))


def cut(eng, toks, sizes):
    return su.replay(eng, {"a": toks}, [[("a", c)] for c in su.portions(len(toks), sizes)])["a"]


# ---- mechanisms, through the layer captures
@BOTH
@pytest.mark.parametrize("name", SINGLE)
def test_layers(name, fp32):
    """What goes into and on from each layer, of a prompt over several pages; the attentions' own outputs."""
    folder, cfg, w = su.model(name, 3)
    toks, kept = prompt(cfg, 210, 1), {}
    eng = su.engine(folder, fp32)
    out, caps = eng.step_capture([E.Run(eng.new_seq(), toks)], E.StepOptions(head=E.Rows.ALL, read_logits=True))
    eng.close()
    logits, runs = ref.forward(cfg, w, toks)
    x, tol = w["embed"][toks] * cfg["embedding"]["scale"], 2e-5 if fp32 else 4e-2
    for i in range(len(cfg["layers"])):
        assert np.abs(caps[i]["resid_in"] - x).max() < tol * np.abs(x).max()
        h = ref.layer_norm(x, w[f"l{i}.norm1"], w[f"l{i}.norm1.b"], cfg["norm"]["eps"])
        want = ref.heads(h, w, i, cfg, kept)
        assert np.abs(caps[i]["sdpa_out"] - want).max() < tol * np.abs(want).max()
        x = runs[i]
        assert np.abs(caps[i]["resid_out"] - x).max() < tol * np.abs(x).max()
    close(out.logits, logits, fp32)


@BOTH
@pytest.mark.parametrize("name", [n for n in su.CONFIGS if n.startswith("rank")])
def test_latent_sizes(name, fp32):
    """Every size the latent kernel is laid out for, and others, in prompts and token by token, across a window's edge."""
    folder, cfg, w = su.model(name, 4, su.standing_keys([7]), "standing")
    toks = [t if t != 7 else 8 for t in prompt(cfg, 190, 2)]
    toks[5] = toks[70] = 7
    want, _ = ref.forward(cfg, w, toks)
    eng = su.engine(folder, fp32, tokens=256)
    for sizes in ([190], [33, 2, 1, 17, 64], [160] + [1] * 30):
        close(cut(eng, toks, sizes), want, fp32)
    eng.close()


# ---- whole prompts, decoding, portions, batches
@BOTH
@pytest.mark.parametrize("name", ["odd", "fast"] + SINGLE)
def test_prompt_decode_and_portions(name, fp32):
    folder, cfg, w = su.model(name, 1)
    toks = prompt(cfg, 230, 2)
    want, _ = ref.forward(cfg, w, toks)
    eng = su.engine(folder, fp32, tokens=256)
    whole = cut(eng, toks, [230])
    close(whole, want, fp32)
    for sizes in ([2], [150] + [1] * 80, [3, 2, 17, 64, 9, 1, 1, 5], [63, 2, 65]):
        got = cut(eng, toks, sizes)
        close(got, want, fp32)
        if fp32:
            close(got, whole, fp32)
    eng.close()


@BOTH
@pytest.mark.parametrize("name", ["kept", "latent", "mixed_odd"])
def test_nothing_is_lost_at_any_cut(name, fp32):
    """Cuts at every place around a tile's and a page's edge."""
    folder, cfg, w = su.model(name, 2)
    toks = prompt(cfg, 140, 4)
    want, _ = ref.forward(cfg, w, toks)
    eng = su.engine(folder, fp32, tokens=256)
    for first in (1, 2, 7, 8, 9, 15, 16, 17, 31, 32, 33, 63, 64, 65):
        close(cut(eng, toks, [first, 2, 1, 9, 140]), want, fp32)
        close(cut(eng, toks, [first, first, 3, 140]), want, fp32)
    eng.close()


@BOTH
@pytest.mark.parametrize("name", ["odd", "fast"])
def test_unequal_batches_and_reused_pages_and_slots(name, fp32):
    """Portions of prompts beside single tokens of others, requests left out of steps, ended and replaced in a pool that holds
    only the live ones: every request as if it were alone."""
    folder, cfg, w = su.model(name, 1)
    lens = {"a": 140, "b": 9, "c": 65, "d": 100, "e": 130, "f": 3, "g": 64}
    prompts = {n: prompt(cfg, k, 10 + i) for i, (n, k) in enumerate(lens.items())}
    steps = [[("a", 50), ("b", 1), ("c", 2)], [("b", 2), ("c", 3), ("d", 20)], [("a", 1), ("c", 1), ("b", 6)], [("a", 1), ("c", 59), ("d", 1)],
             [("d", 2), ("e", 90), ("a", 70)], [("a", 1), ("d", 1), ("e", 1), ("f", 3)], [("a", 17), ("e", 2), ("d", 76), ("g", 40)], [("e", 37), ("g", 24)]]
    want = {n: ref.forward(cfg, w, toks)[0] for n, toks in prompts.items()}
    eng = su.engine(folder, fp32, tokens=256, kv_tokens=9 * 64)
    for _ in range(2):  # the second time on pages and slots the first has used
        got = su.replay(eng, prompts, steps)
        for n in prompts:
            close(got[n], want[n], fp32)
    assert len(eng.debug_read("free_pages")) == 9
    eng.close()


@BOTH
def test_rows_do_not_depend_on_the_batch(fp32):
    """A row's logits with 0 to 40 other requests in the step stay within rounding of its own alone."""
    folder, cfg, w = su.model("fast", 1)
    toks = prompt(cfg, 90, 8)
    want, _ = ref.forward(cfg, w, toks)
    eng = su.engine(folder, fp32, tokens=256, seqs=41, kv_tokens=64 * 60)
    for others in (0, 3, 8, 40):
        prompts = {"a": toks, **{f"o{i}": prompt(cfg, 6 + i, 50 + i) for i in range(others)}}
        first = [("a", 80)] + [(n, 3) for n in prompts if n != "a"]
        steps = [first] + [[("a", 1)] + [(n, 1) for n in prompts if n != "a"] for _ in range(3)] + [[("a", 1)]] * 7
        close(su.replay(eng, prompts, steps)["a"], want, fp32)
    eng.close()


# ---- windows, first positions, far keys, sinks
@BOTH
@pytest.mark.parametrize("size,keep", su.WINDOWS)
def test_windows_and_first_positions(size, keep, fp32):
    """Keys that outshine all others just inside and just outside the window and the kept positions, at page borders and between, from
    prompts, portions and decoding (test_sopetar_host.py shows that such keys tell a mask that is one off)."""
    for odd in ("", "_odd"):
        folder, cfg, w = su.model(f"window{size}_{keep}{odd}", 1, su.standing_keys([7]), "standing")
        eng = su.engine(folder, fp32, tokens=512)
        for at in {max(keep - 1, 0), keep, 63, 64, 100}:
            toks = [t if t != 7 else 8 for t in prompt(cfg, 270, 3)]
            toks[at] = 7
            want, _ = ref.forward(cfg, w, toks)
            edge = min(at + size, 260)  # the first position that does not see it
            for sizes in ([270], [max(edge - 2, 1)] + [1] * 6 + [270], [max(edge - 1, 1), 2, 270], [50, 2, 100, 3]):
                close(cut(eng, toks, sizes), want, fp32)
        eng.close()


@BOTH
@pytest.mark.parametrize("name", ["kept", "kept_odd"])
def test_a_kept_key_far_back(name, fp32):
    folder, cfg, w = su.model(name, change=su.standing_keys([7]), tag="standing")
    eng = su.engine(folder, fp32, tokens=512)
    for at in (0, 1, 10, 11):
        toks = [t if t != 7 else 8 for t in prompt(cfg, 400, 3)]
        toks[at] = 7
        want, _ = ref.forward(cfg, w, toks)
        for sizes in ([400], [340] + [1] * 60, [100, 2, 150, 3]):
            close(cut(eng, toks, sizes), want, fp32)
    eng.close()


@BOTH
@pytest.mark.parametrize("name", ["latent", "latent_odd"])
def test_sinks(name, fp32):
    """Sinks that take most of the softmax, from the first position on."""
    folder, cfg, w = su.model(name, change=su.standing_sinks, tag="sinks")
    toks = prompt(cfg, 150, 3)
    want, _ = ref.forward(cfg, w, toks)
    eng = su.engine(folder, fp32, tokens=256)
    for sizes in ([150], [1], [40, 2, 90]):
        close(cut(eng, toks, sizes), want, fp32)
    eng.close()


@BOTH
@pytest.mark.parametrize("far", [-300.0, 200.0])
def test_sinks_far_from_the_scores(far, fp32):
    """Sinks far below all scores leave a plain softmax; far above them, nothing: no sum overflows."""
    cfg = sv.config(128, 96, [sv.latent(4, 64, 16, 64, 64, window=40, scale=0.3, mlp=sv.dense(64)), sv.latent(3, 20, 6, 13, 30, window=30)])
    bits = sv.random_weights(cfg, 7)
    bits["l0.mix.sink"] = sv.to_bf16(np.array([far, 1.0, far, -far], np.float32))
    bits["l1.mix.sink"] = sv.to_bf16(np.full(3, far, np.float32))
    folder = sv.write_model(su._TMP / f"far{far}", cfg, bits)
    w = {k: sv.from_bf16(v).reshape(v.shape).astype(np.float64) for k, v in bits.items()}
    toks = prompt(cfg, 120, 3)
    want, _ = ref.forward(cfg, w, toks)
    eng = su.engine(folder, fp32, tokens=128)
    for sizes in ([120], [60] + [1] * 60):
        close(cut(eng, toks, sizes), want, fp32)
    eng.close()


@BOTH
@pytest.mark.parametrize("name", ["kept", "latent", "mixed"])
def test_long_decoding(name, fp32):
    """400 tokens one by one from the first on."""
    folder, cfg, w = su.model(name, 6)
    toks = prompt(cfg, 400, 5)
    eng = su.engine(folder, fp32, tokens=512)
    got = cut(eng, toks, [1])
    eng.close()
    close(got, ref.forward(cfg, w, toks)[0], fp32)


@pytest.mark.parametrize("keys", [64, 128, 0])
def test_key_splits(keys):
    """A row's positions over one to sixteen blocks of a cluster, in decoding and in a prompt's portion: windows and kept positions that
    begin in the middle of a block's share, sinks that count once."""
    cfg = sv.config(128, 128, [sv.latent(10, 64, 32, 64, 512, window=777, scale=0.15), sv.attention(12, 1, 64, 128, window=601, keep=90, scale=0.3, softcap=15.0),
                               sv.latent(40, 64, 64, 64, 168, window=500, scale=0.15), sv.latent(20, 64, 16, 64, 64, window=900, scale=0.15),
                               sv.attention(4, 2, 128, 128, window=300, keep=400, scale=0.3, softcap=15.0, v_mix=False)])
    bits = sv.random_weights(cfg, 9)
    su.standing_keys([7])(cfg, bits)
    folder = sv.write_model(su._TMP / "splits", cfg, bits)
    w = {k: sv.from_bf16(v).reshape(v.shape).astype(np.float64) for k, v in bits.items()}
    toks = [t if t != 7 else 8 for t in prompt(cfg, 1015, 4)]
    toks[333] = toks[40] = 7
    want, _ = ref.forward(cfg, w, toks)
    eng = su.engine(folder, False, tokens=1024, tuning=E.Tuning(attn_keys_per_cta=keys))
    got = su.replay(eng, {"a": toks, "b": toks[:40]}, [[("a", 880), ("b", 39)], [("a", 1), ("b", 1)]] + [[("a", 1)]] * 12 + [[("a", 3)], [("a", 1)], [("a", 118)]])
    eng.close()
    close(got["a"], want, False)
    close(got["b"], want[:40], False)


def test_averages_over_many_layers():
    """More results than an average's loads go out together for, a share of every one, rows that are no multiple of four."""
    for width in (128, 90):
        cfg = sv.config(width, 96, [sv.attention(2, 1, 16, 16, window=20) if i % 3 == 0 else sv.latent(2, 8, 4, 8, 16, window=11, mlp=sv.dense(32) if i % 2 else None) for i in range(11)], embed_scale=0.5)
        bits = sv.random_weights(cfg, 12)
        for i in range(11):
            share = np.random.default_rng(i).standard_normal(i + 2)
            bits[f"l{i}.dwa"] = sv.to_bf16((0.8 * share).astype(np.float32))
        folder = sv.write_model(su._TMP / f"deep{width}", cfg, bits)
        w = {k: sv.from_bf16(v).reshape(v.shape).astype(np.float64) for k, v in bits.items()}
        toks = prompt(cfg, 70, 3)
        want, _ = ref.forward(cfg, w, toks)
        for fp32 in (True, False):
            eng = su.engine(folder, fp32, tokens=128)
            for sizes in ([70], [33, 1, 2, 5]):
                close(cut(eng, toks, sizes), want, fp32, 2.0)
            eng.close()


# ---- verified drafts
node = lambda depth, parent, sees: depth | parent << 8 | sees << 16


@BOTH
@pytest.mark.parametrize("name", ["odd", "fast"] + ATTENDING + ["mixed"])
def test_draft_tree_rows(name, fp32):
    """A draft tree: each row's logits are those of its own path -- rows lie in the cache at other places than their positions, on both
    sides of a window's edge; the accepted path, which is not a prefix of the rows, is what the caches go on from."""
    folder, cfg, w = su.model(name, 1)
    tried = 0
    for start in (1, 19, 43, 62, 64):
        eng = su.engine(folder, fp32, tokens=256, head_rows=256)
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
            tried += 1
            eng.settle(s, 6 - 3)
            seq = toks + [feed[i] for i in (0, 2, 4)]
            more = prompt(cfg, 9, 99)
            got = [eng.step_rows([E.Run(s, [t])], [[0]], E.StepOptions(read_logits=True)).logits[0] for t in more[:5]]
            got += list(eng.step_rows([E.Run(s, more[5:])], [[0, 1, 2, 3]], E.StepOptions(read_logits=True)).logits)
            close(np.stack(got), ref.forward(cfg, w, seq + more)[0][len(seq):], fp32)
        eng.close()
    assert tried


@BOTH
@pytest.mark.parametrize("name", ["kept", "latent", "mixed_odd"])
def test_a_verified_run_from_the_first_token_beside_a_prompt(name, fp32):
    """A chain verified from an empty sequence in a slot that was used before, in a step with another request's prompt: what is
    rejected leaves no trace."""
    folder, cfg, w = su.model(name, 2)
    eng = su.engine(folder, fp32, tokens=256, head_rows=256)
    used = eng.new_seq()
    eng.step([E.Run(used, prompt(cfg, 30, 1))])
    eng.free_seq(used)
    s, other = eng.new_seq(), eng.new_seq()
    chain, beside, more = prompt(cfg, 5, 2), prompt(cfg, 90, 3), prompt(cfg, 6, 4)
    eng.debug_write("feed", s * 16, chain)
    eng.debug_write("tree", s * 16, [node(i, i - 1 if i else 255, (2 << i) - 1) for i in range(5)])
    out = eng.debug_step([(s, [E.FEED_ROW + i for i in range(5)], E.Rows.LAST, True), (other, beside, E.Rows.LAST, False)], E.StepOptions(read_logits=True))
    close(out.logits[:5], ref.forward(cfg, w, chain)[0], fp32)
    close(out.logits[5:], ref.forward(cfg, w, beside)[0][-1:], fp32)
    n = int(eng.debug_read("path_len")[0])
    assert 1 <= n < 5
    eng.settle(s, 5 - n)
    got = eng.step_rows([E.Run(s, more)], [list(range(6))], E.StepOptions(read_logits=True)).logits
    close(got, ref.forward(cfg, w, chain[:n] + more)[0][n:], fp32)
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
    folder, cfg, w = su.model(name, 2)
    prompts = [prompt(cfg, k, 30 + k) for k in (37, 5, 70, 1, 20)]
    want = [greedy(cfg, w, p, 12) for p in prompts]
    eng = su.engine(folder, True, tokens=32, seqs=3, head_rows=32, kv_tokens=64 * 6)
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
    folder, cfg, w = su.model("odd", 2)
    prompts = {"x": prompt(cfg, 12, 1), "y": prompt(cfg, 33, 2)}
    files.write_requests(tmp_path / "reqs.txt", [files.RequestLine(n, "max_tokens=6,temperature=0", p) for n, p in prompts.items()])
    r = subprocess.run([sys.executable, str(ROOT / "bin" / "generate"), str(folder), str(tmp_path / "reqs.txt"), str(tmp_path / "out.jsonl"), "--dtype", "float32", "--chunk", "16"],
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert files.read_outputs(tmp_path / "out.jsonl") == {n: greedy(cfg, w, p, 6) for n, p in prompts.items()}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay(tmp_path, dtype):
    folder, cfg, w = su.model("fast", 1)
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
    close(np.concatenate([read(0), read(1), read(3)]), np.concatenate([wa[[0, 29]], wb[[29, 5]], wa[[39]]]), dtype == "float32")
    assert not (tmp_path / "2.f32").exists()
