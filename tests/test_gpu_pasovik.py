"""The Pasovik design on the GPU against the slow restatement (pasovik_ref.py): its mechanisms, prompts, decoding, portions, batches,
far keys, reused pages and slots, verified drafts, generation, and the trace replay program; in 32-bit and in bf16."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest

from silicon_violetto_b200 import engine as E, files, pasovik as pv
from tests import pasovik_ref as ref, pasovik_util as pu

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parents[1]
BOTH = pytest.mark.parametrize("fp32", [True, False], ids=["fp32", "bf16"])
SINGLE = ["capped", "capped_odd", "latent", "latent_odd", "latent_pair", "fade", "fade_odd", "experts", "experts_odd", "dense"]
prompt = pu.prompt


def close(got, want, fp32, factor=1.0):
    """In bf16 a few positions feel the rounding more than others: those whose sublayers leave little in front of their norms. (Mistakes
    cost more: test_pasovik_host.py.)"""
    e = pu.error(got, want)
    assert e.max() < (1 if fp32 else 2) * factor * pu.LIMIT[fp32], (int(e.argmax()), float(e.max()))
    assert np.median(e) < 0.5 * factor * pu.LIMIT[fp32], float(np.median(e))


def cut(eng, toks, sizes):
    return pu.replay(eng, {"a": toks}, [[("a", c)] for c in pu.portions(len(toks), sizes)])["a"]


# ---- mechanisms, through the layer captures
@BOTH
@pytest.mark.parametrize("name", SINGLE)
def test_layers(name, fp32):
    """The stream before and after each layer, of a prompt over several pages; the attentions' own outputs."""
    folder, cfg, w = pu.model(name, 3)
    toks, eps = prompt(cfg, 210, 1), cfg["norm"]["eps"]
    eng = pu.engine(folder, fp32)
    out, caps = eng.step_capture([E.Run(eng.new_seq(), toks)], E.StepOptions(head=E.Rows.ALL, read_logits=True))
    eng.close()
    logits, runs = ref.forward(cfg, w, toks)
    x, kept, tol = w["embed"][toks], {}, 2e-5 if fp32 else 4e-2
    for i, lc in enumerate(cfg["layers"]):
        assert np.abs(caps[i]["resid_in"] - x).max() < tol * np.abs(x).max()
        m, pre = lc["mixer"], f"l{i}.mix."
        if lc["type"] != "lightning":
            if lc["type"] == "attention":
                want = ref.attention_heads(x, w, pre, m, eps)
            else:
                if m.get("kv_from") is None:
                    kept[i] = ref.latent_rows(x, w, pre, m, eps)
                want = ref.latent_heads(x, w, pre, m, eps, kept[m.get("kv_from", i)])
            assert np.abs(caps[i]["sdpa_out"] - want).max() < tol * np.abs(want).max()
        x = runs[i]
        assert np.abs(caps[i]["resid_out"] - x).max() < tol * np.abs(x).max()
    close(out.logits, logits, fp32)


@BOTH
@pytest.mark.parametrize("name", [n for n in pu.CONFIGS if n.startswith("rank")])
def test_latent_sizes(name, fp32):
    """Every size the latent kernel is laid out for, and others, in prompts and token by token."""
    folder, cfg, w = pu.model(name, 4, pu.standing_keys([7]), "standing")
    toks = [t if t != 7 else 8 for t in prompt(cfg, 150, 2)]
    toks[5] = toks[70] = 7
    want, _ = ref.forward(cfg, w, toks)
    eng = pu.engine(folder, fp32, tokens=256)
    for sizes in ([150], [33, 2, 1, 17, 64], [140] + [1] * 10):
        close(cut(eng, toks, sizes), want, fp32)
    eng.close()


@BOTH
@pytest.mark.parametrize("name", [n for n in pu.CONFIGS if n.startswith("wide")])
def test_key_channels(name, fp32):
    """Every size of state a kernel is built for, in prompts and token by token."""
    folder, cfg, w = pu.model(name, 4)
    toks = prompt(cfg, 70, 2)
    want, _ = ref.forward(cfg, w, toks)
    eng = pu.engine(folder, fp32, tokens=128)
    for sizes in ([70], [33, 2, 1, 17], [1]):
        close(cut(eng, toks, sizes), want, fp32)
    eng.close()


@pytest.mark.parametrize("decays", [[1.0, 1e-30, 0.999, 0.5], [1.5e-5, 1.0, 0.9999, 1.0], [0.0, 1.0, 0.3, 0.9], [1.02, 0.5, 1.0, 0.9]], ids=["tiny", "ones", "zero", "growing"])
def test_decays_at_their_ends(decays):
    """Decays that keep everything and nothing, in chunks on the tensor cores where they take them, beside the recurrence token by token."""
    cfg = pv.config(128, 160, [pv.lightning(64, 32, decays), pv.lightning(128, 64, decays[::-1])])
    bits = pv.random_weights(cfg, 21)
    folder = pv.write_model(pu._TMP / f"ends_{decays[0]}", cfg, bits)
    w = {k: pv.from_bf16(v).astype(np.float64) for k, v in bits.items()}
    toks, other = prompt(cfg, 300, 6), prompt(cfg, 40, 7)
    want, want_other = ref.forward(cfg, w, toks)[0], ref.forward(cfg, w, other)[0]
    fast, plain, exact = pu.engine(folder, False), pu.engine(folder, False, tuning=E.Tuning(plain_attention=True)), pu.engine(folder, True)
    for sizes in ([300], [31, 32, 33], [64, 1, 63, 65, 2], [1, 127, 129], [200, 100]):
        got = cut(fast, toks, sizes)
        close(got, want, False, 0.5)
        close(got, cut(plain, toks, sizes), False, 0.5)
        close(cut(exact, toks, sizes), want, True)
    got = pu.replay(fast, {"a": toks, "b": other}, [[("a", 100), ("b", 3)], [("b", 30), ("a", 33)], [("b", 1), ("a", 167)], [("b", 6)]])
    close(got["a"], want, False, 0.5)
    close(got["b"], want_other, False, 0.5)
    for e in (fast, plain, exact):
        e.close()


@pytest.mark.parametrize("dim,vdim", [(64, 32), (128, 64)])
def test_chunks_of_many_heads(dim, vdim):
    """Enough heads, or runs, that a block of the tensor cores' recurrence has 32 value channels; fewer give it 16."""
    cfg = pv.config(64, 96, [pv.lightning(dim, vdim, list(np.linspace(0.4, 0.999, 80)))], side=9)
    bits = pv.random_weights(cfg, 22)
    folder = pv.write_model(pu._TMP / f"many_{dim}", cfg, bits)
    w = {k: pv.from_bf16(v).astype(np.float64) for k, v in bits.items()}
    prompts = {n: prompt(cfg, k, 8 + k) for n, k in (("a", 150), ("b", 97), ("c", 40))}
    eng = pu.engine(folder, False)
    got = pu.replay(eng, prompts, [[("a", 70), ("b", 64), ("c", 33)], [("c", 1), ("a", 33), ("b", 1)], [("b", 32), ("a", 47), ("c", 6)]])
    eng.close()
    for n, toks in prompts.items():
        close(got[n], ref.forward(cfg, w, toks)[0], False)


@BOTH
@pytest.mark.parametrize("top,experts", [(1, 1), (4, 4), (2, 40)])
def test_choices_of_experts(top, experts, fp32):
    """One expert, all of them, and more than a warp holds; scores near 0 and 1."""
    cfg = pv.config(128, 160, [pv.lightning(32, 32, [0.9], mlp=pv.moe(experts, top, 64, limit=0.6))])
    bits = pv.random_weights(cfg, 5)
    pu.decided_routing(cfg, bits)
    bits["l0.mlp.router"] = pv.to_bf16(pv.from_bf16(bits["l0.mlp.router"]) * 4).reshape(bits["l0.mlp.router"].shape)
    folder = pv.write_model(pu._TMP / f"choices_{top}_{experts}", cfg, bits)
    w = {k: pv.from_bf16(v).astype(np.float64) for k, v in bits.items()}
    toks = prompt(cfg, 300, 3)
    want, _ = ref.forward(cfg, w, toks)
    eng = pu.engine(folder, fp32)
    for sizes in ([300], [100, 7, 1, 2, 150]):
        close(cut(eng, toks, sizes), want, fp32)
    eng.close()


# ---- whole prompts, decoding, portions, batches
@BOTH
@pytest.mark.parametrize("name", ["odd", "fast"] + SINGLE)
def test_prompt_decode_and_portions(name, fp32):
    folder, cfg, w = pu.model(name, 1)
    toks = prompt(cfg, 230, 2)
    want, _ = ref.forward(cfg, w, toks)
    eng = pu.engine(folder, fp32, tokens=256)
    whole = cut(eng, toks, [230])
    close(whole, want, fp32)
    for sizes in ([2], [150] + [1] * 80, [3, 2, 17, 64, 9, 1, 1, 5], [63, 2, 65]):
        got = cut(eng, toks, sizes)
        close(got, want, fp32)
        if fp32:
            close(got, whole, fp32)
    eng.close()


@BOTH
@pytest.mark.parametrize("name", ["fade", "fade_odd", "latent_pair"])
def test_nothing_is_lost_at_any_cut(name, fp32):
    """Cuts at every place around a page's and a chunk's edge: what a cut loses of the states or the shared latents would show."""
    folder, cfg, w = pu.model(name, 2)
    toks = prompt(cfg, 140, 4)
    want, _ = ref.forward(cfg, w, toks)
    eng = pu.engine(folder, fp32, tokens=256)
    for first in (1, 2, 7, 8, 9, 15, 16, 17, 31, 32, 33, 63, 64, 65):
        close(cut(eng, toks, [first, 2, 1, 9, 140]), want, fp32)
        close(cut(eng, toks, [first, first, 3, 140]), want, fp32)
    eng.close()


@BOTH
@pytest.mark.parametrize("name", ["odd", "fast"])
def test_unequal_batches_and_reused_pages_and_slots(name, fp32):
    """Portions of prompts beside single tokens of others, requests left out of steps, ended and replaced in a pool that holds
    only the live ones: every request as if it were alone."""
    folder, cfg, w = pu.model(name, 1)
    lens = {"a": 140, "b": 9, "c": 65, "d": 100, "e": 130, "f": 3, "g": 64}
    prompts = {n: prompt(cfg, k, 10 + i) for i, (n, k) in enumerate(lens.items())}
    steps = [[("a", 50), ("b", 1), ("c", 2)], [("b", 2), ("c", 3), ("d", 20)], [("a", 1), ("c", 1), ("b", 6)], [("a", 1), ("c", 59), ("d", 1)],
             [("d", 2), ("e", 90), ("a", 70)], [("a", 1), ("d", 1), ("e", 1), ("f", 3)], [("a", 17), ("e", 2), ("d", 76), ("g", 40)], [("e", 37), ("g", 24)]]
    want = {n: ref.forward(cfg, w, toks)[0] for n, toks in prompts.items()}
    eng = pu.engine(folder, fp32, tokens=256, kv_tokens=9 * 64)
    for _ in range(2):  # the second time on pages and slots the first has used
        got = pu.replay(eng, prompts, steps)
        for n in prompts:
            close(got[n], want[n], fp32)
    assert len(eng.debug_read("free_pages")) == 9
    eng.close()


@BOTH
def test_rows_do_not_depend_on_the_batch(fp32):
    """A row's logits with 0 to 40 other requests in the step stay within rounding of its own alone."""
    folder, cfg, w = pu.model("fast", 1)
    toks = prompt(cfg, 90, 8)
    want, _ = ref.forward(cfg, w, toks)
    eng = pu.engine(folder, fp32, tokens=256, seqs=41, kv_tokens=64 * 60)
    for others in (0, 3, 8, 40):
        prompts = {"a": toks, **{f"o{i}": prompt(cfg, 6 + i, 50 + i) for i in range(others)}}
        first = [("a", 80)] + [(n, 3) for n in prompts if n != "a"]
        steps = [first] + [[("a", 1)] + [(n, 1) for n in prompts if n != "a"] for _ in range(3)] + [[("a", 1)]] * 7
        close(pu.replay(eng, prompts, steps)["a"], want, fp32)
    eng.close()


# ---- far keys, long runs
@BOTH
@pytest.mark.parametrize("name", ["capped", "capped_odd", "latent", "latent_odd", "latent_pair"])
def test_a_far_key(name, fp32):
    """A key that outshines all others hundreds of tokens back, at page borders and at the very start, from prompts and decoding
    (test_pasovik_host.py shows that these models tell its loss)."""
    folder, cfg, w = pu.model(name, change=pu.standing_keys([7]), tag="standing")
    eng = pu.engine(folder, fp32, tokens=512)
    for at in (0, 1, 63, 64, 200):
        toks = [t if t != 7 else 8 for t in prompt(cfg, 340, 3)]
        toks[at] = 7
        want, _ = ref.forward(cfg, w, toks)
        for sizes in ([340], [300] + [1] * 40, [100, 2, 150, 3]):
            close(cut(eng, toks, sizes), want, fp32)
    eng.close()


@BOTH
@pytest.mark.parametrize("name", ["capped", "latent_pair", "fade"])
def test_long_decoding(name, fp32):
    """400 tokens one by one from the first on."""
    folder, cfg, w = pu.model(name, 6)
    toks = prompt(cfg, 400, 5)
    eng = pu.engine(folder, fp32, tokens=512)
    got = cut(eng, toks, [1])
    eng.close()
    close(got, ref.forward(cfg, w, toks)[0], fp32)


@pytest.mark.parametrize("keys", [64, 128, 0])
def test_key_splits(keys):
    """A row's positions over one to sixteen blocks of a cluster, in decoding and in a prompt's portion, with ranks between those the
    kernel is laid out for; a key that outshines all others in one block's share."""
    cfg = pv.config(128, 128, [pv.latent(10, 64, 32, 64, 512, 64, scale=0.15), pv.latent(40, 64, 64, 64, 168, 64, scale=0.15), pv.latent(20, 64, 16, 64, 64, 64, scale=0.15),
                               pv.attention(12, 1, 64, 128, 0.3, softcap=15.0, rot_dims=32)])
    bits = pv.random_weights(cfg, 9)
    pu.standing_keys([7])(cfg, bits)
    folder = pv.write_model(pu._TMP / "splits", cfg, bits)
    w = {k: pv.from_bf16(v).astype(np.float64) for k, v in bits.items()}
    toks = [t if t != 7 else 8 for t in prompt(cfg, 1015, 4)]
    toks[333] = 7
    want, _ = ref.forward(cfg, w, toks)
    eng = pu.engine(folder, False, tokens=1024, tuning=E.Tuning(attn_keys_per_cta=keys))
    got = pu.replay(eng, {"a": toks, "b": toks[:40]}, [[("a", 880), ("b", 39)], [("a", 1), ("b", 1)]] + [[("a", 1)]] * 12 + [[("a", 3)], [("a", 1)], [("a", 118)]])
    eng.close()
    close(got["a"], want, False)
    close(got["b"], want[:40], False)


# ---- verified drafts
node = lambda depth, parent, sees: depth | parent << 8 | sees << 16


@BOTH
@pytest.mark.parametrize("name", ["odd", "fast", "capped", "latent_pair", "fade", "fade_odd"])
def test_draft_tree_rows_and_states(name, fp32):
    """A draft tree: each row's logits are those of its own path; the accepted path, which is not a prefix of the rows, is what
    caches (those that several layers read, too) and states go on from."""
    folder, cfg, w = pu.model(name, 1)
    tried = 0
    for start in (1, 19, 62, 64):
        eng = pu.engine(folder, fp32, tokens=256, head_rows=256)
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
@pytest.mark.parametrize("name", ["latent_pair", "fade"])
def test_a_verified_run_from_the_first_token_beside_a_prompt(name, fp32):
    """A chain verified from an empty sequence in a slot that was used before, in a step with another request's prompt: what is
    rejected leaves no trace."""
    folder, cfg, w = pu.model(name, 2)
    eng = pu.engine(folder, fp32, tokens=256, head_rows=256)
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


@BOTH
def test_a_finished_sequence_keeps_its_state(fp32):
    """The step queued behind the one that ended a sequence does not move it: it may go on later."""
    folder, cfg, w = pu.model("odd", 3)
    eng = pu.engine(folder, fp32)
    s, toks, more = eng.new_seq(), prompt(cfg, 20, 1), prompt(cfg, 10, 2)
    eng.step([E.Run(s, toks)])
    eng.set_gen(s, 0xFFFFFFFF)
    per = len(eng.debug_read("gen")) // 4
    eng.debug_write("gen", s * per + 1, [1])  # done
    eng.step([E.Run(s, [5])])
    eng.settle(s, 1)
    eng.debug_write("gen", s * per + 1, [0])
    got = eng.step_rows([E.Run(s, more)], [list(range(10))], E.StepOptions(read_logits=True)).logits
    eng.close()
    close(got, ref.forward(cfg, w, toks + more)[0][20:], fp32)


# ---- generation
def greedy(cfg, w, toks, n):
    out = list(toks)
    for _ in range(n):
        out.append(int(ref.forward(cfg, w, out)[0][-1].argmax()))
    return out[len(toks):]


@pytest.mark.parametrize("name", ["odd", "fast"])
def test_greedy_generation_through_the_scheduler(name):
    """More requests than slots through Generator: prompts in chunks beside decoding, plain and with replayed drafts."""
    folder, cfg, w = pu.model(name, 2)
    prompts = [prompt(cfg, k, 30 + k) for k in (37, 5, 70, 1, 20)]
    want = [greedy(cfg, w, p, 12) for p in prompts]
    eng = pu.engine(folder, True, tokens=32, seqs=3, head_rows=32, kv_tokens=64 * 6)
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
    folder, cfg, w = pu.model("odd", 2)
    prompts = {"x": prompt(cfg, 12, 1), "y": prompt(cfg, 33, 2)}
    files.write_requests(tmp_path / "reqs.txt", [files.RequestLine(n, "max_tokens=6,temperature=0", p) for n, p in prompts.items()])
    r = subprocess.run([sys.executable, str(ROOT / "bin" / "generate"), str(folder), str(tmp_path / "reqs.txt"), str(tmp_path / "out.jsonl"), "--dtype", "float32", "--chunk", "16"],
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert files.read_outputs(tmp_path / "out.jsonl") == {n: greedy(cfg, w, p, 6) for n, p in prompts.items()}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay(tmp_path, dtype):
    folder, cfg, w = pu.model("fast", 1)
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
