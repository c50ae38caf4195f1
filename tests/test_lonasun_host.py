"""The Lonasun design without a GPU: the slow restatement's mechanisms against hand-worked values and against each other,
the folder reader's errors, and the planner over a Lonasun model."""
import json

import numpy as np
import pytest

from tests import lonasun_ref as ref
from silicon_violetto_b200 import build, engine as E, lonasun
from tests import lonasun_util as lu, util


@pytest.fixture(scope="module", autouse=True)
def built():
    build.build()


def test_rms_norm_weight_is_around_zero():
    x = np.array([[3.0, -4.0]])
    assert np.allclose(ref.rms_norm(x, np.array([0.0, 0.5]), 0.0), [[3 / np.sqrt(12.5), -6 / np.sqrt(12.5)]])
    assert np.allclose(ref.rms_norm(np.zeros((1, 2)) + 1e-3, np.zeros(2), 1.0), 1e-3 / np.sqrt(1 + 1e-6))


def test_short_conv_is_causal_and_starts_from_zeros():
    y = ref.short_conv(np.array([[1.0], [10.0], [100.0]]), np.array([[2.0, 3.0]]))
    assert y[:, 0].tolist() == [3.0, 32.0, 320.0]


def test_rotation_pairs_half_a_rotation_apart():
    x = np.arange(1.0, 7.0).reshape(1, 1, 6)
    y = ref.rotate(x, np.array([2.0]), 9.0, 4)[0, 0]
    for i, f in ((0, 1.0), (1, 9.0 ** -0.5)):
        c, s = np.cos(2 * f), np.sin(2 * f)
        assert np.allclose([y[i], y[i + 2]], [x[0, 0, i] * c - x[0, 0, i + 2] * s, x[0, 0, i + 2] * c + x[0, 0, i] * s])
    assert y[4] == 5.0 and y[5] == 6.0


def test_chunks_are_counted_from_the_first_position():
    q = np.zeros((5, 1, 2))
    v = np.arange(5.0).reshape(5, 1, 1)
    o = ref.chunked_attention(q, q, v, 1.0, 3)[:, 0, 0]
    assert np.allclose(o, [0, 0.5, 1, 3, 3.5])


def test_router_chooses_by_corrected_scores_and_weighs_by_scores():
    z = np.log(np.array([[0.5, 0.3, 0.2]]))
    ids, w = ref.route(z, np.eye(3), np.array([-0.4, 0.0, 0.0]), 2)
    assert ids[0].tolist() == [1, 2] and np.allclose(w[0], [0.6, 0.4])


def test_loop_order():
    cfg = {"layers": [0, 1, 2, 3], "loop": {"start": 1, "stop": 3, "times": 2}}
    assert ref.layer_order(cfg) == [(0, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    assert ref.layer_order({"layers": [0, 1], "loop": None}) == [(0, False), (1, False)]


@pytest.mark.parametrize("name", ["one", "one_odd"])
def test_standing_keys_tell_every_edge(name):
    """The models the edge tests use do show a chunk that is one position off, a lost key and a lost convolution row: planted
    in the restatement, each moves the logits by far more than the engines' limits."""
    folder, cfg, w = lu.model(name, change=lu.standing_keys([7]), tag="standing")
    size, taps = cfg["layers"][0]["mixer"]["mask"]["size"], cfg["layers"][0]["mixer"]["conv"]
    rng = np.random.default_rng(1)
    toks = rng.integers(10, 200, size + 12)
    toks[size - 1] = 7   # the last of the first chunk
    toks[1] = 7          # far from the chunk's end
    right, _ = ref.forward(cfg, w, toks)
    for other, at in ((size + 1, [size]), (size - 1, [size, size + 1, size + 3])):
        wrong = json.loads(json.dumps(cfg))
        wrong["layers"][0]["mixer"]["mask"]["size"] = other
        got, _ = ref.forward(wrong, w, toks)
        assert lu.error(got, right)[at].min() > 5 * lu.LIMIT[False]
    lost = toks.copy()
    lost[1] = 11
    got, _ = ref.forward(cfg, w, lost)
    assert lu.error(got, right)[20:size - 1].min() > 3 * lu.LIMIT[False]
    if taps > 1:  # the rows before position 30 lost from the convolution's state
        cut = dict(w)
        a, b = (ref.forward(cfg, cut, toks[lo:40])[0][30 - lo] for lo in (0, 30))
        assert lu.error(b[None], a[None])[0] > 2 * lu.LIMIT[False]


def test_reader_takes_every_layers_own_sizes():
    for name, cfg in lu.CONFIGS.items():
        folder, _, _ = lu.model(name)
        eng = E.Engine(folder, E.EngineConfig(host_only=True, max_seq_len=256, global_kv_tokens=256))
        runs = len(ref.layer_order(cfg))
        assert (eng.desc.n_layers, eng.desc.d_model, eng.desc.vocab, eng.desc.page_size) == (runs, cfg["width"], cfg["vocab"], 64)
        eng.close()


def test_reader_errors(tmp_path):
    cfg = lu.CONFIGS["one"]
    bits = lonasun.random_weights(cfg)
    host = E.EngineConfig(host_only=True, max_seq_len=128, global_kv_tokens=128)

    def fails(match, c=cfg, b=bits):
        lonasun.write_model(tmp_path / "m", c, b)
        with pytest.raises(E.EngineError, match=match):
            E.Engine(tmp_path / "m", host)

    fails("no architecture named Other", dict(cfg, architecture="Other"))
    fails("no tensor l0.mix.g", b={k: v for k, v in bits.items() if k != "l0.mix.g"})
    fails(r"l0.mix.o: expected BF16 \[128, 256\], found BF16 \[256, 128\]", b=dict(bits, **{"l0.mix.o": bits["l0.mix.o"].T}))
    fails("no mixer named other", dict(cfg, layers=[dict(cfg["layers"][0], type="other")]))
    fails("no feed-forward named dense", dict(cfg, layers=[dict(cfg["layers"][0], mlp={"kind": "dense"})]), dict(bits, **{"l0.norm2": bits["l0.norm1"]}))
    fails("no field `width`", {k: v for k, v in cfg.items() if k != "width"})
    fails("the loop does not fit the layers", dict(cfg, loop={"start": 0, "stop": 2, "times": 1}))
    lonasun.write_model(tmp_path / "m", cfg, bits)
    (tmp_path / "m" / "config.json").write_text("{")
    with pytest.raises(E.EngineError, match="not valid JSON"):
        E.Engine(tmp_path / "m", host)
    (tmp_path / "m" / "config.json").write_text(json.dumps(cfg))
    (tmp_path / "m" / "model.safetensors").write_bytes(b"\xff" * 64)
    with pytest.raises(E.EngineError, match="longer than the file"):
        E.Engine(tmp_path / "m", host)


def test_fp32_is_refused_where_there_is_no_such_path():
    with pytest.raises(E.EngineError, match="no fp32 path"):
        E.Engine(util.weights("micro"), E.EngineConfig(host_only=True, fp32=True, max_seq_len=128, global_kv_tokens=128))


def test_planner_pages_of_64_and_their_reuse():
    folder, _, _ = lu.model("one")
    eng = E.Engine(folder, E.EngineConfig(host_only=True, max_seqs=3, max_step_tokens=128, max_chunk=128, max_seq_len=256, global_kv_tokens=256, max_head_rows=64))
    a, b = eng.new_seq(), eng.new_seq()
    eng.debug_plan([(a, [1] * 64, E.Rows.NONE, False), (b, [1] * 3, E.Rows.LAST, False)])
    assert eng.debug_read("free_pages").tolist() == [3, 2]
    eng.debug_plan([(a, [1], E.Rows.LAST, False)])
    assert eng.debug_read("page_table").reshape(3, -1)[a][:2].tolist() == [0, 2]
    eng.free_seq(a)
    c = eng.new_seq()
    assert c == a and len(eng.debug_read("free_pages")) == 3
    with pytest.raises(E.EngineError, match="KV pool exhausted"):
        for _ in range(3):
            eng.debug_plan([(c, [1] * 80, E.Rows.NONE, False)])
    with pytest.raises(E.EngineError, match="row 3 of a run of 3"):
        eng.step_rows([E.Run(b, [1, 2, 3])], [[3]])
    eng.close()
