"""The Leduvik design without a GPU: the slow restatement's mechanisms against hand-worked values, mistakes planted in it that
the GPU tests' models must reveal, the folder reader's errors, and the planner over a Leduvik model."""
import json

import numpy as np
import pytest

from silicon_violetto_b200 import build, engine as E, leduvik as lv
from tests import leduvik_ref as ref, leduvik_util as lu

HOST = dict(host_only=True, max_seq_len=128, global_kv_tokens=128)


@pytest.fixture(scope="module", autouse=True)
def built():
    build.build()


def test_norm_is_plain_with_eps_under_the_root():
    assert np.allclose(ref.unit_rms(np.array([[3.0, -4.0]]), 0.0), [[3 / np.sqrt(12.5), -4 / np.sqrt(12.5)]])
    assert np.allclose(ref.unit_rms(np.full((1, 2), 1e-3), 1.0), 1e-3 / np.sqrt(1 + 1e-6))


def test_temperature_steps():
    t = ref.temperature(np.array([0, 8, 9, 18, 19]), 0.5, 10)
    assert np.allclose(t, [1, 1, 1 + 0.5 * np.log(2), 1 + 0.5 * np.log(2), 1 + 0.5 * np.log(3)])


def test_window_counts_its_own_position():
    q, v = np.zeros((5, 1, 2)), np.arange(5.0).reshape(5, 1, 1)
    assert np.allclose(ref.attend(q, q, v, 1.0, 2)[:, 0, 0], [0, 0.5, 1.5, 2.5, 3.5])
    assert np.allclose(ref.attend(q, q, v, 1.0)[:, 0, 0], [0, 0.5, 1, 1.5, 2])


def test_query_heads_share_kv_heads_in_order():
    v = np.array([[[1.0], [2.0]]])
    assert ref.attend(np.zeros((1, 4, 1)), np.zeros((1, 2, 1)), v, 1.0)[0, :, 0].tolist() == [1, 1, 2, 2]


def test_time_mix_reads_before_it_writes():
    one = np.ones((3, 1, 1))
    o = ref.time_mix_core(one, one, np.array([1.0, 10.0, 100.0]).reshape(3, 1, 1), one * 0.5, np.array([[0.25]]))[:, 0, 0]
    assert np.allclose(o, [0.25, 1 + 2.5, (0.5 + 10) + 25])


def test_token_shift_starts_from_zeros():
    assert ref.token_shift(np.array([[2.0], [6.0]]), np.array([0.25]))[:, 0].tolist() == [1.5, 5.0]


def test_state_space_writes_before_it_reads():
    x, B, C, dt = (np.array(v, float).reshape(2, 1, -1) for v in ([1, 10], [2, 3], [1, 1], [0.5, 0.5]))
    y = ref.state_space_core(x, B, C, dt[:, :, 0], np.array([np.log(2.0)]), np.array([0.1]))[:, 0, 0]
    assert np.allclose(y, [1 + 0.1, np.exp(-1.0) * 1 + 0.5 * 30 + 1])


def test_short_conv_and_gate_before_norm():
    assert ref.causal_conv(np.array([[1.0], [10.0], [100.0]]), np.array([[2.0, 3.0]]), np.array([0.5]))[:, 0].tolist() == [3.5, 32.5, 320.5]
    assert np.isclose(ref.softplus(0.0), np.log(2)) and ref.softplus(800.0) == 800.0 and np.isclose(ref.silu(0.0), 0)
    assert ref.feed_forward(np.array([[1.0, -1.0]]), {"up": np.eye(2) * 3, "down": np.eye(2)}, "").tolist() == [[9.0, 0.0]]


def test_loop_order():
    cfg = {"layers": [0, 1, 2, 3], "loop": {"start": 1, "stop": 3, "times": 3}}
    assert ref.layer_order(cfg) == [(0, False), (1, False), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    assert ref.layer_order({"layers": [0, 1], "loop": None}) == [(0, False), (1, False)]


@pytest.mark.parametrize("name", ["window", "window_odd", "window_few"])
def test_standing_keys_tell_a_window_one_token_off(name):
    folder, cfg, w = lu.model(name, change=lu.standing_keys([7]), tag="standing")
    size = cfg["layers"][0]["mixer"]["mask"]["size"]
    toks = [t if t != 7 else 8 for t in lu.prompt(cfg, 20 + size + 6, 3)]
    toks[20] = 7
    right, _ = ref.forward(cfg, w, toks)
    for other, at in ((size + 1, 20 + size), (size - 1, 20 + size - 1)):
        wrong = json.loads(json.dumps(cfg))
        wrong["layers"][0]["mixer"]["mask"]["size"] = other
        assert lu.error(ref.forward(wrong, w, toks)[0], right)[at] > 5 * lu.LIMIT[False]


@pytest.mark.parametrize("name", ["beside", "beside_odd"])
def test_standing_keys_tell_a_lost_far_key(name):
    folder, cfg, w = lu.model(name, change=lu.standing_keys([7]), tag="standing")
    toks = [t if t != 7 else 8 for t in lu.prompt(cfg, 200, 3)]
    lost = list(toks)
    toks[3] = 7
    assert lu.error(ref.forward(cfg, w, lost)[0], ref.forward(cfg, w, toks)[0])[60:].min() > 5 * lu.LIMIT[False]


@pytest.mark.parametrize("name", ["state", "state_odd", "beside", "beside_odd"])
def test_long_memories_tell_a_lost_state(name):
    """The rows before position 40 gone from a state (and, just behind the cut, from the ring beside it)."""
    folder, cfg, w = lu.model(name, 2, lu.long_memory, "memory")
    toks = lu.prompt(cfg, 60, 4)
    cut = dict(w, pos=w["pos"][40:])
    e = lu.error(ref.forward(cfg, cut, toks[40:])[0], ref.forward(cfg, w, toks)[0][40:])
    assert e[:8].min() > 3 * lu.LIMIT[False] and e.min() > 1000 * lu.LIMIT[True]


def test_reader_takes_every_layers_own_sizes():
    for name, cfg in lu.CONFIGS.items():
        folder, _, _ = lu.model(name)
        eng = E.Engine(folder, E.EngineConfig(**HOST))
        assert (eng.desc.n_layers, eng.desc.d_model, eng.desc.vocab, eng.desc.page_size) == (len(ref.layer_order(cfg)), cfg["width"], cfg["vocab"], 64)
        eng.close()


def test_reader_errors(tmp_path):
    cfg = lu.CONFIGS["odd"]
    bits = lv.random_weights(cfg)

    def fails(match, c=cfg, b=bits):
        lv.write_model(tmp_path / "m", c, b)
        with pytest.raises(E.EngineError, match=match):
            E.Engine(tmp_path / "m", E.EngineConfig(**HOST))

    def changed(i, **kw):
        c = json.loads(json.dumps(cfg))
        c["layers"][i].update({k: v for k, v in kw.items() if k in ("type", "mlp")})
        c["layers"][i]["mixer"].update({k: v for k, v in kw.items() if k not in ("type", "mlp")})
        return c

    fails("no tensor l2.mix.right.w1", b={k: v for k, v in bits.items() if k != "l2.mix.right.w1"})
    fails("no tensor pos", b={k: v for k, v in bits.items() if k != "pos"})
    fails(r"l0.mix.o: expected BF16 \[88, 168\], found BF16 \[168, 88\]", b=dict(bits, **{"l0.mix.o": bits["l0.mix.o"].T}))
    fails(r"l2.mix.right.w2: expected BF16 \[27, 16\]", b=dict(bits, **{"l2.mix.right.w2": bits["l2.mix.right.w2"][:, :5]}))
    fails("no mixer named other", changed(1, type="other"))
    fails("no feed-forward named moe", changed(0, mlp={"kind": "moe"}))
    fails("a window of 0 positions", changed(0, mask={"size": 0}))
    fails("the heads do not fit the groups", changed(1, groups=4))
    fails("the norm's groups do not fit the heads", changed(1, norm_groups=4))
    fails("a state of at most 512 channels", changed(1, state=513))
    fails("a convolution takes 1 to 32 taps", changed(1, conv=33))
    fails("the heads do not fit the kv heads", changed(0, kv_heads=4))
    fails("no field `max_positions`", {k: v for k, v in cfg.items() if k != "max_positions"})
    fails("no field `logit_scale`", {k: v for k, v in cfg.items() if k != "logit_scale"})
    fails("the loop does not fit the layers", dict(cfg, loop={"start": 0, "stop": 7, "times": 2}))


def test_planner_pages_and_the_last_position():
    folder, _, _ = lu.model("odd")
    eng = E.Engine(folder, E.EngineConfig(host_only=True, max_seqs=3, max_step_tokens=1024, max_chunk=1024, max_seq_len=4096, global_kv_tokens=1024, max_head_rows=64))
    a, b = eng.new_seq(), eng.new_seq()
    eng.debug_plan([(a, [1] * 64, E.Rows.NONE, False), (b, [1] * 65, E.Rows.LAST, False)])
    assert len(eng.debug_read("free_pages")) == 16 - 3
    with pytest.raises(E.EngineError, match=r"would reach 701 tokens \(max 700\)"):
        eng.debug_plan([(a, [1] * 637, E.Rows.NONE, False)])
    eng.close()
