"""The Pasovik design without a GPU: the slow restatement's mechanisms against hand-worked values, mistakes planted in it that the
GPU tests' models must reveal, the folder reader's errors, and the planner over a Pasovik model."""
import json

import numpy as np
import pytest

from silicon_violetto_b200 import build, engine as E, pasovik as pv
from tests import pasovik_ref as ref, pasovik_util as pu

HOST = dict(host_only=True, max_seq_len=128, global_kv_tokens=128)
TELLS = 5 * pu.LIMIT[False]


@pytest.fixture(scope="module", autouse=True)
def built():
    build.build()


def test_norm_is_plain_with_eps_under_the_root():
    assert np.allclose(ref.rms_norm(np.array([[3.0, -4.0]]), np.array([2.0, 1.0]), 0.0), [[6 / np.sqrt(12.5), -4 / np.sqrt(12.5)]])
    assert np.allclose(ref.rms_norm(np.full((1, 2), 1e-3), 1.0, 1.0), 1e-3 / np.sqrt(1 + 1e-6))


def test_neighbours_turn_by_the_scaled_position():
    x = np.zeros((3, 1, 5))
    x[:, 0] = [1, 0, 0, 2, 7]
    y = ref.rotate(x, {"dims": 4, "base": 100.0, "scaling": {"factor": 2.0}})[:, 0]
    assert np.allclose(y[0], [1, 0, 0, 2, 7])
    assert np.allclose(y[2], [np.cos(1.0), np.sin(1.0), -2 * np.sin(0.1), 2 * np.cos(0.1), 7])
    assert np.allclose(ref.rotate(x, {"dims": 2, "base": 100.0})[2, 0], [np.cos(2.0), np.sin(2.0), 0, 2, 7])


def test_scores_are_capped_before_the_softmax():
    q, k, v = np.full((2, 1, 1), 1.0), np.array([[[0.0]], [[100.0]]]), np.array([[[0.0]], [[1.0]]])
    assert np.isclose(ref.causal(q, k, v, 1.0, 2.0)[1, 0, 0], 1 / (1 + np.exp(-2.0)))
    assert ref.causal(q, k, v, 1.0)[0, 0, 0] == 0


def test_query_heads_share_kv_heads_in_order():
    v = np.array([[[1.0], [2.0]]])
    assert ref.causal(np.zeros((1, 4, 1)), np.zeros((1, 2, 1)), v, 1.0)[0, :, 0].tolist() == [1, 1, 2, 2]


def test_linear_attention_fades_writes_then_reads():
    one = np.ones((3, 1, 1))
    assert np.allclose(ref.lightning_core(one * 2, one, np.array([1.0, 10.0, 100.0]).reshape(3, 1, 1), [0.5])[:, 0, 0], [2, 21, 210.5])


def test_experts_take_scaled_inputs():
    w = {"router": np.array([[1.0], [-1.0], [0.5]]), **{f"e{e}.{c}": np.array([[float(e + 1)]]) for e in range(3) for c in ("gate", "up", "down")}}
    m = {"router": {"top": 2}, "expert": {"limit": 0.75}}
    ids, s = ref.chosen(np.array([[2.0]]), w, "", m)
    assert ids.tolist() == [[0, 2]] and np.allclose(s, [[1 / (1 + np.exp(-2.0)), 1 / (1 + np.exp(-1.0))]])
    g = 0.75  # (both experts' inputs are past the limit)
    assert np.allclose(ref.experts(np.array([[2.0]]), w, "", m), g * ref.sigmoid(1.702 * g) * 1.75 * (1 + 3))
    assert np.allclose(ref.expert(np.array([[-3.0]]), w, "e0.", 0.75), -3 * ref.sigmoid(-1.702 * 3) * 0.25)


def test_side_input_reads_its_layers_span():
    w = {"side.embed": np.array([[1.0, 2, 3, 4], [5, 6, 7, 8]]), "l1.side.gate": np.full((2, 1), 30.0), "l1.side.proj": np.array([[1.0, 0.0]]), "l1.side.norm": np.array([2.0])}
    y = ref.side_input(np.ones((2, 1)), w, 1, [1, 0], 2, 0.0)
    assert np.allclose(y, [[2.0], [2.0]]) and np.isclose(ref.gelu_tanh(1.0), 0.841192, atol=1e-6)
    assert np.allclose(ref.side_input(np.ones((2, 1)), w, 1, [1, 0], 2, 1e4)[:, 0], [2 * 210 / np.sqrt(210 ** 2 + 1e4), 2 * 90 / np.sqrt(90 ** 2 + 1e4)])


def test_dense_is_gated_by_silu():
    w = {"gate": np.array([[1.0]]), "up": np.array([[3.0]]), "down": np.array([[2.0]])}
    assert np.isclose(ref.dense(np.array([[2.0]]), w, "")[0, 0], 2 * 6 * 2 / (1 + np.exp(-2.0)))


# ---- the models tell mistakes
def differs(name, toks, monkeypatch=None, wrong_cfg=None, **wrong):
    """The error per position of the restatement with some of its functions replaced, or with another configuration."""
    folder, cfg, w = pu.model(name, 1)
    right, _ = ref.forward(cfg, w, toks)
    for k, f in wrong.items():
        monkeypatch.setattr(ref, k, f)
    return pu.error(ref.forward(wrong_cfg or cfg, w, toks)[0], right)


def edited(name, i, path, value):
    cfg = json.loads(json.dumps(pu.CONFIGS[name]))
    at = cfg["layers"][i]
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    return cfg


@pytest.mark.parametrize("name,path,value", [("capped", ("mixer", "softcap"), 1e6), ("capped", ("mixer", "rot", "scaling", "factor"), 1.0), ("capped", ("mixer", "rot", "dims"), 30),
                                             ("capped", ("mixer", "rot", "base"), 20000.0), ("capped", ("mixer", "scale"), 0.3), ("latent", ("mixer", "rot", "base"), 20000.0),
                                             ("latent", ("mixer", "scale"), 0.25), ("fade", ("mixer", "decay"), [0.99, 0.99, 0.7]), ("experts", ("mlp", "expert", "limit"), 1.0),
                                             ("experts", ("mlp", "router", "top"), 2)])
def test_models_tell_a_wrong_constant(name, path, value):
    e = differs(name, pu.prompt(pu.CONFIGS[name], 120, 2), wrong_cfg=edited(name, 0, path, value))
    assert e[20:].min() > 50 * pu.LIMIT[True]


def test_models_tell_a_wrong_mechanism(monkeypatch):
    def halves(x, rot):
        half, out = rot["dims"] // 2, np.array(x)
        perm = [i for p in range(half) for i in (p, p + half)]
        out[..., :rot["dims"]] = x[..., perm]
        return right(out, rot)[..., [perm.index(i) for i in range(rot["dims"])] + list(range(rot["dims"], x.shape[-1]))]
    right = ref.rotate
    toks = pu.prompt(pu.CONFIGS["capped"], 120, 2)
    assert differs("capped", toks, monkeypatch, rotate=halves)[20:].mean() > 0.05
    monkeypatch.undo()
    assert differs("latent", toks, monkeypatch, rotate=halves)[20:].mean() > 0.05
    monkeypatch.undo()

    def scales_output(x, w, pre, m):
        ids, s = ref.chosen(x, w, pre, m)
        return np.stack([sum(wt * ref.expert(x[t:t + 1], w, f"{pre}e{e}.", m["expert"]["limit"])[0] for e, wt in zip(ids[t], s[t])) for t in range(len(x))])
    assert differs("experts", toks, monkeypatch, experts=scales_output).mean() > 0.03
    monkeypatch.undo()
    chosen = ref.chosen
    assert differs("experts", toks, monkeypatch, chosen=lambda *a: (chosen(*a)[0], chosen(*a)[1] / chosen(*a)[1].sum(axis=1, keepdims=True))).mean() > 2 * pu.LIMIT[False]
    monkeypatch.undo()
    assert differs("latent", toks, monkeypatch, latent_rows=lambda x, w, pre, m, eps: (x @ w[pre + "dkv"][:m["kv_rank"]].T, ref.rotate(x @ w[pre + "dkv"][m["kv_rank"]:].T, m["rot"]))).mean() > 0.03


@pytest.mark.parametrize("name", ["capped", "capped_odd", "latent", "latent_odd", "latent_pair"])
def test_standing_keys_tell_a_lost_far_key(name):
    folder, cfg, w = pu.model(name, change=pu.standing_keys([7]), tag="standing")
    toks = [t if t != 7 else 8 for t in pu.prompt(cfg, 340, 3)]
    lost = list(toks)
    toks[3] = 7
    assert pu.error(ref.forward(cfg, w, lost)[0], ref.forward(cfg, w, toks)[0])[60:].min() > TELLS


@pytest.mark.parametrize("name", ["fade", "fade_odd"])
def test_a_lost_state_shows(name):
    """The rows before position 40 gone from the state."""
    folder, cfg, w = pu.model(name, 2)
    toks = pu.prompt(cfg, 60, 4)
    e = pu.error(ref.forward(cfg, w, toks[40:])[0], ref.forward(cfg, w, toks)[0][40:])
    assert e[:8].min() > TELLS and e.min() > 1000 * pu.LIMIT[True]


def test_no_choice_of_experts_is_close():
    for name in ("odd", "fast", "experts", "experts_odd"):
        folder, cfg, w = pu.model(name, 1)
        toks = pu.prompt(cfg, 40, 1)
        _, runs = ref.forward(cfg, w, toks)
        for i, lc in enumerate(cfg["layers"]):
            if lc.get("mlp") and lc["mlp"]["kind"] == "moe":
                s = np.sort(ref.sigmoid(runs[i] @ w[f"l{i}.mlp.router"].T), axis=1)
                assert np.diff(s, axis=1).min() > 0.01


# ---- the reader, the planner
def test_reader_takes_every_layers_own_sizes():
    for name, cfg in pu.CONFIGS.items():
        folder, _, _ = pu.model(name)
        eng = E.Engine(folder, E.EngineConfig(**HOST))
        assert (eng.desc.n_layers, eng.desc.d_model, eng.desc.vocab, eng.desc.page_size) == (len(cfg["layers"]), cfg["width"], cfg["vocab"], 64)
        eng.close()


def test_reader_errors(tmp_path):
    cfg = pu.CONFIGS["odd"]
    bits = pv.random_weights(cfg)

    def fails(match, c=cfg, b=bits):
        pv.write_model(tmp_path / "m", c, b)
        with pytest.raises(E.EngineError, match=match):
            E.Engine(tmp_path / "m", E.EngineConfig(**HOST))

    change = lambda i, *path: edited("odd", i, path[:-1], path[-1])
    without = lambda name: {k: v for k, v in bits.items() if k != name}
    fails("no tensor l1.mix.dkv.norm", b=without("l1.mix.dkv.norm"))
    fails("no tensor side.embed", b=without("side.embed"))
    fails("no tensor l0.mlp.e4.up", b=without("l0.mlp.e4.up"))
    fails(r"l0.mix.o: expected BF16 \[88, 168\], found BF16 \[168, 88\]", b=dict(bits, **{"l0.mix.o": bits["l0.mix.o"].T}))
    fails(r"l1.mix.uk: expected BF16 \[110, 35\]", b=dict(bits, **{"l1.mix.uk": bits["l1.mix.uk"][:, :5]}))
    fails("no mixer named other", change(1, "type", "other"))
    fails("no feed-forward named other", change(1, "mlp", "kind", "other"))
    fails("softcap must be positive", change(0, "mixer", "softcap", 0))
    fails("rot.dims does not fit the heads", change(0, "mixer", "rot", "dims", 22))
    fails("rot.dims is not rot_dim", change(1, "mixer", "rot", "dims", 4))
    fails("must be positive", change(0, "mixer", "rot", "scaling", "factor", 0))
    fails("the heads do not fit the kv heads", change(0, "mixer", "kv_heads", 4))
    fails("kv_from 3 is no latent layer before this one", change(3, "mixer", "kv_from", 3))
    fails("kv_from 2 is no latent layer before this one", change(3, "mixer", "kv_from", 2))
    fails("kv_from 3 has no latents of its own", change(6, "mixer", "kv_from", 3))
    fails("the latents of layer 4 do not fit", change(6, "mixer", "kv_from", 4))
    fails("2 decays for 3 heads", change(2, "mixer", "decay", [0.5, 0.5]))
    fails("heads of 1 to 512 channels", change(2, "mixer", "dim", 513))
    fails("the router does not fit its experts", change(0, "mlp", "router", "top", 6))
    fails("no field `limit`", change(0, "mlp", "expert", {"ff": 24}))
    fails("token_side.dim must be positive", dict(cfg, token_side={"dim": 0}))


def test_planner_pages():
    folder, _, _ = pu.model("odd")
    eng = E.Engine(folder, E.EngineConfig(host_only=True, max_seqs=3, max_step_tokens=1024, max_chunk=1024, max_seq_len=4096, global_kv_tokens=1024, max_head_rows=64))
    a, b = eng.new_seq(), eng.new_seq()
    eng.debug_plan([(a, [1] * 64, E.Rows.NONE, False), (b, [1] * 65, E.Rows.LAST, False)])
    assert len(eng.debug_read("free_pages")) == 16 - 3
    eng.close()
