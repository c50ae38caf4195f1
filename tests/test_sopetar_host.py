"""The Sopetar design without a GPU: the slow restatement's mechanisms against hand-worked values, mistakes planted in it that the
GPU tests' models must reveal, the folder reader's errors, and the planner over a Sopetar model."""
import json

import numpy as np
import pytest

from silicon_violetto_b200 import build, engine as E, sopetar as sv
from tests import sopetar_ref as ref, sopetar_util as su

HOST = dict(host_only=True, max_seq_len=128, global_kv_tokens=128)
TELLS = 5 * su.LIMIT[False]


@pytest.fixture(scope="module", autouse=True)
def built():
    build.build()


def test_norms():
    assert np.allclose(ref.over_rms(np.array([[3.0, -4.0]]), 0.0), [[3 / np.sqrt(12.5), -4 / np.sqrt(12.5)]])
    assert np.allclose(ref.over_rms(np.full((1, 2), 1e-3), 1.0), 1e-3 / np.sqrt(1 + 1e-6))
    assert np.allclose(ref.layer_norm(np.array([[1.0, 5.0]]), np.array([2.0, 1.0]), np.array([0.5, -0.5]), 0.0), [[-1.5, 0.5]])
    assert np.allclose(ref.layer_norm(np.array([[1.0, 5.0]]), 1.0, 0.0, 12.0), [[-0.5, 0.5]])


def test_neighbours_turn_by_the_position():
    x = np.zeros((3, 1, 5))
    x[:, 0] = [1, 0, 0, 2, 7]
    y = ref.rotate(x, {"dims": 4, "base": 100.0})[:, 0]
    assert np.allclose(y[0], [1, 0, 0, 2, 7])
    assert np.allclose(y[2], [np.cos(2.0), np.sin(2.0), -2 * np.sin(0.2), 2 * np.cos(0.2), 7])


def test_windows_and_kept_positions():
    seen = ref.visible(6, {"size": 2, "keep_first": 1})
    assert seen.astype(int).tolist() == [[1, 0, 0, 0, 0, 0], [1, 1, 0, 0, 0, 0], [1, 1, 1, 0, 0, 0], [1, 0, 1, 1, 0, 0], [1, 0, 0, 1, 1, 0], [1, 0, 0, 0, 1, 1]]
    assert np.array_equal(ref.visible(4, {"size": 1}), np.eye(4, dtype=bool))


def test_slopes_halve_from_head_to_head():
    assert np.allclose(ref.slopes(8), [0.5 ** (h + 1) for h in range(8)]) and np.allclose(ref.slopes(3), [2 ** (-8 / 3), 2 ** (-16 / 3), 2 ** -8])
    assert np.allclose(ref.farther(np.zeros((3, 3)), 0.5)[2], [-1, -0.5, 0])


def test_scores_are_capped_before_distance_counts():
    m = {"scale": 1.0, "softcap": 2.0, "mask": {"size": 9}}
    q, k, v = np.ones((2, 1, 1)), np.array([[[100.0]], [[0.0]]]), np.array([[[1.0]], [[0.0]]])
    assert np.isclose(ref.attention_core(q, k, v, m)[1, 0, 0], 1 / (1 + np.exp(-2.0 + 2.0 ** -8)))


def test_a_sink_takes_its_share_unscaled():
    assert np.allclose(ref.weights(np.zeros((1, 2)), np.array([[True, False]]), np.log(3.0)), [[0.25, 0.0]])
    assert np.allclose(ref.weights(np.array([[-900.0, -900.0]]), np.array([[True, True]]), 0.0), 0.0)


def test_query_heads_share_kv_heads_in_order():
    v = np.array([[[1.0], [2.0]]])
    assert ref.attention_core(np.zeros((1, 4, 1)), np.zeros((1, 2, 1)), v, {"scale": 1.0, "softcap": 1.0, "mask": {"size": 1}})[0, :, 0].tolist() == [1, 1, 2, 2]


def test_feed_forward_is_cut_off():
    w = {f"{c}": np.array([[float(x)]]) for c, x in (("gate", 1), ("up", 1), ("down", 2))} | {f"{c}.b": np.array([b]) for c, b in (("gate", 1.0), ("up", -0.5), ("down", 0.25))}
    f = lambda x: ref.feed_forward(np.array([[x]]), w, "", 0.75)[0, 0]
    assert np.isclose(f(2.0), 2 * 0.75 * ref.sigmoid(1.702 * 0.75) * 1.75 + 0.25)
    assert np.isclose(f(-3.0), 2 * -2 * ref.sigmoid(-1.702 * 2) * 0.25 + 0.25)


def test_values_mix_and_results_average():
    assert ref.mix_values(4.0, 8.0, 0.25) == 5.0
    assert ref.depth_average([np.array([1.0]), np.array([10.0]), np.array([100.0])], [0.5, 2.0, 1.0])[0] == 120.5


# ---- the models tell mistakes
def differs(name, toks, monkeypatch=None, wrong_cfg=None, model=None, **wrong):
    """The error per position of the restatement with some of its functions replaced, or with another configuration."""
    folder, cfg, w = model or su.model(name, 1)
    right, _ = ref.forward(cfg, w, toks)
    for k, f in wrong.items():
        monkeypatch.setattr(ref, k, f)
    return su.error(ref.forward(wrong_cfg or cfg, w, toks)[0], right)


def edited(name, i, path, value):
    cfg = json.loads(json.dumps(su.CONFIGS[name]))
    at = cfg["layers"][i] if i is not None else cfg
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    return cfg


@pytest.mark.parametrize("name,i,path,value", [("kept", 0, ("mixer", "softcap"), 1e6), ("kept", 0, ("mixer", "scale"), 0.25), ("kept_odd", 0, ("mixer", "mask", "keep_first"), 0),
                                               ("latent", 0, ("mixer", "rot", "base"), 20000.0), ("latent", 0, ("mixer", "scale"), 0.25), ("dense", 0, ("mlp", "limit"), 1.0),
                                               ("mixed", None, ("embedding", "scale"), 1.0), ("mixed", 0, ("mixer", "v_mix"), True), ("dense", None, ("norm", "eps"), 1e-2)])
def test_models_tell_a_wrong_constant(name, i, path, value):
    model = None
    if path[-1] == "v_mix":  # (the layer has a share of its own then)
        folder, cfg, w = su.model(name, 1)
        model = folder, cfg, {**w, "l0.mix.vmix": np.array(0.5)}
    e = differs(name, su.prompt(su.CONFIGS[name], 120, 2), wrong_cfg=edited(name, i, path, value), model=model)
    assert e[60:].min() > 50 * su.LIMIT[True]


def test_models_tell_a_wrong_mechanism(monkeypatch):
    def tells(name, least=0.01, **wrong):
        toks = su.prompt(su.CONFIGS[name], 120, 2)
        assert differs(name, toks, monkeypatch, **wrong)[20:].mean() > least, wrong
        monkeypatch.undo()
    for name in ("latent", "latent_odd"):
        rotate, weights = ref.rotate, ref.weights
        def halves(x, rot):
            half = rot["dims"] // 2
            perm = [i for p in range(half) for i in (p, p + half)] + list(range(rot["dims"], x.shape[-1]))
            return rotate(x[..., perm], rot)[..., np.argsort(perm)]
        tells(name, rotate=halves)
        tells(name, weights=lambda s, seen, sink=None: weights(s, seen))
        tells(name, sigmoid=lambda z: np.ones_like(z))
        tells(name, over_rms=lambda x, eps: x)
    for name in ("kept", "kept_odd"):
        soften, farther = ref.soften, ref.farther
        tells(name, farther=lambda s, slope: s)
        tells(name, slopes=lambda heads: 2.0 ** (-8.0 * np.arange(heads) / heads))
        tells(name, soften=lambda s, cap: s, farther=lambda s, slope: soften(farther(s, slope), 13.0), least=2e-4)
    for name in ("mixed", "mixed_odd"):
        tells(name, mix_values=lambda v, first, share: v)
        tells(name, mix_values=lambda v, first, share: share * v + (1 - share) * first)
        tells(name, mix_values=lambda v, first, share: ref.over_rms((1 - share) * v + share * first, 0.0))
        tells(name, depth_average=lambda results, share: results[-1])
        tells(name, depth_average=lambda results, share: sum(s * x for s, x in zip(share[::-1], results)))
        tells(name, layer_norm=lambda x, w, b, eps: ref.over_rms(x, eps) * w + b, least=0.003)
        tells(name, layer_norm=lambda x, w, b, eps: ref.over_rms(x - x.mean(axis=-1, keepdims=True), eps) * w)
    for name in ("dense", "dense_odd"):
        right = ref.feed_forward
        tells(name, feed_forward=lambda x, w, pre, limit: right(x, {**w, pre + "down.b": 0.0}, pre, limit))
        tells(name, feed_forward=lambda x, w, pre, limit: right(x, {**w, pre + "gate.b": 0.0}, pre, limit))
        tells(name, feed_forward=lambda x, w, pre, limit: right(x, w, pre, 1e9))


STANDING = ["kept", "kept_odd", "latent", "latent_odd"]


@pytest.mark.parametrize("name", STANDING)
def test_standing_keys_tell_a_window_that_is_one_off(name):
    """At the first position that does not see a standing key any more, and at the last that does."""
    folder, cfg, w = su.model(name, change=su.standing_keys([7]), tag="standing")
    toks = [t if t != 7 else 8 for t in su.prompt(cfg, 140, 3)]
    toks[30] = 7
    m = cfg["layers"][0]["mixer"]["mask"]
    size = m["size"]
    assert differs(name, toks, wrong_cfg=edited(name, 0, ("mixer", "mask", "size"), size + 1), model=(folder, cfg, w))[30 + size] > TELLS
    assert differs(name, toks, wrong_cfg=edited(name, 0, ("mixer", "mask", "size"), size - 1), model=(folder, cfg, w))[30 + size - 1] > TELLS


@pytest.mark.parametrize("name", ["latent", "latent_odd"])
def test_standing_sinks_tell_their_loss(name, monkeypatch):
    weights = ref.weights
    model = su.model(name, change=su.standing_sinks, tag="sinks")
    assert np.median(differs(name, su.prompt(model[1], 140, 3), monkeypatch, model=model, weights=lambda s, seen, sink=None: weights(s, seen))) > TELLS


@pytest.mark.parametrize("name", ["kept", "kept_odd"])
def test_standing_keys_tell_first_positions_one_off(name):
    folder, cfg, w = su.model(name, change=su.standing_keys([7]), tag="standing")
    keep = cfg["layers"][0]["mixer"]["mask"]["keep_first"]
    for at, wrong in ((keep, keep + 1), (keep - 1, keep - 1)):
        toks = [t if t != 7 else 8 for t in su.prompt(cfg, 340, 3)]
        toks[at] = 7
        assert differs(name, toks, wrong_cfg=edited(name, 0, ("mixer", "mask", "keep_first"), wrong), model=(folder, cfg, w))[100:].min() > 0.5 * TELLS


# ---- the reader, the planner
def test_reader_takes_every_layers_own_sizes():
    for name, cfg in su.CONFIGS.items():
        folder, _, _ = su.model(name)
        eng = E.Engine(folder, E.EngineConfig(**HOST))
        assert (eng.desc.n_layers, eng.desc.d_model, eng.desc.vocab, eng.desc.page_size) == (len(cfg["layers"]), cfg["width"], cfg["vocab"], 64)
        eng.close()


def test_reader_errors(tmp_path):
    cfg = su.CONFIGS["odd"]
    bits = sv.random_weights(cfg)

    def fails(match, c=cfg, b=bits):
        sv.write_model(tmp_path / "m", c, b)
        with pytest.raises(E.EngineError, match=match):
            E.Engine(tmp_path / "m", E.EngineConfig(**HOST))

    change = lambda i, *path: edited("odd", i, path[:-1], path[-1])
    without = lambda name: {k: v for k, v in bits.items() if k != name}
    for name in ("l0.norm1.b", "l0.mix.k.b", "l0.mlp.up.b", "l1.mix.sink", "l1.mix.dkv.norm", "l1.mix.g", "l2.mix.vmix", "l3.dwa", "l4.mlp.down.b", "final.norm.b", "head"):
        fails(f"no tensor {name}", b=without(name))
    fails(r"l0.mix.o: expected BF16 \[88, 80\], found BF16 \[80, 88\]", b=dict(bits, **{"l0.mix.o": bits["l0.mix.o"].T}))
    fails(r"l1.mix.uk: expected BF16 \[110, 35\]", b=dict(bits, **{"l1.mix.uk": bits["l1.mix.uk"][:, :5]}))
    fails(r"l4.dwa: expected BF16 \[6\]", b=dict(bits, **{"l4.dwa": bits["l4.dwa"][1:]}))
    fails("no mixer named other", change(1, "type", "other"))
    fails("no feed-forward named other", change(1, "mlp", "kind", "other"))
    fails("a feed-forward of width 0", change(1, "mlp", "ff", 0))
    fails("softcap must be positive", change(0, "mixer", "softcap", 0))
    fails("mask.size must be positive", change(0, "mixer", "mask", "size", 0))
    fails("mask.size must be positive", change(1, "mixer", "mask", "size", 0))
    fails("`mask.size` is not a size", change(1, "mixer", "mask", "size", 2.5))
    fails("rot.dims is not rot_dim", change(1, "mixer", "rot", "dims", 4))
    fails("must be positive", change(1, "mixer", "rot", "base", 0))
    fails("the heads do not fit the kv heads", change(2, "mixer", "kv_heads", 4))
    fails("neither true nor false", change(2, "mixer", "v_mix", 1))
    fails("its values do not fit those of the first layer", change(0, "mixer", "v_mix", True), dict(bits, **{"l0.mix.vmix": bits["l2.mix.vmix"]}))
    fails("a size of 0", change(1, "mixer", "kv_rank", 0))
    fails("no field `limit`", change(0, "mlp", {"kind": "dense", "ff": 50}))
    fails("no field `embedding`", {k: v for k, v in cfg.items() if k != "embedding"})


def test_planner_pages():
    folder, _, _ = su.model("odd")
    eng = E.Engine(folder, E.EngineConfig(host_only=True, max_seqs=3, max_step_tokens=1024, max_chunk=1024, max_seq_len=4096, global_kv_tokens=1024, max_head_rows=64))
    a, b = eng.new_seq(), eng.new_seq()
    eng.debug_plan([(a, [1] * 64, E.Rows.NONE, False), (b, [1] * 65, E.Rows.LAST, False)])
    assert len(eng.debug_read("free_pages")) == 16 - 3
    eng.close()
