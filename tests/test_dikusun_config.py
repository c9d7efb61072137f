"""Dikusun without a GPU: the configuration reader, the tensors the builder names, layers that use another layer's weights, what
the cache manager is asked for, and the plain implementation on cases worked out by hand."""
import copy

import numpy as np
import pytest

import plain_dikusun as plain
from llmx_b200.cache.manager import KVSpec, StateSpec
from llmx_b200.config import ConfigError, DikusunConfig
from llmx_b200.registry import architecture_of


def raw_config():
    lat = {"type": "latent_attention", "mlp": {"kind": "dense", "ff": 40, "limit": 0.7},
           "mixer": {"heads": 3, "dim": 12, "vdim": 20, "q_rank": 28, "kv_rank": 36, "scale": 0.3}}
    att = {"type": "attention", "mlp": None,
           "mixer": {"heads": 6, "kv_heads": 2, "dim": 10, "vdim": 14, "scale": 0.25, "softcap": 7.0, "diff": 0.3, "mask": {"size": 9},
                     "rot": {"base": 300.0, "dims": 8}}}
    gla = {"type": "gla", "mixer": {"heads": 4, "dim": 6, "vdim": 18, "tau": 5.0}, "mlp": {"kind": "dense", "ff": 24, "limit": 1.3}}
    return {"architecture": "Dikusun", "vocab": 200, "width": 96, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.5},
            "layers": [lat, att, gla, dict(copy.deepcopy(att), weights_of=1), dict(copy.deepcopy(lat), weights_of=0)]}


def test_every_value_is_read_and_written_back():
    cfg = DikusunConfig.from_dict(raw_config())
    assert (cfg.vocab, cfg.width, cfg.norm_eps, cfg.embedding_scale, cfg.ignored) == (200, 96, 1e-5, 1.5, ())
    m = cfg.layers[0].mixer
    assert (m.heads, m.dim, m.vdim, m.q_rank, m.kv_rank, m.scale) == (3, 12, 20, 28, 36, 0.3)
    m = cfg.layers[1].mixer
    assert (m.heads, m.kv_heads, m.dim, m.vdim, m.scale, m.softcap, m.diff, m.window, m.rot_base, m.rot_dims) == (6, 2, 10, 14, 0.25, 7.0, 0.3, 9, 300.0, 8)
    m = cfg.layers[2].mixer
    assert (m.heads, m.dim, m.vdim, m.tau) == (4, 6, 18, 5.0)
    assert (cfg.layers[0].mlp.ff, cfg.layers[0].mlp.limit, cfg.layers[1].mlp, cfg.layers[2].mlp.limit) == (40, 0.7, None, 1.3)
    assert [layer.weights_of for layer in cfg.layers] == [None, None, None, 1, 0]
    assert DikusunConfig.from_dict(cfg.to_dict()) == cfg
    assert architecture_of(raw_config()).config_cls is DikusunConfig


def test_what_config_json_does_not_mention_is_not_there():
    raw = raw_config()
    raw.pop("embedding")
    raw["something_else"] = 1
    for layer in (1, 3):
        for key in ("mask", "rot", "softcap"):
            raw["layers"][layer]["mixer"].pop(key)
    cfg = DikusunConfig.from_dict(raw)
    m = cfg.layers[1].mixer
    assert (cfg.embedding_scale, cfg.ignored, m.window, m.rot_dims, m.softcap) == (1.0, ("something_else",), None, 0, None)
    part = architecture_of(raw).build(cfg).blocks[1].mixer
    assert (part.window, part.rot_dims, part.softcap, part.maps) == (None, 0, None, 2)


@pytest.mark.parametrize("change, what", [
    (lambda r: r["layers"][0].update(type="retention"), "mixer type"),
    (lambda r: r["layers"][1]["mixer"].update(heads=5), "multiple of kv_heads"),
    (lambda r: r["layers"][1]["mixer"]["rot"].update(dims=7), "even"),
    (lambda r: r["layers"][1]["mixer"]["rot"].update(dims=12), "at most dim"),
    (lambda r: r["layers"][1]["mixer"].update(softcap=0.0), "positive"),
    (lambda r: r["layers"][1]["mixer"]["mask"].update(size=0), "size"),
    (lambda r: r["layers"][1]["mixer"].pop("diff"), "diff"),
    (lambda r: r["layers"][2]["mixer"].update(tau=-1.0), "positive"),
    (lambda r: r["layers"][0]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda r: r["layers"][0]["mlp"].update(kind="moe"), "kind"),
    (lambda r: r["layers"][0]["mlp"].pop("limit"), "limit"),
    (lambda r: r["layers"][3].update(weights_of=3), "another layer"),
    (lambda r: r["layers"][3].update(weights_of=9), "another layer"),
    (lambda r: r["layers"][3].update(weights_of=True), "weights_of"),
    (lambda r: r["layers"][3].update(weights_of=0), "differs"),
    (lambda r: r["layers"][4]["mlp"].update(limit=0.8), "differs"),
    (lambda r: r["layers"][1].update(weights_of=3), "back to itself"),
    (lambda r: r.update(layers=[]), "at least one layer"),
    (lambda r: r["norm"].update(eps=-1.0), "eps"),
    (lambda r: r.update(vocab=1.5), "vocab"),
])
def test_what_does_not_fit_is_refused_by_name(change, what):
    raw = raw_config()
    change(raw)
    with pytest.raises(ConfigError, match=what):
        DikusunConfig.from_dict(raw)


def test_tensor_names_shapes_and_the_order_of_blocks():
    cfg = DikusunConfig.from_dict(raw_config())
    model = architecture_of(raw_config()).build(cfg)
    shapes = {n: s.shape for n, s in model.tensor_specs().items()}
    E = 96
    want = {"embed": (200, E), "head": (200, E), "final.norm": (E,),
            "l0.norm1": (E,), "l0.norm2": (E,), "l0.mix.dq": (28, E), "l0.mix.dq.norm": (28,), "l0.mix.uq": (36, 28), "l0.mix.dkv": (36, E),
            "l0.mix.dkv.norm": (36,), "l0.mix.uk": (36, 36), "l0.mix.uv": (60, 36), "l0.mix.o": (E, 60),
            "l0.mlp.gate": (40, E), "l0.mlp.up": (40, E), "l0.mlp.down": (E, 40),
            "l1.norm1": (E,), "l1.mix.q": (120, E), "l1.mix.q.b": (120,), "l1.mix.k": (40, E), "l1.mix.k.b": (40,), "l1.mix.v": (28, E),
            "l1.mix.v.b": (28,), "l1.mix.q.norm": (10,), "l1.mix.k.norm": (10,), "l1.mix.lq1": (10,), "l1.mix.lk1": (10,), "l1.mix.lq2": (10,),
            "l1.mix.lk2": (10,), "l1.mix.g": (6, E), "l1.mix.o": (E, 84), "l1.mix.o.b": (E,),
            "l2.norm1": (E,), "l2.norm2": (E,), "l2.mix.q": (24, E), "l2.mix.k": (24, E), "l2.mix.v": (72, E), "l2.mix.g": (72, E),
            "l2.mix.o": (E, 72), "l2.mix.norm": (18,), "l2.mix.a1": (-1, E), "l2.mix.a2": (24, -1), "l2.mix.a2.b": (24,),
            "l2.mlp.gate": (24, E), "l2.mlp.up": (24, E), "l2.mlp.down": (E, 24)}
    assert shapes == want
    assert [(s.block, s.cache_entry, s.write_cache) for s in model.order] == [(0, 0, True), (1, 1, True), (2, 2, True), (1, 3, True), (0, 4, True)]


def test_a_layer_may_use_the_weights_of_a_later_one_or_through_another():
    raw = raw_config()
    lat, att = raw["layers"][0], raw["layers"][1]
    raw["layers"] = [dict(copy.deepcopy(att), weights_of=2), lat, att, dict(copy.deepcopy(att), weights_of=0)]
    cfg = DikusunConfig.from_dict(raw)
    model = architecture_of(raw).build(cfg)
    assert [cfg.owner(i) for i in range(4)] == [2, 1, 2, 2] == [plain.owner(raw, i) for i in range(4)]
    assert [s.block for s in model.order] == [1, 0, 1, 1] and {n.split(".")[0] for n in model.tensor_specs()} == {"embed", "head", "final", "l1", "l2"}


def test_every_layer_run_has_a_cache_or_state_of_its_own():
    model = architecture_of(raw_config()).build(DikusunConfig.from_dict(raw_config()))
    specs = model.cache_entry_specs()
    kv = KVSpec(2, 2 * 10 + 14, 9, planes=1)
    assert specs == [KVSpec(1, 36, None, planes=1), kv, StateSpec((4 * 18 * 6,), "float32"), kv, KVSpec(1, 36, None, planes=1)]


# ---- the plain implementation on cases worked out by hand ------------------------------------------------------------------
def test_plain_difference_of_two_maps():
    """One head, two keys whose scores are 0 in both maps: both attentions are the mean of the values, so the output is the mean's
    sign pattern over its size, times 1 - diff, flipped when the factor exceeds one."""
    q = np.zeros((2, 1, 2, 3))
    k, v = np.ones((2, 1, 2, 3)), np.array([[[1.0, 3.0]], [[3.0, -1.0]]])
    for factor, sign in ((0.25, 1.0), (2.0, -1.0)):
        o = plain.differential_attention(q, k, v, 1.0, factor, 0.2, 0.0)
        mean = np.array([2.0, 1.0])
        assert np.allclose(o[1, 0], sign * mean / np.sqrt(2.5) * 0.8) and np.allclose(o[0, 0], sign * np.array([1.0, 3.0]) / np.sqrt(5.0) * 0.8)


def test_plain_difference_factor():
    w = {"m.lq1": np.array([1.0, 0.0]), "m.lk1": np.array([np.log(2.0), 5.0]), "m.lq2": np.array([0.0, 1.0]), "m.lk2": np.array([7.0, np.log(3.0)])}
    assert np.isclose(plain.difference_factor(w, "m.", 0.5), 2.0 - 3.0 + 0.5)


def test_plain_gated_recurrence_in_closed_form():
    """o_t = sum_s (prod_{s < r <= t} alpha_r * k_s . q_t) v_s, the decay channel by channel."""
    rng = np.random.default_rng(0)
    T, H, D, V = 7, 2, 3, 4
    q, k, v, a = rng.normal(size=(T, H, D)), rng.normal(size=(T, H, D)), rng.normal(size=(T, H, V)), rng.uniform(0.3, 1.0, size=(T, H, D))
    got = plain.gated_recurrence(q, k, v, a)
    for t in range(T):
        want = sum(((np.prod(a[s + 1:t + 1], axis=0) * k[s] * q[t]).sum(axis=-1))[:, None] * v[s] for s in range(t + 1))
        assert np.allclose(got[t], want)


def test_plain_window_and_cap():
    q = k = np.zeros((5, 2))
    v = np.eye(5)
    o = plain.softmax_attention(q, k, v, 1.0, window=2)
    assert np.allclose(o[0], v[0]) and np.allclose(o[4], 0.5 * (v[3] + v[4]))
    q, k = np.array([[0.0], [100.0]]), np.array([[1.0], [0.0]])
    o = plain.softmax_attention(q, k, np.eye(2), 1.0, softcap=2.0)[1]          # a score of 100 is capped at 2
    assert np.allclose(o[0] / o[1], np.exp(2.0))
