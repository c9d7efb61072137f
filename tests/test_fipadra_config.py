"""Fipadra without a GPU: the configuration reader, the tensors the builder names, what the cache manager is asked for, and
the plain implementation's own choices of experts on cases worked out by hand."""
import copy

import numpy as np
import pytest

import plain_fipadra as plain
from llmx_b200.cache.manager import CacheManager, KVSpec, StateSpec
from llmx_b200.config import ConfigError, FipadraConfig
from llmx_b200.registry import architecture_of


def raw_config():
    lat = {"type": "latent_attention", "mlp": {"kind": "dense", "ff": 40},
           "mixer": {"heads": 3, "dim": 12, "rot_dim": 8, "vdim": 20, "q_rank": 28, "kv_rank": 40, "scale": 0.3, "mask": {"size": 9},
                     "rot": {"base": 500.0, "dims": 8}}}
    ret = {"type": "retention", "mixer": {"heads": 2, "dim": 16, "vdim": 24, "decay": [0.5, 0.99], "rot": {"base": 300.0, "dims": 8}},
           "mlp": {"kind": "moe", "expert": {"ff": 24, "limit": 0.7}, "shared": {"ff": 40, "limit": 1.1},
                   "router": {"experts": 7, "identity": 2, "top": 3, "scale": 1.7, "groups": {"count": 3, "keep": 2}}}}
    delta = {"type": "delta", "mlp": None, "mixer": {"heads": 6, "kv_heads": 2, "dim": 20, "vdim": 12, "conv": 3}}
    return {"architecture": "Fipadra", "vocab": 200, "width": 96, "norm": {"eps": 1e-5}, "logit_scale": 1.5, "layers": [lat, ret, delta, copy.deepcopy(lat)]}


def test_every_value_is_read_and_written_back():
    cfg = FipadraConfig.from_dict(raw_config())
    assert (cfg.vocab, cfg.width, cfg.norm_eps, cfg.logit_scale, cfg.ignored) == (200, 96, 1e-5, 1.5, ())
    m = cfg.layers[0].mixer
    assert (m.heads, m.dim, m.rot_dim, m.vdim, m.q_rank, m.kv_rank, m.scale, m.window, m.rot_base, m.rot_dims) == (3, 12, 8, 20, 28, 40, 0.3, 9, 500.0, 8)
    m = cfg.layers[1].mixer
    assert (m.heads, m.dim, m.vdim, m.decay, m.rot_base, m.rot_dims) == (2, 16, 24, (0.5, 0.99), 300.0, 8)
    f = cfg.layers[1].mlp
    assert (f.experts, f.identity, f.outputs, f.top, f.scale, f.group_count, f.group_keep) == (7, 2, 9, 3, 1.7, 3, 2)
    assert (f.expert.ff, f.expert.limit, f.shared.ff, f.shared.limit) == (24, 0.7, 40, 1.1)
    assert cfg.layers[0].mlp.ff == 40 and cfg.layers[2].mlp is None and cfg.layers[2].mixer.conv == 3
    assert FipadraConfig.from_dict(cfg.to_dict()) == cfg
    assert architecture_of(raw_config()).config_cls is FipadraConfig


def test_what_config_json_does_not_mention_is_not_there():
    raw = raw_config()
    raw.pop("logit_scale")
    raw["something_else"] = 1
    raw["layers"][0]["mixer"].pop("mask")
    raw["layers"][1]["mixer"].pop("rot")
    for key in ("identity", "scale", "groups"):
        raw["layers"][1]["mlp"]["router"].pop(key)
    raw["layers"][1]["mlp"].pop("shared")
    cfg = FipadraConfig.from_dict(raw)
    f = cfg.layers[1].mlp
    assert cfg.logit_scale == 1.0 and cfg.ignored == ("something_else",) and cfg.layers[0].mixer.window is None
    assert (f.identity, f.scale, f.group_count, f.group_keep, f.shared) == (0, 1.0, 1, 1, None) and cfg.layers[1].mixer.rot_dims == 0
    names = set(architecture_of(raw).build(cfg).tensor_specs())
    assert not any(".shared." in n for n in names) and "l1.mlp.correction" in names


@pytest.mark.parametrize("change, what", [
    (lambda r: r["layers"][0].update(type="lightning"), "mixer type"),
    (lambda r: r["layers"][2]["mixer"].update(heads=5), "multiple of kv_heads"),
    (lambda r: r["layers"][1]["mixer"]["rot"].update(dims=7), "even"),
    (lambda r: r["layers"][1]["mixer"]["rot"].update(dims=18), "at most"),
    (lambda r: r["layers"][1]["mixer"].update(decay=[0.5]), "decay"),
    (lambda r: r["layers"][1]["mlp"]["router"].update(top=7), "exceeds"),
    (lambda r: r["layers"][1]["mlp"]["router"]["groups"].update(count=2), "equal groups"),
    (lambda r: r["layers"][1]["mlp"]["router"]["groups"].update(keep=4), "keep"),
    (lambda r: r["layers"][1]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda r: r["layers"][1]["mlp"]["shared"].pop("ff"), "ff"),
    (lambda r: r["layers"][1]["mlp"].update(kind="other"), "not supported"),
    (lambda r: r["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda r: r["layers"][0]["mixer"].pop("q_rank"), "q_rank"),
    (lambda r: r.update(width="96"), "width"),
    (lambda r: r.update(layers=[]), "layers"),
])
def test_wrong_values_are_refused_by_name(change, what):
    raw = raw_config()
    change(raw)
    with pytest.raises(ConfigError, match=what):
        FipadraConfig.from_dict(raw)


def test_tensors_and_cache_entries():
    raw = raw_config()
    model = architecture_of(raw).build(FipadraConfig.from_dict(raw))
    specs = model.tensor_specs()
    shapes = {"embed": (200, 96), "embed.norm": (96,), "final.norm": (96,), "l0.norm1": (96,), "l0.norm2": (96,), "l0.mix.uq": (60, 28),
              "l0.mix.dkv": (48, 96), "l0.mix.uv": (60, 40), "l0.mlp.up": (40, 96), "l0.mlp.down": (96, 40), "l1.mix.q": (32, 96), "l1.mix.g": (48, 96),
              "l1.mlp.router": (9, 96), "l1.mlp.correction": (9,), "l1.mlp.e6.gate": (24, 96), "l1.mlp.shared.down": (96, 40), "l1.mlp.shared.sg": (1, 96),
              "l2.mix.k.conv": (40, 3), "l2.mix.dt_bias": (6,), "l2.mix.norm": (12,)}
    assert {n: tuple(specs[n].shape) for n in shapes} == shapes
    for n in ("head", "l1.mix.norm", "l1.mlp.e7.gate", "l1.mlp.router.b", "l2.norm2", "l2.mlp.up", "l0.mlp.gate", "l0.mix.q"):
        assert n not in specs, n
    entries = model.cache_entry_specs()
    assert entries[0] == entries[3] == KVSpec(1, 48, 9, planes=1) and entries[1] == StateSpec((2 * 24 * 16,), "float32")
    assert entries[2] == StateSpec((6 * 12 * 20 + 2 * (2 * 40 + 72),), "float32")
    manager = CacheManager(entries, page_size=4, kv_tokens=64, max_requests=2)
    assert len(manager.groups) == 1 and len(manager.groups[0].members) == 2
    rc = manager.new_request("r")
    rc.prepare(40)
    rc.commit()
    assert rc.held_pages()[0] <= 4                       # the window gives back the pages it has passed
    manager.free_request("r")
    manager.check()


def test_the_choice_of_experts_by_hand():
    """Six outputs in three groups of two, one group kept: the best choice score decides the group, also when all are negative;
    weights are the plain scores; with two groups kept the order is by choice score."""
    s = np.array([0.30, 0.05, 0.10, 0.25, 0.20, 0.10])
    c = s + np.array([-1.0, -0.9, -0.2, -0.9, -0.95, -0.8])            # -0.70 -0.85 | -0.10 -0.65 | -0.75 -0.70
    chosen, p, _ = plain.choose(s, c, 2, 3, 1, 2.0)
    assert list(chosen) == [2, 3] and np.allclose(p, np.array([0.10, 0.25]) / 0.35 * 2.0)
    chosen, p, margin = plain.choose(s, c, 3, 3, 2, 1.0)
    assert list(chosen) == [2, 3, 0] and np.allclose(p.sum(), 1.0) and np.isclose(margin * c.std(), 0.0)      # groups 0 and 2 tie at -0.70
