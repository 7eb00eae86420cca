"""Dekalorn pieces that need no GPU: the oracle's own consistency (mechanisms by hand), config parsing and validation,
tensor shapes, the order of layer runs, the registry entry and the family's source list."""
import copy
import math
import os

import numpy as np
import pytest

from tests import dekalorn_oracle as orc
from tests.test_dekalorn_gpu import CFG_FLAT, CFG_ODD, CFG_ONES, CFG_TILES, CONFIGS
from zhilight_b200.dekalorn import DekalornConfig


def _weights(cfg, seed=0):
    return {k: v.astype(np.float64) for k, v in orc.random_weights(cfg, seed).items()}


def test_config_round_trip_and_shapes():
    for d in CONFIGS.values():
        cfg = DekalornConfig.from_dict(d)
        again = DekalornConfig.from_dict(cfg.to_dict())
        assert cfg.layers == again.layers and cfg.loop == again.loop and cfg.norm_eps == again.norm_eps
        shapes = cfg.tensor_shapes()
        assert shapes["embed"] == (cfg.vocab, cfg.width) and ("loop.in" in shapes) == (cfg.loop is not None)
    s = DekalornConfig.from_dict(CFG_ODD).tensor_shapes()
    assert s["loop.in"] == (44, 88)
    assert s["l0.mix.q"] == (4 * 2 * 12, 44) and s["l0.mix.k"] == (2 * 2 * 12, 44) and s["l0.mix.v"] == (2 * 10, 44)
    assert s["l0.mix.g"] == (40, 44) and s["l0.mix.lq1"] == (12,)
    assert s["l1.mix.q"] == (3 * 16, 44) and s["l1.mix.dkv"] == (26, 44) and s["l1.mix.dkv.norm"] == (20,)
    assert s["l1.mix.uk"] == (30, 20) and s["l1.mix.uv"] == (42, 20) and s["l1.mix.g"] == (3, 44) and s["l1.mix.o"] == (44, 42)
    assert s["l2.mix.talk"] == (6, 6) and s["l2.mix.temp"] == (6,) and "l2.mix.g" not in s
    assert "l3.norm2" not in s and "l3.norm1" in s and s["l2.mlp.router"] == (5, 44) and "l2.mlp.e5.up" not in s


def test_run_order_of_a_loop():
    cfg = DekalornConfig.from_dict(CFG_ODD)                         # 0, (1, 2) three times, 3
    assert cfg.num_runs == 8 and [cfg.run_layer(r) for r in range(8)] == [0, 1, 2, 1, 2, 1, 2, 3]
    assert [i for i, _ in orc.schedule(cfg)] == [0, 1, 2, 1, 2, 1, 2, 3]
    assert [e for _, e in orc.schedule(cfg)] == [False, True, False, True, False, True, False, False]
    cfg = DekalornConfig.from_dict(CFG_FLAT)
    assert cfg.num_runs == 3 and orc.schedule(cfg) == [(0, False), (1, False), (2, False)]
    cfg = DekalornConfig.from_dict(CFG_TILES)                       # the loop ends the model
    assert [cfg.run_layer(r) for r in range(cfg.num_runs)] == [0, 1, 2, 1, 2]


def test_config_validation():
    def bad(edit):
        d = copy.deepcopy(CFG_ODD)
        edit(d)
        with pytest.raises(ValueError):
            DekalornConfig.from_dict(d)

    bad(lambda d: d["loop"].update(stop=5))
    bad(lambda d: d["loop"].update(start=3))
    bad(lambda d: d["loop"].update(times=0))
    bad(lambda d: d["layers"][0]["mixer"].update(kv_heads=3))
    bad(lambda d: d["layers"][0].update(type="general_delta"))
    bad(lambda d: d["layers"][1]["mlp"].update(kind="glu"))
    bad(lambda d: d["layers"][1]["mixer"]["rot"].update(dims=4))           # not all of rot_dim
    bad(lambda d: d["layers"][2]["mixer"]["rot"].update(dims=16))          # more than the head
    bad(lambda d: d["layers"][2]["mixer"]["rot"].update(dims=5))
    bad(lambda d: d["layers"][0]["mlp"]["router"].update(top=7))
    bad(lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(count=4))
    bad(lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(keep=4))
    bad(lambda d: d["layers"][0]["mlp"]["router"].update(top=5))           # two groups of two hold four


def test_config_defaults():
    d = copy.deepcopy(CFG_TILES)
    r = d["layers"][1]["mlp"]["router"]
    del r["groups"], r["scale"], d["layers"][1]["mixer"]["mask"], d["layers"][0]["mixer"]["rot"]["scaling"], d["loop"]
    cfg = DekalornConfig.from_dict(d)
    assert (cfg.layers[1]["groups"], cfg.layers[1]["keep"], cfg.layers[1]["router_scale"]) == (1, 1, 1.0)
    assert cfg.layers[1]["window"] == 0 and cfg.layers[0]["scaling"] is None and cfg.loop is None


def test_registry_and_family_sources():
    from zhilight_b200 import build, registry
    assert "Dekalorn" in registry.registered()
    assert registry.supported_dtypes(CFG_ONES) == ("bfloat16", "float32")
    for name in build.FAMILY_SOURCES["dekalorn"]:
        assert os.path.exists(os.path.join(build.CSRC, name + ".cu")), name


# ---------------------------------------------------------------------------------------------- the oracle by hand
def test_frequencies_by_hand():
    f = orc.frequencies(4, 100.0)
    assert np.allclose(f, [1.0, 0.1])
    sc = dict(factor=4.0, low=1.0, high=4.0, original=2 * math.pi * 40)
    # wavelengths over 2 pi: 1 and 10 (boundaries: original / high = 10, original / low = 40)
    assert np.allclose(orc.frequencies(4, 100.0, sc), [1.0, 0.1])
    sc["original"] = 2 * math.pi * 20                                # boundaries 5 and 20: 10 lies between, s = (2 - 1) / 3
    assert np.allclose(orc.frequencies(4, 100.0, sc), [1.0, (2 / 3) * 0.1 / 4 + 0.1 / 3])
    sc["original"] = 2 * math.pi * 5                                 # boundaries 1.25 and 5: the long one is divided
    assert np.allclose(orc.frequencies(4, 100.0, sc), [1.0, 0.025])


def test_rotation_by_hand():
    x = np.zeros((3, 1, 5))
    x[:, 0] = [1.0, 0.0, 0.0, 2.0, 9.0]
    y = orc.rotate_adjacent(x, np.array([1.0, 0.1]))
    assert np.allclose(y[2, 0], [math.cos(2), math.sin(2), -2 * math.sin(0.2), 2 * math.cos(0.2), 9.0])
    assert np.allclose(y[0], x[0])


def test_window_mask():
    v = orc.visible(6, 3)
    assert v[5].tolist() == [False, False, False, True, True, True] and v[1].tolist() == [True, True] + [False] * 4
    assert np.array_equal(orc.visible(4, 1), np.eye(4, dtype=bool)) and np.array_equal(orc.visible(4, 0), np.tril(np.ones((4, 4), bool)))


def test_differential_attention_by_hand():
    rng = np.random.default_rng(0)
    q, k, v = rng.standard_normal((5, 2, 2, 3)), rng.standard_normal((5, 1, 2, 3)), rng.standard_normal((5, 1, 4))
    o = orc.differential_attention(q, k, v, 0.5, 2, 0.25, 0.4, 0.0)
    # the first token sees itself only: both maps give v, (1 - lambda) v over its own root mean square
    assert np.allclose(o[0, 1], v[0, 0] / math.sqrt(np.mean(v[0, 0] ** 2)) * 0.6)
    e = [np.exp(0.5 * np.array([q[3, 1, m] @ k[j, 0, m] for j in (2, 3)])) for m in (0, 1)]
    a = [(w[0] * v[2, 0] + w[1] * v[3, 0]) / w.sum() for w in e]
    r = a[0] - 0.25 * a[1]
    assert np.allclose(o[3, 1], r / math.sqrt(np.mean(r * r)) * 0.6)
    W = {"lq1": np.array([1.0, 2.0]), "lk1": np.array([0.5, 0.0]), "lq2": np.array([0.0, 1.0]), "lk2": np.array([3.0, -1.0])}
    assert np.isclose(orc.diff_lambda(W, "", 0.7), math.exp(0.5) - math.exp(-1.0) + 0.7)


def test_mixed_heads_by_hand():
    rng = np.random.default_rng(1)
    q, k, v = rng.standard_normal((4, 2, 3)), rng.standard_normal((4, 1, 3)), rng.standard_normal((4, 1, 2))
    talk, temp = np.array([[0.0, 2.0], [1.0, -0.5]]), np.array([3.0, 0.5])
    o = orc.mixed_head_attention(q, k, v, 0.1, 0, temp, talk)
    s = 0.1 * np.array([[q[2, h] @ k[j, 0] * temp[h] for j in range(3)] for h in range(2)])
    for h, m in ((0, 2.0 * s[1]), (1, s[0] - 0.5 * s[1])):
        e = np.exp(m)
        assert np.allclose(o[2, h], (e[:, None] * v[:3, 0]).sum(0) / e.sum())


def test_route_by_hand():
    logit = lambda s: np.log(np.array(s) / (1 - np.array(s)))
    z = logit([0.9, 0.1, 0.6, 0.55, 0.2, 0.3])                       # group sums 1.0, 1.15, 0.5
    ch, w = orc.route_two_best(z, 2, 3, 1, 2.0)
    assert list(ch) == [2, 3] and np.allclose(w, 2.0 * np.array([0.6, 0.55]) / 1.15)     # the best expert's group lost
    ch, w = orc.route_two_best(z, 3, 3, 2, 1.0)
    assert list(ch) == [0, 2, 3] and np.allclose(w.sum(), 1.0)
    z = logit([0.4, 0.4, 0.4, 0.5, 0.31, 0.1])                       # only the two best of a group count, not its sum
    ch, _ = orc.route_two_best(z, 1, 2, 1, 1.0)
    assert list(ch) == [3]


def test_feed_forwards_by_hand():
    W = {"gate": np.array([[1.0], [-1.0]]), "up": np.array([[2.0], [5.0]]), "down": np.array([[1.0, 1.0]])}
    assert np.allclose(orc.relu_gated_ff(W, "", np.array([[3.0]])), [[18.0]])
    want = 3 * orc.sigmoid(3.0) * 6.0 - 3 * orc.sigmoid(-3.0) * 15.0
    assert np.allclose(orc.silu_expert(W, "", np.array([3.0])), [want])


def test_forward_is_causal_and_latent_rows_are_what_is_cached():
    cfg = DekalornConfig.from_dict(CFG_ODD)
    W = _weights(cfg, 1)
    toks = np.random.default_rng(3).integers(0, cfg.vocab, 17).tolist()
    full, streams, cached = orc.forward(cfg, W, toks)
    part = orc.forward(cfg, W, toks[:9])[0]
    assert np.allclose(full[:9], part, rtol=0, atol=1e-10)
    assert streams.shape == (8, 17, 44) and cached[1][0].shape == (17, 20) and cached[1][1].shape == (17, 6)
    # a loop input that returns its second half restarts every pass from the embedding
    Z = dict(W)
    Z["loop.in"] = np.concatenate([np.zeros((44, 44)), np.eye(44)], axis=1)
    _, s, c = orc.forward(cfg, Z, toks)
    assert np.allclose(s[2], s[4]) and np.allclose(s[4], s[6]) and np.allclose(c[1][0], c[3][0])
