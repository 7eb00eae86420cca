"""Bezasun without a GPU: configuration, registry, source list, and the restatement the GPU tests are held against."""
import math

import numpy as np
import pytest

from tests import bezasun_oracle as orc
from zhilight_b200.bezasun import BezasunConfig

ATT = {"type": "attention", "mixer": {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 5, "scale": 0.4, "softcap": 9.0,
                                      "q_temp": {"coef": 0.2, "every": 8}},
       "mlp": {"kind": "moe", "expert": {"ff": 12}, "router": {"experts": 4, "top": 2}, "shared": {"ff": 20}}}
LAT = {"type": "latent_attention", "mlp": None,
       "mixer": {"heads": 3, "dim": 6, "rot_dim": 4, "vdim": 5, "q_rank": 11, "kv_rank": 9, "scale": 0.3, "mask": {"size": 7},
                 "rot": {"base": 700.0, "dims": 4, "scaling": {"factor": 2.0, "original": 64, "fast": 8.0, "slow": 1.0}}}}
SSM = {"type": "mamba2", "mixer": {"heads": 4, "vdim": 5, "state": 7, "groups": 2, "conv": 4, "norm_groups": 2},
       "mlp": {"kind": "moe", "expert": {"ff": 10}, "router": {"experts": 3, "top": 1}}}
CONFIG = {"architecture": "Bezasun", "vocab": 23, "width": 18, "streams": 3, "residual_mult": 0.9, "logit_scale": 0.5,
          "embedding": {"scale": 4.0}, "norm": {"eps": 1e-5}, "layers": [ATT, LAT, SSM]}


def test_config_round_trip_and_shapes():
    cfg = BezasunConfig.from_dict(CONFIG)
    assert BezasunConfig.from_dict(cfg.to_dict()).to_dict() == cfg.to_dict()
    assert cfg.to_dict()["layers"] == [ATT, LAT, SSM]
    s = cfg.tensor_shapes()
    assert s["l0.mix.q"] == (24, 18) and s["l0.mix.k.norm"] == (6,) and s["l0.mix.sink"] == (4,) and s["l0.mix.o"] == (18, 20)
    assert s["l0.mlp.shared.gate"] == (20, 18) and s["l0.mlp.e3.down"] == (18, 12) and s["l0.hc2.mix"] == (3, 3)
    assert s["l1.mix.uq"] == (30, 11) and s["l1.mix.dkv"] == (13, 18) and s["l1.mix.uv"] == (15, 9)
    assert "l1.norm2" not in s and "l1.hc2.in" not in s and "l1.mlp.router" not in s
    assert s["l2.mix.in"] == (2 * 20 + 2 * 14 + 4, 18) and s["l2.mix.conv"] == (48, 4) and s["l2.mix.norm"] == (20,)
    assert "l2.mlp.shared.gate" not in s


def test_config_optional_parts():
    bare = {"architecture": "Bezasun", "vocab": 9, "width": 8, "streams": 2,
            "layers": [{"type": "attention", "mixer": {"heads": 2, "dim": 4, "vdim": 4, "scale": 0.5}},
                       {"type": "latent_attention",
                        "mixer": {"heads": 2, "dim": 4, "rot_dim": 2, "vdim": 4, "q_rank": 4, "kv_rank": 4, "scale": 0.5,
                                  "rot": {"base": 100.0, "dims": 2}}}]}
    cfg = BezasunConfig.from_dict(bare)
    a, l = cfg.layers
    assert a["kv_heads"] == 2 and a["softcap"] == 0 and a["temp_coef"] == 0 and a["ff_kind"] is None
    assert l["window"] == 0 and l["scaling"] is None
    assert cfg.embed_scale == cfg.residual_mult == cfg.logit_scale == 1.0


@pytest.mark.parametrize("layer,path,value", [(0, ("mixer", "kv_heads"), 3), (0, ("mlp", "kind"), "other"), (0, ("type",), "other"),
                                              (0, ("mlp", "router", "top"), 9), (1, ("mixer", "rot", "dims"), 2),
                                              (1, ("mixer", "mask", "size"), -1), (2, ("mixer", "groups"), 3),
                                              (2, ("mixer", "norm_groups"), 3), (2, ("mixer", "conv"), 0)])
def test_config_rejects(layer, path, value):
    import copy
    d = copy.deepcopy(CONFIG)
    at = d["layers"][layer]
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    with pytest.raises(ValueError):
        BezasunConfig.from_dict(d)


def test_registry_and_sources():
    import os
    from zhilight_b200 import build, registry
    assert "Bezasun" in registry.registered() and registry.supported_dtypes(CONFIG) == ("bfloat16", "float32")
    for name in build.FAMILY_SOURCES["bezasun"]:
        assert os.path.exists(os.path.join(build.CSRC, name + ".cu")), name


def test_struct_matches_header():
    """The ctypes structures list the header's fields in order."""
    import re
    from zhilight_b200 import _lib, bezasun
    src = re.sub(r"/\*.*?\*/", " ", open(_lib.HEADER).read(), flags=re.S)
    for cls, name in ((bezasun.BezasunLayer, "zl_bezasun_layer"), (bezasun.BezasunCConfig, "zl_bezasun_config")):
        body = re.search(r"typedef struct %s \{(.*?)\}" % name, src, flags=re.S).group(1)
        want = []
        for decl in body.split(";"):
            if decl.strip():
                kind, names = decl.split(None, 1)
                want += [(n.strip(), kind) for n in names.split(",")]
        got = [(n, {"c_int": "int", "c_float": "float", "c_double": "double"}[t.__name__]) for n, t in cls._fields_]
        assert got == want


# ---- the restatement, by hand ------------------------------------------------------------------------------------------
def test_oracle_streams_and_mix_orientation():
    x = np.arange(6, dtype=np.float64).reshape(2, 1, 3)
    mix, out, y = np.array([[1.0, 2.0], [3.0, 4.0]]), np.array([5.0, 7.0]), np.ones((1, 3))
    n = orc.hyper_write(x, mix, out, 0.5, y)
    assert np.allclose(n[0], 1 * x[0] + 3 * x[1] + 2.5) and np.allclose(n[1], 2 * x[0] + 4 * x[1] + 3.5)
    assert np.allclose(orc.hyper_read(x, np.array([2.0, -1.0])), 2 * x[0] - x[1])


def test_oracle_attention_pieces():
    t = orc.query_temperature(25, 0.5, 8)
    assert t[6] == 1.0 and t[7] == t[14] == 1 + 0.5 * math.log(2) and t[15] == 1 + 0.5 * math.log(3)
    assert np.allclose(orc.distance_slopes(8), [2.0 ** -i for i in range(1, 9)])
    q, k, v = np.array([[[1.0]], [[2.0]]]), np.array([[[3.0]], [[-1.0]]]), np.array([[[1.0]], [[10.0]]])
    o = orc.sink_attention(q, k, v, 2.0, 4.0, np.array([0.25]), np.array([0.3]))
    s0, s1 = 4 * math.tanh(12 / 4) - 0.25, 4 * math.tanh(-4 / 4)
    e = [math.exp(s) for s in (s0, s1, 0.3)]
    assert np.isclose(o[1, 0, 0], (e[0] * 1 + e[1] * 10) / sum(e))
    e = [math.exp(s) for s in (4 * math.tanh(6 / 4), 0.3)]
    assert np.isclose(o[0, 0, 0], e[0] / sum(e))


def test_oracle_yarn():
    f, m = orc.yarn(8, 100.0)
    assert m == 1.0 and np.allclose(f, [1, 100 ** -0.25, 100 ** -0.5, 100 ** -0.75])
    sc = dict(factor=4.0, original=100.0, fast=10.0, slow=1.0)
    f2, m = orc.yarn(8, 100.0, sc)
    # 8 ln(100 / (2 pi 10)) / (2 ln 100) = 0.40 -> 0;  8 ln(100 / (2 pi)) / (2 ln 100) = 2.40 -> 3
    assert np.isclose(m, 1 + 0.1 * math.log(4)) and np.allclose(f2 / f, [1 - 0.75 * r for r in (0, 1 / 3, 2 / 3, 1)])


def test_oracle_recurrence_and_convolution():
    x = np.array([[1.0], [2.0], [3.0]])
    assert np.allclose(orc.short_convolution(x, np.array([[10.0, 1.0]]), np.array([0.5]))[:, 0], [1.5, 12.5, 23.5])
    a, dt = 0.3, np.array([[0.5], [2.0]])
    xs, B, C = np.array([[[2.0]], [[-1.0]]]), np.array([[[3.0]], [[4.0]]]), np.array([[[5.0]], [[6.0]]])
    y, S = orc.state_space(xs, B, C, dt, np.array([a]), np.array([0.7]))
    s1 = 0.5 * 3 * 2
    s2 = math.exp(-math.exp(a) * 2.0) * s1 + 2.0 * 4 * -1
    assert np.allclose(y[:, 0, 0], [5 * s1 + 0.7 * 2, 6 * s2 - 0.7]) and np.allclose(S, s2)


def test_oracle_routing_keeps_the_scores():
    chosen, s = orc.route_softmax(np.array([0.0, 2.0, 1.0, -1.0]), 2)
    e = np.exp([0.0, 2.0, 1.0, -1.0])
    assert chosen.tolist() == [1, 2] and np.allclose(s, e[[1, 2]] / e.sum())


def test_oracle_is_causal():
    cfg = BezasunConfig.from_dict(CONFIG)
    W = {k: v.astype(np.float64) for k, v in orc.random_weights(cfg, 2).items()}
    toks = np.random.default_rng(0).integers(0, cfg.vocab, 20).tolist()
    full = orc.forward(cfg, W, toks)[0]
    assert np.allclose(orc.forward(cfg, W, toks[:13])[0], full[:13])
    other = toks[:12] + [(toks[12] + 1) % cfg.vocab] + toks[13:]
    moved = orc.forward(cfg, W, other)[0]
    assert np.allclose(moved[:12], full[:12]) and np.abs(moved[12:] - full[12:]).max(-1).min() > 1e-6
