"""Dekalorn on the GPU against the plain numpy restatement in tests/dekalorn_oracle.py.

Small configurations of their own (all sizes different from one another; grouped and single key/value heads; the three
mixers in several orders with dense, routed and no feed-forward; loops at the start, in the middle, over everything and
none; windows of 1 and of sizes around the kernels' tiles; head counts with and without a tensor-core tile), random
bfloat16-exact weights.  float32 runs are held to a tight tolerance, bfloat16 runs to a loose one; the measure is the RMS
over the vocabulary of the mean-free difference of the logits, relative to the RMS of the logits.
"""
import json
import math

import numpy as np
import pytest

from tests import dekalorn_oracle as orc

pytestmark = pytest.mark.gpu

TOL = {"float32": 2e-4, "bfloat16": 5e-2}


def LATENT(heads, dim, rot_dim, vdim, kv_rank, scale, base=10000.0, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=scale,
                          rot=dict(base=base, dims=rot_dim))}


def DIFF(heads, kv_heads, dim, vdim, scale, diff, window, mlp=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, diff=diff, mask={"size": window})}


def MIXED(heads, kv_heads, dim, vdim, scale, window, rot_dims, base=10000.0, scaling=None, mlp=None):
    rot = dict(base=base, dims=rot_dims)
    if scaling:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"type": "attention_2", "mlp": mlp,
            "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, mask={"size": window}, rot=rot)}


def DENSE(ff):
    return {"kind": "dense", "ff": ff}


def MOE(experts, top, count, keep, ff, scale):
    return {"kind": "moe", "expert": {"ff": ff},
            "router": {"experts": experts, "top": top, "scale": scale, "groups": {"count": count, "keep": keep}}}


def CFG(vocab, width, layers, loop=None, eps=1e-5):
    d = {"architecture": "Dekalorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


# sizes without tensor-core tiles; the loop runs the middle three times
CFG_ODD = CFG(67, 44, [DIFF(4, 2, 12, 10, 0.3, 0.3, 9, mlp=MOE(6, 2, 3, 2, 20, 1.5)),
                       LATENT(3, 10, 6, 14, 20, 0.25, base=500.0, mlp=DENSE(52)),
                       MIXED(6, 3, 14, 9, 0.28, 13, 8, base=3000.0, scaling=(3.0, 1.0, 5.0, 40), mlp=MOE(5, 3, 1, 1, 24, 0.7)),
                       LATENT(2, 7, 4, 5, 9, 0.3)], loop=(1, 3, 3))
CFG_ONES = CFG(40, 32, [DIFF(1, 1, 6, 4, 0.4, 0.8, 1, mlp=DENSE(8)), MIXED(1, 1, 2, 6, 0.5, 1, 2, base=300.0, mlp=MOE(1, 1, 1, 1, 16, 1.0)),
                        LATENT(1, 1, 2, 1, 1, 0.7)], loop=(0, 1, 1), eps=1e-6)
# tensor-core sizes: heads of 16 / 32, a latent that is padded, windows around the 32- and 64-key tiles; the loop ends the model
CFG_TILES = CFG(96, 64, [MIXED(8, 2, 32, 16, 0.18, 40, 16, base=2e4, scaling=(2.0, 1.0, 4.0, 64), mlp=DENSE(72)),
                         DIFF(8, 2, 16, 32, 0.25, 0.45, 65, mlp=MOE(8, 3, 4, 2, 40, 2.5)),
                         LATENT(4, 16, 8, 24, 48, 0.2, mlp=MOE(6, 2, 2, 1, 16, 1.2))], loop=(1, 3, 2))
# no loop, one key/value head per query head
CFG_FLAT = CFG(80, 96, [LATENT(5, 32, 16, 32, 64, 0.14), DIFF(4, 4, 32, 16, 0.17, 0.6, 31, mlp=DENSE(64)),
                        MIXED(4, 4, 16, 32, 0.25, 64, 12, mlp=MOE(4, 2, 2, 2, 24, 1.0))])
CONFIGS = {"odd": CFG_ODD, "ones": CFG_ONES, "tiles": CFG_TILES, "flat": CFG_FLAT}


def row_err(got, want):
    d = np.asarray(got, dtype=np.float64) - want
    d = d - d.mean(-1, keepdims=True)
    w = want - want.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / np.sqrt((w * w).mean(-1))


def rel_err(got, want, dtype="float32"):
    """float32: the worst row.  bfloat16: the row at the 90th percentile -- a rounding can flip the choice of an expert
    where two scores nearly tie, which moves that token by far more than rounding does and says nothing about the
    kernels; what a float32 run finds at one position only, it finds with the worst-row measure."""
    e = row_err(got, want)
    return float(np.max(e) if dtype == "float32" else np.quantile(e, 0.9))


def make(cfg_dict, dtype, seed=0, max_batch=4, max_seq=400, max_step_tokens=64, **kw):
    from zhilight_b200.dekalorn import DekalornConfig, DekalornDecoder
    from zhilight_b200.safetensors_io import f32_to_bf16
    cfg = DekalornConfig.from_dict(cfg_dict)
    W = orc.random_weights(cfg, seed)
    m = DekalornDecoder(cfg, dtype=dtype, max_batch=max_batch, max_seq=max_seq, max_step_tokens=max_step_tokens, **kw)
    m.load_state_dict({k: f32_to_bf16(v) for k, v in W.items()})
    return cfg, {k: v.astype(np.float64) for k, v in W.items()}, m


def tokens_for(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg.vocab, n).tolist()


def dev(a, cuda, dtype=None):
    import torch
    t = torch.as_tensor(np.ascontiguousarray(a))
    if dtype is not None:
        t = t.to(dtype)
    return t.to(cuda)


def i32(a, cuda):
    import torch
    return torch.tensor(list(a), dtype=torch.int32, device=cuda)


def b16(a):
    return orc.bf16_round(np.asarray(a, dtype=np.float32))


# ---------------------------------------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_relu_and_silu_gated_units(cuda, lib, dtype):
    """relu(gate) * up in the few-rows, tile and fp32 kernels; silu experts as the clamped unit without its clamp."""
    import torch
    from zhilight_b200 import ops
    td = getattr(torch, dtype)
    tol = 1e-5 if dtype == "float32" else 2e-2
    rng = np.random.default_rng(0)
    for m, f, k in ((5, 7, 16), (70, 65, 80), (3, 48, 64), (40, 10, 24)):
        x, gate, up = b16(rng.standard_normal((m, k))), b16(rng.standard_normal((f, k)) / math.sqrt(k)), b16(rng.standard_normal((f, k)) / math.sqrt(k))
        w = np.empty((2 * f, k), np.float32)
        w[0::2], w[1::2] = gate, up
        W = {"gate": gate.astype(np.float64), "up": up.astype(np.float64), "down": np.eye(f)}
        y = ops.gemm_nt_reglu(dev(x, cuda, td), dev(w, cuda, td), out_dtype=torch.float32)
        assert np.abs(y.cpu().numpy() - orc.relu_gated_ff(W, "", x.astype(np.float64))).max() < tol, (m, f, k)
        off = i32([0, m], cuda)
        y = ops.gemm_nt_grouped(dev(x, cuda, td), dev(w[None], cuda, td), off, m, epilogue=ops.GEMM_EPI_GLU_CLAMP, limit=math.inf,
                                alpha=1.0, beta=0.0, out_dtype=torch.float32)
        want = np.stack([orc.silu_expert(W, "", r) for r in x.astype(np.float64)])
        assert np.abs(y.cpu().numpy() - want).max() < tol, (m, f, k)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_router_ranks_groups_by_their_two_best(cuda, lib, dtype):
    """12 experts in 4 groups of which 2 count, 5 chosen.  In many rows the single best expert sits in a group that loses
    to a group with two good ones; the weights are the scores over their sum times a constant; the lists sort the pairs."""
    import torch
    from zhilight_b200 import ops
    rng = np.random.default_rng(3)
    T, D, E, top, groups, keep, scale = 61, 40, 12, 5, 4, 2, 2.25
    x = b16(rng.standard_normal((T, D)))
    w = b16(2 * rng.standard_normal((E, D)) / math.sqrt(D))
    td = getattr(torch, dtype)
    te, tw, off, lt, lp = (t.cpu().numpy() for t in ops.moe_route_ex(dev(x, cuda, td), dev(w, cuda, td), top, groups, keep,
                                                                     renorm_eps=1e-20, weight_scale=scale))
    z = x.astype(np.float64) @ w.T.astype(np.float64)
    best_lost = 0
    for t in range(T):
        chosen, weight = orc.route_two_best(z[t], top, groups, keep, scale)
        assert (te[t] == chosen).all(), t
        assert np.abs(tw[t] - weight).max() < 2e-6 and abs(tw[t].sum() - scale) < 1e-5
        best_lost += int(np.argmax(z[t])) not in chosen
    assert best_lost > 3
    assert off[0] == 0 and off[-1] == T * top and sorted(lp.tolist()) == list(range(T * top)) and (lt == lp // top).all()
    for e in range(E):
        assert (te.reshape(-1)[lp[off[e]:off[e + 1]]] == e).all()
    # groups of one expert rank by it alone; the largest-member rank gives another choice somewhere
    te1 = ops.moe_route_ex(dev(x, cuda, td), dev(w, cuda, td), 3, E, 3)[0].cpu().numpy()
    assert (te1 == np.argsort(-z, axis=1, kind="stable")[:, :3]).all()
    te2 = ops.moe_route_ex(dev(x, cuda, td), dev(w, cuda, td), top, groups, keep, group_rank=ops.MOE_GROUP_MAX)[0].cpu().numpy()
    assert (te2 != te).any()


@pytest.mark.parametrize("D", [40, 301, 4100])
def test_residual_norm_and_embedding(cuda, lib, D):
    import torch
    from zhilight_b200 import ops
    rng = np.random.default_rng(4)
    T, P, eps = 7, 3, 1e-3
    x, parts, coef = (rng.standard_normal(s).astype(np.float32) for s in ((T, D), (T, P, D), (T, P)))
    x[2] *= 1e-2                                                  # eps inside the root matters in this row
    parts[2] *= 1e-2
    nw = rng.standard_normal(D).astype(np.float32)
    want = x + np.einsum("tp,tpd->td", coef.astype(np.float64), parts)
    ref = orc.rms(want, eps) * nw
    xd, cat = dev(x, cuda), torch.full((T, 2 * D), 7.0, dtype=torch.bfloat16, device=cuda)
    h = ops.residual_norm(xd, dev(parts, cuda), dev(coef, cuda), dev(nw, cuda), cat, eps, torch.bfloat16)
    assert np.abs(xd.cpu().numpy() - want).max() < 3e-6 * np.abs(want).max()
    assert np.abs(h.float().cpu().numpy() - ref).max() < 2.0 ** -8 * np.abs(ref).max()
    assert np.abs(cat[:, :D].float().cpu().numpy() - want).max() < 2.0 ** -8 * np.abs(want).max() and bool((cat[:, D:] == 7.0).all())
    xd = dev(x, cuda)                                             # no parts: x stays, its norm in float32
    h = ops.residual_norm(xd, next_w=dev(nw, cuda), eps=eps)
    assert np.array_equal(xd.cpu().numpy(), x) and np.abs(h.cpu().numpy() - orc.rms(x.astype(np.float64), eps) * nw).max() < 1e-4
    xd = dev(x, cuda)                                             # one part without a coefficient, no norm
    assert ops.residual_norm(xd, dev(parts[:, :1], cuda)) is None
    assert np.abs(xd.cpu().numpy() - (x + parts[:, 0])).max() < 1e-6
    table = dev(b16(rng.standard_normal((9, D))), cuda, torch.bfloat16)
    cat = torch.zeros((T, 2 * D), dtype=torch.bfloat16, device=cuda)
    ids = [0, 8, 3, 3, 1, 7, 2]
    xe, he = ops.embed_norm(i32(ids, cuda), table, dev(nw, cuda), cat[:, D:], cat, eps)
    assert torch.equal(xe, table[ids].float()) and torch.equal(cat, torch.cat([table[ids], table[ids]], 1))
    ref = orc.rms(table[ids].double().cpu().numpy(), eps) * nw
    assert np.abs(he.float().cpu().numpy() - ref).max() < 2.0 ** -8 * np.abs(ref).max()


ATT = [(8, 2, 16, 32), (4, 2, 32, 24), (2, 2, 12, 10), (4, 4, 64, 64), (4, 1, 128, 128), (6, 2, 16, 40), (16, 1, 16, 16)]


def _runs(cuda, rows_runs):
    row0 = np.concatenate([[0], np.cumsum(rows_runs)[:-1]])
    return dict(run_row0=i32(row0, cuda), run_len=i32(rows_runs, cuda), max_run_len=max(rows_runs))


def _caches(k, v, n, cuda, td):
    """Slot 1 of two holds the rows; everything else -- the other slot, rows past the end -- is a huge finite number."""
    import torch
    kc = torch.full((2, n + 5, k.shape[1]), 3e4, dtype=td, device=cuda)
    vc = torch.full((2, n + 5, v.shape[1]), 3e4, dtype=td, device=cuda)
    kc[1, :n], vc[1, :n] = dev(k, cuda, td), dev(v, cuda, td)
    return kc, vc


@pytest.mark.parametrize("shape", ATT)
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_differential_window_attention(cuda, lib, dtype, shape):
    """Two maps per head in windows of 1, 63, 64, 65, 200 and everything; the key just inside the window of token 250
    carries the first map of one head, the key just outside would carry the second one if it were seen; gate and no gate;
    splits; single rows, runs of one and two runs whose tiles straddle the window."""
    import torch
    from zhilight_b200 import ops
    H, G, d, vd = shape
    td = getattr(torch, dtype)
    n, scale, diff, lam, eps = 290, 0.7 / math.sqrt(d), 0.35, 0.62, 1e-5
    rng = np.random.default_rng(7)
    q0, k0, v = b16(rng.standard_normal((n, H, 2, d))), b16(rng.standard_normal((n, G, 2, d))), b16(rng.standard_normal((n, G, vd)))
    gate = rng.standard_normal((n, H * vd)).astype(np.float32)
    tol = 3e-5 if dtype == "float32" else 2e-2
    for window in (1, 63, 64, 65, 200, 0):
        q, k = q0.copy(), k0.copy()
        if window > 1:
            k[250 - window + 1, 0, 0] = b16(np.sign(q[250, 0, 0]) * 8.0)       # just inside: map 1 of head 0
            k[250 - window, 0, 1] = b16(np.sign(q[250, 0, 1]) * 8.0)           # just outside: map 2 of head 0
        att = orc.differential_attention(q.astype(np.float64), k.astype(np.float64), v.astype(np.float64), scale, window, lam, diff, eps)
        want = att.reshape(n, H * vd)
        gated = want * orc.sigmoid(gate.astype(np.float64))
        if window in (63, 64, 65, 200):
            off = orc.differential_attention(q.astype(np.float64), k.astype(np.float64), v.astype(np.float64), scale, window - 1, lam, diff, eps)
            on = orc.differential_attention(q.astype(np.float64), k.astype(np.float64), v.astype(np.float64), scale, window + 1, lam, diff, eps)
            assert np.abs(off[250, 0] - att[250, 0]).max() > 0.2 and np.abs(on[250, 0] - att[250, 0]).max() > 0.2
        kc, vc = _caches(k.reshape(n, -1), v.reshape(n, -1), n, cuda, td)
        args = (ops.slot_table(kc), ops.slot_table(vc))

        def run(rows, g, **kw):
            return ops.window_attention(dev(q[rows].reshape(len(rows), -1), cuda, td), *args, i32([1] * len(rows), cuda), i32(rows, cuda),
                                        scale, window, H, G, d, vd, maps=2, lam=lam, out_eps=eps, out_mul=1 - diff,
                                        gate=dev(gate[rows], cuda) if g else None, **kw).float().cpu().numpy()

        rows = [0, 1, 2, 31, 62, 63, 64, 65, 66, 127, 128, 199, 200, 249, 250, 251, 289]
        seq = list(range(7)) + list(range(170, 290))
        for splits in (1, 2, 5):
            assert np.abs(run(rows, True, splits=splits) - gated[rows]).max() < tol, (window, splits)
            assert np.abs(run(rows, False, splits=splits, **_runs(cuda, [1] * len(rows))) - want[rows]).max() < tol, (window, splits, "ones")
            assert np.abs(run(seq, True, splits=splits, **_runs(cuda, [7, 120])) - gated[seq]).max() < tol, (window, splits, "runs")
        # one map: plain window attention over the first maps' keys of the same shape
        k1 = np.ascontiguousarray(k[:, :, 0])
        kc1, _ = _caches(k1.reshape(n, -1), v.reshape(n, -1), n, cuda, td)
        plain = orc.mixed_head_attention(q[:, :, 0].astype(np.float64), k1.astype(np.float64), v.astype(np.float64), scale, window,
                                         np.ones(H), np.eye(H)).reshape(n, H * vd)
        got = ops.window_attention(dev(q[seq, :, 0].reshape(len(seq), -1), cuda, td), ops.slot_table(kc1), args[1], i32([1] * len(seq), cuda),
                                   i32(seq, cuda), scale, window, H, G, d, vd, splits=2, **_runs(cuda, [7, 120])).float().cpu().numpy()
        assert np.abs(got - plain[seq]).max() < tol, (window, "one map")


@pytest.mark.parametrize("shape", [(8, 2, 16, 16), (4, 4, 32, 48), (6, 2, 16, 32), (16, 8, 64, 64), (12, 12, 16, 16), (3, 1, 12, 10),
                                   (32, 8, 32, 128), (40, 4, 16, 16), (1, 1, 16, 16)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_attention_with_mixed_heads(cuda, lib, dtype, shape):
    """The scores of all heads mixed before the softmax, windows around the tiles and everything; the key just inside and
    the one just outside the window of token 250 stand out through ANOTHER head's query; splits, single rows and runs."""
    import torch
    from zhilight_b200 import ops
    H, G, d, vd = shape
    td = getattr(torch, dtype)
    n, scale = 290, 0.5 / math.sqrt(d)
    rng = np.random.default_rng(11)
    q0, k0, v = b16(rng.standard_normal((n, H, d))), b16(rng.standard_normal((n, G, d))), b16(rng.standard_normal((n, G, vd)))
    temp, talk = 1 + 0.3 * rng.standard_normal(H), np.eye(H) + 0.5 * rng.standard_normal((H, H)) / math.sqrt(H)
    talk[0] = 0.0
    talk[0, H - 1] = 1.5                                            # head 0 scores by the last head's query and keys only
    talk = b16(talk).astype(np.float64)                             # a weight: exact in bfloat16
    factor = (temp * scale).astype(np.float32)
    tol = 4e-5 if dtype == "float32" else 2e-2
    for window in (1, 31, 32, 33, 64, 0):
        q, k = q0.copy(), k0.copy()
        if window > 1:
            k[250 - window + 1, G - 1] = b16(np.sign(q[250, H - 1]) * 6.0 * np.sign(temp[H - 1]))
            k[250 - window, G - 1] = b16(np.sign(q[250, H - 1]) * 12.0 * np.sign(temp[H - 1]))
        ref = lambda w: orc.mixed_head_attention(q.astype(np.float64), k.astype(np.float64), v.astype(np.float64), scale, w, temp, talk)
        att = ref(window)
        if window in (31, 32, 33, 64):
            assert np.abs(ref(window - 1)[250, 0] - att[250, 0]).max() > 0.2 and np.abs(ref(window + 1)[250, 0] - att[250, 0]).max() > 0.2
        want = att.reshape(n, H * vd)
        kc, vc = _caches(k.reshape(n, -1), v.reshape(n, -1), n, cuda, td)
        tabs = (ops.slot_table(kc), ops.slot_table(vc))

        def run(rows, **kw):
            return ops.mixed_head_attention(dev(q[rows].reshape(len(rows), -1), cuda, td), *tabs, i32([1] * len(rows), cuda),
                                            i32(rows, cuda), dev(talk.astype(np.float32), cuda), dev(factor, cuda), window, H, G, d, vd, **kw).float().cpu().numpy()

        rows = [0, 1, 15, 16, 17, 31, 32, 33, 63, 64, 65, 127, 249, 250, 251, 289]
        seq = list(range(9)) + list(range(200, 290))
        for splits in (1, 3):
            assert np.abs(run(rows, splits=splits) - want[rows]).max() < tol, (window, splits)
            assert np.abs(run(rows, splits=splits, **_runs(cuda, [1] * len(rows))) - want[rows]).max() < tol, (window, splits, "ones")
            assert np.abs(run(seq, splits=splits, **_runs(cuda, [9, 90])) - want[seq]).max() < tol, (window, splits, "runs")


@pytest.mark.parametrize("shape", [(3, 20, 20, 6), (4, 64, 64, 16), (20, 64, 128, 48), (16, 48, 64, 16), (5, 100, 128, 64), (2, 512, 512, 64)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_latent_attention_with_rotated_part(cuda, lib, dtype, shape):
    """Score over latent and rotated columns, value the latent alone.  One far key is found by one head through its rotated
    part only, one by another head through its latent; padding columns of the cached row are zero and must not count;
    gate, sink and neither; splits 1 / 2 / 7."""
    import torch
    from zhilight_b200 import ops
    H, R, RC, r = shape
    td = getattr(torch, dtype)
    RS = RC + (r if RC == R and R % 64 else (r + 15) // 16 * 16)
    n, scale = 300, 0.3
    rng = np.random.default_rng(13)
    qa = np.zeros((n, H, RS), np.float32)
    qa[:, :, :R], qa[:, :, RC:RC + r] = b16(rng.standard_normal((n, H, R)) / math.sqrt(R)), b16(rng.standard_normal((n, H, r)) / math.sqrt(r))
    c = np.zeros((n, RS), np.float32)
    c[:, :R], c[:, RC:RC + r] = b16(rng.standard_normal((n, R))), b16(rng.standard_normal((n, r)))
    rows = [0, 1, 31, 32, 33, 63, 64, 65, 127, 128, 255, 256, 280, 299]
    c[11, RC:RC + r] *= 4
    c[23, :R] *= 2
    qa[280, 0, RC:RC + r] = b16(c[11, RC:RC + r] * 40 / np.sum(c[11, RC:RC + r] ** 2))
    qa[280, H - 1, :R] = b16(c[23, :R] * 40 / np.sum(c[23, :R] ** 2))
    s = np.einsum("thc,jc->thj", qa[rows].astype(np.float64), c.astype(np.float64)) * scale
    sink, gate = rng.standard_normal(H).astype(np.float32) + 2, rng.standard_normal((n, H)).astype(np.float32)
    cache = torch.full((2, n + 3, RS), 3e4, dtype=td, device=cuda)
    cache[1, :n] = dev(c, cuda, td)
    for use_sink in (False, True):
        want = np.zeros((len(rows), H, R))
        for i, t in enumerate(rows):
            e = np.exp(s[i, :, :t + 1])
            want[i] = e @ c[:t + 1, :R] / (e.sum(-1, keepdims=True) + (np.exp(sink)[:, None] if use_sink else 0.0))
            if t == 280 and not use_sink:
                assert e[0, 11] / e[0].sum() > 0.9 and e[H - 1, 23] / e[H - 1].sum() > 0.9
        tol = (3e-5 if dtype == "float32" else 2.5e-2)
        for splits in (1, 2, 7):
            for g in (False, True):
                out = ops.latent_attention_ex(dev(qa[rows], cuda), cache, ops.slot_table(cache), i32([1] * len(rows), cuda), i32(rows, cuda),
                                              scale, RC, sink=dev(sink, cuda) if use_sink else None,
                                              gate=dev(gate[rows], cuda) if g else None, splits=splits).float().cpu().numpy()
                ref = want * orc.sigmoid(gate[rows].astype(np.float64))[:, :, None] if g else want
                assert np.abs(out[:, :, :R] - ref).max() < tol and np.abs(out[:, :, R:]).max(initial=0.0) == 0.0, (splits, g, use_sink)
    # two runs of consecutive tokens: the tiles of a prompt
    seq = list(range(5)) + list(range(230, 300))
    s = np.einsum("thc,jc->thj", qa[seq].astype(np.float64), c.astype(np.float64)) * scale
    for use_sink in (False, True):
        want = np.zeros((len(seq), H, R))
        for i, t in enumerate(seq):
            e = np.exp(s[i, :, :t + 1])
            want[i] = e @ c[:t + 1, :R] / (e.sum(-1, keepdims=True) + (np.exp(sink)[:, None] if use_sink else 0.0))
        want *= orc.sigmoid(gate[seq].astype(np.float64))[:, :, None]
        for splits in (1, 3):
            out = ops.latent_attention_ex(dev(qa[seq], cuda), cache, ops.slot_table(cache), i32([1] * len(seq), cuda), i32(seq, cuda), scale,
                                          RC, sink=dev(sink, cuda) if use_sink else None, gate=dev(gate[seq], cuda), splits=splits,
                                          **_runs(cuda, [5, 70])).float().cpu().numpy()
            assert np.abs(out[:, :, :R] - want).max() < tol and np.abs(out[:, :, R:]).max(initial=0.0) == 0.0, (splits, use_sink, "runs")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_latent_rows_and_frequencies(cuda, lib, dtype):
    """Norm of the latent, rotation of the queries' last and the shared key's dimensions at positions near 900, the rows
    appended with padding columns untouched; frequencies by wavelength in all three ranges."""
    import torch
    from zhilight_b200 import ops
    td = getattr(torch, dtype)
    scaling = (3.0, 1.0, 5.0, 200.0)
    for dims, base in ((16, 1e4), (6, 500.0), (64, 5e5)):
        for sc in (None, scaling):
            got = ops.rope_inv_freq_wavelength(base, dims, sc)
            want = orc.frequencies(dims, base, dict(zip(("factor", "low", "high", "original"), sc)) if sc else None)
            assert np.allclose(got, want, rtol=1e-14, atol=0)
    f = orc.frequencies(64, 1e4, dict(zip(("factor", "low", "high", "original"), scaling)))
    ratio = f / orc.frequencies(64, 1e4)
    assert (ratio == 1).any() and np.isclose(ratio, 1 / 3).any() and ((ratio > 0.34) & (ratio < 0.99)).any()
    H, d, r, R, RC, RS, eps = 3, 10, 6, 20, 24, 40, 1e-2
    freqs = orc.frequencies(r, 100.0)
    slots, pos = [2, 2, 2, 0, 1], [898, 899, 900, 0, 37]
    T, n_in = 5, H * (d + r) + R + r + 3
    rng = np.random.default_rng(17)
    proj = rng.standard_normal((T, n_in)).astype(np.float32)
    proj[1, H * (d + r):H * (d + r) + R] *= 0.05                     # eps matters in this row
    w = rng.standard_normal(R).astype(np.float32)
    tab = ops.rope_table(i32(pos, cuda), dev(freqs, cuda))
    cache = torch.full((3, 950, RS), 5.0, dtype=td, device=cuda)
    qa = torch.full((T, H, RS), 5.0, dtype=torch.float32, device=cuda)
    q = ops.latent_rope_append(dev(proj, cuda), 0, H, d, r, tab, H * (d + r), R, dev(w, cuda), RC, qa, cache, ops.slot_table(cache),
                               i32(slots, cuda), i32(pos, cuda), eps)
    p = proj.astype(np.float64)
    wq = p[:, :H * (d + r)].reshape(T, H, d + r)
    ckv = p[:, H * (d + r):H * (d + r) + R + r]
    ang = np.array(pos)[:, None] * freqs[None, :]

    def turn(x, a):
        y = x.copy()
        y[..., 0::2] = x[..., 0::2] * np.cos(a) - x[..., 1::2] * np.sin(a)
        y[..., 1::2] = x[..., 1::2] * np.cos(a) + x[..., 0::2] * np.sin(a)
        return y

    tol = 3e-6 if dtype == "float32" else 2e-2
    assert np.abs(q.float().cpu().numpy() - wq[..., :d]).max() < tol
    qa = qa.cpu().numpy()
    assert np.abs(qa[..., RC:RC + r] - turn(wq[..., d:], ang[:, None, :])).max() < 3e-6
    assert (qa[..., :RC] == 5).all() and (qa[..., RC + r:] == 5).all()
    row = np.stack([cache[s, t].float().cpu().numpy() for s, t in zip(slots, pos)])
    assert np.abs(row[:, :R] - orc.rms(ckv[:, :R], eps) * w).max() < tol * 3
    assert np.abs(row[:, RC:RC + r] - turn(ckv[:, R:], ang)).max() < tol
    assert (row[:, R:RC] == 5).all() and (row[:, RC + r:] == 5).all() and bool((cache[1, 36] == 5).all())


# ---------------------------------------------------------------------------------------------- the whole model
@pytest.mark.parametrize("name", sorted(CONFIGS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prompt_layers_caches_and_logits(cuda, lib, name, dtype):
    cfg, W, m = make(CONFIGS[name], dtype, seed=1, max_step_tokens=128)
    toks = tokens_for(cfg, 97, 5)
    want, streams, caches = orc.forward(cfg, W, toks)
    m.capture_layers(True)
    _, logits = m.step(toks, [2] * len(toks), range(len(toks)), range(len(toks)))
    got_streams = m.read_layers(len(toks))
    assert got_streams.shape == streams.shape and len(caches) == cfg.num_runs
    for i in range(cfg.num_runs):   # the first run that differs is the one to look at
        rows = np.abs(got_streams[i] - streams[i]).max(-1) / np.abs(streams[i]).max()
        d = rows.max() if dtype == "float32" else np.quantile(rows, 0.9)
        assert d < (1e-4 if dtype == "float32" else 6e-2), (name, dtype, "run", i, d)
        for got, ref in zip(m.read_cache(i, 2, len(toks)), caches[i]):
            rows = np.abs(got - ref).max(-1) / np.abs(ref).max()
            d = rows.max() if dtype == "float32" else np.quantile(rows, 0.9)
            assert d < (1e-4 if dtype == "float32" else 6e-2), (name, dtype, "cache of run", i, d)
    assert rel_err(logits, want, dtype) < TOL[dtype]
    m.close()


@pytest.mark.parametrize("name", sorted(CONFIGS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prefill_vs_token_by_token_and_portions(cuda, lib, name, dtype):
    """The same prompt whole, token by token, and in portions down to two tokens: every position (the first tokens of the
    sequence among them) against the oracle and the three runs against one another."""
    from zhilight_b200.engine import Engine
    cfg, W, m = make(CONFIGS[name], dtype, seed=2, max_step_tokens=64)
    eng = Engine(m)
    n = 131
    toks = tokens_for(cfg, n, 9)
    want = orc.forward(cfg, W, toks)[0]
    runs = {}
    for label, sizes in (("whole", [n]), ("single", [1] * n), ("portions", [2, 3, 2, 17, 1, 2, 31, 5, 2, 40, 2, 2, 22])):
        assert sum(sizes) == n
        eng.open(label)
        rows, at = [], 0
        for s in sizes:
            rows.append(eng.forward_step([(label, toks[at:at + s], list(range(s)))])[label][1])
            at += s
        eng.close(label)
        runs[label] = np.concatenate(rows)
        assert rel_err(runs[label], want, dtype) < TOL[dtype], (name, dtype, label)
        assert rel_err(runs[label][:3], want[:3], "float32") < TOL[dtype], (name, dtype, label, "first tokens")
    cut = 2e-5 if dtype == "float32" else 3e-2      # the cuts change the order of sums, no more
    assert rel_err(runs["single"], runs["whole"].astype(np.float64), dtype) < cut
    assert rel_err(runs["portions"], runs["whole"].astype(np.float64), dtype) < cut
    m.close()


@pytest.mark.parametrize("name", ["odd", "tiles"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_batch_against_each_alone_and_slot_reuse(cuda, lib, name, dtype):
    """Three requests of different lengths share steps (prompt portions next to single decode tokens); afterwards their
    slots -- caches of every pass still in them -- are handed to new requests.  Every logit row equals the request alone."""
    from zhilight_b200.engine import Engine
    cfg, W, m = make(CONFIGS[name], dtype, seed=3, max_batch=3, max_step_tokens=16)
    eng = Engine(m)
    prompts = {"a": tokens_for(cfg, 41, 1), "b": tokens_for(cfg, 9, 2), "c": tokens_for(cfg, 26, 3)}
    later = {"d": tokens_for(cfg, 30, 4), "e": tokens_for(cfg, 5, 5)}
    want = {k: orc.forward(cfg, W, v)[0] for k, v in {**prompts, **later}.items()}
    got = {k: [] for k in want}
    at = {k: 0 for k in want}
    for k in prompts:
        eng.open(k)
    plan = [{"a": 7, "b": 2, "c": 1}, {"a": 1, "b": 1, "c": 12}, {"a": 20, "b": 1, "c": 1}, {"a": 1, "b": 5, "c": 2},
            {"a": 12, "c": 10}]
    for step in plan:
        entries = [(k, prompts[k][at[k]:at[k] + n], list(range(n))) for k, n in step.items()]
        res = eng.forward_step(entries)
        for k, n in step.items():
            got[k].append(res[k][1])
            at[k] += n
    assert at == {"a": 41, "b": 9, "c": 26, "d": 0, "e": 0}
    used = {eng.seqs[k].slot for k in prompts}
    for k in prompts:
        eng.close(k)
    for k in later:
        assert eng.open(k).slot in used
    res = eng.forward_step([("d", later["d"][:11], list(range(11))), ("e", later["e"], list(range(5)))])
    got["d"].append(res["d"][1]); got["e"].append(res["e"][1])
    got["d"].append(eng.forward_step([("d", later["d"][11:], list(range(19)))])["d"][1])
    for k in want:
        assert rel_err(np.concatenate(got[k]), want[k], dtype) < TOL[dtype], (dtype, k)
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_through_graphs_and_splits(cuda, lib, dtype):
    """A short prompt and then 330 single-token steps: the windows pass over decoded tokens, the decode graph, the length
    buckets (256, 512) and the key splits of the attention kernels all change on the way."""
    cfg, W, m = make(CFG_TILES, dtype, seed=4, max_batch=2, max_seq=512, max_step_tokens=16)
    toks = tokens_for(cfg, 340, 11)
    want = orc.forward(cfg, W, toks)[0]
    _, first = m.step(toks[:10], [1] * 10, range(10), range(10))
    rows = [first]
    for p in range(10, 340):
        rows.append(m.step([toks[p]], [1], [p], [0])[1])
    assert rel_err(np.concatenate(rows), want, dtype) < TOL[dtype]
    assert m.stats()[1] > 0          # the single-token steps were replayed as graphs
    m.close()


def test_far_token_is_found_through_the_model(cuda, lib):
    """Token 7 of 300 moves the last logits by far more than the float32 tolerance (the oracle says so first) although it
    is far outside every window: the latent layers' caches carry it through prompt portions and decoding."""
    cfg, W, m = make(CFG_TILES, "float32", seed=5, max_batch=2, max_seq=320, max_step_tokens=64)
    toks = tokens_for(cfg, 300, 13)
    base = orc.forward(cfg, W, toks)[0][-1]
    other = list(toks)
    other[7] = (toks[7] + 1) % cfg.vocab
    moved = orc.forward(cfg, W, other)[0][-1]
    assert rel_err(moved[None], base[None]) > 10 * TOL["float32"]   # the oracle says token 7 matters at the end
    for seq, want in ((toks, base), (other, moved)):
        for c0 in range(0, 256, 64):
            m.step(seq[c0:c0 + 64], [0] * 64, range(c0, c0 + 64))
        for p in range(256, 299):
            m.step([seq[p]], [0], [p])
        got = m.step([seq[299]], [0], [299], [0])[1]
        assert rel_err(got, want[None]) < TOL["float32"]
    m.close()


def test_passes_of_a_loop_keep_their_own_caches(cuda, lib):
    """The same layer caches different rows in every pass, and a loop of one pass still goes through the input mix."""
    cfg, W, m = make(CFG_ODD, "float32", seed=9, max_step_tokens=32)
    toks = tokens_for(cfg, 12, 2)
    m.step(toks, [0] * 12, range(12), [11])
    runs = [r for r in range(cfg.num_runs) if cfg.run_layer(r) == 1]
    assert runs == [1, 3, 5]
    a = [m.read_cache(r, 0, 12)[0] for r in runs]
    assert np.abs(a[0] - a[1]).max() > 0.05 and np.abs(a[1] - a[2]).max() > 0.05
    m.close()
    once = dict(CFG_ODD, loop={"start": 1, "stop": 3, "times": 1})
    none = {k: v for k, v in CFG_ODD.items() if k != "loop"}
    outs = []
    for d in (once, none):
        cfg, W, m = make(d, "float32", seed=9, max_step_tokens=32)
        want = orc.forward(cfg, W, toks)[0]
        _, got = m.step(toks, [0] * 12, range(12), range(12))
        assert rel_err(got, want) < TOL["float32"]
        outs.append(got)
        m.close()
    assert rel_err(outs[0], outs[1].astype(np.float64)) > 0.1


def test_device_resident_decode_loop(cuda, lib):
    """set_state / step_device (greedy picks fed back on the device) give the tokens of step-by-step greedy decoding."""
    cfg, W, m = make(CFG_TILES, "float32", seed=7, max_batch=2, max_seq=64, max_step_tokens=16)
    prompts = [tokens_for(cfg, 9, 1), tokens_for(cfg, 9, 2)]
    nxt = []
    for s, p in enumerate(prompts):
        nxt.append(int(m.step(p, [s] * 9, range(9), [8])[0][0]))
    ref = [list(p) + [n] for p, n in zip(prompts, nxt)]
    m.set_state(nxt, [9, 9])
    for _ in range(5):
        m.step_device(2)
    m.sync()
    for s in range(2):
        for _ in range(5):
            logits = orc.forward(cfg, W, ref[s])[0][-1]
            ref[s].append(int(np.argmax(logits)))
    # replay the same on the host path against the device loop's caches: position 14 sees what the loop wrote
    for s in range(2):
        got = m.step([ref[s][14]], [s], [14], [0])[1]
        want = orc.forward(cfg, W, ref[s][:15])[0][-1]
        assert rel_err(got, want[None]) < TOL["float32"], s
    m.close()


def test_greedy_generation_through_the_scheduler(cuda, lib):
    """Engine.generate (admission, portions, mixed steps, retiring, slot reuse: 5 prompts on 2 slots) against greedy
    decoding with the oracle; float32 so that near-ties do not flip."""
    from zhilight_b200.engine import Engine
    cfg, W, m = make(CFG_ODD, "float32", seed=6, max_batch=2, max_seq=128, max_step_tokens=8)
    prompts = [tokens_for(cfg, n, 20 + n) for n in (3, 19, 1, 11, 6)]
    seen = []
    outs = Engine(m).generate(prompts, max_new_tokens=7, on_step=lambda e: seen.append([len(t) for _, t, _ in e]))
    assert any(len(s) > 1 and max(s) > 1 and min(s) == 1 for s in seen)    # a prompt portion beside a decode token
    for p, out in zip(prompts, outs):
        seq = list(p)
        for tok in out:
            logits = orc.forward(cfg, W, seq)[0][-1]
            top = np.sort(logits)[-2:]
            assert tok == int(np.argmax(logits)) or top[1] - top[0] < 1e-4
            seq.append(tok)
        assert len(out) == 7
    m.close()


def test_model_folder_registry_and_trace_replay(cuda, lib, tmp_path):
    """config.json + model.safetensors on disk -> registry -> trace replay: the written logits are the oracle's."""
    from zhilight_b200 import registry, safetensors_io, trace
    from zhilight_b200.dekalorn import DekalornConfig
    cfg = DekalornConfig.from_dict(CFG_ODD)
    W = orc.random_weights(cfg, 8)
    (tmp_path / "m").mkdir()
    (tmp_path / "m" / "config.json").write_text(json.dumps(CFG_ODD))
    safetensors_io.save_file({k: safetensors_io.f32_to_bf16(v) for k, v in W.items()}, str(tmp_path / "m" / "model.safetensors"))
    model = registry.load_model(str(tmp_path / "m"), "float32", max_batch=2, max_seq=64, max_step_tokens=8)
    toks = tokens_for(cfg, 21, 3)
    lines = [json.dumps({"step": 0, "entries": [{"id": "x", "tokens": toks[:13], "want": [12, 0, 5]}], "end": []}),
             json.dumps({"step": 1, "entries": [{"id": "x", "tokens": toks[13:20], "want": []}], "end": []}),
             json.dumps({"step": 2, "entries": [{"id": "x", "tokens": toks[20:], "want": [0]}], "end": ["x"]})]
    said = []
    trace.replay(model, lines, str(tmp_path), emit=said.append)
    assert said == ["done 0", "done 1", "done 2"] and not (tmp_path / "1.f32").exists()
    want = orc.forward(cfg, {k: v.astype(np.float64) for k, v in W.items()}, toks)[0]
    got0 = np.fromfile(tmp_path / "0.f32", dtype="<f4").reshape(3, cfg.vocab)
    got2 = np.fromfile(tmp_path / "2.f32", dtype="<f4").reshape(1, cfg.vocab)
    assert rel_err(got0, want[[12, 0, 5]]) < TOL["float32"] and rel_err(got2, want[[20]]) < TOL["float32"]
    model.close()
