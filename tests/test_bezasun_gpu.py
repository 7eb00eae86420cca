"""Bezasun on the GPU against the plain numpy restatement in tests/bezasun_oracle.py.

Small configurations of their own (all sizes different from one another, and all ones; the three mixers in several orders with
and without experts, with and without a shared one; one to five streams; windows of 1 and of sizes around the kernels' tiles;
head counts with and without a tensor-core tile), random bfloat16-exact weights.  float32 runs are held to a tight tolerance,
bfloat16 runs to a loose one; the measure is the RMS over the vocabulary of the mean-free difference of the logits, relative to
the RMS of the logits.
"""
import json
import math

import numpy as np
import pytest

from tests import bezasun_oracle as orc

pytestmark = pytest.mark.gpu

TOL = {"float32": 2e-4, "bfloat16": 5e-2}


def ATT(heads, kv_heads, dim, vdim, scale, softcap=None, temp=None, mlp=None):
    mx = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale)
    if softcap:
        mx["softcap"] = softcap
    if temp:
        mx["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "attention", "mixer": mx, "mlp": mlp}


def LATENT(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, window, base=10000.0, scaling=None, mlp=None):
    rot = dict(base=base, dims=rot_dim)
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    mx = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale, rot=rot)
    if window:
        mx["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": mx, "mlp": mlp}


def SSM(heads, vdim, state, groups, conv, norm_groups, mlp=None):
    return {"type": "mamba2", "mlp": mlp,
            "mixer": dict(heads=heads, vdim=vdim, state=state, groups=groups, conv=conv, norm_groups=norm_groups)}


def MOE(experts, top, ff, shared=0):
    d = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        d["shared"] = {"ff": shared}
    return d


def CFG(vocab, width, streams, layers, residual_mult=0.8, logit_scale=0.6, embed_scale=9.0, eps=1e-5):
    return {"architecture": "Bezasun", "vocab": vocab, "width": width, "streams": streams, "residual_mult": residual_mult,
            "logit_scale": logit_scale, "embedding": {"scale": embed_scale}, "norm": {"eps": eps}, "layers": layers}


# sizes without tensor-core tiles
CFG_ODD = CFG(67, 44, 2, [LATENT(3, 10, 6, 14, 22, 20, 0.25, 9, base=500.0, scaling=(3.0, 60, 8.0, 1.0), mlp=MOE(6, 2, 20, 28)),
                          SSM(6, 5, 9, 3, 4, 2, mlp=MOE(5, 3, 24)),
                          ATT(4, 2, 12, 10, 0.3, 7.0, (0.6, 13), mlp=MOE(7, 4, 12, 36)),
                          SSM(2, 7, 18, 1, 2, 2)])
CFG_ONES = CFG(40, 32, 1, [SSM(1, 1, 1, 1, 1, 1, mlp=MOE(1, 1, 8, 1)), LATENT(1, 1, 2, 1, 1, 1, 0.7, 1),
                           ATT(1, 1, 6, 4, 0.4, mlp=MOE(2, 2, 16))], 1.0, 1.0, 1.0, 1e-6)
# tensor-core sizes: heads of 16 / 32 / 64, a latent that is padded, windows around the 32-row tiles
CFG_TILES = CFG(96, 64, 4, [SSM(8, 16, 32, 2, 4, 4, mlp=MOE(8, 3, 40, 64)),
                            ATT(8, 2, 32, 32, 0.18, 20.0, (0.4, 50), mlp=MOE(6, 2, 32, 48)),
                            LATENT(4, 16, 16, 24, 32, 48, 0.2, 40, base=2e4, scaling=(4.0, 256, 16.0, 1.0), mlp=MOE(4, 2, 16, 24)),
                            LATENT(8, 32, 32, 32, 64, 64, 0.12, 65, base=2e4, scaling=(8.0, 512, 32.0, 1.0)),
                            ATT(4, 4, 16, 64, 0.25, None, None, mlp=MOE(4, 1, 24))])
# five streams (the general residual kernel), no window, no scaling, groups = heads, a state over one compiled size
CFG_WIDE = CFG(80, 96, 5, [ATT(6, 2, 24, 40, 0.2, 15.0, (0.3, 7)), LATENT(5, 32, 8, 16, 40, 64, 0.15, 0, mlp=MOE(9, 4, 32)),
                           SSM(4, 36, 20, 4, 3, 1, mlp=MOE(3, 3, 16, 40))], 0.5, 2.0, 20.0)
CONFIGS = {"odd": CFG_ODD, "ones": CFG_ONES, "tiles": CFG_TILES, "wide": CFG_WIDE}


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
    from zhilight_b200.bezasun import BezasunConfig, BezasunDecoder
    from zhilight_b200.safetensors_io import f32_to_bf16
    cfg = BezasunConfig.from_dict(cfg_dict)
    W = orc.random_weights(cfg, seed)
    m = BezasunDecoder(cfg, dtype=dtype, max_batch=max_batch, max_seq=max_seq, max_step_tokens=max_step_tokens, **kw)
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


def f64(a):
    return np.asarray(a, dtype=np.float64)


def _runs(cuda, lens):
    row0 = np.concatenate([[0], np.cumsum(lens)[:-1]])
    return dict(run_row0=i32(row0, cuda), run_len=i32(lens, cuda), max_run_len=max(lens))


# ---------------------------------------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("shape", [(1, 40), (2, 301), (3, 48), (4, 4100), (3, 1030), (6, 64), (16, 33), (2, 9000)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_streams(cuda, lib, dtype, shape):
    """Write and read of the streams (mix indexed [from, to]: an asymmetric matrix), one result and several weighted ones with a
    dense one added, the sum of the streams, no update at all, a row whose norm eps decides; the embedding as the start."""
    import torch
    from zhilight_b200 import ops
    S, D = shape
    td = getattr(torch, dtype)
    T, P, eps = 5, 3, 1e-2
    rng = np.random.default_rng(S * 1000 + D)
    x = rng.standard_normal((S, T, D)).astype(np.float32)
    x[:, 3] *= 0.03
    parts, coef = rng.standard_normal((T, P, D)).astype(np.float32), rng.standard_normal((T, P)).astype(np.float32)
    parts[3] *= 0.03
    dense = rng.standard_normal((T, D)).astype(np.float32) * np.where(np.arange(T) == 3, 0.03, 1.0)[:, None].astype(np.float32)
    mix, out, w_in = (rng.standard_normal(s).astype(np.float32) for s in ((S, S), (S,), (S,)))
    nw = rng.standard_normal(D).astype(np.float32)
    tol = 2e-5 if dtype == "float32" else 3e-2
    for many in (False, True):
        y = np.einsum("tp,tpd->td", f64(coef), f64(parts)) + dense if many else f64(parts[:, 0])
        want = orc.hyper_write(f64(x), f64(mix), f64(out), 1.0, y)
        u = orc.hyper_read(want, f64(w_in))
        dx = dev(x.transpose(1, 0, 2), cuda)
        pd = dev(parts if many else parts[:, :1], cuda)
        h, gu = ops.hyper_update(dx, pd, dev(mix, cuda), dev(out, cuda), dev(w_in, cuda), coef=dev(coef, cuda) if many else None,
                                 dense=dev(dense, cuda) if many else None, next_w=dev(nw, cuda), want_u=True, eps=eps, act_dtype=td)
        assert np.abs(dx.cpu().numpy().transpose(1, 0, 2) - want).max() < 2e-5 * np.abs(want).max()
        assert np.abs(gu.cpu().numpy() - u).max() < 2e-5 * np.abs(u).max()
        ref = orc.rms(u, eps) * nw
        assert np.abs(h.float().cpu().numpy() - ref).max() < tol * np.abs(ref).max()
        _, total = ops.hyper_update(dx, None, None, None, want_u=True, eps=eps)
        assert np.abs(total.cpu().numpy() - want.sum(0)).max() < 2e-5 * np.abs(want).max() * S
    table = b16(rng.standard_normal((11, D)))
    ids = [3, 10, 0, 7, 3]
    ex, eh, eu = ops.hyper_embed(i32(ids, cuda), dev(table, cuda, td), 3.5, S, dev(w_in, cuda), dev(nw, cuda), True, eps)
    want = np.stack([f64(table[ids]) * 3.5] * S)
    u = orc.hyper_read(want, f64(w_in))
    assert np.abs(ex.cpu().numpy().transpose(1, 0, 2) - want).max() < 1e-5
    assert np.abs(eu.cpu().numpy() - u).max() < 1e-5 * max(1.0, np.abs(u).max())
    ref = orc.rms(u, eps) * nw
    assert np.abs(eh.float().cpu().numpy() - ref).max() < tol * np.abs(ref).max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_head_norms_and_query_temperature(cuda, lib, dtype):
    """Norms per head with plain weights, values as projected, the temperature at positions on both sides of its steps."""
    import torch
    from zhilight_b200 import ops
    td = getattr(torch, dtype)
    H, G, d, vd, eps, coef, every = 6, 3, 20, 9, 1e-2, 0.7, 13
    pos = [0, 11, 12, 13, 24, 25, 26, 500, 597]
    T = len(pos)
    rng = np.random.default_rng(3)
    proj = rng.standard_normal((T, H * d + G * d + G * vd + 5)).astype(np.float32)
    proj[2] *= 0.02
    qw, kw = rng.standard_normal(d).astype(np.float32), rng.standard_normal(d).astype(np.float32)
    slot = [1, 0, 0, 0, 1, 1, 1, 0, 1]
    kc, vc = torch.full((2, 600, G * d), 5.0, dtype=td, device=cuda), torch.full((2, 600, G * vd), 5.0, dtype=td, device=cuda)
    temp = orc.query_temperature(600, coef, every)[pos]
    assert temp[1] == 1.0 and temp[2] > 1.4 and temp[3] == temp[2] and temp[4] == temp[2] < temp[5] == temp[6]
    for c in (coef, 0.0):
        q = ops.qkv_headnorm_append_ex(dev(proj, cuda), 0, H * d, H * d + G * d, H, G, d, vd, dev(qw, cuda), dev(kw, cuda),
                                       ops.slot_table(kc), ops.slot_table(vc), i32(slot, cuda), i32(pos, cuda), td, eps, temp_coef=c,
                                       temp_every=every)
        p = f64(proj)
        want = orc.rms(p[:, :H * d].reshape(T, H, d), eps) * qw * (temp if c else np.ones(T))[:, None, None]
        tol = 3e-6 if dtype == "float32" else 1e-2
        assert np.abs(q.float().cpu().numpy().reshape(T, H, d) - want).max() < tol * np.abs(want).max()
        k = np.stack([kc[s, t].float().cpu().numpy() for s, t in zip(slot, pos)])
        v = np.stack([vc[s, t].float().cpu().numpy() for s, t in zip(slot, pos)])
        kw_ = (orc.rms(p[:, H * d:H * d + G * d].reshape(T, G, d), eps) * kw).reshape(T, -1)
        assert np.abs(k - kw_).max() < tol * np.abs(kw_).max()
        vw = p[:, H * d + G * d:H * d + G * d + G * vd]
        assert np.abs(v - vw).max() < tol * np.abs(vw).max()
        assert bool((kc[0, 0] == 5).all()) and bool((kc[1, 12] == 5).all())


def _caches(k, v, n, cuda, td):
    """Slot 1 of two holds the rows; everything else -- the other slot, rows past the end -- is a huge finite number."""
    import torch
    kc = torch.full((2, n + 5, k.shape[1]), 3e4, dtype=td, device=cuda)
    vc = torch.full((2, n + 5, v.shape[1]), 3e4, dtype=td, device=cuda)
    kc[1, :n], vc[1, :n] = dev(k, cuda, td), dev(v, cuda, td)
    return kc, vc


@pytest.mark.parametrize("shape", [(8, 2, 32, 32), (4, 2, 12, 10), (2, 2, 64, 128), (4, 4, 16, 64), (6, 2, 16, 40), (16, 1, 128, 24), (1, 1, 5, 3)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_biased_sink_attention(cuda, lib, dtype, shape):
    """Cap, slope and sink, together and each left out: a far key whose raw score is far above the cap, the same key losing to the
    slope in the first head, a sink that outweighs all keys in the last; windows; splits; single rows and runs."""
    import torch
    from zhilight_b200 import ops
    H, G, d, vd = shape
    td = getattr(torch, dtype)
    n, scale = 300, 1.0 / math.sqrt(d)
    rng = np.random.default_rng(5)
    q, k, v = (b16(rng.standard_normal(s)) for s in ((n, H, d), (n, G, d), (n, G, vd)))
    sink = rng.standard_normal(H).astype(np.float32)
    sink[H - 1] = 6.0
    k[9] = b16(np.sign(q[280].reshape(G, H // G, d)[:, 0]) * 3.0)       # stands out for the first head of every group at token 280
    slopes = orc.distance_slopes(H)
    rows = [0, 1, 2, 31, 62, 63, 64, 65, 127, 128, 129, 255, 256, 280, 299]
    seq = list(range(5)) + list(range(215, 300))
    kc, vc = _caches(k.reshape(n, -1), v.reshape(n, -1), n, cuda, td)
    tabs = (ops.slot_table(kc), ops.slot_table(vc))
    tol = 3e-5 if dtype == "float32" else 2e-2
    base = orc.sink_attention(f64(q), f64(k), f64(v), scale, 0.0, slopes, sink)
    seen = orc.sink_attention(f64(q), f64(k), f64(v), scale, 5.0, slopes, sink)
    assert np.abs(base - seen).max() > 0.05                              # the oracle says the cap shows
    for cap, with_slope, with_sink in ((5.0, True, True), (0.0, True, True), (5.0, False, True), (5.0, True, False), (30.0, True, True)):
        sl = slopes if with_slope else np.zeros(H)
        want = orc.sink_attention(f64(q), f64(k), f64(v), scale, cap, sl, sink if with_sink else np.full(H, -np.inf)).reshape(n, H * vd)

        def run(rs, **kw):
            return ops.biased_sink_attention(dev(q[rs].reshape(len(rs), -1), cuda, td), *tabs, i32([1] * len(rs), cuda), i32(rs, cuda), scale,
                                             H, G, d, vd, sink=dev(sink, cuda) if with_sink else None, no_sink=not with_sink, softcap=cap,
                                             slopes=dev(sl.astype(np.float32), cuda) if with_slope else None, **kw).float().cpu().numpy()

        for splits in (1, 2, 7):
            what = (cap, with_slope, with_sink, splits)
            assert np.abs(run(rows, splits=splits) - want[rows]).max() < tol, what
            assert np.abs(run(rows, splits=splits, **_runs(cuda, [1] * len(rows))) - want[rows]).max() < tol, what + ("ones",)
            assert np.abs(run(seq, splits=splits, **_runs(cuda, [5, 85])) - want[seq]).max() < tol, what + ("runs",)


@pytest.mark.parametrize("shape", [(3, 20, 20, 6), (4, 64, 64, 16), (20, 64, 128, 48), (16, 48, 64, 16), (5, 100, 128, 64), (2, 512, 512, 64)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_latent_window_attention(cuda, lib, dtype, shape):
    """Windows of 1, around the 32-row tiles, 200 and everything.  The row just inside the window of token 280 carries one head
    (through its rotated part), the row just outside would carry another (through its latent); prompts and single rows; splits."""
    import torch
    from zhilight_b200 import ops
    H, R, RC, r = shape
    td = getattr(torch, dtype)
    RS = RC + (r if RC == R and R % 64 else (r + 15) // 16 * 16)
    n, scale = 300, 0.3
    rng = np.random.default_rng(13)
    qa = np.zeros((n, H, RS), np.float32)
    qa[:, :, :R], qa[:, :, RC:RC + r] = b16(rng.standard_normal((n, H, R)) / math.sqrt(R)), b16(rng.standard_normal((n, H, r)) / math.sqrt(r))
    c0 = np.zeros((n, RS), np.float32)
    c0[:, :R], c0[:, RC:RC + r] = b16(rng.standard_normal((n, R))), b16(rng.standard_normal((n, r)))
    rows = [0, 1, 30, 31, 32, 33, 63, 64, 65, 199, 200, 201, 279, 280, 281, 299]
    seq = list(range(5)) + list(range(215, 300))

    def ref(q, c, window, which):
        out = np.zeros((len(which), H, R))
        for i, t in enumerate(which):
            lo = max(0, t - window + 1) if window else 0
            s = q[t].astype(np.float64) @ c[lo:t + 1].T.astype(np.float64) * scale
            out[i] = orc.softmax_rows(s, np.ones_like(s, bool)) @ c[lo:t + 1, :R]
        return out

    for window in (1, 31, 32, 33, 64, 200, 0):
        q, c = qa.copy(), c0.copy()
        if window > 1:
            inside, outside = 280 - window + 1, 280 - window
            c[inside, RC:RC + r] *= 4
            q[280, 0, RC:RC + r] = b16(c[inside, RC:RC + r] * 40 / np.sum(c[inside, RC:RC + r] ** 2))
            q[280, H - 1, :R] = b16(c[outside, :R] * 40 / np.sum(c[outside, :R] ** 2))
            at = rows.index(280)
            assert np.abs(ref(q, c, window - 1, rows)[at, 0] - ref(q, c, window, rows)[at, 0]).max() > 0.3
            assert np.abs(ref(q, c, window + 1, rows)[at, H - 1] - ref(q, c, window, rows)[at, H - 1]).max() > 0.3
        cache = torch.full((2, n + 3, RS), 3e4, dtype=td, device=cuda)
        cache[1, :n] = dev(c, cuda, td)
        tab = ops.slot_table(cache)
        tol = 3e-5 if dtype == "float32" else 2.5e-2
        for splits in (1, 2, 7):
            out = ops.latent_window_attention(dev(q[rows], cuda), cache, tab, i32([1] * len(rows), cuda), i32(rows, cuda), scale, RC,
                                              window, splits=splits).float().cpu().numpy()
            assert np.abs(out[:, :, :R] - ref(q, c, window, rows)).max() < tol, (window, splits)
            out = ops.latent_window_attention(dev(q[seq], cuda), cache, tab, i32([1] * len(seq), cuda), i32(seq, cuda), scale, RC, window,
                                              splits=splits, **_runs(cuda, [5, 85])).float().cpu().numpy()
            assert np.abs(out[:, :, :R] - ref(q, c, window, seq)).max() < tol, (window, splits, "runs")
            assert np.abs(out[:, :, R:]).max(initial=0.0) == 0.0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_latent_rows_with_scaled_rotation(cuda, lib, dtype):
    """Frequencies kept, blended and divided, cos and sin enlarged; queries from a matrix of their own; the norm of the latent;
    padding columns untouched; positions near 900."""
    import torch
    from zhilight_b200 import ops
    td = getattr(torch, dtype)
    scaling = dict(factor=6.0, original=300.0, fast=20.0, slow=1.0)
    for dims, base in ((16, 1e4), (6, 500.0), (64, 5e5), (2, 100.0)):
        for sc in (None, scaling):
            got, mult = ops.rope_inv_freq_yarn(base, dims, *(sc[k] for k in ("factor", "original", "fast", "slow")) if sc else ())
            want, wm = orc.yarn(dims, base, sc)
            assert np.allclose(got, want, rtol=1e-14, atol=0) and abs(mult - wm) < 1e-6
    f, _ = orc.yarn(64, 1e4, scaling)
    ratio = f / orc.yarn(64, 1e4)[0]
    assert (ratio == 1).any() and np.isclose(ratio, 1 / 6).any() and ((ratio > 0.17) & (ratio < 0.99)).any()
    H, d, r, R, RC, RS, eps = 3, 10, 6, 20, 24, 40, 1e-2
    freqs, mult = orc.yarn(r, 100.0, scaling)
    assert mult > 1.15
    slots, pos = [2, 2, 2, 0, 1], [898, 899, 900, 0, 37]
    T, off = 5, 7
    rng = np.random.default_rng(17)
    qp, kv = rng.standard_normal((T, H * (d + r))).astype(np.float32), rng.standard_normal((T, off + R + r + 3)).astype(np.float32)
    kv[1, off:off + R] *= 0.05                                        # eps matters in this row
    w = rng.standard_normal(R).astype(np.float32)
    tab = ops.rope_table_scaled(i32(pos, cuda), dev(freqs, cuda), mult)
    cache = torch.full((3, 950, RS), 5.0, dtype=td, device=cuda)
    qa = torch.full((T, H, RS), 5.0, dtype=torch.float32, device=cuda)
    q = ops.latent_rope_append_split(dev(qp, cuda), H, d, r, tab, dev(kv, cuda), off, R, dev(w, cuda), RC, qa, cache, ops.slot_table(cache),
                                     i32(slots, cuda), i32(pos, cuda), eps)
    full = np.zeros((901, H + 1, r))
    wq, ckv = f64(qp).reshape(T, H, d + r), f64(kv)[:, off:off + R + r]
    tol = 3e-6 if dtype == "float32" else 2e-2
    assert np.abs(q.float().cpu().numpy() - wq[..., :d]).max() < tol
    qa = qa.cpu().numpy()
    row = np.stack([cache[s, t].float().cpu().numpy() for s, t in zip(slots, pos)])
    for i, p in enumerate(pos):
        full[:] = 0
        full[p, :H], full[p, H] = wq[i, :, d:], ckv[i, R:]
        turned = orc.rotate_adjacent(full, freqs, mult)[p]
        assert np.abs(qa[i, :, RC:RC + r] - turned[:H]).max() < 3e-6
        assert np.abs(row[i, RC:RC + r] - turned[H]).max() < tol * 1.5
    assert (qa[..., :RC] == 5).all() and (qa[..., RC + r:] == 5).all()
    assert np.abs(row[:, :R] - orc.rms(ckv[:, :R], eps) * w).max() < tol * 3
    assert (row[:, R:RC] == 5).all() and (row[:, RC + r:] == 5).all() and bool((cache[1, 36] == 5).all())


@pytest.mark.parametrize("shape", [(6, 48, 40, 3, 3), (4, 5, 9, 2, 4), (2, 64, 128, 1, 4), (3, 40, 20, 3, 2), (1, 1, 1, 1, 1), (8, 16, 256, 4, 4),
                                   (2, 34, 96, 2, 7), (2, 12, 272, 1, 3), (4, 8, 64, 4, 1)])
def test_state_space_scan(cuda, lib, shape):
    """Convolution, step sizes, decays and the recurrence over a plan of portions and single tokens of three sequences on slots full
    of leftovers: outputs, final states and the convolutions' last inputs; heads that forget within a few tokens and heads that
    remember hundreds; sizes with and without 16-byte rows, state sizes compiled, padded and general."""
    import torch
    from zhilight_b200 import ops
    H, vd, N, G, taps = shape
    inner, C = H * vd, H * vd + 2 * G * N
    n = {0: 130, 1: 7, 2: 41}
    rng = np.random.default_rng(H * 100 + N)
    ld, col_x = inner + C + H + (-(inner + C + H)) % 8, inner
    proj = {s: rng.standard_normal((k, ld)).astype(np.float32) for s, k in n.items()}
    cw, cb = (rng.standard_normal(s).astype(np.float32) / math.sqrt(taps) for s in ((C, taps), (C,)))
    dt_bias, a_log = rng.uniform(-5, 0.5, H).astype(np.float32), rng.uniform(-2, 1, H).astype(np.float32)
    skip = rng.standard_normal(H).astype(np.float32)
    want, final = {}, {}
    for s in n:
        p = f64(proj[s])
        u = orc.silu(orc.short_convolution(p[:, col_x:col_x + C], f64(cw), f64(cb)))
        want[s], final[s] = orc.state_space(u[:, :inner].reshape(-1, H, vd), u[:, inner:inner + G * N].reshape(-1, G, N),
                                            u[:, inner + G * N:].reshape(-1, G, N), orc.softplus(p[:, col_x + C:col_x + C + H] + dt_bias),
                                            f64(a_log), f64(skip))
    slot_of = {0: 2, 1: 0, 2: 3}
    state = torch.full((4, H, vd, N), 1e3, dtype=torch.float32, device=cuda)
    ring = torch.full((4, max(taps - 1, 1), C), 1e3, dtype=torch.float32, device=cuda)
    got = {s: [] for s in n}
    at = dict.fromkeys(n, 0)
    for step in ([(0, 3), (1, 1)], [(1, 1), (0, 2), (2, 40)], [(0, 1), (1, 1), (2, 1)], [(0, 1)], [(0, 70), (1, 4)], [(0, 17)], [(0, 36)]):
        rows = np.concatenate([proj[s][at[s]:at[s] + k] for s, k in step])
        slots = [slot_of[s] for s, k in step for _ in range(k)]
        pos = [at[s] + i for s, k in step for i in range(k)]
        r = _runs(cuda, [k for _, k in step])
        o = ops.ssm_scan(dev(rows, cuda), col_x, col_x + C, dev(np.ascontiguousarray(cw.T), cuda), dev(cb, cuda), dev(dt_bias, cuda),
                         dev(a_log, cuda), dev(skip, cuda), ops.slot_table(ring), r["run_row0"], r["run_len"], i32(slots, cuda),
                         i32(pos, cuda), ops.slot_table(state), H, vd, N, G).cpu().numpy()
        b = 0
        for s, k in step:
            got[s].append(o[b:b + k])
            b += k
            at[s] += k
    assert at == n
    for s in n:
        g, w = np.concatenate(got[s]), want[s].reshape(n[s], inner)
        assert np.abs(g - w).max() < 2e-5 * np.abs(w).max(), s
        st = state[slot_of[s]].cpu().numpy().transpose(0, 2, 1)
        assert np.abs(st - final[s]).max() < 2e-5 * np.abs(final[s]).max(), s
        for j in range(1, taps):
            if n[s] - j >= 0:
                assert np.array_equal(ring[slot_of[s], (n[s] - j) % (taps - 1)].cpu().numpy(), proj[s][n[s] - j, col_x:col_x + C]), (s, j)
    assert bool((state[1] == 1e3).all())


@pytest.mark.parametrize("shape", [(48, 4), (35, 5), (192, 1), (8200, 2), (30, 30)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_silu_gate_and_norm_in_groups(cuda, lib, dtype, shape):
    import torch
    from zhilight_b200 import ops
    D, groups = shape
    T, eps = 4, 1e-2
    rng = np.random.default_rng(D)
    o, z, w = (rng.standard_normal(s).astype(np.float32) for s in ((T, D), (T, D + 3), (D,)))
    o[:, :D // groups] *= 0.05                                        # one group's own mean, and eps, decide
    want = orc.gated_group_norm(f64(o), f64(z)[:, :D], f64(w), groups, eps)
    got = ops.silu_gate_group_rmsnorm(dev(o, cuda), dev(z, cuda), dev(w, cuda), groups, eps, getattr(torch, dtype)).float().cpu().numpy()
    assert np.abs(got - want).max() < (1e-5 if dtype == "float32" else 1e-2) * np.abs(want).max()


@pytest.mark.parametrize("shape", [(16, 3), (5, 5), (1, 1), (70, 6)])
def test_router_weights_are_the_softmax_scores(cuda, lib, shape):
    """The chosen experts' scores over all experts, not renormalised."""
    import torch
    from zhilight_b200 import ops
    E, top = shape
    T, D = 9, 40
    rng = np.random.default_rng(E)
    x, w = b16(rng.standard_normal((T, D))), b16(rng.standard_normal((E, D)) / math.sqrt(D) * 3)
    for td in (torch.float32, torch.bfloat16):
        te, tw, off, lt, lp = ops.moe_route_ex(dev(x, cuda, td), dev(w, cuda, td), top, group_rank=ops.MOE_GROUP_MAX,
                                               score_fn=ops.MOE_SCORE_SOFTMAX, renormalize=False)
        for t in range(T):
            chosen, s = orc.route_softmax(f64(w) @ f64(x[t]), top)
            assert te[t].cpu().tolist() == chosen.tolist()
            assert np.abs(tw[t].cpu().numpy() - s).max() < 1e-5
            assert E == top or s.sum() < 1 - 1e-5
        assert off.cpu().numpy()[-1] == T * top and sorted(lp.cpu().tolist()) == list(range(T * top))


# ---------------------------------------------------------------------------------------------- the whole model
@pytest.mark.parametrize("name", sorted(CONFIGS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prompt_layers_caches_and_logits(cuda, lib, name, dtype):
    cfg, W, m = make(CONFIGS[name], dtype, seed=3, max_step_tokens=128)
    toks = tokens_for(cfg, 97, 5)
    want, sums, kept = orc.forward(cfg, W, toks)
    m.capture_layers(True)
    _, logits = m.step(toks, [2] * len(toks), range(len(toks)), range(len(toks)))
    got = m.read_layers(len(toks))
    tol = 1e-4 if dtype == "float32" else 6e-2

    def close(a, b, what):
        rows = np.abs(a - b).reshape(len(b), -1).max(-1) / np.abs(b).max()
        d = rows.max() if dtype == "float32" else np.quantile(rows, 0.9)
        assert d < tol, (name, dtype) + what + (d,)

    assert got.shape == sums.shape
    for i, l in enumerate(cfg.layers):   # the first layer that differs is the one to look at
        close(got[i], sums[i], ("layer", i))
        if l["type"] == "mamba2":
            close(m.read_state(i, 2), kept[i][0], ("state of layer", i))
        else:
            for a, b in zip(m.read_cache(i, 2, len(toks)), kept[i]):
                close(a, b, ("cache of layer", i))
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
    cut = 3e-5 if dtype == "float32" else 3e-2      # the cuts change the order of sums, no more
    assert rel_err(runs["single"], runs["whole"].astype(np.float64), dtype) < cut
    assert rel_err(runs["portions"], runs["whole"].astype(np.float64), dtype) < cut
    m.close()


@pytest.mark.parametrize("name", ["odd", "tiles"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_batch_against_each_alone_and_slot_reuse(cuda, lib, name, dtype):
    """Three requests of different lengths share steps (prompt portions next to single decode tokens); afterwards their
    slots -- caches, states and convolution inputs still in them -- are handed to new requests.  Every logit row equals the
    request alone."""
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
    is far outside every window: states and key caches carry it through prompt portions and decoding."""
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
    # replay the same on the host path against the device loop's caches and states: position 14 sees what the loop wrote
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
    from zhilight_b200.bezasun import BezasunConfig
    cfg = BezasunConfig.from_dict(CFG_ODD)
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
