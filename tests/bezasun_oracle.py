"""Plain, slow restatement of the Bezasun layer equations in numpy float64, one function per mechanism.

Nothing here is shared with the product path: keys and values of the latent layers are expanded per head, attention is
a full score matrix per head, the recurrence and the convolution are loops over tokens, the experts a loop over tokens and
chosen experts.  A whole prompt is computed at once; by causality the value at a position is also the truth for any way of
cutting the prompt or decoding it token by token.
"""
import math

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def yarn(dims, base, scaling=None):
    """(frequencies, factor on cos and sin): base^(-2i/dims); with scaling (factor, original, fast, slow) pairs that turn at
    least `fast` times over `original` positions keep their frequency, those below `slow` turns have it divided by factor,
    the ones between are blended, linearly in the pair's index."""
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=np.float64)
    if not scaling:
        return f, 1.0

    def index_of(turns):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    low = max(math.floor(index_of(scaling["fast"])), 0)
    high = min(math.ceil(index_of(scaling["slow"])), dims - 1)
    out = np.empty_like(f)
    for i in range(len(f)):
        r = min(max((i - low) / max(high - low, 0.001), 0.0), 1.0)
        out[i] = f[i] / scaling["factor"] * r + f[i] * (1.0 - r)
    return out, 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_adjacent(x, freqs, mult):
    """x (n, heads, d) at positions 0 .. n-1: dimensions (2i, 2i+1) turn by p * freqs[i] and grow by mult; the rest pass."""
    n, k = x.shape[0], len(freqs)
    a = np.arange(n, dtype=np.float64)[:, None, None] * freqs[None, None, :]
    c, s = np.cos(a) * mult, np.sin(a) * mult
    y = x.copy()
    u, v = x[..., 0:2 * k:2], x[..., 1:2 * k:2]
    y[..., 0:2 * k:2] = u * c - v * s
    y[..., 1:2 * k:2] = v * c + u * s
    return y


def visible(n, window):
    """(n, n) mask: i sees j <= i, and with a window only i - j < window."""
    d = np.arange(n)[:, None] - np.arange(n)[None, :]
    return (d >= 0) & ((d < window) if window else True)


def softmax_rows(s, mask, sink=None):
    """Softmax over the visible keys; a sink adds exp(sink) to the denominator."""
    s = np.where(mask, s, -np.inf)
    top = s.max(axis=-1, keepdims=True)
    if sink is not None:
        top = np.maximum(top, sink)
    e = np.exp(s - top)
    return e / (e.sum(axis=-1, keepdims=True) + (0.0 if sink is None else np.exp(sink - top)))


def query_temperature(n, coef, every):
    return np.array([1.0 + coef * math.log(math.floor((p + 1) / every) + 1) for p in range(n)])


def distance_slopes(heads):
    return np.array([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)])


def sink_attention(q, k, v, scale, softcap, slopes, sink):
    """q (n, H, d), k (n, G, d), v (n, G, dv): scores scaled, soft-capped, lowered by slope times the distance; causal; a sink."""
    n, H = q.shape[:2]
    G = k.shape[1]
    dist = (np.arange(n)[:, None] - np.arange(n)[None, :]).astype(np.float64)
    out = np.zeros((n, H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if softcap:
            s = softcap * np.tanh(s / softcap)
        out[:, h] = softmax_rows(s - slopes[h] * dist, visible(n, 0), sink[h]) @ v[:, g]
    return out


def attention_mixer(W, p, l, h, eps):
    n = h.shape[0]
    H, G, d, dv = l["heads"], l["kv_heads"], l["dim"], l["vdim"]
    q = rms((h @ W[p + "q"].T).reshape(n, H, d), eps) * W[p + "q.norm"]
    k = rms((h @ W[p + "k"].T).reshape(n, G, d), eps) * W[p + "k.norm"]
    v = (h @ W[p + "v"].T).reshape(n, G, dv)
    if l["temp_coef"]:
        q = q * query_temperature(n, l["temp_coef"], l["temp_every"])[:, None, None]
    o = sink_attention(q, k, v, l["scale"], l["softcap"], distance_slopes(H), W[p + "sink"])
    return o.reshape(n, H * dv) @ W[p + "o"].T, (k.reshape(n, G * d), v.reshape(n, G * dv))


def latent_mixer(W, p, l, h, eps):
    """Queries through a normed latent; keys and values are linear maps of another, beside a rotated key part for all heads."""
    n = h.shape[0]
    H, d, r, R, dv = l["heads"], l["dim"], l["rot_dim"], l["kv_rank"], l["vdim"]
    f, mult = yarn(r, l["rot_base"], l["scaling"]) if r else (np.zeros(0), 1.0)
    cq = rms(h @ W[p + "dq"].T, eps) * W[p + "dq.norm"]
    q = (cq @ W[p + "uq"].T).reshape(n, H, d + r)
    ckv = h @ W[p + "dkv"].T
    c = rms(ckv[:, :R], eps) * W[p + "dkv.norm"]
    qr, kr = rotate_adjacent(q[:, :, d:], f, mult), rotate_adjacent(ckv[:, None, R:], f, mult)[:, 0]
    k = (c @ W[p + "uk"].T).reshape(n, H, d)
    v = (c @ W[p + "uv"].T).reshape(n, H, dv)
    o = np.zeros((n, H, dv))
    for j in range(H):
        s = (q[:, j, :d] @ k[:, j].T + qr[:, j] @ kr.T) * l["scale"]
        o[:, j] = softmax_rows(s, visible(n, l["window"])) @ v[:, j]
    return o.reshape(n, H * dv) @ W[p + "o"].T, (c, kr)


def short_convolution(x, w, b):
    """x (n, C), w (C, taps) with the last tap for the current token, zeros before the start."""
    n, taps = x.shape[0], w.shape[1]
    y = np.tile(b, (n, 1)).astype(np.float64)
    for t in range(n):
        for j in range(taps):
            if t - j >= 0:
                y[t] += w[:, taps - 1 - j] * x[t - j]
    return y


def state_space(x, B, C, dt, a_log, d_skip):
    """x (n, H, dv), B / C (n, G, N), dt (n, H) step sizes -> (y (n, H, dv), final state (H, N, dv))."""
    n, H, dv = x.shape
    G, N = B.shape[1:]
    y, final = np.zeros_like(x), np.zeros((H, N, dv))
    for h in range(H):
        g = h // (H // G)
        S = np.zeros((N, dv))
        for t in range(n):
            S = math.exp(-math.exp(a_log[h]) * dt[t, h]) * S + dt[t, h] * np.outer(B[t, g], x[t, h])
            y[t, h] = C[t, g] @ S + d_skip[h] * x[t, h]
        final[h] = S
    return y, final


def gated_group_norm(y, z, w, groups, eps):
    v = y * silu(z)
    n, D = v.shape
    return rms(v.reshape(n, groups, D // groups), eps).reshape(n, D) * w


def mamba2_mixer(W, p, l, h, eps):
    n = h.shape[0]
    H, dv, N, G = l["heads"], l["vdim"], l["state"], l["groups"]
    inner, bc = H * dv, G * N
    proj = h @ W[p + "in"].T
    z, xbc, dt = proj[:, :inner], proj[:, inner:2 * inner + 2 * bc], proj[:, 2 * inner + 2 * bc:]
    u = silu(short_convolution(xbc, W[p + "conv"], W[p + "conv.b"]))
    x, B, C = u[:, :inner].reshape(n, H, dv), u[:, inner:inner + bc].reshape(n, G, N), u[:, inner + bc:].reshape(n, G, N)
    y, final = state_space(x, B, C, softplus(dt + W[p + "dt_bias"]), W[p + "A_log"], W[p + "D"])
    o = gated_group_norm(y.reshape(n, inner), z, W[p + "norm"], l["norm_groups"], eps)
    return o @ W[p + "o"].T, (final, xbc)


MIXERS = {"attention": attention_mixer, "latent_attention": latent_mixer, "mamba2": mamba2_mixer}


def gated_unit(W, p, h):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def route_softmax(z, top):
    """z (experts,) logits of one token -> (chosen experts, their softmax scores over all experts, as they are)."""
    e = np.exp(z - z.max())
    s = e / e.sum()
    chosen = np.argsort(-s, kind="stable")[:top]
    return chosen, s[chosen]


def experts_ff(W, p, l, h):
    out = np.zeros_like(h)
    z = h @ W[p + "router"].T
    for t in range(h.shape[0]):
        for e, s in zip(*route_softmax(z[t], l["top"])):
            out[t] += s * gated_unit(W, p + "e%d." % e, h[t])
    return out + (gated_unit(W, p + "shared.", h) if l["shared_ff"] else 0.0)


def hyper_read(x, w_in):
    """x (streams, n, D) -> the sublayer's input."""
    return sum(w_in[s] * x[s] for s in range(len(x)))


def hyper_write(x, mix, out, mult, y):
    """Every new stream from the old ones (mix is indexed [from, to]) and the sublayer's result."""
    S = len(x)
    return np.stack([sum(mix[s, t] * x[s] for s in range(S)) + mult * out[t] * y for t in range(S)])


def layer(cfg, W, i, x):
    l, p = cfg.layers[i], "l%d." % i
    h = rms(hyper_read(x, W[p + "hc1.in"]), cfg.norm_eps) * (1.0 + W[p + "norm1"])
    y, cached = MIXERS[l["type"]](W, p + "mix.", l, h, cfg.norm_eps)
    x = hyper_write(x, W[p + "hc1.mix"], W[p + "hc1.out"], cfg.residual_mult, y)
    if l["ff_kind"]:
        h = rms(hyper_read(x, W[p + "hc2.in"]), cfg.norm_eps) * (1.0 + W[p + "norm2"])
        x = hyper_write(x, W[p + "hc2.mix"], W[p + "hc2.out"], cfg.residual_mult, experts_ff(W, p + "mlp.", l, h))
    return x, cached


def forward(cfg, W, tokens):
    """cfg: BezasunConfig; W: name -> float64 array.  -> (logits (n, vocab), sum of the streams after every layer
    (layers, n, width), [what each layer keeps])."""
    x = np.stack([W["embed"][np.asarray(tokens)] * cfg.embed_scale] * cfg.streams)
    per_layer, kept = [], []
    for i in range(len(cfg.layers)):
        x, c = layer(cfg, W, i, x)
        per_layer.append(x.sum(axis=0))
        kept.append(c)
    out = rms(x.sum(axis=0), cfg.norm_eps) * (1.0 + W["final.norm"])
    return (out @ W["head"].T) * cfg.logit_scale, np.stack(per_layer), kept


def bf16_round(a):
    """float32 array rounded to the nearest bfloat16 (ties to even), still float32."""
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    u = (u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000
    return u.astype(np.uint32).view(np.float32).reshape(np.shape(a))


def random_weights(cfg, seed=0, router_gain=3.0):
    """name -> float32 array whose values are exact in bfloat16.  Router rows are scaled up so that the choice of experts
    does not hang on a rounding; queries and keys so that attention is not flat; the state-space step sizes so that some
    heads forget within a few tokens and some remember hundreds; the streams mix differently in every sublayer."""
    rng = np.random.default_rng(seed)
    W = {}
    for name, shp in sorted(cfg.tensor_shapes().items()):
        last = name.rsplit(".", 1)[-1]
        norm = rng.standard_normal(shp)
        if last in ("norm1", "norm2") or name == "final.norm":
            a = 0.2 * norm
        elif name.endswith(("q.norm", "k.norm")):
            a = 1.2 + 0.2 * norm
        elif last == "norm":
            a = 1.0 + 0.2 * norm
        elif ".hc" in name:
            a = np.eye(shp[0]) * 0.8 + 0.2 * norm if last == "mix" else (0.5 + 0.3 * norm if last == "out" else 1.0 / shp[0] + 0.3 * norm)
        elif last in ("sink", "D"):
            a = 0.5 + norm
        elif last == "A_log":
            a = rng.uniform(-2.0, 1.0, shp)
        elif last == "dt_bias":
            a = rng.uniform(-5.0, 0.5, shp)
        elif name == "embed":
            a = 0.12 * norm
        elif last == "b":
            a = 0.2 * norm
        elif last == "conv":
            a = norm / math.sqrt(shp[-1])
        elif last == "router":
            a = router_gain * norm / math.sqrt(shp[-1])
        elif last in ("uq", "uk"):
            a = 1.3 * norm / math.sqrt(shp[-1])
        else:
            a = norm / math.sqrt(shp[-1])
        W[name] = bf16_round(a.astype(np.float32))
    return W
