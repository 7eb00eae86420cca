"""Plain, slow restatement of the Dekalorn layer equations in numpy float64, one function per mechanism.

Nothing here is shared with the product path: keys and values of the latent layers are expanded per head, attention is
a full score matrix per head, the experts a loop over tokens and chosen experts.  A whole prompt is computed at once; by
causality the value at a position is also the truth for any way of cutting the prompt or decoding it token by token.
"""
import math

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def frequencies(dims, base, scaling=None):
    """base^(-2i/dims); with scaling (factor, low, high, original) long wavelengths are divided by factor, short ones
    kept, those between original/high and original/low blended."""
    f = base ** (-2.0 * np.arange(dims // 2, dtype=np.float64) / dims)
    if not scaling:
        return f
    factor, low, high, original = (float(scaling[k]) for k in ("factor", "low", "high", "original"))
    out = np.empty_like(f)
    for i, fi in enumerate(f):
        wave = 2.0 * math.pi / fi
        if wave < original / high:
            out[i] = fi
        elif wave > original / low:
            out[i] = fi / factor
        else:
            s = (original / wave - low) / (high - low)
            out[i] = (1.0 - s) * fi / factor + s * fi
    return out


def rotate_adjacent(x, freqs):
    """x (n, heads, d) at positions 0 .. n-1: dimensions (2i, 2i+1) turn by p * freqs[i]; the rest pass."""
    n, k = x.shape[0], len(freqs)
    a = np.arange(n, dtype=np.float64)[:, None, None] * freqs[None, None, :]
    y = x.copy()
    u, v = x[..., 0:2 * k:2], x[..., 1:2 * k:2]
    y[..., 0:2 * k:2] = u * np.cos(a) - v * np.sin(a)
    y[..., 1:2 * k:2] = v * np.cos(a) + u * np.sin(a)
    return y


def visible(n, window):
    """(n, n) mask: i sees j <= i, and with a window only i - j < window."""
    d = np.arange(n)[:, None] - np.arange(n)[None, :]
    return (d >= 0) & ((d < window) if window else True)


def softmax_rows(s, mask):
    s = np.where(mask, s, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def latent_mixer(W, p, l, h, eps):
    """Keys and values are linear maps of a normed latent; a separately projected rotated key part is shared by the heads."""
    n = h.shape[0]
    H, d, r, R, dv = l["heads"], l["dim"], l["rot_dim"], l["kv_rank"], l["vdim"]
    f = frequencies(r, l["rot_base"]) if r else np.zeros(0)
    q = (h @ W[p + "q"].T).reshape(n, H, d + r)
    ckv = h @ W[p + "dkv"].T
    c = rms(ckv[:, :R], eps) * W[p + "dkv.norm"]
    qr, kr = rotate_adjacent(q[:, :, d:], f), rotate_adjacent(ckv[:, None, R:], f)[:, 0]
    k = (c @ W[p + "uk"].T).reshape(n, H, d)
    v = (c @ W[p + "uv"].T).reshape(n, H, dv)
    gate = sigmoid(h @ W[p + "g"].T)
    o = np.zeros((n, H, dv))
    for j in range(H):
        s = (q[:, j, :d] @ k[:, j].T + qr[:, j] @ kr.T) * l["scale"]
        o[:, j] = softmax_rows(s, visible(n, 0)) @ v[:, j] * gate[:, j:j + 1]
    return o.reshape(n, H * dv) @ W[p + "o"].T, (c, kr)


def diff_lambda(W, p, diff):
    return math.exp(float(W[p + "lq1"] @ W[p + "lk1"])) - math.exp(float(W[p + "lq2"] @ W[p + "lk2"])) + diff


def differential_attention(q, k, v, scale, window, lam, diff, eps):
    """q (n, H, 2, d), k (n, G, 2, d), v (n, G, dv): two softmax maps per head over the same values, the second taken off
    lam times, the head's result divided by its root mean square and times 1 - diff."""
    n, H = q.shape[:2]
    G = k.shape[1]
    out = np.zeros((n, H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        a = [softmax_rows((q[:, h, m] @ k[:, g, m].T) * scale, visible(n, window)) @ v[:, g] for m in (0, 1)]
        out[:, h] = rms(a[0] - lam * a[1], eps) * (1.0 - diff)
    return out


def diff_mixer(W, p, l, h, eps):
    n = h.shape[0]
    H, G, d, dv = l["heads"], l["kv_heads"], l["dim"], l["vdim"]
    q = (h @ W[p + "q"].T).reshape(n, H, 2, d)
    k = (h @ W[p + "k"].T).reshape(n, G, 2, d)
    v = (h @ W[p + "v"].T).reshape(n, G, dv)
    o = differential_attention(q, k, v, l["scale"], l["window"], diff_lambda(W, p, l["diff"]), l["diff"], eps)
    o = o.reshape(n, H * dv) * sigmoid(h @ W[p + "g"].T)
    return o @ W[p + "o"].T, (k.reshape(n, G * 2 * d), v.reshape(n, G * dv))


def mixed_head_attention(q, k, v, scale, window, temp, talk):
    """q (n, H, d), k (n, G, d), v (n, G, dv): every head's scaled scores times its temp, then talk (H, H) mixes the
    heads' scores before the softmax."""
    n, H = q.shape[:2]
    G = k.shape[1]
    s = np.stack([(q[:, h] @ k[:, h // (H // G)].T) * scale * temp[h] for h in range(H)])
    out = np.zeros((n, H, v.shape[2]))
    for h in range(H):
        mixed = sum(talk[h, g] * s[g] for g in range(H))
        out[:, h] = softmax_rows(mixed, visible(n, window)) @ v[:, h // (H // G)]
    return out


def talking_mixer(W, p, l, h, eps):
    n = h.shape[0]
    H, G, d, dv = l["heads"], l["kv_heads"], l["dim"], l["vdim"]
    f = frequencies(l["rot_dims"], l["rot_base"], l["scaling"]) if l["rot_dims"] else np.zeros(0)
    q = rotate_adjacent((h @ W[p + "q"].T).reshape(n, H, d), f)
    k = rotate_adjacent((h @ W[p + "k"].T).reshape(n, G, d), f)
    v = (h @ W[p + "v"].T).reshape(n, G, dv)
    o = mixed_head_attention(q, k, v, l["scale"], l["window"], W[p + "temp"], W[p + "talk"])
    return o.reshape(n, H * dv) @ W[p + "o"].T, (k.reshape(n, G * d), v.reshape(n, G * dv))


MIXERS = {"latent_attention": latent_mixer, "attention": diff_mixer, "attention_2": talking_mixer}


def relu_gated_ff(W, p, h):
    return (np.maximum(h @ W[p + "gate"].T, 0.0) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def silu_expert(W, p, h):
    z = W[p + "gate"] @ h
    return W[p + "down"] @ (z * sigmoid(z) * (W[p + "up"] @ h))


def route_two_best(z, top, groups, keep, scale):
    """z (experts,) logits of one token -> (chosen experts, weights).  Sigmoid scores; a group of neighbours ranks by the
    sum of its two largest scores; the best `top` of the `keep` best groups, weights = scores over their sum, times scale."""
    s = sigmoid(z)
    per = len(z) // groups
    rank = np.sort(s.reshape(groups, per), axis=-1)[:, -2:].sum(axis=-1)
    masked = np.full_like(s, -np.inf)
    for g in np.argsort(-rank, kind="stable")[:keep]:
        masked[g * per:(g + 1) * per] = s[g * per:(g + 1) * per]
    chosen = np.argsort(-masked, kind="stable")[:top]
    return chosen, s[chosen] / (s[chosen].sum() + 1e-20) * scale


def experts_ff(W, p, l, h):
    out = np.zeros_like(h)
    z = h @ W[p + "router"].T
    for t in range(h.shape[0]):
        for e, s in zip(*route_two_best(z[t], l["top"], l["groups"], l["keep"], l["router_scale"])):
            out[t] += s * silu_expert(W, p + "e%d." % e, h[t])
    return out


def layer(cfg, W, i, x):
    l, p = cfg.layers[i], "l%d." % i
    y, cached = MIXERS[l["type"]](W, p + "mix.", l, rms(x, cfg.norm_eps) * W[p + "norm1"], cfg.norm_eps)
    x = x + y
    if l["ff_kind"]:
        h = rms(x, cfg.norm_eps) * W[p + "norm2"]
        x = x + (relu_gated_ff(W, p + "mlp.", h) if l["ff_kind"] == "dense" else experts_ff(W, p + "mlp.", l, h))
    return x, cached


def schedule(cfg):
    """[(layer, first of a pass of the loop)] in running order."""
    n = len(cfg.layers)
    a, b, times = cfg.loop if cfg.loop else (0, 0, 0)
    runs = [(i, False) for i in range(a)]
    for _ in range(times):
        runs += [(i, i == a) for i in range(a, b)]
    return runs + [(i, False) for i in range(b, n)]


def forward(cfg, W, tokens):
    """cfg: DekalornConfig; W: name -> float64 array.  -> (logits (n, vocab), residual stream after every layer run
    (runs, n, width), [what each run caches])."""
    x0 = W["embed"][np.asarray(tokens)]
    x, per_run, cached = x0, [], []
    for i, enters in schedule(cfg):
        if enters:
            x = np.concatenate([x, x0], axis=-1) @ W["loop.in"].T
        x, c = layer(cfg, W, i, x)
        per_run.append(x.copy())
        cached.append(c)
    return (rms(x, cfg.norm_eps) * W["final.norm"]) @ W["head"].T, np.stack(per_run), cached


def bf16_round(a):
    """float32 array rounded to the nearest bfloat16 (ties to even), still float32."""
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    u = (u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000
    return u.astype(np.uint32).view(np.float32).reshape(np.shape(a))


def random_weights(cfg, seed=0, router_gain=4.0):
    """name -> float32 array whose values are exact in bfloat16.  Router rows are scaled up so that the choice of
    experts does not hang on a rounding."""
    rng = np.random.default_rng(seed)
    W = {}
    for name, shp in sorted(cfg.tensor_shapes().items()):
        last = name.rsplit(".", 1)[-1]
        if last in ("norm", "norm1", "norm2"):
            a = 1.0 + 0.2 * rng.standard_normal(shp)
        elif last in ("lq1", "lk1", "lq2", "lk2"):
            a = 0.5 * rng.standard_normal(shp) / math.sqrt(shp[-1])
        elif last == "temp":
            a = 1.0 + 0.3 * rng.standard_normal(shp)
        elif last == "talk":
            a = np.eye(shp[0]) + 0.4 * rng.standard_normal(shp)
        elif name == "embed":
            a = rng.standard_normal(shp)
        elif last == "router":
            a = router_gain * rng.standard_normal(shp) / math.sqrt(shp[-1])
        else:
            a = rng.standard_normal(shp) / math.sqrt(shp[-1])
        W[name] = bf16_round(a.astype(np.float32))
    return W
