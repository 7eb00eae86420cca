"""Bezasun front end (zl_bezasun_* C-ABI): configuration from config.json, weight loading, and the step call.

Bezasun is a decoder-only family whose config.json lists the layers one by one.  The residual is a set of `streams` fp32
copies that all start as the scaled embedding (hyper-connections): sublayer q of a layer reads u = sum_s in[s] x_s through
an RMS norm (multipliers 1 + w) and its result y goes back as x_t <- sum_s mix[s, t] x_s + residual_mult out[t] y, all
streams at once; the model's output reads the sum of the streams.  Mixers:

  * "attention": grouped-query attention without positions: RMS norm per query / key head, queries times
    1 + coef ln(floor((p + 1) / every) + 1), scores soft-capped, a linear bias by distance per head, a softmax with a
    learned sink per head.
  * "latent_attention": queries through a normed latent, keys and values as linear maps of a normed latent, which is cached
    beside one rotated key part shared by the heads (YaRN frequencies); sliding window, ordinary softmax.
  * "mamba2": a selective state space per head behind a short causal convolution, a silu gate and a norm in groups.

The feed-forward is absent (mlp null) or a mixture of silu-gated experts weighted by their softmax scores as they are, plus
an optional expert shared by all tokens.  config.json:

    {"architecture": "Bezasun", "vocab": V, "width": D, "streams": s, "residual_mult": m, "logit_scale": c,
     "embedding": {"scale": a}, "norm": {"eps": e},
     "layers": [{"type": "attention",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "softcap", "q_temp": {"coef", "every"}},
                 "mlp": null | {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"}, "shared": {"ff"}}},
                {"type": "latent_attention",
                 "mixer": {"heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale", "mask": {"size"},
                           "rot": {"base", "dims", "scaling": {"factor", "original", "fast", "slow"}}}, "mlp": ...},
                {"type": "mamba2",
                 "mixer": {"heads", "vdim", "state", "groups", "conv", "norm_groups"}, "mlp": ...}]}

Checkpoint tensors: embed, head, final.norm, per layer l<i>.norm1 and l<i>.hc1.{in, out, mix} (norm2 and hc2 with a
feed-forward), l<i>.mix.{q, k, v, q.norm, k.norm, sink, o} | {dq, dq.norm, uq, dkv, dkv.norm, uk, uv, o} |
{in, conv, conv.b, dt_bias, A_log, D, norm, o}, l<i>.mlp.{router, e<j>.gate, e<j>.up, e<j>.down, shared.gate, shared.up,
shared.down}; Linears are (out, in).
"""
import ctypes

import numpy as np

from . import _lib
from .safetensors_io import is_bf16

MIXERS = {"attention": 0, "latent_attention": 1, "mamba2": 2}
FF_KINDS = {None: 0, "moe": 2}
SCALING_KEYS = ("factor", "original", "fast", "slow")


class BezasunLayer(ctypes.Structure):
    """zl_bezasun_layer_t"""
    _fields_ = [("type", ctypes.c_int), ("heads", ctypes.c_int), ("kv_heads", ctypes.c_int), ("dim", ctypes.c_int),
                ("vdim", ctypes.c_int), ("scale", ctypes.c_float), ("softcap", ctypes.c_float), ("temp_coef", ctypes.c_float),
                ("temp_every", ctypes.c_double), ("rot_dim", ctypes.c_int), ("q_rank", ctypes.c_int), ("kv_rank", ctypes.c_int),
                ("window", ctypes.c_int), ("rot_base", ctypes.c_double), ("rot_factor", ctypes.c_double),
                ("rot_original", ctypes.c_double), ("rot_fast", ctypes.c_double), ("rot_slow", ctypes.c_double),
                ("state", ctypes.c_int), ("groups", ctypes.c_int), ("conv", ctypes.c_int), ("norm_groups", ctypes.c_int),
                ("ff_kind", ctypes.c_int), ("ff", ctypes.c_int), ("experts", ctypes.c_int), ("top", ctypes.c_int),
                ("shared_ff", ctypes.c_int)]


class BezasunCConfig(ctypes.Structure):
    """zl_bezasun_config_t"""
    _fields_ = [("num_layers", ctypes.c_int), ("width", ctypes.c_int), ("vocab", ctypes.c_int), ("streams", ctypes.c_int),
                ("eps", ctypes.c_float), ("embed_scale", ctypes.c_float), ("residual_mult", ctypes.c_float),
                ("logit_scale", ctypes.c_float), ("dtype", ctypes.c_int), ("max_batch", ctypes.c_int), ("max_seq", ctypes.c_int),
                ("max_step_tokens", ctypes.c_int), ("use_pdl", ctypes.c_int), ("use_graph", ctypes.c_int)]


class BezasunConfig:
    """Parsed config.json of a Bezasun model.  `layers` is a list of dicts: type and ff_kind as in config.json and every size
    and constant of zl_bezasun_layer_t that the type has (scaling: None or a dict, window 0: none, softcap 0: none)."""

    def __init__(self, vocab, width, layers, streams=1, norm_eps=1e-6, embed_scale=1.0, residual_mult=1.0, logit_scale=1.0):
        self.vocab, self.width, self.streams, self.norm_eps = int(vocab), int(width), int(streams), float(norm_eps)
        self.embed_scale, self.residual_mult, self.logit_scale = float(embed_scale), float(residual_mult), float(logit_scale)
        self.layers = layers
        if not 1 <= self.streams <= 16:
            raise ValueError("streams must be between 1 and 16")
        for i, l in enumerate(layers):
            if l["type"] == "attention":
                if l["heads"] < 1 or l["kv_heads"] < 1 or l["heads"] % l["kv_heads"]:
                    raise ValueError("layer %d: heads is not a multiple of kv_heads" % i)
                if l["softcap"] < 0 or (l["temp_coef"] and l["temp_every"] <= 0):
                    raise ValueError("layer %d: softcap and q_temp.every must be positive" % i)
            elif l["type"] == "latent_attention":
                if l["rot_dim"] % 2 or l["rot_dims"] != l["rot_dim"]:
                    raise ValueError("layer %d: rot.dims must be even and equal to rot_dim" % i)
                if l["window"] < 0:
                    raise ValueError("layer %d: mask.size must be positive" % i)
            else:
                if l["groups"] < 1 or l["heads"] % l["groups"]:
                    raise ValueError("layer %d: heads is not a multiple of groups" % i)
                if l["norm_groups"] < 1 or (l["heads"] * l["vdim"]) % l["norm_groups"]:
                    raise ValueError("layer %d: norm_groups does not divide heads * vdim" % i)
                if l["conv"] < 1:
                    raise ValueError("layer %d: conv must be at least 1" % i)
            if l["ff_kind"] == "moe" and not 0 < l["top"] <= l["experts"]:
                raise ValueError("layer %d: router.top must be between 1 and experts" % i)

    @classmethod
    def from_dict(cls, d):
        layers = []
        for i, l in enumerate(d["layers"]):
            kind, mx, mlp = l.get("type"), l["mixer"], l.get("mlp")
            if kind not in MIXERS:
                raise ValueError("layer %d: unknown mixer type %r" % (i, kind))
            out = dict(type=kind, heads=int(mx["heads"]), vdim=int(mx["vdim"]), ff_kind=None, ff=0, experts=0, top=0, shared_ff=0)
            if kind == "attention":
                temp = mx.get("q_temp") or {}
                out.update(kv_heads=int(mx.get("kv_heads", mx["heads"])), dim=int(mx["dim"]), scale=float(mx["scale"]),
                           softcap=float(mx.get("softcap") or 0.0), temp_coef=float(temp.get("coef", 0.0)),
                           temp_every=float(temp.get("every", 1.0)))
            elif kind == "latent_attention":
                rot = mx.get("rot") or {}
                sc = rot.get("scaling") or None
                out.update(dim=int(mx["dim"]), rot_dim=int(mx["rot_dim"]), q_rank=int(mx["q_rank"]), kv_rank=int(mx["kv_rank"]),
                           scale=float(mx["scale"]), window=int((mx.get("mask") or {}).get("size", 0)),
                           rot_dims=int(rot.get("dims", mx["rot_dim"])), rot_base=float(rot.get("base", 10000.0)),
                           scaling={k: float(sc[k]) for k in SCALING_KEYS} if sc else None)
            else:
                out.update(state=int(mx["state"]), groups=int(mx.get("groups", 1)), conv=int(mx["conv"]),
                           norm_groups=int(mx.get("norm_groups", 1)))
            if mlp is not None:
                if mlp.get("kind") != "moe":
                    raise ValueError("layer %d: unknown feed-forward kind %r" % (i, mlp.get("kind")))
                r = mlp["router"]
                out.update(ff_kind="moe", ff=int(mlp["expert"]["ff"]), experts=int(r["experts"]), top=int(r["top"]),
                           shared_ff=int((mlp.get("shared") or {}).get("ff", 0)))
            layers.append(out)
        return cls(d["vocab"], d["width"], layers, d.get("streams", 1), (d.get("norm") or {}).get("eps", 1e-6),
                   (d.get("embedding") or {}).get("scale", 1.0), d.get("residual_mult", 1.0), d.get("logit_scale", 1.0))

    def to_dict(self):
        out = []
        for l in self.layers:
            keys = {"attention": ("heads", "kv_heads", "dim", "vdim", "scale"),
                    "latent_attention": ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale"),
                    "mamba2": ("heads", "vdim", "state", "groups", "conv", "norm_groups")}[l["type"]]
            mx = {k: l[k] for k in keys}
            if l["type"] == "attention":
                if l["softcap"]:
                    mx["softcap"] = l["softcap"]
                if l["temp_coef"]:
                    mx["q_temp"] = {"coef": l["temp_coef"], "every": l["temp_every"]}
            elif l["type"] == "latent_attention":
                mx["rot"] = {"base": l["rot_base"], "dims": l["rot_dims"]}
                if l["scaling"]:
                    mx["rot"]["scaling"] = dict(l["scaling"])
                if l["window"]:
                    mx["mask"] = {"size": l["window"]}
            mlp = None
            if l["ff_kind"]:
                mlp = {"kind": "moe", "expert": {"ff": l["ff"]}, "router": {"experts": l["experts"], "top": l["top"]}}
                if l["shared_ff"]:
                    mlp["shared"] = {"ff": l["shared_ff"]}
            out.append({"type": l["type"], "mixer": mx, "mlp": mlp})
        return {"architecture": "Bezasun", "vocab": self.vocab, "width": self.width, "streams": self.streams,
                "residual_mult": self.residual_mult, "logit_scale": self.logit_scale, "embedding": {"scale": self.embed_scale},
                "norm": {"eps": self.norm_eps}, "layers": out}

    def tensor_shapes(self):
        """name -> shape of every checkpoint tensor."""
        D, s = self.width, {}
        s["embed"] = s["head"] = (self.vocab, D)
        s["final.norm"] = (D,)
        for i, l in enumerate(self.layers):
            p, H, vd = "l%d." % i, l["heads"], l["vdim"]
            m = p + "mix."
            for q in (1, 2) if l["ff_kind"] else (1,):
                s[p + "norm%d" % q] = (D,)
                s[p + "hc%d.in" % q] = s[p + "hc%d.out" % q] = (self.streams,)
                s[p + "hc%d.mix" % q] = (self.streams, self.streams)
            if l["type"] == "attention":
                G, d = l["kv_heads"], l["dim"]
                s[m + "q"], s[m + "k"], s[m + "v"] = (H * d, D), (G * d, D), (G * vd, D)
                s[m + "q.norm"] = s[m + "k.norm"] = (d,)
                s[m + "sink"] = (H,)
            elif l["type"] == "latent_attention":
                R, Q = l["kv_rank"], l["q_rank"]
                s[m + "dq"], s[m + "dq.norm"], s[m + "uq"] = (Q, D), (Q,), (H * (l["dim"] + l["rot_dim"]), Q)
                s[m + "dkv"], s[m + "dkv.norm"] = (R + l["rot_dim"], D), (R,)
                s[m + "uk"], s[m + "uv"] = (H * l["dim"], R), (H * vd, R)
            else:
                inner, bc = H * vd, l["groups"] * l["state"]
                s[m + "in"] = (2 * inner + 2 * bc + H, D)
                s[m + "conv"], s[m + "conv.b"] = (inner + 2 * bc, l["conv"]), (inner + 2 * bc,)
                s[m + "dt_bias"] = s[m + "A_log"] = s[m + "D"] = (H,)
                s[m + "norm"] = (inner,)
            s[m + "o"] = (D, H * vd)
            if l["ff_kind"]:
                s[p + "mlp.router"] = (l["experts"], D)
                units = [("e%d." % e, l["ff"]) for e in range(l["experts"])]
                if l["shared_ff"]:
                    units.append(("shared.", l["shared_ff"]))
                for u, f in units:
                    s[p + "mlp." + u + "gate"] = s[p + "mlp." + u + "up"] = (f, D)
                    s[p + "mlp." + u + "down"] = (D, f)
        return s


DTYPES = {"bf16": 1, "bfloat16": 1, "f32": 2, "float32": 2}


class BezasunDecoder:
    """One model instance on the current CUDA device.  Slots (0..max_batch-1) each own `max_seq` rows of every attention layer's
    caches and one state per state-space layer; the engine's scheduler decides which sequence lives in which slot."""

    architecture = "Bezasun"
    supports_dtypes = ("bfloat16", "float32")
    supports_ragged_steps = True

    def __init__(self, config, dtype="bf16", max_batch=1, max_seq=512, max_step_tokens=512, use_pdl=True, use_graph=True):
        self.lib = _lib.load()
        self.config = config
        self.vocab_size = config.vocab
        self.dtype = dtype
        self.max_batch, self.max_seq = int(max_batch), int(max_seq)
        self.max_step_tokens = max(int(max_step_tokens), self.max_batch)
        c = config
        self.cfg = BezasunCConfig(len(c.layers), c.width, c.vocab, c.streams, c.norm_eps, c.embed_scale, c.residual_mult,
                                  c.logit_scale, DTYPES[dtype], self.max_batch, self.max_seq, self.max_step_tokens, int(use_pdl),
                                  int(use_graph))
        arr = (BezasunLayer * len(c.layers))()
        for i, l in enumerate(c.layers):
            sc = l.get("scaling") or dict.fromkeys(SCALING_KEYS, 0.0)
            latent = l["type"] == "latent_attention"
            arr[i] = BezasunLayer(MIXERS[l["type"]], l["heads"], l.get("kv_heads", l["heads"]), l.get("dim", 0), l["vdim"],
                                  l.get("scale", 0.0), l.get("softcap", 0.0), l.get("temp_coef", 0.0), l.get("temp_every", 1.0),
                                  l.get("rot_dim", 0), l.get("q_rank", 0), l.get("kv_rank", 0), l.get("window", 0),
                                  l["rot_base"] if latent else 0.0, sc["factor"], sc["original"], sc["fast"], sc["slow"],
                                  l.get("state", 0), l.get("groups", 0), l.get("conv", 0), l.get("norm_groups", 0),
                                  FF_KINDS[l["ff_kind"]], l["ff"], l["experts"], l["top"], l["shared_ff"])
        h = ctypes.c_void_p()
        _lib.check(self.lib.zl_bezasun_create(ctypes.byref(self.cfg), arr, ctypes.byref(h)))
        self.h = h

    @classmethod
    def from_config_dict(cls, d, **kw):
        return cls(BezasunConfig.from_dict(d), **kw)

    def close(self):
        if getattr(self, "h", None):
            self.lib.zl_bezasun_destroy(self.h)
            self.h = None

    def __del__(self):
        try:
            self.close()
        except Exception:
            pass

    def load_state_dict(self, state_dict):
        """name -> numpy array: bfloat16 bit patterns (safetensors_io.Bf16Array) or float32."""
        needed = self.config.tensor_shapes()
        for name, arr in state_dict.items():
            a = np.ascontiguousarray(arr)
            if name not in needed:
                continue                      # a checkpoint may carry tensors this family does not use
            if not (is_bf16(arr) or a.dtype == np.float32):
                raise ValueError("tensor %s: expected bfloat16 or float32, got %s" % (name, a.dtype))
            if tuple(a.shape) != tuple(needed[name]):
                raise ValueError("tensor %s: shape %s, expected %s" % (name, tuple(a.shape), tuple(needed[name])))
            rows, cols = (1, a.size) if a.ndim <= 1 else (a.shape[0], a.size // a.shape[0])
            _lib.check(self.lib.zl_bezasun_load_tensor(self.h, name.encode(), a.ctypes.data_as(ctypes.c_void_p), rows, cols,
                                                       a.itemsize))
        _lib.check(self.lib.zl_bezasun_finalize(self.h))

    def init_synthetic(self, seed=0):
        _lib.check(self.lib.zl_bezasun_init_synthetic(self.h, seed))

    def step(self, tokens, slots, positions, want_rows=(), want_logits=True):
        """One step over T rows.  Returns (next tokens (n_want), logits (n_want, vocab) or None) for the wanted rows."""
        t = np.ascontiguousarray(tokens, dtype=np.int32)
        s = np.ascontiguousarray(slots, dtype=np.int32)
        p = np.ascontiguousarray(positions, dtype=np.int32)
        w = np.ascontiguousarray(want_rows, dtype=np.int32)
        nxt = np.empty(w.size, dtype=np.int32)
        logits = np.empty((w.size, self.vocab_size), dtype=np.float32) if want_logits else None
        _lib.check(self.lib.zl_bezasun_step(
            self.h, t.ctypes.data_as(ctypes.c_void_p), s.ctypes.data_as(ctypes.c_void_p), p.ctypes.data_as(ctypes.c_void_p),
            t.size, w.ctypes.data_as(ctypes.c_void_p) if w.size else None, w.size,
            logits.ctypes.data_as(ctypes.c_void_p) if (want_logits and w.size) else None,
            nxt.ctypes.data_as(ctypes.c_void_p) if w.size else None))
        return nxt, logits

    # the two calls LlamaDecoder offers, on top of step()
    def prefill(self, task, tokens, pos0=0, want_logits=False):
        n = len(tokens)
        nxt, logits = None, None
        for c0 in range(0, n, self.max_step_tokens):
            chunk = tokens[c0:c0 + self.max_step_tokens]
            last = c0 + len(chunk) == n
            nxt, logits = self.step(chunk, [task] * len(chunk), range(pos0 + c0, pos0 + c0 + len(chunk)),
                                    [len(chunk) - 1] if last else [], want_logits)
        return (int(nxt[0]), logits) if want_logits else int(nxt[0])

    def decode(self, tokens, positions, want_logits=False):
        b = len(tokens)
        nxt, logits = self.step(tokens, range(b), positions, range(b), want_logits)
        return (nxt, logits) if want_logits else nxt

    def set_state(self, tokens, positions):
        t = np.ascontiguousarray(tokens, dtype=np.int32)
        p = np.ascontiguousarray(positions, dtype=np.int32)
        _lib.check(self.lib.zl_bezasun_set_state(self.h, t.ctypes.data_as(ctypes.c_void_p), p.ctypes.data_as(ctypes.c_void_p),
                                                 t.size))

    def step_device(self, b):
        _lib.check(self.lib.zl_bezasun_step_device(self.h, b))

    def sync(self):
        _lib.check(self.lib.zl_bezasun_sync(self.h))

    def stream(self):
        return self.lib.zl_bezasun_stream(self.h)

    def capture_layers(self, on=True):
        _lib.check(self.lib.zl_bezasun_capture_layers(self.h, int(on)))

    def read_layers(self, n_tokens):
        """Sum of the residual streams after every layer of the last step (layers, n_tokens, width)."""
        out = np.empty((len(self.config.layers), n_tokens, self.config.width), dtype=np.float32)
        _lib.check(self.lib.zl_bezasun_read_layers(self.h, out.ctypes.data_as(ctypes.c_void_p), n_tokens))
        return out

    def read_cache(self, layer, slot, n_rows):
        """What an attention layer caches for the slot's first rows, as float32: latent attention (latents (n_rows, kv_rank),
        rotated key parts (n_rows, rot_dim)), otherwise (keys (n_rows, kv_heads * dim), values (n_rows, kv_heads * vdim))."""
        l = self.config.layers[layer]
        if l["type"] == "latent_attention":
            na, nb = l["kv_rank"], l["rot_dim"]
        else:
            na, nb = l["kv_heads"] * l["dim"], l["kv_heads"] * l["vdim"]
        a, b = np.empty((n_rows, na), dtype=np.float32), np.empty((n_rows, nb), dtype=np.float32)
        _lib.check(self.lib.zl_bezasun_read_cache(self.h, layer, slot, n_rows, a.ctypes.data_as(ctypes.c_void_p),
                                                  b.ctypes.data_as(ctypes.c_void_p)))
        return a, b

    def read_state(self, layer, slot):
        """The slot's state of a state-space layer, (heads, state, vdim)."""
        l = self.config.layers[layer]
        out = np.empty((l["heads"], l["vdim"], l["state"]), dtype=np.float32)
        _lib.check(self.lib.zl_bezasun_read_state(self.h, layer, slot, out.ctypes.data_as(ctypes.c_void_p)))
        return out.transpose(0, 2, 1)

    def stats(self):
        wb, kn = ctypes.c_double(), ctypes.c_int()
        _lib.check(self.lib.zl_bezasun_stats(self.h, ctypes.byref(wb), ctypes.byref(kn)))
        return wb.value, kn.value
