"""Dekalorn front end (zl_dekalorn_* C-ABI): configuration from config.json, weight loading, and the step call.

Dekalorn is a decoder-only family whose config.json lists the layers one by one; the residual stream is fp32 and every
sublayer is pre-norm, x += sublayer(w * rms(x)).  A range of layers may be *looped*: it runs `times` times with the same
weights, each pass with caches of its own, and before each pass x <- W_in [x; x0] with x0 the token's embedding.  Mixers:

  * "latent_attention": queries with an unrotated and a rotated part; one normed latent row and one rotated key part per
    position are all that is cached, keys and values of a head being linear maps of the latent; causal softmax; one
    sigmoid gate per head.
  * "attention": differential attention in a sliding window without positions: two softmax maps per head over the same
    values, o = a1 - lambda a2 with one learned lambda per layer, o divided by its root mean square over vdim and times
    (1 - diff); a full-width sigmoid gate before the output projection.
  * "attention_2": rotated queries and keys in a sliding window (adjacent pairs; frequencies scaled by wavelength), the
    scores of a head times a learned number, then mixed over all heads by a learned matrix before the softmax.

The feed-forward is absent (mlp null), "dense": W_down (relu(W_gate h) * W_up h), or "moe": silu-gated experts chosen by
sigmoid scores inside the best groups (a group ranks by the sum of its two largest scores), weights = scores over their
sum times router.scale.  config.json:

    {"architecture": "Dekalorn", "vocab": V, "width": D, "norm": {"eps": e},
     "loop": {"start", "stop", "times"} or absent,
     "layers": [{"type": "latent_attention",
                 "mixer": {"heads", "dim", "rot_dim", "vdim", "kv_rank", "scale", "rot": {"base", "dims"}},
                 "mlp": null | {"kind": "dense", "ff"}
                      | {"kind": "moe", "expert": {"ff"},
                         "router": {"experts", "top", "scale", "groups": {"count", "keep"}}}},
                {"type": "attention",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "diff", "mask": {"size"}}, "mlp": ...},
                {"type": "attention_2",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "mask": {"size"},
                           "rot": {"base", "dims", "scaling": {"factor", "low", "high", "original"}}}, "mlp": ...}]}

Checkpoint tensors: embed, head, final.norm, loop.in (D, 2 D), per layer l<i>.norm1 (and norm2 with a feed-forward),
l<i>.mix.{q, dkv, dkv.norm, uk, uv, g, o} | {q, k, v, lq1, lk1, lq2, lk2, g, o} | {q, k, v, temp, talk, o},
l<i>.mlp.{gate, up, down} | {router, e<j>.gate, e<j>.up, e<j>.down}; Linears are (out, in).
"""
import ctypes

import numpy as np

from . import _lib
from .safetensors_io import is_bf16

MIXERS = {"latent_attention": 0, "attention": 1, "attention_2": 2}
FF_KINDS = {None: 0, "dense": 1, "moe": 2}
SCALING_KEYS = ("factor", "low", "high", "original")


class DekalornLayer(ctypes.Structure):
    """zl_dekalorn_layer_t"""
    _fields_ = [("type", ctypes.c_int), ("heads", ctypes.c_int), ("kv_heads", ctypes.c_int), ("dim", ctypes.c_int),
                ("vdim", ctypes.c_int), ("rot_dim", ctypes.c_int), ("kv_rank", ctypes.c_int), ("window", ctypes.c_int),
                ("rot_dims", ctypes.c_int), ("scale", ctypes.c_float), ("diff", ctypes.c_float), ("rot_base", ctypes.c_double),
                ("rot_factor", ctypes.c_double), ("rot_low", ctypes.c_double), ("rot_high", ctypes.c_double),
                ("rot_original", ctypes.c_double), ("ff_kind", ctypes.c_int), ("ff", ctypes.c_int), ("experts", ctypes.c_int),
                ("top", ctypes.c_int), ("groups", ctypes.c_int), ("keep", ctypes.c_int), ("router_scale", ctypes.c_float)]


class DekalornCConfig(ctypes.Structure):
    """zl_dekalorn_config_t"""
    _fields_ = [("num_layers", ctypes.c_int), ("width", ctypes.c_int), ("vocab", ctypes.c_int), ("eps", ctypes.c_float),
                ("loop_start", ctypes.c_int), ("loop_stop", ctypes.c_int), ("loop_times", ctypes.c_int),
                ("dtype", ctypes.c_int), ("max_batch", ctypes.c_int), ("max_seq", ctypes.c_int), ("max_step_tokens", ctypes.c_int),
                ("use_pdl", ctypes.c_int), ("use_graph", ctypes.c_int)]


class DekalornConfig:
    """Parsed config.json of a Dekalorn model.  `layers` is a list of dicts (type, ff_kind as in config.json, every size of
    zl_dekalorn_layer_t; scaling is None or a dict), `loop` is None or (start, stop, times)."""

    def __init__(self, vocab, width, layers, norm_eps=1e-6, loop=None):
        self.vocab, self.width, self.norm_eps = int(vocab), int(width), float(norm_eps)
        self.layers, self.loop = layers, loop
        if loop is not None and not (0 <= loop[0] < loop[1] <= len(layers) and loop[2] >= 1):
            raise ValueError("loop: start < stop must lie inside the layers and times be at least 1")
        for i, l in enumerate(layers):
            if l["heads"] < 1 or l["kv_heads"] < 1 or l["heads"] % l["kv_heads"]:
                raise ValueError("layer %d: heads is not a multiple of kv_heads" % i)
            n = l["rot_dim"] if l["type"] == "latent_attention" else l["dim"]
            if l["rot_dims"] % 2 or l["rot_dims"] > n:
                raise ValueError("layer %d: rot.dims must be even and at most the rotated size" % i)
            if l["type"] == "latent_attention" and l["rot_dims"] != l["rot_dim"]:
                raise ValueError("layer %d: latent attention rotates all of rot_dim" % i)
            if l["window"] < 0:
                raise ValueError("layer %d: mask.size must be positive" % i)
            if l["ff_kind"] == "moe":
                if not 0 < l["top"] <= l["experts"]:
                    raise ValueError("layer %d: router.top must be between 1 and experts" % i)
                if l["groups"] < 1 or l["experts"] % l["groups"] or not 0 < l["keep"] <= l["groups"]:
                    raise ValueError("layer %d: groups.count must divide experts and keep lie in 1..count" % i)
                if l["keep"] * (l["experts"] // l["groups"]) < l["top"]:
                    raise ValueError("layer %d: the kept groups hold fewer experts than router.top" % i)

    @classmethod
    def from_dict(cls, d):
        layers = []
        for i, l in enumerate(d["layers"]):
            kind, mx, mlp = l.get("type"), l["mixer"], l.get("mlp")
            if kind not in MIXERS:
                raise ValueError("layer %d: unknown mixer type %r" % (i, kind))
            rot = mx.get("rot") or {}
            scaling = rot.get("scaling") or None
            latent = kind == "latent_attention"
            out = dict(type=kind, heads=int(mx["heads"]), kv_heads=int(mx["heads"] if latent else mx.get("kv_heads", mx["heads"])),
                       dim=int(mx["dim"]), vdim=int(mx["vdim"]), rot_dim=int(mx.get("rot_dim", 0)) if latent else 0,
                       kv_rank=int(mx["kv_rank"]) if latent else 0,
                       window=0 if latent else int((mx.get("mask") or {}).get("size", 0)),
                       rot_dims=0, rot_base=float(rot.get("base", 10000.0)), scaling=None, scale=float(mx["scale"]),
                       diff=float(mx["diff"]) if kind == "attention" else 0.0, ff_kind=None, ff=0, experts=0, top=0, groups=1,
                       keep=1, router_scale=1.0)
            if kind != "attention":
                out["rot_dims"] = int(rot.get("dims", out["rot_dim"]))
                if scaling:
                    out["scaling"] = {k: float(scaling[k]) for k in SCALING_KEYS}
            if mlp is not None:
                ff = mlp.get("kind")
                if ff == "dense":
                    out.update(ff_kind="dense", ff=int(mlp["ff"]))
                elif ff == "moe":
                    r = mlp["router"]
                    g = r.get("groups") or {}
                    out.update(ff_kind="moe", ff=int(mlp["expert"]["ff"]), experts=int(r["experts"]), top=int(r["top"]),
                               groups=int(g.get("count", 1)), keep=int(g.get("keep", g.get("count", 1))),
                               router_scale=float(r.get("scale", 1.0)))
                else:
                    raise ValueError("layer %d: unknown feed-forward kind %r" % (i, ff))
            layers.append(out)
        loop = d.get("loop")
        if loop is not None:
            loop = (int(loop["start"]), int(loop["stop"]), int(loop["times"]))
        return cls(d["vocab"], d["width"], layers, (d.get("norm") or {}).get("eps", 1e-6), loop)

    def to_dict(self):
        out = []
        for l in self.layers:
            keys = {"latent_attention": ("heads", "dim", "rot_dim", "vdim", "kv_rank", "scale"),
                    "attention": ("heads", "kv_heads", "dim", "vdim", "scale", "diff"),
                    "attention_2": ("heads", "kv_heads", "dim", "vdim", "scale")}[l["type"]]
            mx = {k: l[k] for k in keys}
            if l["type"] != "attention":
                mx["rot"] = {"base": l["rot_base"], "dims": l["rot_dims"]}
                if l["scaling"]:
                    mx["rot"]["scaling"] = dict(l["scaling"])
            if l["window"]:
                mx["mask"] = {"size": l["window"]}
            mlp = None
            if l["ff_kind"] == "dense":
                mlp = {"kind": "dense", "ff": l["ff"]}
            elif l["ff_kind"] == "moe":
                mlp = {"kind": "moe", "expert": {"ff": l["ff"]},
                       "router": {"experts": l["experts"], "top": l["top"], "scale": l["router_scale"],
                                  "groups": {"count": l["groups"], "keep": l["keep"]}}}
            out.append({"type": l["type"], "mixer": mx, "mlp": mlp})
        d = {"architecture": "Dekalorn", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps}, "layers": out}
        if self.loop:
            d["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        return d

    @property
    def num_runs(self):
        """Layer runs of a step: a looped layer counts once per pass (each run has caches of its own)."""
        n = len(self.layers)
        return n if not self.loop else n + (self.loop[1] - self.loop[0]) * (self.loop[2] - 1)

    def run_layer(self, run):
        """The layer that runs as number `run` of a step."""
        if not self.loop:
            return run
        a, b, times = self.loop
        if run < a:
            return run
        if run < a + (b - a) * times:
            return a + (run - a) % (b - a)
        return run - (b - a) * (times - 1)

    def tensor_shapes(self):
        """name -> shape of every checkpoint tensor."""
        D, s = self.width, {}
        s["embed"] = s["head"] = (self.vocab, D)
        s["final.norm"] = (D,)
        if self.loop:
            s["loop.in"] = (D, 2 * D)
        for i, l in enumerate(self.layers):
            p, H, G, d, vd = "l%d." % i, l["heads"], l["kv_heads"], l["dim"], l["vdim"]
            m = p + "mix."
            s[p + "norm1"] = (D,)
            if l["type"] == "latent_attention":
                R = l["kv_rank"]
                s[m + "q"] = (H * (d + l["rot_dim"]), D)
                s[m + "dkv"], s[m + "dkv.norm"] = (R + l["rot_dim"], D), (R,)
                s[m + "uk"], s[m + "uv"], s[m + "g"] = (H * d, R), (H * vd, R), (H, D)
            elif l["type"] == "attention":
                s[m + "q"], s[m + "k"], s[m + "v"] = (H * 2 * d, D), (G * 2 * d, D), (G * vd, D)
                for n in ("lq1", "lk1", "lq2", "lk2"):
                    s[m + n] = (d,)
                s[m + "g"] = (H * vd, D)
            else:
                s[m + "q"], s[m + "k"], s[m + "v"] = (H * d, D), (G * d, D), (G * vd, D)
                s[m + "temp"], s[m + "talk"] = (H,), (H, H)
            s[m + "o"] = (D, H * vd)
            if l["ff_kind"]:
                s[p + "norm2"] = (D,)
            if l["ff_kind"] == "dense":
                s[p + "mlp.gate"] = s[p + "mlp.up"] = (l["ff"], D)
                s[p + "mlp.down"] = (D, l["ff"])
            elif l["ff_kind"] == "moe":
                s[p + "mlp.router"] = (l["experts"], D)
                for e in range(l["experts"]):
                    s[p + "mlp.e%d.gate" % e] = s[p + "mlp.e%d.up" % e] = (l["ff"], D)
                    s[p + "mlp.e%d.down" % e] = (D, l["ff"])
        return s


DTYPES = {"bf16": 1, "bfloat16": 1, "f32": 2, "float32": 2}


class DekalornDecoder:
    """One model instance on the current CUDA device.  Slots (0..max_batch-1) each own `max_seq` rows of every layer run's
    caches (a looped layer has caches per pass); the engine's scheduler decides which sequence lives in which slot."""

    architecture = "Dekalorn"
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
        loop = c.loop or (0, 0, 0)
        self.cfg = DekalornCConfig(len(c.layers), c.width, c.vocab, c.norm_eps, loop[0], loop[1], loop[2], DTYPES[dtype],
                                   self.max_batch, self.max_seq, self.max_step_tokens, int(use_pdl), int(use_graph))
        arr = (DekalornLayer * len(c.layers))()
        for i, l in enumerate(c.layers):
            sc = l["scaling"] or dict.fromkeys(SCALING_KEYS, 0.0)
            arr[i] = DekalornLayer(MIXERS[l["type"]], l["heads"], l["kv_heads"], l["dim"], l["vdim"], l["rot_dim"], l["kv_rank"],
                                   l["window"], l["rot_dims"], l["scale"], l["diff"], l["rot_base"], sc["factor"], sc["low"],
                                   sc["high"], sc["original"], FF_KINDS[l["ff_kind"]], l["ff"], l["experts"], l["top"],
                                   l["groups"], l["keep"], l["router_scale"])
        h = ctypes.c_void_p()
        _lib.check(self.lib.zl_dekalorn_create(ctypes.byref(self.cfg), arr, ctypes.byref(h)))
        self.h = h

    @classmethod
    def from_config_dict(cls, d, **kw):
        return cls(DekalornConfig.from_dict(d), **kw)

    def close(self):
        if getattr(self, "h", None):
            self.lib.zl_dekalorn_destroy(self.h)
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
            _lib.check(self.lib.zl_dekalorn_load_tensor(self.h, name.encode(), a.ctypes.data_as(ctypes.c_void_p), rows, cols,
                                                       a.itemsize))
        _lib.check(self.lib.zl_dekalorn_finalize(self.h))

    def init_synthetic(self, seed=0):
        _lib.check(self.lib.zl_dekalorn_init_synthetic(self.h, seed))

    def step(self, tokens, slots, positions, want_rows=(), want_logits=True):
        """One step over T rows.  Returns (next tokens (n_want), logits (n_want, vocab) or None) for the wanted rows."""
        t = np.ascontiguousarray(tokens, dtype=np.int32)
        s = np.ascontiguousarray(slots, dtype=np.int32)
        p = np.ascontiguousarray(positions, dtype=np.int32)
        w = np.ascontiguousarray(want_rows, dtype=np.int32)
        nxt = np.empty(w.size, dtype=np.int32)
        logits = np.empty((w.size, self.vocab_size), dtype=np.float32) if want_logits else None
        _lib.check(self.lib.zl_dekalorn_step(
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
        _lib.check(self.lib.zl_dekalorn_set_state(self.h, t.ctypes.data_as(ctypes.c_void_p), p.ctypes.data_as(ctypes.c_void_p),
                                                 t.size))

    def step_device(self, b):
        _lib.check(self.lib.zl_dekalorn_step_device(self.h, b))

    def sync(self):
        _lib.check(self.lib.zl_dekalorn_sync(self.h))

    def stream(self):
        return self.lib.zl_dekalorn_stream(self.h)

    def capture_layers(self, on=True):
        _lib.check(self.lib.zl_dekalorn_capture_layers(self.h, int(on)))

    def read_layers(self, n_tokens):
        """Residual stream after every layer run of the last step (runs, n_tokens, width)."""
        out = np.empty((self.config.num_runs, n_tokens, self.config.width), dtype=np.float32)
        _lib.check(self.lib.zl_dekalorn_read_layers(self.h, out.ctypes.data_as(ctypes.c_void_p), n_tokens))
        return out

    def read_cache(self, run, slot, n_rows):
        """What layer run `run` caches for the slot's first rows, as float32: latent attention (latents (n_rows, kv_rank),
        rotated key parts (n_rows, rot_dim)), otherwise (keys (n_rows, kv_heads * dim, twice that for differential
        attention), values (n_rows, kv_heads * vdim))."""
        l = self.config.layers[self.config.run_layer(run)]
        if l["type"] == "latent_attention":
            na, nb = l["kv_rank"], l["rot_dim"]
        else:
            na, nb = l["kv_heads"] * l["dim"] * (2 if l["type"] == "attention" else 1), l["kv_heads"] * l["vdim"]
        a, b = np.empty((n_rows, na), dtype=np.float32), np.empty((n_rows, nb), dtype=np.float32)
        _lib.check(self.lib.zl_dekalorn_read_cache(self.h, run, slot, n_rows, a.ctypes.data_as(ctypes.c_void_p),
                                                   b.ctypes.data_as(ctypes.c_void_p)))
        return a, b

    def stats(self):
        wb, kn = ctypes.c_double(), ctypes.c_int()
        _lib.check(self.lib.zl_dekalorn_stats(self.h, ctypes.byref(wb), ctypes.byref(kn)))
        return wb.value, kn.value
