"""Plain, slow restatement of the Latodra decoder: a sandwich-normed stack (a norm before and after every sublayer, the sublayer's
normed result scaled per channel before it joins the stream) whose layers are latent attentions -- one kind with a rotated shared
key part, YaRN frequencies and a learned softmax sink per head, the other without positions and with a sigmoid gate on the
concatenated heads, both with queries that go through a normed latent of their own --, a tanh-gelu gated feed-forward, a span of
layers that runs several times with the same weights (each pass with its own cache, a learned vector in front of every pass, the
embedding output once more in front of every pass but the first), a normed embedding and an output projection that is the
embedding table.  Test infrastructure only: numpy, one function per mechanism, token by token, float64.  Nothing of the product
imports this file and this file imports nothing of the product.

Notation: x = the residual row, h = what a sublayer reads, W matrices are [out, in] and applied as W @ h.
"""
from __future__ import annotations

import math

import numpy as np


# ---- small pieces ----------------------------------------------------------------------------------------------------
def rms_norm(x, w, eps):
    """x / sqrt(mean(x^2) + eps) * w over the last axis"""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def yarn_frequencies(dims, base, scaling=None):
    """-> (f [dims/2], magnitude).  f_i = base^(-2i/dims); with YaRN the pairs that turn often within the original context keep
    their frequency, slow ones are divided by the factor, a ramp between the two indices; cos and sin grow with the factor"""
    i = np.arange(dims // 2, dtype=np.float64)
    f = float(base) ** (-2.0 * i / dims) if dims else np.zeros(0)
    if not scaling:
        return f, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def index_of(turns):            # the (real-valued) pair index whose wave turns that often within the original context
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(float(base)))
    lo = max(math.floor(index_of(float(scaling["fast"]))), 0)
    hi = min(math.ceil(index_of(float(scaling["slow"]))), dims - 1)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / factor * ramp + f * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def rotate_interleaved(v, pos, f, magnitude=1.0):
    """v [..., R]: channel 2i turns with channel 2i + 1 by pos * f_i; channels behind the 2 len(f) rotated ones pass"""
    out = np.array(v, dtype=np.float64, copy=True)
    n = 2 * len(f)
    c, s = np.cos(pos * f) * magnitude, np.sin(pos * f) * magnitude
    u, w = v[..., 0:n:2], v[..., 1:n:2]
    out[..., 0:n:2], out[..., 1:n:2] = u * c - w * s, w * c + u * s
    return out


def softmax_weights(s, sink=None):
    """softmax over the scores; sink: one more term exp(sink) in the denominator that has no value"""
    m = s.max() if sink is None else max(s.max(), sink)
    e = np.exp(s - m)
    return e / (e.sum() + (0.0 if sink is None else np.exp(sink - m)))


def latent_heads(q, qr, lat, kr, Wuk, Wuv, scale, sinks=None):
    """q [H, D] plain query parts, qr [H, R] rotated ones; lat [n, C] cached latents, kr [n, R] cached shared key parts (rotated);
    Wuk [H, D, C], Wuv [H, Dv, C]: per head the keys and values are expanded from the latents.  -> [H, Dv]"""
    out = []
    for h in range(q.shape[0]):
        k, v = lat @ Wuk[h].T, lat @ Wuv[h].T
        s = (k @ q[h] + kr @ qr[h]) * scale
        out.append(softmax_weights(s, None if sinks is None else sinks[h]) @ v)
    return np.stack(out)


def gelu_glu(h, gate, up, down):
    return down @ (gelu_tanh(gate @ h) * (up @ h))


def run_order(n_layers, loop):
    """(layer, pass, first of its pass) of every layer run; pass is -1 outside the loop"""
    if not loop:
        return [(i, -1, False) for i in range(n_layers)]
    a, b, n = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    return [(i, -1, False) for i in range(a)] + [(i, t, i == a) for t in range(n) for i in range(a, b)] + [(i, -1, False) for i in range(b, n_layers)]


# ---- the model -------------------------------------------------------------------------------------------------------
class Latodra:
    """weights: dict name -> float array holding the values the product sees (bf16-representable).  cache_round: optional function
    applied to the latents and shared key parts the attentions cache."""

    def __init__(self, config: dict, weights: dict, cache_round=None):
        self.cfg = config
        self.w = {k: np.asarray(v, dtype=np.float64) for k, v in weights.items()}
        self.eps = float(config["norm"]["eps"])
        self.layers = config["layers"]
        self.W = int(config["width"])
        self.cache_round = cache_round
        self.order = run_order(len(self.layers), config.get("loop"))
        self.freqs = {}

    def new_state(self):
        return {"pos": 0, "kv": [([], []) for _ in self.order]}

    def attention(self, i, run, h, st):
        m, w, p = self.layers[i]["mixer"], self.w, f"l{i}.mix."
        first = self.layers[i]["type"] == "latent_attention"
        if not first and self.layers[i]["type"] != "latent_attention_2":
            raise ValueError(self.layers[i]["type"])
        H, D, Dv, C = m["heads"], m["dim"], m["vdim"], m["kv_rank"]
        R = int(m["rot_dim"]) if first else 0
        cq = rms_norm(w[p + "dq"] @ h, w[p + "dq.norm"], self.eps)
        q = (w[p + "uq"] @ cq).reshape(H, D + R)
        kv = w[p + "dkv"] @ h
        lat, kr = rms_norm(kv[:C], w[p + "dkv.norm"], self.eps), kv[C:]
        qr = q[:, D:]
        if R:
            if i not in self.freqs:
                rot = m["rot"]
                self.freqs[i] = yarn_frequencies(int(rot["dims"]), float(rot["base"]), rot.get("scaling"))
            f, mag = self.freqs[i]
            qr, kr = rotate_interleaved(qr, st["pos"], f, mag), rotate_interleaved(kr, st["pos"], f, mag)
        if self.cache_round is not None:
            lat, kr = np.asarray(self.cache_round(lat), dtype=np.float64), np.asarray(self.cache_round(kr), dtype=np.float64)
        st["kv"][run][0].append(lat)
        st["kv"][run][1].append(kr)
        o = latent_heads(q[:, :D], qr, np.stack(st["kv"][run][0]), np.stack(st["kv"][run][1]), w[p + "uk"].reshape(H, D, C), w[p + "uv"].reshape(H, Dv, C),
                         float(m["scale"]), w[p + "sink"] if first else None).reshape(-1)
        if not first:
            o = o * sigmoid(w[p + "g"] @ h)
        return w[p + "o"] @ o

    def feed_forward(self, i, h):
        w, p = self.w, f"l{i}.mlp."
        return gelu_glu(h, w[p + "gate"], w[p + "up"], w[p + "down"])

    # -- one token through every layer run --
    def step(self, token, st, layer_trace=None):
        w, eps = self.w, self.eps
        x0 = rms_norm(w["embed"][int(token)], w["embed.norm"], eps)
        x = x0
        for run, (i, t, first) in enumerate(self.order):
            if first:
                x = x + (x0 if t > 0 else 0.0) + w["loop.step"][t]
            p = f"l{i}."
            x = x + rms_norm(self.attention(i, run, rms_norm(x, w[p + "norm1"], eps), st), w[p + "norm1b"], eps) * w[p + "ls1"]
            if self.layers[i].get("mlp"):
                x = x + rms_norm(self.feed_forward(i, rms_norm(x, w[p + "norm2"], eps)), w[p + "norm2b"], eps) * w[p + "ls2"]
            if layer_trace is not None:
                layer_trace.append(x.copy())
        st["pos"] += 1
        return w["embed"] @ rms_norm(x, w["final.norm"], eps)

    def run(self, tokens, st=None, layer_trace=False):
        """-> logits [len(tokens), vocab] (and the residual stream after every layer run [runs, tokens, width] if asked)"""
        st = st if st is not None else self.new_state()
        out, tr = [], []
        for t in tokens:
            lt = [] if layer_trace else None
            out.append(self.step(t, st, lt))
            if layer_trace:
                tr.append(lt)
        logits = np.stack(out)
        if layer_trace:
            return logits, np.transpose(np.asarray(tr), (1, 0, 2))
        return logits


# ---- random models for tests -----------------------------------------------------------------------------------------
def to_bf16(a):
    """round-to-nearest-even to bfloat16, returned as float32"""
    shape = np.shape(a)
    b = np.ascontiguousarray(a, dtype=np.float32).reshape(-1).view(np.uint32)
    r = ((b + 0x7FFF + ((b >> 16) & 1)) >> 16).astype(np.uint32) << 16
    return r.view(np.float32).reshape(shape)


def tensor_shapes(cfg: dict) -> dict:
    """name -> shape of every tensor the configuration asks for"""
    W, V, out = cfg["width"], cfg["vocab"], {}
    out["embed"], out["embed.norm"], out["final.norm"] = (V, W), (W,), (W,)
    if cfg.get("loop"):
        out["loop.step"] = (cfg["loop"]["times"], W)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        H, D, Dv, C, Q = m["heads"], m["dim"], m["vdim"], m["kv_rank"], m["q_rank"]
        R = m["rot_dim"] if l["type"] == "latent_attention" else 0
        out[p + "norm1"], out[p + "norm1b"], out[p + "ls1"] = (W,), (W,), (W,)
        out[p + "mix.dq"], out[p + "mix.dq.norm"], out[p + "mix.uq"] = (Q, W), (Q,), (H * (D + R), Q)
        out[p + "mix.dkv"], out[p + "mix.dkv.norm"] = (C + R, W), (C,)
        out[p + "mix.uk"], out[p + "mix.uv"], out[p + "mix.o"] = (H * D, C), (H * Dv, C), (W, H * Dv)
        if l["type"] == "latent_attention":
            out[p + "mix.sink"] = (H,)
        else:
            out[p + "mix.g"] = (H * Dv, W)
        if l.get("mlp"):
            F = l["mlp"]["ff"]
            out[p + "norm2"], out[p + "norm2b"], out[p + "ls2"] = (W,), (W,), (W,)
            out[p + "mlp.gate"], out[p + "mlp.up"], out[p + "mlp.down"] = (F, W), (F, W), (W, F)
    return out


def random_weights(cfg: dict, seed: int = 0) -> dict:
    """bf16-representable random weights: matrices N(0, 1/in); norm weights around 1; layer scales away from 0 and 1; sinks of order
    one; loop vectors of the stream's size"""
    rng = np.random.default_rng(seed)
    w = {}
    for name, shp in tensor_shapes(cfg).items():
        if name.endswith((".ls1", ".ls2")):
            a = rng.uniform(0.3, 1.5, shp) * np.where(rng.uniform(size=shp) < 0.2, -1.0, 1.0)
        elif "norm" in name:
            a = 1.0 + rng.normal(0.0, 0.25, shp)
        elif name.endswith(".sink"):
            a = rng.normal(0.0, 1.5, shp)
        elif name == "loop.step":
            a = rng.normal(0.0, 0.7, shp)
        elif name == "embed":
            a = rng.normal(0.0, 1.0, shp)
        else:
            a = rng.normal(0.0, 1.0, shp) / math.sqrt(shp[1])
        w[name] = to_bf16(a)
    return w
