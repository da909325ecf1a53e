"""Plain, slow restatement of the Tufazen decoder: layers whose mixer and feed-forward both read ONE normed copy of the stream and
join it together, the norm being an element-wise tanh; latent attention (a query latent, rotate-half key part shared by the heads,
one sigmoid gate per head) and grouped-query attention whose values are its un-rotated keys (interleaved rotation with YaRN
frequencies, capped scores, a learned softmax sink per head, a sigmoid gate per channel); a clamped-swish dense feed-forward or silu
experts chosen from the best groups by softmax scores that stay as they are, plus an always-on expert; a bigram embedding, a per-layer
vector looked up by token id behind every layer, a span of layers that runs several times.  Test infrastructure only: numpy, one
function per mechanism, token by token, float64.  Nothing of the product imports this file and this file imports nothing of the
product.

Notation: x = the residual row, h = what the sublayers read, W matrices are [out, in] and applied as W @ h.
"""
from __future__ import annotations

import math

import numpy as np


# ---- small pieces ----------------------------------------------------------------------------------------------------
def rms_norm(x, w, eps):
    """x / sqrt(mean(x^2) + eps) * w over the last axis"""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def tanh_norm(x, alpha, w, b):
    return np.tanh(alpha * x) * w + b


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def bigram_row(token, previous, buckets, mul_prev, mul_cur):
    """row of the bigram table: a hash of (previous token, token); the row behind the hashed ones for a sequence's first token"""
    return buckets if previous is None else (int(previous) * mul_prev + int(token) * mul_cur) % buckets


def frequencies(dims, base, scaling=None):
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


def rotate_pairs(v, pos, f, magnitude=1.0):
    """v [..., D]: channel 2i turns with channel 2i + 1 by pos * f_i; channels behind the 2 len(f) rotated ones pass"""
    out = np.array(v, dtype=np.float64, copy=True)
    n = 2 * len(f)
    c, s = np.cos(pos * f) * magnitude, np.sin(pos * f) * magnitude
    u, w = v[..., 0:n:2], v[..., 1:n:2]
    out[..., 0:n:2], out[..., 1:n:2] = u * c - w * s, w * c + u * s
    return out


def rotate_halves(v, pos, f, magnitude=1.0):
    """the same with channel i turning with channel i + len(f)"""
    out = np.array(v, dtype=np.float64, copy=True)
    n = len(f)
    c, s = np.cos(pos * f) * magnitude, np.sin(pos * f) * magnitude
    u, w = v[..., :n], v[..., n:2 * n]
    out[..., :n], out[..., n:2 * n] = u * c - w * s, w * c + u * s
    return out


def softmax_weights(s, sink=None):
    """softmax over the scores; sink: one more term exp(sink) in the denominator that has no value"""
    m = s.max() if sink is None else max(s.max(), sink)
    e = np.exp(s - m)
    return e / (e.sum() + (0.0 if sink is None else np.exp(sink - m)))


def latent_heads(q, qr, k, kr, v, scale):
    """q [H, D] plain query parts, qr [H, R] rotated ones; k [n, H, D], v [n, H, Dv] expanded from the cached latents, kr [n, R] the
    shared key parts (rotated) -> [H, Dv]"""
    s = (np.einsum("nhd,hd->hn", k, q) + qr @ kr.T) * scale
    return np.stack([softmax_weights(s[h]) @ v[:, h] for h in range(q.shape[0])])


def grouped_heads(q, k, v, scale, cap, sinks):
    """q [H, D]; k, v [n, G, D]: query head h reads key/value head h // (H / G) -> [H, D]"""
    H, rep = q.shape[0], q.shape[0] // k.shape[1]
    out = []
    for h in range(H):
        s = k[:, h // rep] @ q[h] * scale
        out.append(softmax_weights(cap * np.tanh(s / cap), sinks[h]) @ v[:, h // rep])
    return np.stack(out)


def clamped_swish_glu(h, gate, up, down, limit):
    g, u = np.minimum(gate @ h, limit), np.clip(up @ h, -limit, limit)
    return down @ (g * sigmoid(1.702 * g) * (u + 1.0))


def silu_glu(h, gate, up, down):
    return down @ (silu(gate @ h) * (up @ h))


def choose_experts(scores, top, groups, keep):
    """-> indices of the `top` largest scores among the experts of the `keep` groups (equal runs of neighbours) whose largest score
    is largest; lower index first among equals"""
    per = len(scores) // groups
    marks = [max(scores[g * per:(g + 1) * per]) for g in range(groups)]
    kept = sorted(range(groups), key=lambda g: -marks[g])[:keep]
    pool = [e for e in range(len(scores)) if e // per in kept]
    return sorted(pool, key=lambda e: -scores[e])[:top]


def run_order(n_layers, loop):
    """(layer, pass, first of its pass) of every layer run; pass is -1 outside the loop"""
    if not loop:
        return [(i, -1, False) for i in range(n_layers)]
    a, b, n = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    return [(i, -1, False) for i in range(a)] + [(i, t, i == a) for t in range(n) for i in range(a, b)] + [(i, -1, False) for i in range(b, n_layers)]


# ---- the model -------------------------------------------------------------------------------------------------------
class Tufazen:
    """weights: dict name -> float array holding the values the product sees (bf16-representable).  cache_round: optional function
    applied to what the attentions cache (latents and shared key parts; rotated keys and values)."""

    def __init__(self, config: dict, weights: dict, cache_round=None):
        self.cfg = config
        self.w = {k: np.asarray(v, dtype=np.float64) for k, v in weights.items()}
        self.eps = float(config["norm"]["eps"])
        self.layers = config["layers"]
        self.W = int(config["width"])
        self.cache_round = cache_round or (lambda a: a)
        self.order = run_order(len(self.layers), config.get("loop"))
        self.freqs = {}

    def new_state(self):
        return {"pos": 0, "prev": None, "kv": [([], [], []) for _ in self.order]}

    def norm(self, x, name):
        return tanh_norm(x, float(self.w[name + ".alpha"].reshape(())), self.w[name], self.w[name + ".b"])

    def rot(self, i):
        if i not in self.freqs:
            r = self.layers[i]["mixer"]["rot"]
            self.freqs[i] = frequencies(int(r["dims"]), float(r["base"]), r.get("scaling"))
        return self.freqs[i]

    def cached(self, a):
        return np.asarray(self.cache_round(a), dtype=np.float64)

    def latent_attention(self, i, run, h, st):
        m, w, p = self.layers[i]["mixer"], self.w, f"l{i}.mix."
        H, D, R, Dv, C = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        q = (w[p + "uq"] @ rms_norm(w[p + "dq"] @ h, w[p + "dq.norm"], self.eps)).reshape(H, D + R)
        kv = w[p + "dkv"] @ h
        f, mag = self.rot(i)
        lat = self.cached(rms_norm(kv[:C], w[p + "dkv.norm"], self.eps))
        ks, krs, vs = st["kv"][run]
        ks.append((w[p + "uk"] @ lat).reshape(H, D))
        krs.append(self.cached(rotate_halves(kv[C:], st["pos"], f, mag)))
        vs.append((w[p + "uv"] @ lat).reshape(H, Dv))
        o = latent_heads(q[:, :D], rotate_halves(q[:, D:], st["pos"], f, mag), np.stack(ks), np.stack(krs), np.stack(vs), float(m["scale"]))
        return w[p + "o"] @ (o * sigmoid(w[p + "g"] @ h)[:, None]).reshape(-1)

    def attention(self, i, run, h, st):
        m, w, p = self.layers[i]["mixer"], self.w, f"l{i}.mix."
        H, G, D = m["heads"], m["kv_heads"], m["dim"]
        f, mag = self.rot(i)
        q, k = (w[p + "q"] @ h).reshape(H, D), (w[p + "k"] @ h).reshape(G, D)
        ks, vs, _ = st["kv"][run]
        ks.append(self.cached(rotate_pairs(k, st["pos"], f, mag)))
        vs.append(self.cached(k))
        o = grouped_heads(rotate_pairs(q, st["pos"], f, mag), np.stack(ks), np.stack(vs), float(m["scale"]), float(m["softcap"]), w[p + "sink"])
        return w[p + "o"] @ (o.reshape(-1) * sigmoid(w[p + "g"] @ h))

    def feed_forward(self, i, h):
        w, p, m = self.w, f"l{i}.mlp.", self.layers[i]["mlp"]
        if m["kind"] == "dense":
            return clamped_swish_glu(h, w[p + "gate"], w[p + "up"], w[p + "down"], float(m["limit"]))
        z = w[p + "router"] @ h
        s = np.exp(z - z.max())
        s = s / s.sum()
        r = m["router"]
        g = r.get("groups") or {"count": 1, "keep": 1}
        y = silu_glu(h, w[p + "shared.gate"], w[p + "shared.up"], w[p + "shared.down"]) if m.get("shared") else 0.0
        for e in choose_experts(s, r["top"], g["count"], g["keep"]):
            y = y + s[e] * silu_glu(h, w[f"{p}e{e}.gate"], w[f"{p}e{e}.up"], w[f"{p}e{e}.down"])
        return y

    def token_side(self, i, x, token):
        w, p, d = self.w, f"l{i}.side.", int(self.cfg["token_side"]["dim"])
        e = w["side.embed"][int(token)][i * d:(i + 1) * d]
        return rms_norm(w[p + "proj"] @ (gelu_tanh(w[p + "gate"] @ x) * e), w[p + "norm"], self.eps)

    def embedding(self, token, previous):
        x = self.w["embed"][int(token)]
        b = (self.cfg.get("embedding") or {}).get("bigram")
        if b:
            x = x + self.w["bigram"][bigram_row(token, previous, int(b["buckets"]), int(b["mul_prev"]), int(b["mul_cur"]))]
        return x

    # -- one token through every layer run --
    def step(self, token, st, layer_trace=None):
        x = self.embedding(token, st["prev"])
        for run, (i, t, first) in enumerate(self.order):
            if first:
                x = x + self.w["loop.step"][t]
            h = self.norm(x, f"l{i}.norm1")
            y = {"latent_attention": self.latent_attention, "attention": self.attention}[self.layers[i]["type"]](i, run, h, st)
            if self.layers[i].get("mlp"):
                y = y + self.feed_forward(i, h)
            x = x + y
            if self.cfg.get("token_side"):
                x = x + self.token_side(i, x, token)
            if layer_trace is not None:
                layer_trace.append(x.copy())
        st["pos"] += 1
        st["prev"] = token
        return self.w["head"] @ self.norm(x, "final.norm") * float(self.cfg.get("logit_scale", 1.0))

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

    def norm(name):
        out[name], out[name + ".b"], out[name + ".alpha"] = (W,), (W,), ()

    def glu(p, F):
        out[p + "gate"], out[p + "up"], out[p + "down"] = (F, W), (F, W), (W, F)
    out["embed"], out["head"] = (V, W), (V, W)
    norm("final.norm")
    b = (cfg.get("embedding") or {}).get("bigram")
    if b:
        out["bigram"] = (b["buckets"] + 1, W)
    if cfg.get("loop"):
        out["loop.step"] = (cfg["loop"]["times"], W)
    side = (cfg.get("token_side") or {}).get("dim")
    if side:
        out["side.embed"] = (V, len(cfg["layers"]) * side)
    for i, l in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", l["mixer"], l.get("mlp")
        H, D = m["heads"], m["dim"]
        norm(p + "norm1")
        if l["type"] == "latent_attention":
            Dv, C, Q, R = m["vdim"], m["kv_rank"], m["q_rank"], m["rot_dim"]
            out[p + "mix.dq"], out[p + "mix.dq.norm"], out[p + "mix.uq"] = (Q, W), (Q,), (H * (D + R), Q)
            out[p + "mix.dkv"], out[p + "mix.dkv.norm"] = (C + R, W), (C,)
            out[p + "mix.uk"], out[p + "mix.uv"], out[p + "mix.g"], out[p + "mix.o"] = (H * D, C), (H * Dv, C), (H, W), (W, H * Dv)
        else:
            out[p + "mix.q"], out[p + "mix.k"], out[p + "mix.sink"] = (H * D, W), (m["kv_heads"] * D, W), (H,)
            out[p + "mix.g"], out[p + "mix.o"] = (H * D, W), (W, H * D)
        if f and f["kind"] == "dense":
            glu(p + "mlp.", f["ff"])
        elif f:
            out[p + "mlp.router"] = (f["router"]["experts"], W)
            for e in range(f["router"]["experts"]):
                glu(f"{p}mlp.e{e}.", f["expert"]["ff"])
            if f.get("shared"):
                glu(p + "mlp.shared.", f["shared"]["ff"])
        if side:
            out[p + "side.gate"], out[p + "side.proj"], out[p + "side.norm"] = (side, W), (W, side), (W,)
    return out


def random_weights(cfg: dict, seed: int = 0) -> dict:
    """bf16-representable random weights: matrices N(0, 1/in), gates and routers sharper; norm weights around 1 with biases; alphas
    off 1; sinks of order one; embeddings, bigram and loop vectors of the stream's size"""
    rng = np.random.default_rng(seed)
    w = {}
    for name, shp in tensor_shapes(cfg).items():
        if name.endswith(".alpha"):
            a = rng.uniform(0.4, 1.3, shp)
        elif name.endswith("norm1.b") or name == "final.norm.b":
            a = rng.normal(0.0, 0.3, shp)
        elif "norm" in name:
            a = 1.0 + rng.normal(0.0, 0.25, shp)
        elif name.endswith(".sink"):
            a = rng.normal(0.0, 1.5, shp)
        elif name in ("embed", "bigram", "side.embed"):
            a = rng.normal(0.0, 1.0, shp)
        elif name == "loop.step":
            a = rng.normal(0.0, 0.7, shp)
        elif name.endswith((".router", "mix.g")):
            a = rng.normal(0.0, 2.0, shp) / math.sqrt(shp[1])
        else:
            a = rng.normal(0.0, 1.0, shp) / math.sqrt(shp[1])
        w[name] = to_bf16(a)
    return w
