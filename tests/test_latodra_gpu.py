"""The Latodra decoder on the GPU against the plain numpy restatement in oracle/latodra.py.

Small random configurations of the tests' own; the product runs through the C ABI (models.LatodraWithConfig /
DeviceCache.forward_ragged), the oracle token by token in float64.  Two precisions: "f32" (every product and the cache in 32-bit)
against the exact oracle; "bf16" (the serving precision: tensor-core GEMMs over hi | lo activation halves, bf16 latent cache) against
the oracle that rounds the latents and shared key parts it caches to bf16.
"""
import copy
import json
import os
import subprocess

import numpy as np
import pytest

from fastllm_b200 import models
from fastllm_b200._lib import FastllmError
from oracle import latodra as O

pytestmark = pytest.mark.gpu

TOL = {"f32": 4e-5, "bf16": 1e-2}


# ---- configurations ---------------------------------------------------------------------------------------------------------
def rot(dims, base=10000.0, scaling=None):
    r = {"dims": dims, "base": base}
    if scaling:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return r


def rotated(heads=4, dim=8, rot_dim=6, vdim=12, kv_rank=20, q_rank=14, scale=None, yarn=(4.0, 64, 8.0, 1.0), base=500.0):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
            "scale": scale if scale is not None else (dim + rot_dim) ** -0.5, "rot": rot(rot_dim, base, yarn)}


def gated(heads=3, dim=10, vdim=6, kv_rank=16, q_rank=18, scale=None):
    return {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale if scale is not None else dim ** -0.5}


def rlayer(m=None, ff=24):
    return {"type": "latent_attention", "mixer": m or rotated(), "mlp": {"kind": "dense", "ff": ff} if ff else None}


def glayer(m=None, ff=24):
    return {"type": "latent_attention_2", "mixer": m or gated(), "mlp": {"kind": "dense", "ff": ff} if ff else None}


def loop(start, stop, times):
    return {"start": start, "stop": stop, "times": times}


def config(layers, lp=None, vocab=48, width=32, eps=1e-5):
    c = {"architecture": "Latodra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if lp:
        c["loop"] = lp
    return c


def deep_cfg(**kw):
    """five unequal layers, the second to the fourth run twice: with and without feed-forward, other head counts and latent sizes"""
    return config([glayer(),
                   rlayer(),
                   glayer(gated(heads=5, dim=6, vdim=14, kv_rank=24, q_rank=8), ff=None),
                   rlayer(rotated(heads=2, dim=12, rot_dim=10, vdim=8, kv_rank=12, q_rank=22, yarn=(2.0, 32, 4.0, 0.5), base=100.0), ff=40),
                   rlayer(rotated(heads=6, dim=4, rot_dim=2, vdim=4, kv_rank=28, q_rank=6, yarn=None), ff=20)], loop(1, 4, 2), **kw)


# ---- helpers ----------------------------------------------------------------------------------------------------------------
def to_bits(a):
    return (np.ascontiguousarray(a, dtype=np.float32).reshape(-1).view(np.uint32) >> 16).astype(np.uint16).reshape(np.shape(a))


_built = {}


def build(cfg, seed=0, dtype="f32", tweak=None):
    """-> (oracle, product adapter); weights are bf16-representable, handed over as bf16 bit patterns"""
    key = (repr(cfg), seed, dtype, tweak.__name__ if tweak else None)
    if key not in _built:
        w = O.random_weights(cfg, seed)
        if tweak:
            tweak(w)
        model, _ = models.LatodraWithConfig.initialize_model(cfg, {k: to_bits(v) for k, v in w.items()}, dtype)
        _built[key] = (O.Latodra(cfg, w, cache_round=O.to_bf16 if dtype == "bf16" else None), model)
    return _built[key]


def relerr(got, ref):
    """worst position's error: rms over the vocabulary of the logits' difference (means taken off) relative to the rms of the logits"""
    d = np.asarray(got, dtype=np.float64) - ref
    d = d - d.mean(-1, keepdims=True)
    r = ref - ref.mean(-1, keepdims=True)
    return float((np.sqrt((d * d).mean(-1)) / np.sqrt((r * r).mean(-1))).max())


def tokens(cfg, n, seed=1):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def run_whole(model, toks, slot=0, cache=None):
    cache = cache or model.new_device_cache(max_batch=4, max_seq=max(64, len(toks)))
    return cache.forward_ragged([slot], [toks], [list(range(len(toks)))])


def run_cut(model, toks, cuts, slot=0, cache=None):
    """feed the tokens in portions of the given sizes (the rest one by one) and collect every position's logits"""
    cache = cache or model.new_device_cache(max_batch=4, max_seq=max(64, len(toks)))
    out, at = [], 0
    sizes = list(cuts)
    while at < len(toks):
        n = min(sizes.pop(0) if sizes else 1, len(toks) - at)
        out.append(cache.forward_ragged([slot], [toks[at:at + n]], [list(range(n))]))
        at += n
    return np.concatenate(out)


# ---- each mechanism alone ---------------------------------------------------------------------------------------------------
MECHANISMS = {
    "rotated_no_ff": config([rlayer(ff=None)]),
    "rotated_no_scaling": config([rlayer(rotated(yarn=None), ff=None)]),
    "rotated_factor_one": config([rlayer(rotated(yarn=(1.0, 64, 8.0, 1.0)), ff=None)]),
    "rotated_ramp_everywhere": config([rlayer(rotated(rot_dim=16, yarn=(8.0, 40, 16.0, 0.25), base=30.0), ff=None)]),
    "rotated_two_channels": config([rlayer(rotated(heads=1, rot_dim=2, dim=5, yarn=(3.0, 20, 2.0, 1.0), base=7.0), ff=None)]),
    "rotated_one_head_sharp": config([rlayer(rotated(heads=1, dim=16, rot_dim=8, vdim=40, scale=1.5), ff=None)]),
    "gated_no_ff": config([glayer(ff=None)]),
    "gated_one_head": config([glayer(gated(heads=1, dim=1, vdim=1, kv_rank=1, q_rank=1), ff=None)]),
    "gated_wide_values": config([glayer(gated(heads=2, dim=20, vdim=70, kv_rank=40, q_rank=33), ff=None)]),
    "many_heads": config([rlayer(rotated(heads=19), ff=None), glayer(gated(heads=17), ff=None)]),
    "feed_forward": config([glayer(ff=20)]),
    "loop_all_layers": config([glayer(), rlayer()], loop(0, 2, 3)),
    "loop_once": config([glayer(), rlayer()], loop(0, 1, 1)),
    "loop_first_layer": config([rlayer(), glayer()], loop(0, 1, 2)),
    "loop_last_layer_no_ff": config([rlayer(), glayer(ff=None)], loop(1, 2, 4)),
    "loop_middle_behind_no_ff": config([rlayer(ff=None), glayer(), rlayer(ff=None), glayer()], loop(1, 3, 2)),
    "eps_large": config([rlayer(), glayer()], loop(1, 2, 2), eps=0.3),
}


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", sorted(MECHANISMS))
def test_mechanism_alone(name, dtype):
    cfg = MECHANISMS[name]
    oracle, model = build(cfg, seed=3, dtype=dtype)
    toks = tokens(cfg, 37)
    assert relerr(run_whole(model, toks), oracle.run(toks)) < TOL[dtype]


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_odd_sizes_every_mechanism(dtype):
    """sizes that are no multiple of 4 / 8 / 32 anywhere, 70 tokens across a page border"""
    cfg = config([rlayer(rotated(heads=5, dim=9, rot_dim=14, vdim=35, kv_rank=37, q_rank=23), ff=21),
                  glayer(gated(heads=7, dim=11, vdim=13, kv_rank=45, q_rank=19), ff=33)], loop(1, 2, 2), vocab=37, width=50)
    oracle, model = build(cfg, seed=5, dtype=dtype)
    toks = tokens(cfg, 70)
    ref = oracle.run(toks)
    assert relerr(run_whole(model, toks), ref) < TOL[dtype]
    assert relerr(run_cut(model, toks, [3, 2, 30]), ref) < TOL[dtype]


def tc_cfg():
    """widths in whole 64-column blocks: in the serving precision every product runs on the tensor-core GEMM, the per-head products with
    W_uk / W_uv as block-diagonal GEMMs, long portions' scores and weighted sums as GEMMs too"""
    return config([rlayer(rotated(heads=4, dim=32, rot_dim=16, vdim=48, kv_rank=64, q_rank=64), ff=128),
                   glayer(gated(heads=2, dim=64, vdim=64, kv_rank=128, q_rank=128), ff=64),
                   rlayer(rotated(heads=24, dim=16, rot_dim=32, vdim=8, kv_rank=128, q_rank=64), ff=None)], loop(1, 3, 2), vocab=96, width=128)


def tc_cfg_partial_tiles():
    """latents, query latents and head sizes in multiples of 8 that end inside k blocks and inside 128-row tiles"""
    return config([glayer(gated(heads=3, dim=40, vdim=72, kv_rank=136, q_rank=104), ff=320),
                   rlayer(rotated(heads=9, dim=24, rot_dim=8, vdim=16, kv_rank=200, q_rank=72, yarn=(16.0, 128, 32.0, 1.0), base=10000.0), ff=192)],
                  loop(0, 1, 2), vocab=200, width=192)


@pytest.mark.parametrize("dtype", ["bf16", "f32"])
@pytest.mark.parametrize("make", [tc_cfg, tc_cfg_partial_tiles])
def test_tensor_core_projections_and_attention(make, dtype):
    """1 row, a few rows, up to 128 rows (weights as the 128-row operand, split-K) and more (tokens as rows) through the same layers"""
    cfg = make()
    oracle, model = build(cfg, seed=21, dtype=dtype)
    toks = tokens(cfg, 600, seed=9)
    ref = oracle.run(toks)
    assert relerr(run_whole(model, toks, cache=model.new_device_cache(4, 640)), ref) < TOL[dtype]
    assert relerr(run_cut(model, toks, [5, 128, 129, 2, 230, 64, 30], cache=model.new_device_cache(4, 640)), ref) < TOL[dtype]


# ---- schedules: whole prompt, token by token, portions, batches ---------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_prefill_equals_token_by_token(dtype):
    cfg = deep_cfg()
    oracle, model = build(cfg, seed=7, dtype=dtype)
    toks = tokens(cfg, 90)
    ref = oracle.run(toks)
    whole, single = run_whole(model, toks), run_cut(model, toks, [])
    assert relerr(whole, ref) < TOL[dtype] and relerr(single, ref) < TOL[dtype]
    assert relerr(single, np.asarray(whole, dtype=np.float64)) < TOL[dtype]


@pytest.mark.parametrize("cuts", [[2, 2, 2, 3, 2], [5, 64, 2, 17], [63, 2, 64], [1, 66, 2, 2, 2, 40], [3, 1, 1, 2, 1, 3, 1, 1, 1, 4]])
def test_portions(cuts):
    """a prompt cut into portions (down to two tokens and single ones) across page borders, the rest decoded"""
    cfg = deep_cfg()
    oracle, model = build(cfg, seed=8)
    toks = tokens(cfg, 150, seed=4)
    assert relerr(run_cut(model, toks, cuts), oracle.run(toks)) < TOL["f32"]


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("make", [deep_cfg, tc_cfg])
def test_mixed_batch_equals_each_alone(make, dtype):
    """three requests of unequal length advance together: portions of one (also long ones) beside single tokens of another"""
    cfg = make()
    oracle, model = build(cfg, seed=9, dtype=dtype)
    reqs = [tokens(cfg, n, seed=s) for n, s in ((205, 1), (9, 2), (80, 3))]
    cache = model.new_device_cache(max_batch=4, max_seq=256, pool_tokens=7 * 64)
    plan = [[(0, 3), (1, 1)], [(0, 130), (1, 1), (2, 2)], [(2, 78), (1, 7), (0, 1)], [(0, 71)]]
    at, got = [0, 0, 0], [[], [], []]
    slot = {0: 2, 1: 0, 2: 3}
    for step in plan:
        parts = [reqs[r][at[r]:at[r] + n] for r, n in step]
        lg = cache.forward_ragged([slot[r] for r, _ in step], parts, [list(range(len(p))) for p in parts])
        row = 0
        for (r, n), p in zip(step, parts):
            got[r].append(lg[row:row + len(p)])
            row += len(p)
            at[r] += len(p)
    for r in range(3):
        assert at[r] == len(reqs[r])
        alone = run_whole(model, reqs[r])
        together = np.concatenate(got[r])
        assert relerr(together, oracle.run(reqs[r])) < TOL[dtype]
        assert relerr(together, np.asarray(alone, dtype=np.float64)) < TOL[dtype]


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_pages_and_slots_reused(dtype):
    """a pool of three pages and two slots serves seven requests one after another and two at a time; what a finished request left
    in its pages (one set per pass of a looped layer) must not leak into the next one"""
    cfg = deep_cfg()
    oracle, model = build(cfg, seed=10, dtype=dtype)
    tol = TOL[dtype]
    cache = model.new_device_cache(max_batch=2, max_seq=192, pool_tokens=192)
    assert cache.pool_stats() == (3, 3)
    for i, n in enumerate((130, 100, 64, 65, 3, 1, 2)):
        toks = tokens(cfg, n, seed=20 + i)
        slot = i % 2
        assert relerr(run_whole(model, toks, slot=slot, cache=cache), oracle.run(toks)) < tol
        assert cache.slot_len(slot) == n and cache.pool_stats()[1] == 3 - (n + 63) // 64
        cache.slot_reset(slot)
        assert cache.pool_stats() == (3, 3)
    a, b = tokens(cfg, 100, seed=31), tokens(cfg, 60, seed=32)
    lg = cache.forward_ragged([1, 0], [a, b], [list(range(100)), list(range(60))])
    assert cache.pool_stats()[1] == 0
    assert relerr(lg[:100], oracle.run(a)) < tol and relerr(lg[100:], oracle.run(b)) < tol
    with pytest.raises(FastllmError):          # b would need a second page: the pool is empty, nothing is changed
        cache.forward_ragged([0], [tokens(cfg, 10)], None)
    assert cache.slot_len(0) == 60
    cache.slot_reset(1)
    more = tokens(cfg, 10, seed=33)
    lg = cache.forward_ragged([0], [more], [list(range(10))])
    assert relerr(lg, oracle.run(b + more)[60:]) < tol
    cache.slot_reset(0)
    short = tokens(cfg, 6, seed=34)
    assert relerr(run_cut(model, short, [], slot=0, cache=cache), oracle.run(short)) < tol


def test_interrupted_requests_go_on_in_scattered_pages():
    """two requests grow page by page in turns, so that their pages interleave; one ends and a third takes its pages while the other goes on"""
    cfg = deep_cfg()
    oracle, model = build(cfg, seed=11, dtype="bf16")
    a, b, d = tokens(cfg, 260, seed=1), tokens(cfg, 190, seed=2), tokens(cfg, 150, seed=3)
    cache = model.new_device_cache(max_batch=3, max_seq=320, pool_tokens=8 * 64)
    ga, gb, gd = [], [], []
    for k in range(3):
        ga.append(cache.forward_ragged([0], [a[64 * k:64 * k + 64]], [list(range(64))]))
        gb.append(cache.forward_ragged([2], [b[63 * k:63 * k + 63]], [list(range(63))]))
    gb.append(cache.forward_ragged([2], [b[189:]], [[0]]))
    assert relerr(np.concatenate(gb), oracle.run(b)) < TOL["bf16"]
    cache.slot_reset(2)
    for k in range(68):                         # the first goes on token by token, the third comes in portions of two and three
        lo, hi = len(d) * k // 68, len(d) * (k + 1) // 68
        lg = cache.forward_ragged([1, 0], [d[lo:hi], [a[192 + k]]], [list(range(hi - lo)), [0]])
        gd.append(lg[:hi - lo])
        ga.append(lg[hi - lo:])
    assert relerr(np.concatenate(ga), oracle.run(a)) < TOL["bf16"]
    assert relerr(np.concatenate(gd), oracle.run(d)) < TOL["bf16"]


# ---- far keys, sinks, every piece: made to stand out ----------------------------------------------------------------------------
def standout_pair(oracle, cfg):
    """(query token, key token): the pair whose score in a position-free first layer stands out most over every other key's"""
    w, m = oracle.w, cfg["layers"][0]["mixer"]
    H, D, C = m["heads"], m["dim"], m["kv_rank"]
    h = O.rms_norm(O.rms_norm(w["embed"], w["embed.norm"], oracle.eps) + (w["loop.step"][0] if "loop.step" in w and cfg["loop"]["start"] == 0 else 0.0),
                   w["l0.norm1"], oracle.eps)
    q = (O.rms_norm(h @ w["l0.mix.dq"].T, w["l0.mix.dq.norm"], oracle.eps) @ w["l0.mix.uq"].T).reshape(len(h), H, D)
    c = O.rms_norm(h @ w["l0.mix.dkv"].T, w["l0.mix.dkv.norm"], oracle.eps)
    k = (c @ w["l0.mix.uk"].T).reshape(len(h), H, D)
    best = None
    for hd in range(H):
        s = q[:, hd] @ k[:, hd].T * m["scale"]
        top = np.sort(s, axis=1)
        for a in range(len(h)):
            b = int(s[a].argmax())
            if b != a and (best is None or top[a, -1] - top[a, -2] > best[0]):
                best = (top[a, -1] - top[a, -2], a, b)
    assert best[0] > 8.0            # the key holds nearly all of that head's weight even among a thousand others
    return best[1], best[2]


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_far_keys_stand_out(dtype):
    """one key far back takes nearly all the weight of a later query: at the sequence's start, at both sides of page borders and in the
    middle of a page, read from a whole prompt, from a portion and by decoded tokens; the same prompt without it is far away"""
    cfg = config([glayer(gated(heads=2, dim=16, vdim=16, kv_rank=24, q_rank=24, scale=3.0), ff=None), rlayer()], vocab=64, width=64)
    oracle, model = build(cfg, seed=12, dtype=dtype)
    qt, kt = standout_pair(oracle, cfg)
    other = [t for t in range(cfg["vocab"]) if t not in (qt, kt)]
    rng = np.random.default_rng(3)
    for place in (0, 1, 63, 64, 100, 127, 128):
        toks = rng.choice(other, 420).tolist()
        toks[place] = kt
        for p in (129, 191, 192, 300, 418, 419):
            toks[p] = qt
        ref = oracle.run(toks)
        without = list(toks)
        without[place] = other[0]
        moved = oracle.run(without)
        for p in (129, 192, 419):
            assert relerr(moved[p:p + 1], ref[p:p + 1]) > 10 * TOL["bf16"]
        assert relerr(run_whole(model, toks, cache=model.new_device_cache(2, 448)), ref) < TOL[dtype]
        assert relerr(run_cut(model, toks, [64, 64, 2, 3, 280, 2], cache=model.new_device_cache(2, 448)), ref) < TOL[dtype]


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_positions_matter_where_they_should(dtype):
    """sharp rotated scores: the oracle without the scaling, with another base, or with the pairs' magnitude left out is far away; and far
    positions (past the scaling's original context) still agree"""
    cfg = config([rlayer(rotated(heads=2, dim=4, rot_dim=16, vdim=16, kv_rank=24, scale=1.5, yarn=(8.0, 48, 8.0, 1.0), base=100.0), ff=None)], width=48)
    oracle, model = build(cfg, seed=13, dtype=dtype)
    toks = tokens(cfg, 400, seed=5)
    ref = oracle.run(toks)

    def other(change):
        c = copy.deepcopy(cfg)
        change(c["layers"][0]["mixer"]["rot"])
        return relerr(O.Latodra(c, oracle.w).run(toks[:200]), ref[:200])
    assert other(lambda r: r.pop("scaling")) > 10 * TOL["bf16"]
    assert other(lambda r: r.__setitem__("base", 120.0)) > 10 * TOL["bf16"]
    assert other(lambda r: r["scaling"].__setitem__("factor", 7.0)) > TOL["bf16"]
    assert other(lambda r: r["scaling"].__setitem__("fast", 4.0)) > TOL["bf16"]
    assert other(lambda r: r["scaling"].__setitem__("slow", 2.0)) > TOL["bf16"]
    assert other(lambda r: r["scaling"].__setitem__("original", 64)) > TOL["bf16"]
    assert relerr(run_whole(model, toks, cache=model.new_device_cache(2, 448)), ref) < TOL[dtype]
    assert relerr(run_cut(model, toks, [100, 2, 200, 50], cache=model.new_device_cache(2, 448)), ref) < TOL[dtype]


def test_every_piece_would_show():
    """the oracle itself with one piece taken out or changed is far outside the bar the product is held to"""
    cfg = config([glayer(), rlayer(), glayer(ff=None), rlayer()], loop(1, 3, 2))
    w = O.random_weights(cfg, 13)
    toks = tokens(cfg, 40, seed=5)
    ref = O.Latodra(cfg, w).run(toks)
    _, model = build(cfg, seed=13)
    assert relerr(run_whole(model, toks), ref) < TOL["f32"]

    def changed(change=None, cfg_change=None):
        v = {k: np.array(a, copy=True) for k, a in w.items()}
        c = copy.deepcopy(cfg)
        if change:
            change(v)
        if cfg_change:
            cfg_change(c)
        return relerr(O.Latodra(c, v).run(toks), ref)

    def to(pattern, value):
        def f(v):
            hit = [k for k in v if k.endswith(pattern)]
            assert hit
            for k in hit:
                v[k] = np.full_like(v[k], value)
        return f
    bar = 100 * TOL["f32"]
    for name in ("embed.norm", "final.norm", "l0.norm1", "l1.norm1b", "l1.norm2", "l3.norm2b", "l2.ls1", "l1.ls2", "dq.norm", "dkv.norm"):
        assert changed(to(name, 1.0)) > bar, name
    assert changed(to(".sink", -1e9)) > bar
    assert changed(to(".sink", 0.0)) > bar
    assert changed(to("loop.step", 0.0)) > bar
    assert changed(lambda v: v.__setitem__("loop.step", v["loop.step"][::-1].copy())) > bar
    assert changed(to("mix.g", 0.0)) > bar
    assert changed(cfg_change=lambda c: c["loop"].__setitem__("times", 1)) > bar
    assert changed(cfg_change=lambda c: c["layers"][1]["mixer"].__setitem__("scale", 0.3)) > bar
    no_again = O.Latodra(cfg, w)
    no_again.w = dict(no_again.w)
    again = O.Latodra.step

    def without_embedding(self, token, st, layer_trace=None):       # the second pass starts from the stream alone
        saved = self.w["loop.step"]
        x0 = O.rms_norm(self.w["embed"][int(token)], self.w["embed.norm"], self.eps)
        self.w["loop.step"] = saved.copy()
        self.w["loop.step"][1] = saved[1] - x0
        out = again(self, token, st, layer_trace)
        self.w["loop.step"] = saved
        return out
    st = no_again.new_state()
    assert relerr(np.stack([without_embedding(no_again, t, st) for t in toks]), ref) > bar


def test_passes_have_their_own_cache():
    """a looped layer that read one cache for both passes would see the other pass's latents: the oracle with shared lists is far away"""
    cfg = config([glayer(), rlayer()], loop(0, 2, 2))
    oracle, model = build(cfg, seed=16)
    toks = tokens(cfg, 30, seed=2)
    ref = oracle.run(toks)
    st = oracle.new_state()
    st["kv"] = [st["kv"][r % 2] for r in range(4)]
    assert relerr(oracle.run(toks, st), ref) > 100 * TOL["f32"]
    assert relerr(run_cut(model, toks, [7, 2]), ref) < TOL["f32"]


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("sink", [-30.0, 0.0, 9.0])
def test_sinks(sink, dtype):
    """no sink to speak of, one that weighs as much as a key of score zero, one that takes most of the weight"""
    def tweak(w):
        w["l0.mix.sink"][:] = O.to_bf16(np.array([sink, sink - 1.0, 0.5 * sink, 1.0]))
    tweak.__name__ = f"sink{sink}"
    cfg = config([rlayer(ff=None), rlayer()])
    oracle, model = build(cfg, seed=17, dtype=dtype, tweak=tweak)
    toks = tokens(cfg, 200, seed=4)
    ref = oracle.run(toks)
    assert relerr(run_whole(model, toks), ref) < TOL[dtype]
    assert relerr(run_cut(model, toks, [1, 1, 2, 90]), ref) < TOL[dtype]


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_first_tokens(dtype):
    cfg = deep_cfg()
    oracle, model = build(cfg, seed=13, dtype=dtype)
    for n in (1, 2, 3, 5):
        toks = tokens(cfg, n, seed=n)
        assert relerr(run_whole(model, toks), oracle.run(toks)) < TOL[dtype]
        assert relerr(run_cut(model, toks, []), oracle.run(toks)) < TOL[dtype]


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_long_decoding(dtype):
    cfg = deep_cfg()
    oracle, model = build(cfg, seed=14, dtype=dtype)
    toks = tokens(cfg, 330, seed=7)
    assert relerr(run_cut(model, toks, [10]), oracle.run(toks)) < TOL[dtype]


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_long_context_and_steps_of_more_than_a_thousand_rows(dtype):
    """two requests in one long step, then decoded tokens of both over contexts whose keys are split over many blocks"""
    cfg = config([rlayer(rotated(heads=20, dim=8, rot_dim=8, vdim=8, kv_rank=48, q_rank=16)), glayer(gated(heads=2, kv_rank=24), ff=None)], loop(0, 1, 2), width=64)
    oracle, model = build(cfg, seed=19, dtype=dtype)
    a, b = tokens(cfg, 1340, seed=1), tokens(cfg, 75, seed=2)
    ra, rb = oracle.run(a), oracle.run(b)
    cache = model.new_device_cache(max_batch=2, max_seq=1408, pool_tokens=1408 + 128)
    lg = cache.forward_ragged([1, 0], [b[:3], a[:1027]], [list(range(3)), list(range(1027))])
    assert relerr(lg[:3], rb[:3]) < TOL[dtype] and relerr(lg[3:], ra[:1027]) < TOL[dtype]
    lg = cache.forward_ragged([0, 1], [a[1027:1300], b[3:40]], [list(range(273)), list(range(37))])
    assert relerr(lg[:273], ra[1027:1300]) < TOL[dtype] and relerr(lg[273:], rb[3:40]) < TOL[dtype]
    for k in range(35):
        lg = cache.forward_ragged([0, 1], [[a[1300 + k]], [b[40 + k]]], [[0], [0]])
        assert relerr(lg[:1], ra[1300 + k:1301 + k]) < TOL[dtype] and relerr(lg[1:], rb[40 + k:41 + k]) < TOL[dtype]
    lg = cache.forward_ragged([0], [a[1335:]], [list(range(5))])
    assert relerr(lg, ra[1335:]) < TOL[dtype]


# ---- the framework's own entry points -------------------------------------------------------------------------------------------
def oracle_greedy(oracle, prompt, n):
    st = oracle.new_state()
    logits = oracle.run(prompt, st)[-1]
    out = []
    for _ in range(n):
        tok = int(np.flatnonzero(logits == logits.max())[-1])       # last index among equal maxima, as the sampler does
        out.append(tok)
        logits = oracle.step(tok, st)
    return out


def test_greedy_generation_through_model_and_batcher():
    cfg = deep_cfg()
    oracle, model = build(cfg, seed=15)
    prompts = [tokens(cfg, n, seed=40 + n) for n in (5, 70, 23, 9, 31)]
    want = [oracle_greedy(oracle, p, 12) for p in prompts]
    assert models.Model(model, None, eos_token_id=None).generate(prompts[0], 12) == want[0]
    assert models.ContinuousBatcher(model, max_batch=3, eos_token_id=None).generate(prompts, 12) == want
    b = models.ContinuousBatcher(model, max_batch=2, eos_token_id=None, prefill_chunk=16)
    assert b.generate(prompts, 12) == want
    assert b.cache.pool_stats()[0] == b.cache.pool_stats()[1]


def test_uniform_entry_points_and_errors():
    cfg = deep_cfg()
    oracle, model = build(cfg, seed=16)
    toks = tokens(cfg, 20)
    cache = model.new_device_cache(max_batch=2, max_seq=64)
    ref = oracle.run(toks)
    both = cache.forward(np.asarray([toks[:12], toks[:12]], dtype=np.uint32), 0)
    assert relerr(both, np.stack([ref[11], ref[11]])) < TOL["f32"]
    nxt = cache.forward_slots([1], np.asarray([toks[12:]], dtype=np.uint32), [12])
    assert relerr(nxt, ref[19:20]) < TOL["f32"]
    for bad in (loop(1, 6, 2), loop(2, 2, 2), loop(-1, 2, 2)):                     # a loop past the last layer, an empty one, one before the first
        c = dict(cfg, loop=bad)
        with pytest.raises(FastllmError):
            models.LatodraWithConfig.initialize_model(c, None, "f32")
    for name in ("l1.mix.sink", "l0.mix.g", "loop.step", "l2.ls1", "embed.norm", "l4.mix.dq.norm"):
        missing = {k: to_bits(v) for k, v in O.random_weights(cfg).items() if k != name}
        with pytest.raises(FastllmError):
            models.LatodraWithConfig.initialize_model(cfg, missing, "f32")
    clone = model.clone()
    assert relerr(run_whole(clone, toks), ref) < TOL["f32"]


def test_random_init_runs_both_precisions():
    """synthetic weights (the benchmark's way in): finite logits, whole prompt = token by token"""
    cfg = tc_cfg()
    for dtype in ("bf16", "f32"):
        model, _ = models.LatodraWithConfig.initialize_model(cfg, None, dtype, random_seed=3)
        toks = tokens(cfg, 80)
        whole, single = run_whole(model, toks, cache=model.new_device_cache(2, 128)), run_cut(model, toks, [], cache=model.new_device_cache(2, 128))
        assert np.isfinite(whole).all() and np.abs(whole).max() > 0 and relerr(single, np.asarray(whole, dtype=np.float64)) < TOL[dtype]


def test_looped_layers_of_another_design():
    """the loop belongs to the stack: Nifunex layers (a recurrent state and a windowed latent cache) looped through the stack options equal
    the same layers written out twice with the same weights"""
    from oracle import nifunex as N
    base = {"architecture": "Nifunex", "vocab": 40, "width": 32, "norm": {"eps": 1e-5}, "layers": [
        {"type": "gla", "mixer": {"heads": 2, "dim": 8, "vdim": 12, "tau": 8.0, "decay_rank": 5}, "mlp": {"kind": "dense", "ff": 20, "limit": 3.0}},
        {"type": "latent_attention", "mixer": {"heads": 3, "dim": 8, "rot_dim": 4, "vdim": 6, "kv_rank": 20, "scale": 0.4, "mask": {"size": 9},
                                               "rot": {"dims": 4, "base": 50.0}}, "mlp": None}]}
    w = N.random_weights(base, seed=4)
    twice = dict(base, layers=base["layers"] * 2)
    w2 = dict(w)
    for k, v in w.items():
        if k[0] == "l" and k[1].isdigit():
            w2[f"l{int(k[1]) + 2}{k[2:]}"] = v

    class Looped(models.NifunexWithConfig):
        @classmethod
        def stack_options(cls, config, sc):
            sc.loop_start, sc.loop_stop, sc.loop_times = 0, 2, 2
    a, _ = Looped.initialize_model(base, {k: to_bits(v) for k, v in w.items()}, "f32")
    b, _ = models.NifunexWithConfig.initialize_model(twice, {k: to_bits(v) for k, v in w2.items()}, "f32")
    toks = tokens(base, 50)
    assert np.array_equal(run_cut(a, toks, [20, 2]), run_cut(b, toks, [20, 2]))


def _write_checkpoint(folder, cfg, w):
    from fastllm_b200 import safetensors_io
    folder.mkdir(exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    safetensors_io.write_safetensors(str(folder / "model.safetensors"), {k: to_bits(v) for k, v in w.items()})


def test_checkpoint_folder_through_the_registry(tmp_path):
    cfg = deep_cfg()
    w = O.random_weights(cfg, 17)
    _write_checkpoint(tmp_path / "m", cfg, w)
    model, _ = models.load_model(str(tmp_path / "m"), "f32")
    assert isinstance(model, models.LatodraWithConfig)
    toks = tokens(cfg, 30)
    assert relerr(run_whole(model, toks), O.Latodra(cfg, w).run(toks)) < TOL["f32"]


def test_command_line_generate(tmp_path):
    """python -m fastllm_b200 generate: registry, loader, continuous batcher with prompt portions, greedy sampling -- ids in, ids out"""
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg = deep_cfg()
    w = O.random_weights(cfg, 29)
    _write_checkpoint(tmp_path / "m", cfg, w)
    prompts = [tokens(cfg, n, seed=60 + n) for n in (3, 40, 17)]
    cmd = ["python3", "-m", "fastllm_b200", "generate", "--model", str(tmp_path / "m"), "--dtype", "f32", "--max-tokens", "6", "--max-batch", "2",
           "--prefill-chunk", "16"]
    for p in prompts:
        cmd += ["--prompt-ids", ",".join(str(t) for t in p)]
    r = subprocess.run(cmd, capture_output=True, text=True, timeout=600, cwd=root, env=dict(os.environ, PYTHONPATH=root))
    assert r.returncode == 0, r.stderr[-2000:]
    got = [json.loads(l)["generated"] for l in r.stdout.splitlines() if l.startswith("{")]
    oracle = O.Latodra(cfg, w)
    assert got == [oracle_greedy(oracle, p, 6) for p in prompts]


def test_trace_runner_end_to_end(tmp_path):
    """bin/trace_run as a process: steps on standard input (portions beside single tokens, a request that sits out a step, one that
    wants nothing, a fifth request that takes over a finished one's slot and pages), logits files out"""
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg = deep_cfg()
    w = O.random_weights(cfg, 23)
    model_dir, out_dir = tmp_path / "model", tmp_path / "out"
    _write_checkpoint(model_dir, cfg, w)
    reqs = {name: tokens(cfg, n, seed=50 + i) for i, (name, n) in enumerate((("a", 70), ("b", 5), ("c", 33), ("d", 64), ("e", 40)))}
    refs = {"float32": {k: O.Latodra(cfg, w).run(v) for k, v in reqs.items()},
            "bfloat16": {k: O.Latodra(cfg, w, cache_round=O.to_bf16).run(v) for k, v in reqs.items()}}
    plan = [[("a", 3, [0, 2]), ("b", 1, [0])],
            [("a", 60, [59]), ("c", 33, []), ("d", 2, [1])],
            [("b", 4, [0, 3]), ("d", 62, [0, 61])],
            [("a", 1, [0]), ("e", 40, [39])],
            [("a", 6, [0, 5])]]
    at = {k: 0 for k in reqs}
    lines, places = [], {}
    for n, step in enumerate(plan):
        entries, rows, end = [], [], []
        for rid, cnt, want in step:
            entries.append({"id": rid, "tokens": reqs[rid][at[rid]:at[rid] + cnt], "want": want})
            rows += [(rid, at[rid] + p) for p in want]
            at[rid] += cnt
            if at[rid] == len(reqs[rid]):
                end.append(rid)
        lines.append(json.dumps({"step": n, "entries": entries, "end": end}))
        places[n] = rows
    assert all(at[k] == len(reqs[k]) for k in reqs)
    for dtype, tol in (("float32", TOL["f32"]), ("bfloat16", TOL["bf16"])):
        p = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(model_dir), "--dtype", dtype, "--out", str(out_dir), "--max-tokens", "256"],
                           input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=600)
        assert p.returncode == 0, p.stderr[-2000:]
        assert [l for l in p.stdout.splitlines() if l.startswith("done ")] == ["done %d" % n for n in range(len(plan))]
        for n, rows in places.items():
            want = np.stack([refs[dtype][rid][p] for rid, p in rows])
            f = out_dir / ("%d.f32" % n)
            got = np.fromfile(f, dtype="<f4").reshape(-1, cfg["vocab"])
            assert got.shape == want.shape and relerr(got, want) < tol
            f.unlink()
