"""The Tufazen decoder on the GPU against the plain numpy restatement in oracle/tufazen.py.

Small random configurations of the tests' own; the product runs through the C ABI (models.TufazenWithConfig /
DeviceCache.forward_ragged), the oracle token by token in float64.  Two precisions: "f32" (every product and the cache in 32-bit)
against the exact oracle; "bf16" (the serving precision: tensor-core GEMMs over hi | lo activation halves, bf16 cache) against the
oracle that rounds what its attentions cache to bf16.
"""
import copy
import json
import os
import subprocess

import numpy as np
import pytest

from fastllm_b200 import models
from fastllm_b200._lib import FastllmError
from oracle import tufazen as O

pytestmark = pytest.mark.gpu

TOL = {"f32": 4e-5, "bf16": 1e-2}


# ---- configurations ---------------------------------------------------------------------------------------------------------
def rot(dims, base=10000.0, scaling=None):
    r = {"dims": dims, "base": base}
    if scaling:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return r


def latent(heads=4, dim=8, rot_dim=6, vdim=12, kv_rank=20, q_rank=14, scale=None, base=500.0):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
            "scale": scale if scale is not None else (dim + rot_dim) ** -0.5, "rot": rot(rot_dim, base)}


def grouped(heads=4, kv_heads=2, dim=12, dims=8, scale=None, softcap=15.0, yarn=(4.0, 64, 8.0, 1.0), base=300.0):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale if scale is not None else 1.3 * dim ** -0.5, "softcap": softcap,
            "rot": rot(dims, base, yarn)}


def dense(ff=24, limit=1.5):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(ff=10, experts=6, top=3, groups=(3, 2), shared=14):
    r = {"experts": experts, "top": top}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    m = {"kind": "moe", "expert": {"ff": ff}, "router": r}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def llayer(m=None, mlp=None):
    return {"type": "latent_attention", "mixer": m or latent(), "mlp": mlp}


def alayer(m=None, mlp=None):
    return {"type": "attention", "mixer": m or grouped(), "mlp": mlp}


def loop(start, stop, times):
    return {"start": start, "stop": stop, "times": times}


BIGRAM = {"buckets": 61, "mul_prev": 31, "mul_cur": 5}


def config(layers, lp=None, vocab=48, width=32, eps=1e-5, side=5, bigram=BIGRAM, logit_scale=1.5):
    c = {"architecture": "Tufazen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers, "logit_scale": logit_scale}
    if lp:
        c["loop"] = lp
    if side:
        c["token_side"] = {"dim": side}
    if bigram:
        c["embedding"] = {"bigram": bigram}
    return c


def bare(layers, **kw):
    """one mechanism without the pieces around it"""
    return config(layers, **{"side": 0, "bigram": None, "logit_scale": 1.0, **kw})


def deep_cfg(**kw):
    """five unequal layers, the second to the fourth run twice: every mixer with every kind of feed-forward, other head counts"""
    return config([alayer(mlp=dense()),
                   llayer(mlp=moe()),
                   alayer(grouped(heads=6, kv_heads=1, dim=10, dims=10, yarn=None), mlp=moe(ff=12, experts=8, top=3, groups=(2, 1), shared=0)),
                   llayer(latent(heads=2, dim=12, rot_dim=10, vdim=8, kv_rank=12, q_rank=22, base=100.0), mlp=dense(40, 0.7)),
                   llayer(latent(heads=6, dim=4, rot_dim=2, vdim=4, kv_rank=28, q_rank=6))], loop(1, 4, 2), **kw)


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
        model, _ = models.TufazenWithConfig.initialize_model(cfg, {k: to_bits(v) for k, v in w.items()}, dtype)
        _built[key] = (O.Tufazen(cfg, w, cache_round=O.to_bf16 if dtype == "bf16" else None), model)
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
    "latent": bare([llayer()]),
    "latent_one_head": bare([llayer(latent(heads=1, dim=1, rot_dim=2, vdim=1, kv_rank=1, q_rank=1))]),
    "latent_wide_values": bare([llayer(latent(heads=2, dim=20, vdim=70, kv_rank=40, q_rank=33))]),
    "latent_wide_rotation_sharp": bare([llayer(latent(heads=3, dim=4, rot_dim=40, scale=0.9, base=50.0))]),
    "latent_many_heads": bare([llayer(latent(heads=19))]),
    "grouped": bare([alayer()]),
    "grouped_all_channels_turn": bare([alayer(grouped(dim=16, dims=16))]),
    "grouped_two_channels_turn": bare([alayer(grouped(dim=9, dims=2, heads=3, kv_heads=3))]),
    "grouped_no_channel_turns": bare([alayer(grouped(dims=0, yarn=None))]),
    "grouped_no_scaling": bare([alayer(grouped(yarn=None))]),
    "grouped_factor_one": bare([alayer(grouped(yarn=(1.0, 64, 8.0, 1.0)))]),
    "grouped_ramp_everywhere": bare([alayer(grouped(dim=16, dims=16, yarn=(8.0, 40, 16.0, 0.25), base=30.0))]),
    "grouped_one_head": bare([alayer(grouped(heads=1, kv_heads=1, dim=4, dims=2))]),
    "grouped_seven_per_head": bare([alayer(grouped(heads=14, kv_heads=2, dim=34, dims=14))]),
    "grouped_tight_cap": bare([alayer(grouped(softcap=0.8, scale=2.0))]),
    "grouped_wide_head": bare([alayer(grouped(heads=2, kv_heads=1, dim=200, dims=72))]),
    "dense": bare([alayer(mlp=dense(20, 0.5))]),
    "dense_odd": bare([llayer(mlp=dense(21, 3.0))]),
    "experts": bare([alayer(mlp=moe(shared=0))]),
    "experts_shared": bare([llayer(mlp=moe())]),
    "experts_no_groups": bare([llayer(mlp=moe(groups=None, experts=5, top=3))]),
    "experts_groups_of_one": bare([alayer(mlp=moe(groups=(6, 2), top=2))]),
    "experts_keep_one": bare([alayer(mlp=moe(experts=9, groups=(3, 1), top=3))]),
    "experts_all_used": bare([alayer(mlp=moe(experts=4, groups=(2, 2), top=4))]),
    "experts_many": bare([alayer(mlp=moe(experts=40, groups=(8, 3), top=6, ff=6))]),
    "token_vectors": bare([alayer(), llayer()], side=7),
    "token_vectors_one": bare([alayer(mlp=dense())], side=1),
    "bigram": bare([alayer()], bigram=BIGRAM),
    "bigram_one_bucket": bare([alayer()], bigram={"buckets": 1, "mul_prev": 3, "mul_cur": 1}),
    "bigram_wide_products": bare([alayer()], bigram={"buckets": 101, "mul_prev": 9_876_543_211, "mul_cur": 1_234_567_891}),
    "logit_scale": bare([llayer()], logit_scale=0.37),
    "loop_all_layers": config([alayer(), llayer()], loop(0, 2, 3)),
    "loop_once": config([llayer(), alayer()], loop(0, 1, 1)),
    "loop_first_layer": config([alayer(mlp=moe()), llayer()], loop(0, 1, 2), side=0),
    "loop_last_layer": config([llayer(), alayer(mlp=dense())], loop(1, 2, 4)),
    "loop_middle": config([llayer(), alayer(mlp=moe()), llayer(mlp=dense()), alayer()], loop(1, 3, 2), bigram=None),
    "eps_large": config([llayer(mlp=dense()), alayer()], loop(1, 2, 2), eps=0.3),
}


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", sorted(MECHANISMS))
def test_mechanism_alone(name, dtype):
    cfg = MECHANISMS[name]
    oracle, model = build(cfg, seed=3, dtype=dtype)
    toks = tokens(cfg, 37)
    assert relerr(run_whole(model, toks), oracle.run(toks)) < TOL[dtype]


def test_logit_scale_is_in_the_logits():
    """the comparison above is relative: here the numbers themselves"""
    cfg = MECHANISMS["logit_scale"]
    oracle, model = build(cfg, seed=3)
    toks = tokens(cfg, 9)
    assert np.allclose(run_whole(model, toks), oracle.run(toks), atol=1e-3)


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_odd_sizes_every_mechanism(dtype):
    """sizes that are no multiple of 4 / 8 / 32 anywhere, 70 tokens across a page border"""
    cfg = config([llayer(latent(heads=5, dim=9, rot_dim=14, vdim=35, kv_rank=37, q_rank=23), mlp=dense(21)),
                  alayer(grouped(heads=9, kv_heads=3, dim=11, dims=6), mlp=moe(ff=13, experts=10, top=3, groups=(5, 2), shared=19))],
                 loop(1, 2, 2), vocab=37, width=50, side=11)
    oracle, model = build(cfg, seed=5, dtype=dtype)
    toks = tokens(cfg, 70)
    ref = oracle.run(toks)
    assert relerr(run_whole(model, toks), ref) < TOL[dtype]
    assert relerr(run_cut(model, toks, [3, 2, 30]), ref) < TOL[dtype]


def tc_cfg():
    """widths in whole 64-column blocks: in the serving precision every product runs on the tensor-core GEMM, long portions' scores and
    weighted sums as GEMMs too"""
    return config([llayer(latent(heads=4, dim=32, rot_dim=16, vdim=48, kv_rank=64, q_rank=64), mlp=dense(128)),
                   alayer(grouped(heads=8, kv_heads=2, dim=64, dims=64), mlp=moe(ff=64, experts=8, top=3, groups=(4, 2), shared=64)),
                   llayer(latent(heads=24, dim=16, rot_dim=32, vdim=8, kv_rank=128, q_rank=64))], loop(1, 3, 2), vocab=96, width=128, side=64)


def tc_cfg_partial_tiles():
    """sizes in multiples of 8 that end inside k blocks and inside 128-row tiles; heads whose turned channels are a part"""
    return config([alayer(grouped(heads=10, kv_heads=5, dim=40, dims=24), mlp=moe(ff=72, experts=6, top=3, groups=(3, 2), shared=136)),
                   llayer(latent(heads=9, dim=24, rot_dim=8, vdim=16, kv_rank=200, q_rank=72, base=10000.0), mlp=dense(200)),
                   alayer(grouped(heads=4, kv_heads=1, dim=72, dims=16))],
                  loop(0, 1, 2), vocab=200, width=200, side=40)


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
    (pages of every pass, the slot's previous token) must not leak into the next one"""
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
    with pytest.raises(FastllmError):          # b would need a second page: the pool is empty, nothing is changed (the previous token neither)
        cache.forward_ragged([0], [tokens(cfg, 10)], None)
    assert cache.slot_len(0) == 60
    cache.slot_reset(1)
    more = tokens(cfg, 10, seed=33)
    lg = cache.forward_ragged([0], [more], [list(range(10))])
    assert relerr(lg, oracle.run(b + more)[60:]) < tol
    cache.slot_reset(0)
    short = tokens(cfg, 6, seed=34)
    assert relerr(run_cut(model, short, [], slot=0, cache=cache), oracle.run(short)) < tol
    cache.reset()
    assert relerr(run_cut(model, short, [2], slot=0, cache=cache), oracle.run(short)) < tol


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


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_previous_token_crosses_every_border(dtype):
    """a bigram table that outweighs the embedding: the token before a portion, a decoded token or a mixed step counts, at page borders
    and after another request used the slot"""
    def tweak(w):
        w["bigram"] = O.to_bf16(4.0 * w["bigram"])
    cfg = bare([alayer()], bigram={"buckets": 211, "mul_prev": 13, "mul_cur": 7})
    oracle, model = build(cfg, seed=18, dtype=dtype, tweak=tweak)
    toks = tokens(cfg, 140, seed=6)
    ref = oracle.run(toks)
    st = oracle.new_state()
    first = oracle.run(toks[:64], st)
    st["prev"] = None
    assert relerr(oracle.run(toks[64:65], st), ref[64:65]) > 10 * TOL["bf16"] and relerr(first, ref[:64]) < 1e-9
    for cuts in ([64], [63, 1, 2, 62], [1, 2, 3, 60, 2], [2] * 70, []):
        assert relerr(run_cut(model, toks, cuts, cache=model.new_device_cache(2, 192)), ref) < TOL[dtype]
    other = tokens(cfg, 90, seed=7)
    ro = oracle.run(other)
    cache = model.new_device_cache(2, 192)
    got, goth = [], []
    for k in range(45):                         # two requests in turns, and together
        got.append(cache.forward_ragged([1], [toks[2 * k:2 * k + 2]], [[0, 1]]))
        goth.append(cache.forward_ragged([0], [other[k:k + 1]], [[0]]))
    lg = cache.forward_ragged([0, 1], [other[45:], toks[90:]], [list(range(45)), list(range(50))])
    assert relerr(np.concatenate(got + [lg[45:]]), ref) < TOL[dtype] and relerr(np.concatenate(goth + [lg[:45]]), ro) < TOL[dtype]
    cache.slot_reset(1)
    assert relerr(run_cut(model, other, [1], slot=1, cache=cache), ro) < TOL[dtype]


# ---- far keys, sinks, routing, every piece: made to stand out -------------------------------------------------------------------
def standout_pair(q, k, scale):
    """q, k [tokens, heads, D]: the (query token, key token) whose score in some head stands out most over every other key's"""
    best = None
    for hd in range(q.shape[1]):
        s = q[:, hd] @ k[:, hd].T * scale
        top = np.sort(s, axis=1)
        for a in range(len(q)):
            b = int(s[a].argmax())
            if b != a and (best is None or top[a, -1] - top[a, -2] > best[0]):
                best = (top[a, -1] - top[a, -2], a, b)
    assert best[0] > 8.0            # the key holds nearly all of that head's weight even among a thousand others
    return best[1], best[2]


def far_latent():
    """a latent attention whose queries' rotated parts are zero (positions do not matter) in front of a rotated layer"""
    cfg = bare([llayer(latent(heads=2, dim=16, rot_dim=4, vdim=16, kv_rank=24, q_rank=24, scale=3.0)), alayer()], vocab=64, width=64)

    def tweak(w):
        w["l0.mix.uq"].reshape(2, 20, 24)[:, 16:] = 0.0
        w["l0.mix.o"][:] *= 2.0
    return cfg, tweak


def far_grouped():
    """a grouped attention without turned channels and a loose cap in front of a latent one"""
    return bare([alayer(grouped(heads=4, kv_heads=2, dim=24, dims=0, yarn=None, scale=3.0, softcap=200.0)), llayer()], vocab=64, width=64), None


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("make", [far_latent, far_grouped])
def test_far_keys_stand_out(make, dtype):
    """one key far back takes nearly all the weight of a later query: at the sequence's start, at both sides of page borders and in the
    middle of a page, read from a whole prompt, from a portion and by decoded tokens; the same prompt without it is far away"""
    cfg, tweak = make()
    oracle, model = build(cfg, seed=12, dtype=dtype, tweak=tweak)
    w, m = oracle.w, cfg["layers"][0]["mixer"]
    h = oracle.norm(w["embed"], "l0.norm1")
    H, D, n = m["heads"], m["dim"], cfg["vocab"]
    if cfg["layers"][0]["type"] == "attention":
        q, k = (h @ w["l0.mix.q"].T).reshape(n, H, D), (h @ w["l0.mix.k"].T).reshape(n, m["kv_heads"], D).repeat(H // m["kv_heads"], axis=1)
    else:
        q = (O.rms_norm(h @ w["l0.mix.dq"].T, w["l0.mix.dq.norm"], oracle.eps) @ w["l0.mix.uq"].T).reshape(n, H, D + m["rot_dim"])[:, :, :D]
        k = (O.rms_norm((h @ w["l0.mix.dkv"].T)[:, :m["kv_rank"]], w["l0.mix.dkv.norm"], oracle.eps) @ w["l0.mix.uk"].T).reshape(n, H, D)
    qt, kt = standout_pair(q, k, m["scale"])
    other = [t for t in range(n) if t not in (qt, kt)]
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
            assert relerr(moved[p:p + 1], ref[p:p + 1]) > 5 * TOL["bf16"]
        assert relerr(run_whole(model, toks, cache=model.new_device_cache(2, 448)), ref) < TOL[dtype]
        assert relerr(run_cut(model, toks, [64, 64, 2, 3, 280, 2], cache=model.new_device_cache(2, 448)), ref) < TOL[dtype]


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_positions_matter_where_they_should(dtype):
    """sharp rotated scores: the oracle without the scaling, with another base, or with another pairing of the channels is far away; and
    far positions (past the scaling's original context) still agree"""
    cfg = bare([alayer(grouped(heads=2, kv_heads=1, dim=20, dims=16, scale=1.0, yarn=(8.0, 48, 8.0, 1.0), base=100.0)),
                llayer(latent(heads=2, dim=4, rot_dim=16, vdim=16, kv_rank=24, scale=1.2, base=60.0))], width=48)
    oracle, model = build(cfg, seed=13, dtype=dtype)
    toks = tokens(cfg, 400, seed=5)
    ref = oracle.run(toks)

    def other(change, layer=0):
        c = copy.deepcopy(cfg)
        change(c["layers"][layer]["mixer"]["rot"])
        return relerr(O.Tufazen(c, oracle.w).run(toks[:200]), ref[:200])
    assert other(lambda r: r.pop("scaling")) > 10 * TOL["bf16"]
    assert other(lambda r: r.__setitem__("base", 120.0)) > 10 * TOL["bf16"]
    assert other(lambda r: r.__setitem__("base", 70.0), 1) > 10 * TOL["bf16"]
    for key, value in (("factor", 7.0), ("fast", 4.0), ("slow", 2.0), ("original", 64)):
        assert other(lambda r: r["scaling"].__setitem__(key, value)) > TOL["bf16"]

    def swapped(a, b):
        saved = getattr(O, a)
        setattr(O, a, getattr(O, b))
        try:
            return relerr(O.Tufazen(cfg, oracle.w).run(toks[:100]), ref[:100])
        finally:
            setattr(O, a, saved)
    assert swapped("rotate_pairs", "rotate_halves") > 10 * TOL["bf16"]
    assert swapped("rotate_halves", "rotate_pairs") > 10 * TOL["bf16"]
    assert relerr(run_whole(model, toks, cache=model.new_device_cache(2, 448)), ref) < TOL[dtype]
    assert relerr(run_cut(model, toks, [100, 2, 200, 50], cache=model.new_device_cache(2, 448)), ref) < TOL[dtype]


def test_every_piece_would_show():
    """the oracle itself with one piece taken out or changed is far outside the bar the product is held to"""
    cfg = config([alayer(mlp=moe()), llayer(mlp=dense(limit=0.6)), alayer(), llayer(mlp=moe())], loop(1, 3, 2))
    w = O.random_weights(cfg, 13)
    toks = tokens(cfg, 40, seed=5)
    ref = O.Tufazen(cfg, w).run(toks)
    _, model = build(cfg, seed=13)
    assert relerr(run_whole(model, toks), ref) < TOL["f32"]

    def changed(change=None, cfg_change=None):
        v = {k: np.array(a, copy=True) for k, a in w.items()}
        c = copy.deepcopy(cfg)
        if change:
            change(v)
        if cfg_change:
            cfg_change(c)
        return relerr(O.Tufazen(c, v).run(toks), ref)

    def to(pattern, value):
        def f(v):
            hit = [k for k in v if k.endswith(pattern)]
            assert hit
            for k in hit:
                v[k] = np.full_like(v[k], value)
        return f
    bar = 100 * TOL["f32"]
    for name in ("final.norm", "l0.norm1", "l1.norm1", "dq.norm", "dkv.norm", "side.norm", ".alpha"):
        assert changed(to(name, 1.0)) > bar, name
    for name in ("final.norm.b", "l0.norm1.b", "l2.norm1.b", "bigram", "side.embed", "l0.mlp.shared.up", "mix.g", "loop.step"):
        assert changed(to(name, 0.0)) > bar, name
    assert changed(to(".sink", -1e9)) > bar
    assert changed(to(".sink", 0.0)) > bar
    assert changed(lambda v: v.__setitem__("loop.step", v["loop.step"][::-1].copy())) > bar
    assert changed(lambda v: v.__setitem__("side.embed", np.roll(v["side.embed"], 5, axis=1))) > bar
    assert changed(lambda v: v.__setitem__("bigram", np.concatenate([v["bigram"][:-1], v["bigram"][:1]]))) > bar          # the first token's row
    for path, value in ((("loop", "times"), 1), (("layers", 1, "mixer", "scale"), 0.3), (("layers", 0, "mixer", "softcap"), 2.0),
                        (("layers", 1, "mlp", "limit"), 0.5), (("layers", 0, "mlp", "router", "groups", "keep"), 1),
                        (("layers", 3, "mlp", "router", "groups", "count"), 2), (("layers", 0, "mlp", "router", "top"), 1),
                        (("embedding", "bigram", "mul_prev"), 30), (("embedding", "bigram", "mul_cur"), 6)):
        def put(c):
            for k in path[:-1]:
                c = c[k]
            c[path[-1]] = value
        assert changed(cfg_change=put) > bar, path

    def patched(name, fn):
        saved = getattr(O, name)
        setattr(O, name, fn)
        try:
            return relerr(O.Tufazen(cfg, w).run(toks), ref)
        finally:
            setattr(O, name, saved)
    rotate = O.rotate_pairs
    heads = O.grouped_heads
    assert patched("grouped_heads", lambda q, k, v, scale, cap, sinks: heads(q, k, k, scale, cap, sinks)) > bar            # values that turn with the keys
    assert patched("rotate_pairs", lambda v, pos, f, mag=1.0: rotate(v, pos, f)) > bar                                     # the magnitude
    assert patched("choose_experts", lambda s, top, groups, keep: sorted(range(len(s)), key=lambda e: -s[e])[:top]) > bar   # no groups
    assert patched("silu", lambda z: O.gelu_tanh(z)) > bar

    class Renormalised(O.Tufazen):
        def feed_forward(self, i, h):
            m = self.layers[i]["mlp"]
            if m["kind"] != "moe":
                return super().feed_forward(i, h)
            z = self.w[f"l{i}.mlp.router"] @ h
            s = np.exp(z - z.max())
            s = s / s.sum()
            e = O.choose_experts(s, m["router"]["top"], m["router"]["groups"]["count"], m["router"]["groups"]["keep"])
            p = f"l{i}.mlp.shared."
            sh = O.silu_glu(h, self.w[p + "gate"], self.w[p + "up"], self.w[p + "down"])
            return sh + (super().feed_forward(i, h) - sh) / s[e].sum()
    assert relerr(Renormalised(cfg, w).run(toks), ref) > bar

    class Serial(O.Tufazen):        # the feed-forward reads a norm of what the mixer made of the stream
        def norm(self, x, name):
            self.x = x
            return super().norm(x, name)

        def attention(self, *a):
            self.y = super().attention(*a)
            return self.y

        def latent_attention(self, *a):
            self.y = super().latent_attention(*a)
            return self.y

        def feed_forward(self, i, h):
            return super().feed_forward(i, self.norm(self.x + self.y, f"l{i}.norm1"))
    assert relerr(Serial(cfg, w).run(toks), ref) > bar


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_best_experts_in_a_dropped_group(dtype):
    """routers made so that the second largest score lies in a group that is dropped for the token (its mark is small beside two others'
    larger ones): choosing without groups, or marking groups by the sum of their two best, picks other experts"""
    cfg = bare([alayer(mlp=moe(ff=12, experts=12, top=3, groups=(4, 2), shared=0))], width=48, vocab=150)

    def tweak(w):
        w["l0.mlp.router"] = O.to_bf16(2.5 * w["l0.mlp.router"])
    oracle, model = build(cfg, seed=22, dtype=dtype, tweak=tweak)
    h = oracle.norm(oracle.w["embed"], "l0.norm1")
    z = h @ oracle.w["l0.mlp.router"].T
    s = np.exp(z - z.max(-1, keepdims=True))
    s /= s.sum(-1, keepdims=True)
    free = sum(set(O.choose_experts(r, 3, 4, 2)) != set(np.argsort(-r)[:3]) for r in s)

    def by_two(r):
        g = r.reshape(4, 3)
        marks = np.sort(g, axis=1)[:, -2:].sum(1)
        kept = np.argsort(-marks)[:2]
        pool = [e for e in range(12) if e // 3 in kept]
        return set(sorted(pool, key=lambda e: -r[e])[:3])
    two = sum(set(O.choose_experts(r, 3, 4, 2)) != by_two(r) for r in s)
    assert free > 5 and two > 2
    toks = list(range(cfg["vocab"]))
    ref = oracle.run(toks)
    assert relerr(run_whole(model, toks), ref) < TOL[dtype]
    assert relerr(run_cut(model, toks, [1, 2, 5, 70]), ref) < TOL[dtype]


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("sink", [-30.0, 0.0, 9.0])
def test_sinks(sink, dtype):
    """no sink to speak of, one that weighs as much as a key of score zero, one that takes most of the weight (not capped: 9 is above the cap)"""
    def tweak(w):
        w["l0.mix.sink"][:] = O.to_bf16(np.array([sink, sink - 1.0, 0.5 * sink, 1.0]))
    tweak.__name__ = f"sink{sink}"
    cfg = config([alayer(grouped(softcap=5.0)), llayer()])
    oracle, model = build(cfg, seed=17, dtype=dtype, tweak=tweak)
    toks = tokens(cfg, 200, seed=4)
    ref = oracle.run(toks)
    assert relerr(run_whole(model, toks), ref) < TOL[dtype]
    assert relerr(run_cut(model, toks, [1, 1, 2, 90]), ref) < TOL[dtype]


def test_passes_have_their_own_cache():
    """a looped layer that read one cache for both passes would see the other pass's keys: the oracle with shared lists is far away"""
    cfg = config([alayer(), llayer()], loop(0, 2, 2))
    oracle, model = build(cfg, seed=16)
    toks = tokens(cfg, 30, seed=2)
    ref = oracle.run(toks)
    st = oracle.new_state()
    st["kv"] = [st["kv"][r % 2] for r in range(4)]
    assert relerr(oracle.run(toks, st), ref) > 100 * TOL["f32"]
    assert relerr(run_cut(model, toks, [7, 2]), ref) < TOL["f32"]


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
    cfg = config([alayer(grouped(heads=6, kv_heads=2, dim=16, dims=8), mlp=moe(ff=8, experts=4, groups=(2, 1), top=1, shared=8)),
                  llayer(latent(heads=18, dim=8, rot_dim=8, vdim=8, kv_rank=48, q_rank=16))], loop(0, 1, 2), width=64, side=8)
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


# ---- the pieces belong to the stack, not to this design ---------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_parallel_sublayers_of_other_mixers(dtype):
    """a recurrent mixer in a parallel layer: with a feed-forward whose down matrix is zero it equals the same layer without one, and what
    the feed-forward adds does not depend on how the prompt is cut"""
    base = {"architecture": "Tufazen", "vocab": 40, "width": 32, "norm": {"eps": 1e-5}, "layers": [{"type": "delta", "mlp": None}, {"type": "mamba2", "mlp": None}]}
    shapes = {"delta": {"q": (16, 32), "k": (16, 32), "v": (48, 32), "g": (48, 32), "b": (4, 32), "a": (4, 32), "q.conv": (16, 3), "k.conv": (16, 3),
                        "v.conv": (48, 3), "A_log": (4,), "dt_bias": (4,), "norm": (12,), "o": (32, 48)},
              "mamba2": {"in": (20 + 20 + 6 + 6 + 4, 32), "conv": (32, 4), "conv.b": (32,), "dt_bias": (4,), "A_log": (4,), "D": (4,), "norm": (20,), "o": (32, 20)}}

    class Other(models.TufazenWithConfig):
        @classmethod
        def layer_descs(cls, config, tensor_shapes):
            arr = (models._lib.FlLayerDesc * 2)()
            for d, l in zip(arr, config["layers"]):
                d.mixer, d.kv_from, d.heads = models._lib.FL_MIXER[l["type"]], -1, 4
                if l["type"] == "delta":
                    d.dim, d.vdim, d.kv_heads, d.conv = 8, 12, 2, 3
                else:
                    d.vdim, d.state, d.groups, d.norm_groups, d.conv = 5, 6, 1, 1, 4
                models._ffn_desc(d, 0, l["mlp"], act="silu")
            return arr

    def weights(ff):
        rng = np.random.default_rng(5)
        w = {}
        for name, shp in (("embed", (40, 32)), ("head", (40, 32)), ("final.norm", (32,)), ("final.norm.b", (32,)), ("final.norm.alpha", ())):
            w[name] = O.to_bf16(rng.normal(0, 0.7, shp))
        for i, l in enumerate(base["layers"]):
            for name, shp in (("norm1", (32,)), ("norm1.b", (32,)), ("norm1.alpha", ())):
                w[f"l{i}.{name}"] = O.to_bf16(rng.normal(1.0, 0.2, shp))
            for name, shp in shapes[l["type"]].items():
                w[f"l{i}.mix.{name}"] = O.to_bf16(rng.normal(0.0, 0.3, shp))
            for name, shp in (("gate", (24, 32)), ("up", (24, 32)), ("down", (32, 24))):
                w[f"l{i}.mlp.{name}"] = O.to_bf16(rng.normal(0.0, 0.3, shp)) * (ff if name == "down" else 1.0)
        return {k: to_bits(v) for k, v in w.items()}

    def model(ff):
        cfg = copy.deepcopy(base)
        for l in cfg["layers"]:
            l["mlp"] = {"kind": "dense", "ff": 24}
        return Other.initialize_model(cfg, weights(ff), dtype)[0]
    toks = tokens(base, 60)
    zero, full = model(0.0), model(1.0)
    w_zero = run_whole(zero, toks)
    assert np.isfinite(w_zero).all()
    without = Other.initialize_model(base, {k: v for k, v in weights(0.0).items() if ".mlp." not in k}, dtype)[0]
    assert relerr(w_zero, np.asarray(run_whole(without, toks), dtype=np.float64)) < TOL[dtype]
    whole = run_whole(full, toks)
    assert relerr(whole, np.asarray(w_zero, dtype=np.float64)) > 0.1
    assert relerr(run_cut(full, toks, [20, 2, 3]), np.asarray(whole, dtype=np.float64)) < TOL[dtype]


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
    bad_moe = copy.deepcopy(cfg)
    bad_moe["layers"][1]["mlp"]["router"]["groups"]["count"] = 4           # six experts do not divide into four groups
    bad_top = copy.deepcopy(cfg)
    bad_top["layers"][1]["mlp"]["router"].update(top=5)                    # two groups of two hold fewer
    for bad in (dict(cfg, loop=loop(1, 6, 2)), dict(cfg, loop=loop(2, 2, 2)), bad_moe, bad_top):
        with pytest.raises(FastllmError):
            models.TufazenWithConfig.initialize_model(bad, None, "f32")
    for name in ("l0.mix.sink", "l0.mix.g", "l1.mix.g", "loop.step", "bigram", "side.embed", "l2.side.proj", "l4.norm1.alpha", "final.norm.b",
                 "l1.mlp.shared.down", "l1.mlp.e3.gate"):
        missing = {k: to_bits(v) for k, v in O.random_weights(cfg).items() if k != name}
        with pytest.raises(FastllmError):
            models.TufazenWithConfig.initialize_model(cfg, missing, "f32")
    clone = model.clone()
    assert relerr(run_whole(clone, toks), ref) < TOL["f32"]


def test_random_init_runs_both_precisions():
    """synthetic weights (the benchmark's way in): finite logits, whole prompt = token by token"""
    cfg = tc_cfg()
    for dtype in ("bf16", "f32"):
        model, _ = models.TufazenWithConfig.initialize_model(cfg, None, dtype, random_seed=3)
        toks = tokens(cfg, 80)
        whole, single = run_whole(model, toks, cache=model.new_device_cache(2, 128)), run_cut(model, toks, [], cache=model.new_device_cache(2, 128))
        assert np.isfinite(whole).all() and np.abs(whole).max() > 0 and relerr(single, np.asarray(whole, dtype=np.float64)) < TOL[dtype]


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
    assert isinstance(model, models.TufazenWithConfig)
    toks = tokens(cfg, 30)
    assert relerr(run_whole(model, toks), O.Tufazen(cfg, w).run(toks)) < TOL["f32"]


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
    oracle = O.Tufazen(cfg, w)
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
    refs = {"float32": {k: O.Tufazen(cfg, w).run(v) for k, v in reqs.items()},
            "bfloat16": {k: O.Tufazen(cfg, w, cache_round=O.to_bf16).run(v) for k, v in reqs.items()}}
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
