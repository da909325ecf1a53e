"""Host-side pieces of the Tufazen decoder that need no GPU: config.json -> layer descriptors and stack options, the registry, and
closed-form checks of the plain restatement (oracle/tufazen.py) that the GPU tests lean on."""
import copy
import math

import numpy as np
import pytest

from fastllm_b200 import _lib, models
from oracle import tufazen as O


def _cfg():
    return {"architecture": "Tufazen", "vocab": 40, "width": 24, "norm": {"eps": 1e-6}, "loop": {"start": 1, "stop": 3, "times": 3}, "logit_scale": 0.75,
            "embedding": {"bigram": {"buckets": 17, "mul_prev": 5, "mul_cur": 3}}, "token_side": {"dim": 6}, "layers": [
                {"type": "latent_attention", "mixer": {"heads": 3, "dim": 8, "rot_dim": 6, "vdim": 10, "kv_rank": 14, "q_rank": 7, "scale": 0.3,
                                                       "rot": {"dims": 6, "base": 777.0}},
                 "mlp": {"kind": "dense", "ff": 20, "limit": 1.25}},
                {"type": "attention", "mixer": {"heads": 4, "kv_heads": 2, "dim": 9, "vdim": 9, "scale": 0.5, "softcap": 12.0,
                                                "rot": {"dims": 4, "base": 99.0, "scaling": {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}}},
                 "mlp": {"kind": "moe", "expert": {"ff": 11}, "router": {"experts": 6, "top": 3, "groups": {"count": 3, "keep": 2}}, "shared": {"ff": 13}}},
                {"type": "attention", "mixer": {"heads": 2, "kv_heads": 1, "dim": 4, "vdim": 4, "scale": 1.0, "softcap": 3.0, "rot": {"dims": 2, "base": 10.0}},
                 "mlp": None}]}


def test_config_to_layer_descs_and_stack_options():
    d = models.tufazen_layer_descs(_cfg())
    a, b, c = d[0], d[1], d[2]
    assert len(d) == 3
    assert (a.mixer, a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank, a.q_rank, a.kv_from) == (_lib.FL_MIXER["latent_attention"], 3, 8, 6, 10, 14, 7, -1)
    assert (a.rot_dims, a.rot_base, a.rot_halves, a.out_gate, a.sink, a.yarn_factor) == (6, 777.0, 1, 2, 0, 0.0) and abs(a.scale - 0.3) < 1e-7
    assert (a.ffn, a.ffn_act, a.ff, a.limit, a.ffn_bias) == (_lib.FL_FFN["dense"], _lib.FL_ACT["swish_clamp"], 20, 1.25, 0)
    assert (b.mixer, b.heads, b.kv_heads, b.dim, b.vdim, b.scale, b.softcap) == (_lib.FL_MIXER["attention"], 4, 2, 9, 9, 0.5, 12.0)
    assert (b.no_qk_norm, b.v_from_k, b.sink, b.out_gate, b.rot_halves, b.rot_dims, b.rot_scaling) == (1, 1, 2, 1, 0, 4, _lib.FL_ROT_SCALE["yarn"])
    assert (b.yarn_factor, b.yarn_original, b.yarn_fast, b.yarn_slow) == (4.0, 64.0, 8.0, 1.0)
    assert (b.ffn, b.ffn_act, b.ff, b.experts, b.top, b.shared_ff, b.shared_plain) == (_lib.FL_FFN["moe"], _lib.FL_ACT["silu"], 11, 6, 3, 13, 1)
    assert (b.router, b.route_groups, b.route_keep, b.route_best, b.route_renorm) == (_lib.FL_ROUTER["softmax_groups"], 3, 2, 1, 0)
    assert (c.ffn, c.yarn_factor, c.kv_heads) == (_lib.FL_FFN["none"], 0.0, 1)
    sc = _lib.FlStackConfig()
    models.TufazenWithConfig.stack_options(_cfg(), sc)
    assert (sc.norm_tanh, sc.parallel_sub, sc.token_side) == (1, 1, 6)
    assert (sc.bigram_buckets, sc.bigram_mul_prev, sc.bigram_mul_cur, sc.logit_scale) == (17, 5, 3, 0.75)
    assert (sc.loop_start, sc.loop_stop, sc.loop_times, sc.loop_reinject, sc.loop_step) == (1, 3, 3, 0, 1)


def test_optional_entries_may_be_missing():
    plain = _cfg()
    for k in ("loop", "embedding", "token_side", "logit_scale"):
        plain.pop(k)
    plain["layers"][1]["mlp"].pop("shared")
    plain["layers"][1]["mlp"]["router"].pop("groups")
    sc = _lib.FlStackConfig()
    models.TufazenWithConfig.stack_options(plain, sc)
    assert (sc.loop_times, sc.loop_step, sc.token_side, sc.bigram_buckets, sc.logit_scale) == (0, 0, 0, 0, 0.0)
    b = models.tufazen_layer_descs(plain)[1]
    assert (b.shared_ff, b.route_groups, b.route_keep) == (0, 1, 1)
    for change in (lambda l: l.__setitem__("type", "mamba2"), lambda l: l.__setitem__("mlp", {"kind": "sparse"})):
        bad = copy.deepcopy(_cfg())
        change(bad["layers"][0])
        with pytest.raises(models.FastllmError):
            models.tufazen_layer_descs(bad)


def test_descriptor_layout_matches_header():
    """the newer fields sit where the header puts them: behind out_gate in the layer descriptor, behind loop_step in the stack's"""
    assert _lib.FlLayerDesc.v_from_k.offset == 104 + 26 * 4 and _lib.FlLayerDesc.route_renorm.offset == 104 + 28 * 4
    assert _lib.FlStackConfig.norm_tanh.offset == 27 * 4 and _lib.FlStackConfig.logit_scale.offset == 31 * 4
    assert _lib.FlStackConfig.bigram_mul_prev.offset == 32 * 4 and _lib.FlStackConfig.bigram_mul_cur.offset == 34 * 4


def test_registry_picks_by_architecture():
    assert models.model_class_for({"architecture": "Tufazen"}) is models.TufazenWithConfig
    assert models.model_class_for({"architecture": "Latodra"}) is models.LatodraWithConfig
    assert models.TufazenWithConfig in models.registered_models()
    assert models.TufazenWithConfig.get_family() == "Tufazen" and not models.TufazenWithConfig.supports_architecture("Latodra")
    assert models.TufazenWithConfig.no_post_norm and not models.TufazenWithConfig.no_pre_norm


# ---- closed forms of the restatement ------------------------------------------------------------------------------------------
def test_norms():
    assert np.allclose(O.tanh_norm(np.array([0.0, 100.0, -0.5]), 2.0, np.array([3.0, 2.0, 1.0]), np.array([1.0, 0.5, 0.0])), [1.0, 2.5, math.tanh(-1.0)])
    assert np.allclose(O.rms_norm(np.array([3.0, 4.0]), np.array([1.0, 2.0]), 12.0), [3.0 / math.sqrt(24.5), 8.0 / math.sqrt(24.5)])


def test_bigram_rows():
    assert O.bigram_row(4, None, 17, 5, 3) == 17
    assert O.bigram_row(4, 9, 17, 5, 3) == (45 + 12) % 17
    assert O.bigram_row(4, 0, 17, 5, 3) == 12
    assert O.bigram_row(39, 39, 101, 10 ** 10, 10 ** 9) == (39 * 10 ** 10 + 39 * 10 ** 9) % 101


def test_frequencies():
    """base 10000 over 8 channels (f = 1, .1, .01, .001): with original 4096, fast 32 and slow 1 the turning points lie at pair indices
    1.31 and 2.81, so the ramp runs from 1 to 3: half way at pair 2"""
    f, mag = O.frequencies(8, 10000.0, {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0})
    assert np.allclose(f, [1.0, 0.1, 0.01 * 0.625, 0.001 / 4.0]) and np.isclose(mag, 0.1 * math.log(4.0) + 1.0)
    f, mag = O.frequencies(8, 10000.0)
    assert np.allclose(f, [1.0, 0.1, 0.01, 0.001]) and mag == 1.0
    assert O.frequencies(0, 10.0)[0].size == 0


def test_the_two_rotations_pair_other_channels():
    """the same rotation up to the channels' order, and only the first channels turn"""
    rng = np.random.default_rng(1)
    v = rng.normal(size=(2, 9))
    f, _ = O.frequencies(6, 50.0)
    order = [0, 3, 1, 4, 2, 5, 6, 7, 8]                 # halves -> neighbours
    assert np.allclose(O.rotate_halves(v, 7, f, 1.2)[:, order], O.rotate_pairs(v[:, order], 7, f, 1.2))
    assert np.allclose(O.rotate_pairs(v, 3, f)[:, 6:], v[:, 6:]) and np.allclose(O.rotate_halves(v, 3, f)[:, 6:], v[:, 6:])
    assert np.allclose(O.rotate_pairs(np.array([1.0, 0.0, 5.0]), 1, np.array([math.pi / 2])), [0.0, 1.0, 5.0])
    assert np.allclose(O.rotate_halves(np.array([1.0, 5.0, 0.0, 5.0]), 1, np.array([math.pi / 2, 0.0])), [0.0, 5.0, 1.0, 5.0])
    q, k = rng.normal(size=6), rng.normal(size=6)
    assert np.isclose(O.rotate_halves(q, 9, f) @ O.rotate_halves(k, 4, f), O.rotate_halves(q, 25, f) @ O.rotate_halves(k, 20, f))


def test_attentions():
    assert np.allclose(O.softmax_weights(np.zeros(3), math.log(5.0)), 1 / 8) and np.allclose(O.softmax_weights(np.zeros(4)), 1 / 4)
    # the cap acts before the softmax and not on the sink; query heads 0, 1 read key head 0, heads 2, 3 key head 1
    q = np.array([[10.0], [-10.0], [0.0], [10.0]])
    k = np.array([[[1.0], [0.0]], [[-1.0], [1.0]]])                            # [keys, key heads, 1]
    v = np.array([[[1.0], [2.0]], [[5.0], [7.0]]])
    o = O.grouped_heads(q, k, v, 100.0, 2.0, np.array([3.0, 3.0, 0.0, 3.0]))
    p = np.exp([2.0, -2.0]) / (np.exp(2.0) + np.exp(-2.0) + np.exp(3.0))
    assert np.allclose(o[:, 0], [p @ [1.0, 5.0], p[::-1] @ [1.0, 5.0], 9.0 / 3.0, (2.0 + math.e ** 2 * 7.0) / (1.0 + math.e ** 2 + math.e ** 3)])
    rng = np.random.default_rng(2)
    q, qr, k, kr, v = rng.normal(size=(2, 3)), rng.normal(size=(2, 4)), rng.normal(size=(5, 2, 3)), rng.normal(size=(5, 4)), rng.normal(size=(5, 2, 6))
    o = O.latent_heads(q, qr, k, kr, v, 0.7)
    for h in range(2):
        assert np.allclose(o[h], O.softmax_weights(np.array([(k[j, h] @ q[h] + kr[j] @ qr[h]) * 0.7 for j in range(5)])) @ v[:, h])


def test_feed_forwards():
    eye = np.array([[1.0, 1.0]])
    assert np.allclose(O.clamped_swish_glu(np.array([2.0]), np.array([[5.0], [-1.0]]), np.array([[9.0], [-9.0]]), eye, 3.0),
                       3.0 * O.sigmoid(1.702 * 3.0) * 4.0 + -2.0 * O.sigmoid(-1.702 * 2.0) * -2.0)
    assert np.allclose(O.silu_glu(np.array([2.0]), np.array([[0.0], [1.0]]), np.array([[7.0], [3.0]]), eye), 2.0 * O.sigmoid(2.0) * 6.0)
    assert np.isclose(O.gelu_tanh(np.array(1.0)), 0.5 * (1 + math.tanh(math.sqrt(2 / math.pi) * 1.044715)))


def test_experts_come_from_the_best_groups():
    s = [0.30, 0.05, 0.20, 0.19, 0.16, 0.10]
    assert O.choose_experts(s, 3, 3, 2) == [0, 2, 3]           # groups marked .30, .20, .16: the last one's .16 and .10 are out, .05 is not needed
    assert O.choose_experts(s, 4, 3, 2) == [0, 2, 3, 1]
    assert O.choose_experts(s, 4, 1, 1) == [0, 2, 3, 4]
    assert O.choose_experts([0.25] * 4, 2, 2, 1) == [0, 1]
    assert O.choose_experts(s, 2, 6, 2) == [0, 2]


def test_run_order():
    assert O.run_order(3, None) == [(0, -1, False), (1, -1, False), (2, -1, False)]
    assert O.run_order(4, {"start": 1, "stop": 3, "times": 2}) == [(0, -1, False), (1, 0, True), (2, 0, False), (1, 1, True), (2, 1, False), (3, -1, False)]


def test_model_shapes_and_the_loop():
    cfg = _cfg()
    w = O.random_weights(cfg, 3)
    assert set(w) == set(O.tensor_shapes(cfg)) and "l1.mix.v" not in w and "l0.norm2" not in w and "l2.mlp.gate" not in w
    assert w["bigram"].shape == (18, 24) and w["side.embed"].shape == (40, 18) and w["l0.mix.g"].shape == (3, 24) and w["l1.mix.g"].shape == (36, 24)
    m = O.Tufazen(cfg, w)
    lg, tr = m.run([1, 2, 3, 4, 5, 6], layer_trace=True)
    assert lg.shape == (6, 40) and tr.shape == (1 + 3 * 2, 6, 24)
    # one pass with a step vector of zeros is no loop at all
    once, flat = dict(cfg, loop={"start": 1, "stop": 3, "times": 1}), {k: v for k, v in cfg.items() if k != "loop"}
    z = dict(w, **{"loop.step": np.zeros((1, 24))})
    assert np.array_equal(O.Tufazen(once, z).run([3, 1, 2]), O.Tufazen(flat, z).run([3, 1, 2]))
    # the state carries the previous token: a cut prompt continues alike
    st = m.new_state()
    assert np.array_equal(np.concatenate([m.run([1, 2, 3], st), m.run([4, 5, 6], st)]), lg)
