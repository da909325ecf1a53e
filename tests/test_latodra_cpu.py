"""Host-side pieces of the Latodra decoder that need no GPU: config.json -> layer descriptors and stack options, the registry, and
closed-form checks of the plain restatement (oracle/latodra.py) that the GPU tests lean on."""
import math

import numpy as np
import pytest

from fastllm_b200 import _lib, models
from oracle import latodra as O


def _cfg():
    return {"architecture": "Latodra", "vocab": 40, "width": 24, "norm": {"eps": 1e-6}, "loop": {"start": 1, "stop": 3, "times": 3}, "layers": [
        {"type": "latent_attention_2", "mixer": {"heads": 3, "dim": 8, "vdim": 10, "kv_rank": 14, "q_rank": 6, "scale": 0.3}, "mlp": {"kind": "dense", "ff": 20}},
        {"type": "latent_attention",
         "mixer": {"heads": 2, "dim": 4, "rot_dim": 6, "vdim": 5, "kv_rank": 9, "q_rank": 7, "scale": 0.5,
                   "rot": {"dims": 6, "base": 777.0, "scaling": {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}}}, "mlp": None},
        {"type": "latent_attention", "mixer": {"heads": 1, "dim": 2, "rot_dim": 2, "vdim": 2, "kv_rank": 3, "q_rank": 4, "scale": 1.0, "rot": {"dims": 2, "base": 10.0}},
         "mlp": {"kind": "dense", "ff": 9}}]}


def test_config_to_layer_descs_and_stack_options():
    d = models.latodra_layer_descs(_cfg())
    a, b, c = d[0], d[1], d[2]
    assert len(d) == 3
    assert (a.mixer, a.heads, a.dim, a.vdim, a.kv_rank, a.q_rank, a.kv_from) == (_lib.FL_MIXER["latent_attention"], 3, 8, 10, 14, 6, -1)
    assert (a.rot_dim, a.rot_dims, a.out_gate, a.sink, a.window) == (0, 0, 1, 0, 0) and abs(a.scale - 0.3) < 1e-7
    assert (a.ffn, a.ffn_act, a.ff, a.ffn_bias) == (_lib.FL_FFN["dense"], _lib.FL_ACT["gelu_tanh"], 20, 0)
    assert (b.mixer, b.heads, b.dim, b.rot_dim, b.vdim, b.kv_rank, b.q_rank) == (_lib.FL_MIXER["latent_attention"], 2, 4, 6, 5, 9, 7)
    assert (b.rot_dims, b.rot_base, b.rot_scaling, b.out_gate, b.sink) == (6, 777.0, _lib.FL_ROT_SCALE["yarn"], 0, 2)
    assert (b.yarn_factor, b.yarn_original, b.yarn_fast, b.yarn_slow, b.ffn) == (4.0, 64.0, 8.0, 1.0, _lib.FL_FFN["none"])
    assert (c.yarn_factor, c.rot_dims, c.ff) == (0.0, 2, 9)
    sc = _lib.FlStackConfig()
    models.LatodraWithConfig.stack_options(_cfg(), sc)
    assert (sc.embed_norm, sc.layer_scale, sc.tied_head) == (1, 1, 1)
    assert (sc.loop_start, sc.loop_stop, sc.loop_times, sc.loop_reinject, sc.loop_step) == (1, 3, 3, 1, 1)
    plain = _cfg()
    plain.pop("loop")
    sc = _lib.FlStackConfig()
    models.LatodraWithConfig.stack_options(plain, sc)
    assert (sc.loop_times, sc.loop_reinject, sc.loop_step) == (0, 0, 0)
    for change in (lambda l: l.__setitem__("type", "attention"), lambda l: l.__setitem__("mlp", {"kind": "moe", "expert": {"ff": 4, "limit": 1.0},
                                                                                              "router": {"experts": 2, "top": 1}})):
        bad = _cfg()
        change(bad["layers"][0])
        with pytest.raises(models.FastllmError):
            models.latodra_layer_descs(bad)


def test_descriptor_layout_matches_header():
    """the newer fields sit where the header puts them: behind shared_plain in the layer descriptor, behind token_shift in the stack's"""
    assert _lib.FlLayerDesc.q_rank.offset == 104 + 24 * 4 and _lib.FlLayerDesc.out_gate.offset == 104 + 25 * 4
    assert _lib.FlStackConfig.embed_norm.offset == 19 * 4 and _lib.FlStackConfig.loop_step.offset == 26 * 4


def test_registry_picks_by_architecture():
    assert models.model_class_for({"architecture": "Latodra"}) is models.LatodraWithConfig
    assert models.model_class_for({"architecture": "Nifunex"}) is models.NifunexWithConfig
    assert models.LatodraWithConfig in models.registered_models()
    assert models.LatodraWithConfig.get_family() == "Latodra" and not models.LatodraWithConfig.supports_architecture("Nifunex")
    assert models.LatodraWithConfig.norm_plain and not models.LatodraWithConfig.no_pre_norm and not models.LatodraWithConfig.no_post_norm


# ---- closed forms of the restatement ------------------------------------------------------------------------------------------
def test_rms_norm_has_eps_inside_the_root():
    assert np.allclose(O.rms_norm(np.array([3.0, 4.0]), np.array([1.0, 2.0]), 12.0), [3.0 / math.sqrt(24.5), 8.0 / math.sqrt(24.5)])
    assert np.allclose(O.rms_norm(np.zeros(3), np.ones(3), 1e-5), 0.0)


def test_yarn_frequencies():
    """base 10000 over 8 channels (f = 1, .1, .01, .001): with original 4096, fast 32 and slow 1 the turning points lie at pair indices
    1.31 and 2.81, so the ramp runs from 1 to 3: half way at pair 2"""
    f, mag = O.yarn_frequencies(8, 10000.0, {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0})
    assert np.allclose(f, [1.0, 0.1, 0.01 * 0.625, 0.001 / 4.0]) and np.isclose(mag, 0.1 * math.log(4.0) + 1.0)
    f, mag = O.yarn_frequencies(8, 10000.0)
    assert np.allclose(f, [1.0, 0.1, 0.01, 0.001]) and mag == 1.0
    f, _ = O.yarn_frequencies(2, 10.0, {"factor": 2.0, "original": 1, "fast": 32.0, "slow": 1.0})      # both turning points clamp to the first pair
    assert f.shape == (1,) and O.yarn_frequencies(0, 10.0)[0].size == 0


def test_rotation_is_relative_interleaved_and_grows_with_the_magnitude():
    rng = np.random.default_rng(1)
    q, k = rng.normal(size=(1, 6)), rng.normal(size=6)
    f, _ = O.yarn_frequencies(6, 50.0)
    a = O.rotate_interleaved(q, 9, f)[0] @ O.rotate_interleaved(k, 4, f)
    b = O.rotate_interleaved(q, 25, f)[0] @ O.rotate_interleaved(k, 20, f)
    assert np.isclose(a, b)
    assert np.allclose(O.rotate_interleaved(q, 3, f, 2.0), 2.0 * O.rotate_interleaved(q, 3, f))
    assert np.allclose(O.rotate_interleaved(np.array([1.0, 0.0, 5.0, 6.0]), 1, np.array([math.pi / 2])), [0.0, 1.0, 5.0, 6.0])


def test_softmax_with_and_without_a_sink():
    assert np.allclose(O.softmax_weights(np.zeros(3)), 1 / 3)
    assert np.allclose(O.softmax_weights(np.zeros(3), math.log(5.0)), 1 / 8)
    assert np.allclose(O.softmax_weights(np.array([-800.0, -801.0]), 0.0), 0.0)
    assert np.allclose(O.softmax_weights(np.array([700.0, 0.0]), -5.0), [1.0, 0.0])


def test_latent_heads_equal_a_query_absorbed_into_the_latent():
    rng = np.random.default_rng(2)
    H, D, R, C, Dv, n = 2, 3, 2, 5, 4, 6
    q, qr, lat, kr = rng.normal(size=(H, D)), rng.normal(size=(H, R)), rng.normal(size=(n, C)), rng.normal(size=(n, R))
    uk, uv = rng.normal(size=(H, D, C)), rng.normal(size=(H, Dv, C))
    o = O.latent_heads(q, qr, lat, kr, uk, uv, 0.7, np.array([0.5, -1.0]))
    for h in range(H):
        p = O.softmax_weights((lat @ (uk[h].T @ q[h]) + kr @ qr[h]) * 0.7, [0.5, -1.0][h])
        assert np.allclose(o[h], uv[h] @ (lat.T @ p))


def test_gelu_and_run_order():
    assert np.isclose(O.gelu_tanh(np.array(1.0)), 0.5 * (1 + math.tanh(math.sqrt(2 / math.pi) * 1.044715)))
    assert np.allclose(O.gelu_glu(np.array([2.0]), np.array([[0.0], [1.0]]), np.array([[7.0], [3.0]]), np.array([[1.0, 1.0]])), [O.gelu_tanh(2.0) * 6.0])
    assert O.run_order(3, None) == [(0, -1, False), (1, -1, False), (2, -1, False)]
    assert O.run_order(4, {"start": 1, "stop": 3, "times": 2}) == [(0, -1, False), (1, 0, True), (2, 0, False), (1, 1, True), (2, 1, False), (3, -1, False)]
    assert O.run_order(1, {"start": 0, "stop": 1, "times": 1}) == [(0, 0, True)]


def test_model_shapes_and_the_loop():
    cfg = _cfg()
    w = O.random_weights(cfg, 3)
    assert set(w) == set(O.tensor_shapes(cfg)) and "head" not in w and "l1.norm2" not in w and "l1.ls2" not in w and "l0.mix.sink" not in w and "l1.mix.g" not in w
    assert w["loop.step"].shape == (3, 24) and w["l1.mix.uq"].shape == (2 * 10, 7) and w["l0.mix.dkv"].shape == (14, 24) and w["l2.mix.dkv"].shape == (5, 24)
    m = O.Latodra(cfg, w)
    lg, tr = m.run([1, 2, 3, 4, 5, 6], layer_trace=True)
    assert lg.shape == (6, 40) and tr.shape == (1 + 3 * 2, 6, 24)
    # one pass with a step vector of zeros is no loop at all
    once, flat = dict(cfg, loop={"start": 1, "stop": 3, "times": 1}), {k: v for k, v in cfg.items() if k != "loop"}
    z = dict(w, **{"loop.step": np.zeros((1, 24))})
    assert np.array_equal(O.Latodra(once, z).run([3, 1, 2]), O.Latodra(flat, z).run([3, 1, 2]))
