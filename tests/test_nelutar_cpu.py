"""CPU-side checks of the Nelutar integration: config reader and registry, rotary frequencies, and the restatement's own properties
(visibility through the window, causality, decays, routing by groups)."""
import os
import sys

import numpy as np
import pytest

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import nelutar_oracle as O  # noqa: E402
import nelutar_testlib as L  # noqa: E402


def test_config_reader(tmp_path):
    from simplellminference_b200.config import DeltaRuleConfig, ExpertsConfig, GatedFeedForwardConfig, NelutarConfig, RotaryConfig, read_model_config
    layers = [L.delta_pair(mlp=L.moe()), L.lightning_pair(), L.retention_layer(mlp=None, rot_dims=0), L.lightning_pair(size=None, conv=0, softcap=0.0, mlp=L.moe(groups=0, shared=0))]
    cfg = L.make_config(layers + [L.again(layers, 1)])
    c = read_model_config(L.write_model(str(tmp_path / "m"), cfg, {"embed": np.zeros((2, 2), np.float32)}))
    assert isinstance(c, NelutarConfig) and (c.vocab, c.width, c.norm_eps) == (83, 48, 1e-5)
    assert (c.pair_buckets, c.pair_mul_prev, c.pair_mul_cur) == (53, 29, 11)
    a, b, r, e, again = c.layers
    assert (a.left.heads, a.left.kv_heads, a.left.dim, a.left.vdim, a.left.scale, a.left.mask.size, a.left.rot) == (4, 2, 16, 12, 0.3, 20, RotaryConfig(8, 1000.0))
    assert a.right == DeltaRuleConfig(6, 3, 10, 14, 3) and a.mlp == ExpertsConfig(8, 0, 3, 12, 20, 0.9, 1.3, 4, 2, 1.5)
    assert (b.left.conv, b.left.softcap, b.left_scale, b.right_scale) == (3, 4.0, 0.7, 1.2) and b.right.decay == tuple(L.decays(3, 0.4, 0.99))
    assert b.mlp == GatedFeedForwardConfig(40) and r.mlp is None and r.mixer.rot is None and r.mixer.decay == tuple(L.decays(3))
    assert e.left.mask.size is None and (e.left.conv, e.left.softcap) == (0, 0.0) and (e.mlp.groups, e.mlp.shared) == (0, 0)
    assert again.weights_of == 1 and again.left == b.left
    bad = lambda msg, ls: pytest.raises(ValueError, NelutarConfig.from_dict, L.make_config(ls)).match(msg)   # noqa: E731
    bad("unknown mixer type", [dict(L.retention_layer(), type="conv")])
    bad("not part of this design", [L.retention_layer(mlp={"kind": "sparse"})])
    bad("weights_of", [dict(layers[0], weights_of=0)])
    bad("weights_of", [layers[0], dict(layers[0], weights_of=2), dict(layers[0], weights_of=0)])
    bad("described like it", [layers[0], dict(layers[1], weights_of=0)])
    bad("do not divide", [L.delta_pair(heads=5, kv_heads=2)])
    bad("do not divide", [L.delta_pair(rheads=5, rkv=2)])
    bad("do not fit", [L.retention_layer(dim=8, rot_dims=12)])
    bad("decays for", [L.retention_layer(heads=3, decay=[0.5, 0.9])])
    bad("groups", [L.retention_layer(mlp=L.moe(experts=8, groups=3))])
    bad("experts", [L.retention_layer(mlp=L.moe(experts=8, groups=4, keep=1, top=3))])


def test_registry_knows_the_design():
    from simplellminference_b200.config import CONFIG_READERS
    from simplellminference_b200.models import MODEL_CLASSES
    assert "Nelutar" in MODEL_CLASSES and set(MODEL_CLASSES) == set(CONFIG_READERS)


def test_rotary_frequencies():
    from simplellminference_b200.config import RotaryConfig
    from simplellminference_b200.layers import rotary_frequencies
    key, freq = rotary_frequencies(RotaryConfig(6, 100.0), "cpu")
    np.testing.assert_allclose(freq.numpy(), [1.0, 100.0 ** (-1 / 3), 100.0 ** (-2 / 3)], rtol=1e-14)
    assert rotary_frequencies(None, "cpu") == ((), None)


def _w(layer, width=24, seed=1):
    return {k: v.astype(np.float64) for k, v in L.random_weights(L.make_config([layer], width=width), seed=seed).items()}


def test_window_and_causality_of_the_restatement():
    rng = np.random.default_rng(0)
    d, n = 24, 30
    for layer, unit in ((L.delta_pair(heads=2, kv_heads=1, dim=8, vdim=8, size=5), False), (L.lightning_pair(heads=2, kv_heads=1, dim=8, vdim=8, size=5, conv=0), True)):
        w, h = _w(layer), rng.standard_normal((n, d))
        base = O.window_attention(h, w, "l0.mix.left.", layer["mixer"]["left"], 1e-5, unit)
        for changed in (10, 29):
            h2 = h.copy()
            h2[changed] += 1.0
            moved = np.abs(O.window_attention(h2, w, "l0.mix.left.", layer["mixer"]["left"], 1e-5, unit) - base).max(axis=1) > 1e-12
            assert moved[:changed].sum() == 0 and moved[changed:changed + 5].all() and moved[changed + 5:].sum() == 0       # nothing earlier, nothing beyond the window


def test_rotation_of_the_restatement_depends_on_distance_only():
    rng = np.random.default_rng(2)
    q, k = rng.standard_normal((1, 1, 12)), rng.standard_normal((1, 1, 12))
    for interleaved in (True, False):
        rot = {"dims": 8, "base": 50.0}
        rq, rk = (O.rotate(np.repeat(x, 20, axis=0), rot, interleaved)[:, 0] for x in (q, k))
        dots = rq @ rk.T
        for off in (0, 3, -5):
            np.testing.assert_allclose(np.diagonal(dots, off), np.diagonal(dots, off)[0])
        np.testing.assert_allclose(rq[:, 8:], np.repeat(q[0, :, 8:], 20, axis=0))       # the rest passes unchanged
    assert np.abs(O.rotate(np.repeat(q, 5, 0), rot, True) - O.rotate(np.repeat(q, 5, 0), rot, False)).max() > 0.1


def test_recurrences_of_the_restatement():
    rng = np.random.default_rng(3)
    q, k, v = rng.standard_normal((20, 4)), rng.standard_normal((20, 4)), rng.standard_normal((20, 3))
    t = np.arange(20)
    weights = np.where(t[:, None] >= t[None, :], 0.9 ** np.maximum(t[:, None] - t[None, :], 0.0), 0.0)
    np.testing.assert_allclose(O.decayed_attention(q, k, v, 0.9), (weights * (q @ k.T)) @ v)      # the sum over all earlier tokens
    beta, g = rng.uniform(0.1, 0.9, 20), rng.uniform(0.5, 1.0, 20)
    k /= np.linalg.norm(k, axis=1, keepdims=True)
    np.testing.assert_allclose(O.channel_delta_rule(q, k, v, beta, np.repeat(g[:, None], 4, 1)), O.delta_rule(q, k, v, beta, g))   # equal decays: the decay per head
    # a channel that forgets at once: what was stored under that key is gone, what was stored under another stays
    e, dec = np.eye(4), np.ones((3, 4))
    dec[:, 1] = 0.0
    o = O.channel_delta_rule(e[[0, 0, 1]], e[[0, 1, 2]], np.array([[1.0], [2.0], [3.0]]), np.ones(3), dec)
    np.testing.assert_allclose(o[:, 0], [1.0, 1.0, 0.0])


def test_routing_by_groups_of_the_restatement():
    z = np.log(np.array([0.9, 0.1, 0.6, 0.59]) / (1 - np.array([0.9, 0.1, 0.6, 0.59])))       # scores 0.9 0.1 | 0.6 0.59
    w = {"r.router": z[:, None], "r.correction": np.zeros(4)}
    h = np.array([[1.0]])
    r = {"experts": 4, "top": 2, "scale": 2.0, "groups": {"count": 2, "keep": 1}}
    chosen, weight = O.route(h, w, "r.", r)
    assert sorted(chosen[0].tolist()) == [2, 3]                                     # the second group's two best sum to more
    np.testing.assert_allclose(weight[0], 2.0 * np.array([0.6, 0.59]) / 1.19)
    chosen, weight = O.route(h, dict(w, **{"r.correction": np.array([0.5, -0.3, -2.0, -2.0])}), "r.", r)
    assert sorted(chosen[0].tolist()) == [0, 1]                                     # the corrected scores decide about groups too (one of them is negative) ...
    np.testing.assert_allclose(sorted(weight[0]), sorted(2.0 * np.array([0.9, 0.1])))   # ... and stay out of the weights
    chosen, _ = O.route(h, w, "r.", {"experts": 4, "top": 2, "scale": 2.0})
    assert sorted(chosen[0].tolist()) == [0, 2]


def test_clamped_expert_of_the_restatement():
    w = {"e.gate": np.array([[10.0], [-10.0]]), "e.up": np.array([[10.0], [-10.0]]), "e.down": np.eye(2)}
    out = O.clamped_expert(np.array([[1.0]]), w, "e.", 2.0)[0]
    np.testing.assert_allclose(out, [2.0 / (1 + np.exp(-1.702 * 2.0)) * 3.0, -10.0 / (1 + np.exp(17.02)) * -1.0])   # the gate is bounded above only


def test_bench_geometries():
    """The throughput option's sizes are valid models: heads of 128, groups of experts, and tensors under the names the model asks for."""
    import torch

    from simplellminference_b200.bench_nelutar import EXPERTS, SIZES, _state_bytes, _used_params, nelutar_config, random_nelutar_weights
    from simplellminference_b200.config import NelutarConfig
    for size in SIZES.values():
        c = NelutarConfig.from_dict(nelutar_config(size["width"], size["repeats"]))
        assert c.width == size["width"] and [l.type for l in c.layers[:4]] == ["parallel_2", "parallel", "retention", "parallel_2"] and len(c.layers) == 4 * size["repeats"]
        assert all(l.mlp.experts == EXPERTS for l in c.layers[1:4])
    cfg = nelutar_config(256, 1, vocab=64)
    cfg["embedding"]["bigram"]["buckets"] = 31
    w = random_nelutar_weights(cfg, torch.device("cpu"))
    used, total = _used_params(cfg, w)
    assert 0 < used < total and _state_bytes(cfg, 4096) == _state_bytes(cfg, 2048) > 0
    names = set(L.random_weights(cfg, seed=0))
    assert set(w) == names
