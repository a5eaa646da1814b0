"""CPU-side checks of the Lovulix integration: config reader and registry, the rotary frequencies of the package against the
restatement's, and the restatement's own properties (visibility by chunks, causality, the sink, the mix of scores, routing)."""
import os
import sys

import numpy as np
import pytest

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import lovulix_oracle as O  # noqa: E402
import lovulix_testlib as L  # noqa: E402


def test_config_reader(tmp_path):
    from simplellminference_b200.config import ExpertsConfig, LovulixConfig, RotaryConfig, ScoreMixingAttentionConfig, read_model_config
    cfg = L.make_config([L.layer(), L.layer(chunk=None, rot_dims=0, v_mix=False, mlp=L.moe(shared=0)), L.layer(mlp=None)])
    folder = L.write_model(str(tmp_path / "m"), cfg, {"embed": np.zeros((2, 2), np.float32)})
    c = read_model_config(folder)
    assert isinstance(c, LovulixConfig) and (c.vocab, c.width, c.norm_eps, c.logit_scale) == (83, 48, 1e-5, 0.7)
    assert c.layers[0].mixer == ScoreMixingAttentionConfig(4, 2, 16, 12, 0.3, RotaryConfig(8, 1000.0, L.BANDS), 20, True)
    assert c.layers[1].mixer == ScoreMixingAttentionConfig(4, 2, 16, 12, 0.3, None, None, False)
    assert c.layers[0].mlp == ExpertsConfig(5, 0, 2, 12, 20) and c.layers[1].mlp == ExpertsConfig(5, 0, 2, 12, 0) and c.layers[2].mlp is None
    bare = LovulixConfig.from_dict({"architecture": "Lovulix", "vocab": 5, "width": 4, "layers": []})      # what is not named does not exist
    assert (bare.logit_scale, bare.norm_eps) == (1.0, 1e-6)
    for bad, text in ((dict(L.layer(), type="conv"), "unknown mixer type"), (L.layer(mlp={"kind": "dense", "ff": 3}), "not part of this design"),
                      (L.layer(heads=5, kv_heads=2), "do not divide"), (L.layer(dim=8, rot_dims=10), "rotary"), (L.layer(rot_dims=7), "rotary"),
                      (L.layer(mlp=L.moe(experts=2, top=4)), "experts")):
        with pytest.raises(ValueError, match=text):
            LovulixConfig.from_dict(L.make_config([bad]))
    with pytest.raises(ValueError, match="same key/value heads"):
        LovulixConfig.from_dict(L.make_config([L.layer(), L.layer(v_mix=False, vdim=3), L.layer(vdim=16)]))


def test_registry_knows_the_design():
    from simplellminference_b200.config import CONFIG_READERS
    from simplellminference_b200.models import MODEL_CLASSES
    assert all(n in MODEL_CLASSES and n in CONFIG_READERS for n in ("Lovulix", "Kodezen", "Vasosun", "Sopetar", "Munazen"))


def test_band_frequencies_against_the_restatement():
    from simplellminference_b200.layers import band_frequencies
    for dims, base, scaling in ((8, 1000.0, L.BANDS), (128, 500000.0, {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}), (30, 77.0, None),
                                (24, 500.0, {"factor": 8.0, "low": 0.5, "high": 0.75, "original": 64})):
        a, b = band_frequencies(dims, base, scaling), O.band_frequencies(dims, base, scaling)
        np.testing.assert_allclose(a, b, rtol=1e-14)
        if scaling:
            plain = np.array(O.band_frequencies(dims, base, None))
            ratio = plain / np.array(a)
            assert ratio[0] == 1.0 and abs(ratio[-1] - scaling["factor"]) < 1e-12      # both ends of the bands are hit
    band = O.band_frequencies(128, 500000.0, {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192})
    plain = O.band_frequencies(128, 500000.0, None)
    assert any(1.01 < p / f < 7.99 for p, f in zip(plain, band)), "no pair falls between the bands"


def test_chunks_and_causality_of_the_restatement():
    rng = np.random.default_rng(0)
    d, n = 24, 30
    layer = L.layer(heads=2, kv_heads=1, dim=8, vdim=8, chunk=7)
    w = {k: v.astype(np.float64) for k, v in L.random_weights(L.make_config([layer], width=d), seed=1).items()}
    h = rng.standard_normal((n, d))
    base = O.attention(h, w, "l0.mix.", layer["mixer"], 1e-5)[0]
    for at in (13, 14, 16):                                     # the last of a chunk, the first, one in the middle
        h2 = h.copy()
        h2[at] += 1.0
        moved = np.abs(O.attention(h2, w, "l0.mix.", layer["mixer"], 1e-5)[0] - base).max(axis=1) > 1e-12
        assert moved.tolist() == [at <= i < (at // 7 + 1) * 7 for i in range(n)]
    see = O.same_chunk(12, 5)
    assert see[9, 5] and not see[10, 9] and see[4, 0] and not see[4, 5] and O.same_chunk(4, None)[3, 0]


def test_sink_and_mixed_scores_of_the_restatement():
    s, see = np.array([[0.0, 0.0], [1.0, 2.0]]), O.same_chunk(2, None)
    p = O.sink_softmax(s, see, 0.5)
    np.testing.assert_allclose(p[0], [1 / (1 + np.exp(0.5)), 0])
    np.testing.assert_allclose(p[1], np.exp([1.0, 2.0]) / (np.exp(1) + np.exp(2) + np.exp(0.5)))
    rng = np.random.default_rng(1)
    q, k = rng.standard_normal((3, 4, 5)), rng.standard_normal((3, 2, 5))
    T = np.zeros((4, 4))
    T[0, 3], T[1, 0], T[1, 2] = 2.0, 1.0, -1.0
    m = O.mixed_scores(q, k, T, 0.5)
    np.testing.assert_allclose(m[0], q[:, 3] @ k[:, 1].T)                      # head 3 reads key head 1
    np.testing.assert_allclose(m[1], 0.5 * (q[:, 0] @ k[:, 0].T - q[:, 2] @ k[:, 1].T))
    assert np.all(m[2] == 0)


def test_rotation_of_the_restatement():
    x = np.zeros((3, 1, 6))
    x[:, 0, 0] = x[:, 0, 4] = 1.0
    y = O.rotate_halves(x, 4, [1.0, 0.1])
    np.testing.assert_allclose(y[2, 0, [0, 2]], [np.cos(2.0), np.sin(2.0)])    # dimension 0 turns with dimension 2
    np.testing.assert_allclose(y[:, 0, 4], 1.0)                                # beyond the rotary dimensions nothing turns


def test_routing_and_shared_expert_of_the_restatement():
    W = {"m.router": np.array([[0.5, 0.5]]), "m.e0.gate": np.ones((1, 2)), "m.e0.up": np.ones((1, 2)), "m.e0.down": np.ones((2, 1)),
         "m.shared.gate": 2 * np.ones((1, 2)), "m.shared.up": np.ones((1, 2)), "m.shared.down": np.ones((2, 1))}
    mlp = {"router": {"experts": 1, "top": 1}, "expert": {"ff": 1}}
    h = np.array([[2.0, -1.0]])
    s = O.sigmoid(0.5)
    routed = O.silu(s) * s                                                     # silu(s * sum h) * (s * sum h)
    np.testing.assert_allclose(O.experts_ff(h, W, "m.", mlp), np.full((1, 2), routed))
    np.testing.assert_allclose(O.experts_ff(h, W, "m.", dict(mlp, shared={"ff": 1})), np.full((1, 2), routed + O.silu(2.0) * 1.0))


def test_bench_geometries_are_valid_configurations():
    """The sizes of ``bench.py --lovulix`` parse and have the width and depth of the sizes they are compared with."""
    from simplellminference_b200 import bench_kodezen
    from simplellminference_b200.bench_lovulix import SIZES, lovulix_config
    from simplellminference_b200.config import LovulixConfig
    for name, size in SIZES.items():
        cfg = LovulixConfig.from_dict(lovulix_config(size["width"], size["layers"]))
        k = bench_kodezen.SIZES[name]
        assert cfg.width == size["width"] == k["width"] and len(cfg.layers) == size["layers"] == 4 * k["repeats"] and size["prompt"] == k["prompt"]
        assert all(l.mixer.heads * l.mixer.vdim == cfg.width and l.mlp.shared == l.mlp.ff for l in cfg.layers)
