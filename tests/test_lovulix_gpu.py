"""Lovulix on the GPU against the plain float64 restatement (tests/lovulix_oracle.py): every mechanism alone, whole prompts with the stream
after every layer, decoding through the cache, portions down to two tokens, unequal requests in one batch, pages and slots that are freed
and used again, keys that stand out just inside and just outside a chunk of positions (in prompts and in decoding, at page borders) and far
back, other sizes (also values that happen to be equal or 1), and greedy generation through the scheduler and the command lines. Small
random models, made here; fp32 mode is compared tightly, bf16 mode within the rounding of bf16 operands."""
import os
import sys

import numpy as np
import pytest

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import lovulix_oracle as O  # noqa: E402
import lovulix_testlib as L  # noqa: E402

pytestmark = pytest.mark.gpu

F32_TOL = 2e-5     # relative rms of a vector, fp32 mode: one mechanism
F32_MODEL = 5e-5   # logits of a whole model
BF16_MIXER = 3e-2  # one mixer with bf16 operands and a bf16 cache
BF16_MODEL_TYPICAL = 8e-2
EPS = 1e-5
TUNE_SEQ_ATTN_MMA = 9   # sllm_tune key of the tensor-core attention switch

# layers that keep and blend values with one between them that does neither, a layer without feed-forward, one without a shared expert
CFG_A = L.make_config([L.layer(), L.layer(heads=6, kv_heads=3, dim=10, vdim=7, chunk=33, v_mix=False, scaling=None, mlp=L.moe(experts=6, top=3, ff=10, shared=8)),
                       L.layer(chunk=None, mlp=None), L.layer(heads=8, dim=12, rot_dims=12, chunk=50, mlp=L.moe(experts=3, top=1, ff=20, shared=0))])
# values that a model may happen to make equal or 1: one head, chunks of one position, one expert of one, all experts chosen, no rotation
CFG_ONES = L.make_config([L.layer(heads=1, kv_heads=1, dim=32, vdim=32, chunk=1, rot_dims=32, mlp=L.moe(experts=1, top=1, ff=32, shared=32)),
                          L.layer(heads=1, kv_heads=1, dim=1, vdim=32, rot_dims=0, chunk=32, mlp=L.moe(experts=4, top=4, ff=1, shared=1)),
                          L.layer(heads=2, kv_heads=2, dim=16, vdim=1, scale=1.0, rot_dims=2, chunk=64, v_mix=False)], vocab=61, width=32, logit_scale=1.0)
# widths the tensor-core attention and products take, enough tokens in the tests for the tensor-core products
CFG_TC = L.make_config([L.layer(heads=4, kv_heads=2, dim=32, vdim=32, chunk=40, rot_dims=32, mlp=L.moe(experts=6, top=2, ff=32, shared=64)),
                        L.layer(heads=8, kv_heads=2, dim=40, vdim=32, chunk=70, rot_dims=16, mlp=L.moe(experts=4, top=1, ff=64, shared=40)),
                        L.layer(heads=6, kv_heads=2, dim=8, vdim=72, chunk=None, rot_dims=8, v_mix=False, mlp=L.moe(experts=3, top=2, ff=48, shared=32))],
                       width=64, vocab=128)
# sizes that are multiples of nothing
CFG_ODD = L.make_config([L.layer(heads=10, kv_heads=1, dim=6, vdim=13, chunk=45, rot_dims=2, scale=0.7, mlp=L.moe(experts=7, top=4, ff=11, shared=9)),
                         L.layer(heads=9, kv_heads=3, dim=10, vdim=5, chunk=17, rot_dims=6, base=77.0, v_mix=False, mlp=None),
                         L.layer(heads=7, kv_heads=1, dim=34, vdim=13, chunk=101, rot_dims=30, mlp=L.moe(experts=2, top=1, ff=5, shared=23))],
                        vocab=67, width=50, eps=1e-6, logit_scale=2.5)
ALL = [CFG_A, CFG_ONES, CFG_TC, CFG_ODD]
IDS = ["mixed", "ones", "tensorcore", "odd"]


def _engine(tmp_path, cfg, w, dtype="float32", max_tokens=512, max_seqs=4, page_len=32, name="m", **kw):
    from simplellminference_b200.models import build_model
    from simplellminference_b200.seqengine import SequenceEngine
    folder = L.write_model(str(tmp_path / name), cfg, w)
    model = build_model(folder, dtype, "cuda")
    return SequenceEngine(model, max_tokens=max_tokens, max_seqs=max_seqs, page_len=page_len, **kw)


def _logits(eng, slot, toks, want=None):
    want = list(range(len(toks))) if want is None else want
    out = eng.run([(slot, toks, want)])
    return None if out is None else out.cpu().numpy()


def _rel(got, want):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    return float(np.sqrt(((got - want) ** 2).mean()) / max(1e-30, np.sqrt((want ** 2).mean())))


def _w64(w):
    return {k: v.astype(np.float64) for k, v in w.items()}


def _forward(cfg, w, toks, layer_outputs=None):
    return O.forward(cfg, _w64(w), toks, layer_outputs)


# ------------------------------------------------------------------------------------------------ mechanisms alone
def _mixer_stub(layer_cfgs, w, width, dtype="float32", eps=EPS, shares=None):
    """Every layer's mixer on the same rows; ``shares``: what each does with its values (None / "keep" / "blend")."""
    import torch

    from simplellminference_b200 import layers
    from simplellminference_b200.config import BF16, F32, LovulixConfig
    from simplellminference_b200.seqops import Ops
    dev = torch.device("cuda")
    ops = Ops(BF16 if dtype == "bfloat16" else F32)
    wt = {k: torch.tensor(v, device=dev, dtype=torch.bfloat16 if dtype == "bfloat16" else torch.float32) for k, v in w.items()}
    cfg = LovulixConfig.from_dict(L.make_config([dict(lc, mixer=dict(lc["mixer"], v_mix=False)) for lc in layer_cfgs], width=width))
    groups = []
    for i, lc in enumerate(cfg.layers):
        mech = layers.ScoreMixingAttention(lc.mixer, wt, f"l{i}.mix.", ops, dev, eps, 1, (shares or [None] * len(layer_cfgs))[i])
        groups.append(layers.MixerGroup([("mix", mech, 1.0)], ops, dev))

    def fn(step, h, states):
        outs = []
        for g, st in zip(groups, states):
            y = step.scratch("sub_out", step.T * width)
            g.forward(step, h, st, y)
            outs.append(y[:step.T * width].view(step.T, width).clone())
        return outs
    return L.Stub([g.state_spec() for g in groups], fn, ops, dev)


def _oracle_mixer(layer_cfg, w, h, pre="l0.mix.", eps=EPS, v_first=None):
    return O.attention(h.astype(np.float64), _w64(w), pre, layer_cfg["mixer"], eps, v_first)[0]


ALONE = [L.layer(), L.layer(heads=3, kv_heads=3, dim=20, vdim=20, chunk=9, rot_dims=20, scaling=None), L.layer(heads=8, kv_heads=1, dim=8, vdim=40, chunk=64, scale=1.0, rot_dims=2),
         L.layer(heads=6, kv_heads=3, dim=12, vdim=16, chunk=None, rot_dims=0), L.layer(heads=2, kv_heads=2, dim=36, vdim=5, chunk=5), L.layer(heads=5, kv_heads=1, dim=7, vdim=130, chunk=31, rot_dims=6),
         L.layer(heads=12, kv_heads=4, dim=128, vdim=128, chunk=32, rot_dims=64), L.layer(heads=1, kv_heads=1, dim=2, vdim=3, chunk=1, rot_dims=2), L.layer(heads=40, kv_heads=20, dim=4, vdim=4, chunk=48, rot_dims=4),
         L.layer(heads=18, kv_heads=2, dim=16, vdim=16, chunk=33, rot_dims=16)]


@pytest.mark.parametrize("portions", [[75], [33, 2, 15, 16, 1, 1, 1, 1, 5], [1] * 75])
def test_each_mixer_alone(portions):
    rng = np.random.default_rng(5)
    d, T = 48, 75
    for layer_cfg in ALONE:
        w = L.random_weights(L.make_config([layer_cfg], width=d), seed=11)
        h = rng.standard_normal((T, d)).astype(np.float32)
        got = L.feed(_mixer_stub([layer_cfg], w, d), h, portions)[0]
        want = _oracle_mixer(layer_cfg, w, h)
        assert _rel(got, want) < F32_TOL, (layer_cfg["mixer"], _rel(got, want))


@pytest.mark.parametrize("portions", [[80], [40, 2, 37, 1], [5] + [1] * 75], ids=["whole", "portions", "decoded"])
def test_each_mixer_alone_bf16(portions):
    """bf16 matrices, operands and cache; portions of a prompt take the tensor-core form where the head widths allow it (with heads of a
    value head in fours, twos and ones, key rows shorter and longer than a piece and than the ring of pieces, an odd number of value
    tiles), single tokens the form that mixes scores."""
    rng = np.random.default_rng(7)
    d, T = 64, 80
    for layer_cfg in (L.layer(heads=4, kv_heads=2, dim=32, vdim=32, chunk=30), L.layer(heads=8, kv_heads=2, dim=56, vdim=48, chunk=70), L.layer(heads=3, kv_heads=1, dim=16, vdim=24, chunk=None),
                      L.layer(heads=6, kv_heads=2, dim=64, vdim=40, chunk=33), L.layer(heads=16, kv_heads=4, dim=128, vdim=128, chunk=64, rot_dims=128),
                      L.layer(heads=4, kv_heads=4, dim=80, vdim=72, chunk=20), L.layer(heads=3, kv_heads=1, dim=13, vdim=12, chunk=None), L.layer(heads=4, kv_heads=1, dim=32, vdim=136, chunk=17),
                      L.layer(heads=18, kv_heads=2, dim=20, vdim=16, chunk=33)):
        w = L.random_weights(L.make_config([layer_cfg], width=d), seed=13)
        h = L.bf16_round(rng.standard_normal((T, d))).astype(np.float32)
        got = L.feed(_mixer_stub([layer_cfg], w, d, dtype="bfloat16"), h, portions)[0]
        want = _oracle_mixer(layer_cfg, w, h)
        assert _rel(got, want) < BF16_MIXER, (layer_cfg["mixer"], _rel(got, want))


def test_the_two_bf16_forms_agree_on_one_step():
    """A step with portions on the tensor cores and the same step with the tensor-core form switched off: the same numbers up to the
    rounding of the mixed queries."""
    rng = np.random.default_rng(17)
    d, T = 64, 150
    layer_cfg = L.layer(heads=8, kv_heads=2, dim=56, vdim=48, chunk=70)
    w = L.random_weights(L.make_config([layer_cfg], width=d), seed=14)
    h = L.bf16_round(rng.standard_normal((T, d))).astype(np.float32)
    stub = _mixer_stub([layer_cfg], w, d, dtype="bfloat16")
    tensor = L.feed(stub, h, [100, 50])[0]
    lib = stub.ops.lib
    assert lib.sllm_tune(TUNE_SEQ_ATTN_MMA, 0) == 0
    try:
        stub = _mixer_stub([layer_cfg], w, d, dtype="bfloat16")
        plain = L.feed(stub, h, [100, 50])[0]
    finally:
        lib.sllm_tune(TUNE_SEQ_ATTN_MMA, 1)
    assert 0 < _rel(tensor, plain) < 1e-2


def _standing_out(d, H, chunk):
    """A layer and weights in which the query of a position reads the first third of its input row and the key the second third, through
    the same map, unrotated: a query row whose first third repeats the second third of an earlier row gives that position (and no other,
    itself included) a score far above the rest. The heads' scores are mixed by a full matrix of positive numbers."""
    t = d // 3
    layer = L.layer(heads=H, kv_heads=H // 2, dim=16, vdim=16, scale=3.0, chunk=chunk, rot_dims=0)
    w = L.random_weights(L.make_config([layer], width=d), seed=3)
    a = w["l0.mix.k"][:, :t].copy()
    w["l0.mix.q"][:] = 0.0
    w["l0.mix.k"][:] = 0.0
    # the query heads of a group read through their key head's map
    w["l0.mix.q"][:, :t] = np.repeat(a.reshape(H // 2, 1, 16, t), 2, axis=1).reshape(H * 16, t)
    w["l0.mix.k"][:, t:2 * t] = a
    for n in ("q", "k"):
        w[f"l0.mix.{n}.norm"][:] = 1.0
    w["l0.mix.talk"] = L.bf16_round(0.6 * np.eye(H) + 0.2 * np.abs(np.random.default_rng(1).standard_normal((H, H))))
    w["l0.mix.sink"][:] = 0.0
    return layer, w, t


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("decode", [False, True], ids=["prompt", "decoded"])
def test_keys_just_inside_and_outside_the_chunk(decode, dtype):
    """The key input of an earlier position is repeated as the query input of a later one: when that position is the first of the query's
    chunk the query's output is essentially its value; when it is the last of the chunk before, it is something else — the restatement
    says so and the engine has to follow it. Chunks that end inside, at and just after a border of pages and tiles of 32; queries at the
    chunk's start, middle and end."""
    rng = np.random.default_rng(9)
    d, T, H = 48, 150, 4
    seen = []
    for chunk in (37, 32, 33, 64, 75):
        layer, w, t = _standing_out(d, H, chunk)
        stub = _mixer_stub([layer], w, d, dtype)
        for query in (149, 2 * chunk - 1, chunk + 1, chunk + 20):
            if query >= T:
                continue
            first = query // chunk * chunk
            for key, visible in ((first, True), (first - 1, False), (max(first, query - 1), True), (0, first == 0)):
                if key < 0 or key == query:
                    continue
                h = L.bf16_round(rng.standard_normal((T, d))).astype(np.float32)
                h[key, t:2 * t] *= 2.0                          # a long key: no other key's chance alignment with the query comes close
                h[query, :t] = h[key, t:2 * t]
                want = _oracle_mixer(layer, w, h)
                got = L.feed(stub, h, [query] + [1] * (T - query) if decode else [T])[0]
                assert _rel(got, want) < (F32_TOL if dtype == "float32" else BF16_MIXER), (chunk, query, key, _rel(got, want))
                # scores far apart turn rounding into differences of the weights: the one row is held a little looser
                assert _rel(got[query], want[query]) < (5 * F32_TOL if dtype == "float32" else 0.1), (chunk, query, key, _rel(got[query], want[query]))
                base = h.copy()
                base[key] = rng.standard_normal(d)
                seen.append((visible, _rel(_oracle_mixer(layer, w, base)[query], want[query])))
    shown = sorted(r for v, r in seen if v)
    assert shown[0] > 0.05 and shown[len(shown) // 2] > 0.3, "a visible repeated position does not stand out: the test would not notice a lost key"
    assert max(r for v, r in seen if not v) < 1e-6, "a hidden position changes the restatement's result"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("decode", [False, True], ids=["prompt", "decoded"])
def test_a_key_far_back_among_hundreds(decode, dtype):
    """One position hundreds of tokens back (the first token, one at a page border, one in the middle of a page) towers over all others."""
    rng = np.random.default_rng(10)
    d, T, H = 48, 420, 4
    layer, w, t = _standing_out(d, H, 421)
    stub = _mixer_stub([layer], w, d, dtype)
    shown = []
    for query, key in ((419, 20), (400, 64), (330, 0), (399, 31)):
        h = L.bf16_round(rng.standard_normal((T, d))).astype(np.float32)
        h[key, t:2 * t] *= 2.0
        h[query, :t] = h[key, t:2 * t]
        want = _oracle_mixer(layer, w, h)
        got = L.feed(stub, h, [320] + [1] * (T - 320) if decode else [200, 220])[0]
        assert _rel(got, want) < (F32_TOL if dtype == "float32" else BF16_MIXER), (query, key, _rel(got, want))
        base = h.copy()
        base[key] = rng.standard_normal(d)
        shown.append(_rel(_oracle_mixer(layer, w, base)[query], want[query]))
    assert min(shown) > 0.3, "the far position does not stand out"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_scores_of_other_heads_are_mixed_before_the_softmax(dtype):
    """With a mixing matrix that gives head 0 the scores of the last head only (a query of another key head), head 0 weighs ITS values by
    that head's attention; and mixing before the softmax differs visibly from mixing the weights after it."""
    rng = np.random.default_rng(12)
    d, T = 48, 60
    layer = L.layer(heads=4, kv_heads=2, dim=16, vdim=16, chunk=None, scale=1.0)
    w = L.random_weights(L.make_config([layer], width=d), seed=5)
    talk = np.eye(4, dtype=np.float32)
    talk[0] = [0, 0, 0, 1]
    w["l0.mix.talk"] = talk
    h = L.bf16_round(rng.standard_normal((T, d))).astype(np.float32)
    want = _oracle_mixer(layer, w, h)
    for portions in ([T], [20] + [1] * 40):
        assert _rel(L.feed(_mixer_stub([layer], w, d, dtype), h, portions)[0], want) < (F32_TOL if dtype == "float32" else BF16_MIXER)
    plain = dict(w)
    plain["l0.mix.talk"] = np.eye(4, dtype=np.float32)
    assert _rel(_oracle_mixer(layer, plain, h), want) > 0.05
    # a matrix of halves: mixed before the softmax every head sees the sum of two heads' scores
    w["l0.mix.talk"] = np.full((4, 4), 0.5, np.float32)
    want = _oracle_mixer(layer, w, h)
    assert _rel(L.feed(_mixer_stub([layer], w, d, dtype), h, [T])[0], want) < (F32_TOL if dtype == "float32" else BF16_MIXER)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sink_in_the_denominator(dtype):
    """Sinks above, among and far below the scores, different for every head, also for a sequence's first tokens (one visible key): they
    count once, whatever the number of shares the keys are cut into."""
    rng = np.random.default_rng(13)
    d, T = 48, 130
    layer = L.layer(heads=4, kv_heads=2, dim=16, vdim=16, chunk=100)
    w = L.random_weights(L.make_config([layer], width=d), seed=6)
    h = L.bf16_round(rng.standard_normal((T, d))).astype(np.float32)
    for sink in ([4.0, -1.0, 0.0, 2.0], [30.0, -30.0, 12.0, 1.0]):
        w["l0.mix.sink"] = np.array(sink, np.float32)
        want = _oracle_mixer(layer, w, h)
        for portions in ([T], [2, 60] + [1] * 68):
            got = L.feed(_mixer_stub([layer], w, d, dtype), h, portions)[0]
            assert _rel(got, want) < (F32_TOL if dtype == "float32" else BF16_MIXER), (sink, portions[:2], _rel(got, want))
    w["l0.mix.sink"] = np.array([0.0, -1.0, 0.0, 2.0], np.float32)
    assert _rel(_oracle_mixer(layer, w, h), want) > 0.05


def test_norm_over_the_whole_projection():
    """One query and key head much longer than the others: the norm over all heads at once keeps that ratio, a norm per head would not."""
    rng = np.random.default_rng(15)
    d, T = 48, 50
    layer = L.layer(heads=4, kv_heads=2, dim=16, vdim=16, chunk=None)
    w = L.random_weights(L.make_config([layer], width=d), seed=7)
    w["l0.mix.q"][16:32] *= 8.0
    w["l0.mix.k"][16:32] *= 8.0
    h = rng.standard_normal((T, d)).astype(np.float32)
    want = _oracle_mixer(layer, w, h)
    for portions in ([T], [1] * T):
        assert _rel(L.feed(_mixer_stub([layer], w, d), h, portions)[0], want) < F32_TOL
    per_head = dict(w)
    per_head["l0.mix.q"], per_head["l0.mix.k"] = w["l0.mix.q"].copy(), w["l0.mix.k"].copy()
    per_head["l0.mix.q"][16:32] /= 8.0
    per_head["l0.mix.k"][16:32] /= 8.0
    assert _rel(_oracle_mixer(layer, per_head, h), want) > 0.05


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_values_blended_with_the_first_layers(dtype):
    """Three mixers on the same rows: the first keeps its values, the second blends them into its own (other head counts and widths of q and
    k), the third neither; the blended values are what the cache holds, so decoded tokens read them for earlier tokens too."""
    rng = np.random.default_rng(16)
    d, T = 48, 70
    layers = [L.layer(heads=4, kv_heads=2, vdim=16), L.layer(heads=6, kv_heads=2, dim=8, vdim=16, chunk=31), L.layer(heads=4, kv_heads=4, vdim=16)]
    w = L.random_weights(L.make_config(layers, width=d), seed=8)
    w["l1.mix.vmix"] = np.float32(0.75)
    h = L.bf16_round(rng.standard_normal((T, d))).astype(np.float32)
    W, eps = _w64(w), EPS
    first, kept = O.attention(h, W, "l0.mix.", layers[0]["mixer"], eps)
    want = [first, O.attention(h, W, "l1.mix.", layers[1]["mixer"], eps, kept)[0], O.attention(h, W, "l2.mix.", layers[2]["mixer"], eps)[0]]
    assert _rel(O.attention(h, W, "l1.mix.", layers[1]["mixer"], eps)[0], want[1]) > 0.05
    for portions in ([T], [30, 2] + [1] * 38):
        got = L.feed(_mixer_stub(layers, w, d, dtype, shares=["keep", "blend", None]), h, portions)
        for a, b in zip(got, want):
            assert _rel(a, b) < (F32_TOL if dtype == "float32" else BF16_MIXER), (portions[:2], _rel(a, b))


def test_rotation_far_from_the_start():
    """Positions up to 600 with frequencies on both sides of the bands and inside the blend: the angle's error does not grow."""
    rng = np.random.default_rng(18)
    d, T = 48, 600
    for scaling in (L.BANDS, {"factor": 8.0, "low": 0.5, "high": 0.75, "original": 64}, None):
        layer = L.layer(heads=2, kv_heads=1, dim=32, vdim=8, chunk=None, rot_dims=24, base=500.0, scaling=scaling)
        w = L.random_weights(L.make_config([layer], width=d), seed=9)
        h = rng.standard_normal((T, d)).astype(np.float32)
        want = _oracle_mixer(layer, w, h)
        got = L.feed(_mixer_stub([layer], w, d), h, [580] + [1] * 20)[0]
        assert _rel(got[-100:], want[-100:]) < F32_TOL, (scaling, _rel(got[-100:], want[-100:]))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_chunks_in_the_plain_attention_kernels(dtype):
    """The chunk option of the attention launch without mixed scores (both bodies: portions of bf16 pools run on the tensor cores), with the
    merge's gate per column and its bf16 rows."""
    import torch

    from simplellminference_b200.config import BF16, F32
    from simplellminference_b200.seqops import Ops
    rng, dev, ops = np.random.default_rng(19), torch.device("cuda"), Ops(BF16 if dtype == "bfloat16" else F32)
    H, G, dk, dv, T = 4, 2, 16, 24, 110
    width = H * dk + G * dk + G * dv + H * dv
    rows = L.bf16_round(rng.standard_normal((T, width))).astype(np.float32)
    r64 = rows.astype(np.float64)
    q, k = r64[:, :H * dk].reshape(T, H, dk), r64[:, H * dk:(H + G) * dk].reshape(T, G, dk)
    v, gate = r64[:, (H + G) * dk:(H + G) * dk + G * dv].reshape(T, G, dv), r64[:, (H + G) * dk + G * dv:]
    for chunk in (1, 20, 32, 45, 200):
        opts = ops.attention_options(chunk=chunk)
        want = np.stack([O.sink_softmax(q[:, hh] @ k[:, hh // 2].T * 0.5, O.same_chunk(T, chunk), -np.inf) @ v[:, hh // 2] for hh in range(H)], axis=1)
        want = want.reshape(T, H * dv) * O.sigmoid(gate)

        def fn(step, h, states):
            n, base = step.T, h.data_ptr()
            ops.unit_kv(step.b, base, width, H, dk, base + 4 * H * dk, width, G, base + 4 * (H + G) * dk, width, dv, 0.0, 0, None, 0, 0.0, states[0]["k"], states[0]["v"], step.st)
            ws = step.scratch("ws", n * H * step.nsplit * (dv + 2))
            ops.attention(step.b, base, width, H, G, dk, dv, 0.5, states[0]["k"], states[0]["v"], step.nsplit, ws, step.st, opts=opts)
            out, out16 = step.scratch("out", n * H * dv), torch.zeros(n, H * dv, dtype=torch.bfloat16, device=dev)
            ops.attention_finish(step.b, ws, step.nsplit, H, dv, None, 0, base + 4 * ((H + G) * dk + G * dv), width, out, H * dv, step.st, gate_channels=True, out16=out16)
            return [out[:n * H * dv].view(n, H * dv), out16.float()]
        stub = L.Stub([{"pages": [("k", G, dk), ("v", G, dv)], "slots": []}], fn, ops, dev)
        for portions in ([T], [30, 2, 33, 1, 44], [60] + [1] * 50):
            got = L.feed(stub, rows, portions)
            assert _rel(got[0], want) < (F32_TOL if dtype == "float32" else 1e-2), (chunk, portions[:2], _rel(got[0], want))
            assert _rel(got[1], want) < 1e-2


def test_seam_with_channel_weights_on_the_sublayers_output():
    """x + w * y / rms(y), the stream as bf16 operand rows, and the model's last norm behind it; rows of a multiple of four floats (in
    registers, one to four groups of channels a thread) and others."""
    import torch

    from simplellminference_b200.config import F32
    from simplellminference_b200.seqops import Ops
    rng, dev, ops = np.random.default_rng(2), torch.device("cuda"), Ops(F32)
    for d, T in ((48, 40), (50, 9), (1000, 70), (4100, 66), (2048, 3), (6144, 2), (9000, 1)):
        x, y = (3 * rng.standard_normal((T, d))).astype(np.float32), rng.standard_normal((T, d)).astype(np.float32)
        pw, nw = (0.5 + 0.3 * rng.standard_normal(d)).astype(np.float32), (1 + 0.3 * rng.standard_normal(d)).astype(np.float32)
        eps = 1e-5
        want = x.astype(np.float64) + O.rms_norm(y, pw, eps)
        normed = 0.25 * O.rms_norm(want, nw, eps)
        pwt, nwt = torch.tensor(pw, device=dev), torch.tensor(nw, device=dev)

        def fn(step, h, states):
            n = step.T
            xy = h.view(n, 2 * d)
            xi, yi = xy[:, :d].contiguous(), xy[:, d:].contiguous()
            xo, xo2, ho, x16 = torch.empty_like(xi), torch.empty_like(xi), torch.empty_like(xi), torch.zeros(n, d, dtype=torch.bfloat16, device=dev)
            ops.seam(step.b, xi, d, step.st, x_out=xo, y=yi, post_w=pwt, eps=eps, h16=x16)
            ops.seam(step.b, xi, d, step.st, x_out=xo2, y=yi, post_w=pwt, eps=eps, pre_g=0.25, pre_w=nwt, h=ho)
            return [xo, xo2, ho, x16.float()]
        got = L.feed(L.Stub([{"pages": [], "slots": []}], fn, ops, dev), np.concatenate([x, y], axis=1), [T])
        assert _rel(got[0], want) < 1e-6 and _rel(got[1], want) < 1e-6 and _rel(got[2], normed) < 2e-6, (d, T)
        assert np.array_equal(got[3], L.bf16_round(got[0])), (d, T)


def _ff_stub(mlp, w, d, dtype="float32"):
    import torch

    from simplellminference_b200 import layers
    from simplellminference_b200.config import BF16, F32, LovulixConfig
    from simplellminference_b200.seqops import Ops
    dev, ops = torch.device("cuda"), Ops(BF16 if dtype == "bfloat16" else F32)
    wt = {k: torch.tensor(v, device=dev, dtype=torch.bfloat16 if dtype == "bfloat16" else torch.float32) for k, v in w.items()}
    c = LovulixConfig.from_dict(L.make_config([L.layer(mlp=mlp)], width=d)).layers[0].mlp
    ff = layers.ExpertsFeedForward(c, wt, "l0.mlp.", ops, dev, activation=2, gated=True, sigmoid_scores=True, scale_input=True)

    def fn(step, h, states):
        y = step.scratch("sub_out", step.T * d)
        ff.forward(step, h, y)
        return [y[:step.T * d].view(step.T, d)]
    return L.Stub([{"pages": [], "slots": []}], fn, ops, dev), ff


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_experts_beside_a_shared_one_in_every_form(dtype, monkeypatch):
    """All experts as two wide products, tokens gathered per expert, and experts chosen on the device in steps of few tokens: the shared
    expert rides along in each, with a width of its own, and the three give the restatement's numbers."""
    from simplellminference_b200 import layers
    F = layers.ExpertsFeedForward
    rng, d = np.random.default_rng(14), 64
    tol = F32_TOL if dtype == "float32" else BF16_MIXER
    for mlp in (L.moe(experts=6, top=2, ff=32, shared=48), L.moe(experts=12, top=1, ff=24, shared=24), L.moe(experts=9, top=3, ff=17, shared=5), L.moe(experts=5, top=2, ff=40, shared=0),
                L.moe(experts=1, top=1, ff=8, shared=16)):
        w = L.random_weights(L.make_config([L.layer(mlp=mlp)], width=d), seed=5)
        stub, ff = _ff_stub(mlp, w, d, dtype)
        for T, form in ((150, "every"), (150, "gathered"), (3, "every"), (2, "indexed"), (1, "indexed")):
            h = L.bf16_round(2 * rng.standard_normal((T, d))).astype(np.float32)
            monkeypatch.setattr(F, "gather_min_tokens", 64 if form == "gathered" else 10 ** 9)
            monkeypatch.setattr(F, "gather_launch_cost", 0.0)
            monkeypatch.setattr(F, "index_launch_cost", 0.0 if form == "indexed" else 1e9)
            possible = mlp["router"]["top"] < mlp["router"]["experts"]
            if form == "gathered":
                assert ff._gathered_pays(T) == possible
            if form == "indexed":
                assert ff._indexed_pays(T) == (possible and T * mlp["router"]["top"] < mlp["router"]["experts"])
            want = O.experts_ff(h, _w64(w), "l0.mlp.", mlp)
            got = L.feed(stub, h, [T])[0]
            assert _rel(got, want) < tol, (mlp, form, T, _rel(got, want))


def test_score_multiplies_the_routed_experts_input_and_not_the_shared_ones():
    rng, d, T = np.random.default_rng(8), 40, 20
    mlp = L.moe(experts=4, top=2, ff=16, shared=24)
    w = L.random_weights(L.make_config([L.layer(mlp=mlp)], width=d), seed=3)
    h = (2 * rng.standard_normal((T, d))).astype(np.float64)
    want = O.experts_ff(h, _w64(w), "l0.mlp.", mlp)
    chosen, score = O.route(h, _w64(w), "l0.mlp.", 2)
    other = O.glu(h, _w64(w), "l0.mlp.shared.")
    for t in range(T):
        for e, s in zip(chosen[t], score[t]):
            other[t] += s * O.glu(h[t:t + 1], _w64(w), f"l0.mlp.e{int(e)}.")[0]
    assert _rel(other, want) > 0.02
    stub, _ = _ff_stub(mlp, w, d)
    assert _rel(L.feed(stub, h.astype(np.float32), [T])[0], want) < F32_TOL


# ------------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("cfg", ALL, ids=IDS)
def test_whole_prompt_matches_oracle_fp32_and_layers(tmp_path, cfg):
    w = L.random_weights(cfg, seed=1)
    toks = np.random.default_rng(2).integers(0, cfg["vocab"], size=140).tolist()
    taps_want = []
    want = _forward(cfg, w, toks, taps_want)
    eng = _engine(tmp_path, cfg, w)
    taps = []
    got = eng.run([(eng.admit(), toks, list(range(len(toks))))], tap=lambda i, x: taps.append((i, x.clone().cpu().numpy()))).cpu().numpy()
    assert [i for i, _ in taps] == list(range(len(cfg["layers"])))
    for (i, a), b in zip(taps, taps_want):
        assert _rel(a, b) < F32_MODEL, (i, _rel(a, b))
    assert L.logit_error(got, want).max() < F32_MODEL
    # the logits' factor is part of the logits (the error measure alone would not see it)
    assert abs(np.std(got) / np.std(want) - 1) < 1e-4


@pytest.mark.parametrize("cfg", [CFG_A, CFG_TC, CFG_ODD], ids=["mixed", "tensorcore", "odd"])
def test_bf16_mode_within_operand_rounding(tmp_path, cfg):
    w = L.random_weights(cfg, seed=3)
    toks = np.random.default_rng(4).integers(0, cfg["vocab"], size=150).tolist()
    want = _forward(cfg, w, toks)
    eng = _engine(tmp_path, cfg, w, dtype="bfloat16")
    s = eng.admit()
    whole = _logits(eng, s, toks)
    eng.release(s)
    s = eng.admit()
    cut = np.concatenate([_logits(eng, s, toks[:100]), _logits(eng, s, toks[100:102])] + [_logits(eng, s, toks[p:p + 1]) for p in range(102, 150)])
    # a choice of experts that is a near tie may fall the other way: the typical position is held to the rounding, outliers are few
    for got in (whole, cut):
        e = L.logit_error(got, want)
        assert np.median(e) < BF16_MODEL_TYPICAL and (e > 0.3).mean() < 0.1, (np.median(e), (e > 0.3).mean())
    e = L.logit_error(cut, whole)
    assert np.median(e) < BF16_MODEL_TYPICAL, np.median(e)


@pytest.mark.parametrize("cfg", ALL, ids=IDS)
def test_prefill_against_token_by_token_and_portions(tmp_path, cfg):
    w = L.random_weights(cfg, seed=5)
    toks = np.random.default_rng(6).integers(0, cfg["vocab"], size=120).tolist()
    want = _forward(cfg, w, toks)
    eng = _engine(tmp_path, cfg, w)
    for portions in ([1] * 120, [2] * 60, [31, 2, 33, 1, 1, 40, 12], [64, 56], [119, 1], [3, 1, 2, 114]):
        s, outs, p = eng.admit(), [], 0
        for n in portions:
            outs.append(_logits(eng, s, toks[p:p + n]))
            p += n
        eng.release(s)
        assert L.logit_error(np.concatenate(outs), want).max() < F32_MODEL, portions[:3]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cfg", [CFG_A, CFG_TC], ids=["mixed", "tensorcore"])
def test_unequal_requests_in_one_batch_and_reuse_of_pages_and_slots(tmp_path, cfg, dtype):
    """Seven requests of unequal length through three slots and ten pages of 32: portions of prompts beside single tokens of others, every
    request's logits equal the restatement's of that request alone; pages and slots go from finished requests to new ones."""
    w = L.random_weights(cfg, seed=7)
    rng = np.random.default_rng(8)
    lens = [70, 33, 5, 96, 64, 1, 47]
    reqs = [rng.integers(0, cfg["vocab"], size=n).tolist() for n in lens]
    want = [_forward(cfg, w, r) for r in reqs]
    eng = _engine(tmp_path, cfg, w, dtype=dtype, max_tokens=320, max_seqs=3, page_len=32)
    waiting, slots, fed, got = list(range(len(reqs))), {}, [0] * len(reqs), [[] for _ in reqs]
    used_slots, page_users, step = [], {}, 0
    sizes = [17, 2, 32, 5, 40, 3]
    while waiting or slots:
        while waiting and len(slots) < 3 and eng.free_pages >= -(-lens[waiting[0]] // 32) + sum(-(-lens[i] // 32) - eng.pages.held(s) for i, s in slots.items()):
            i = waiting.pop(0)
            slots[i] = eng.admit()
            used_slots.append(slots[i])
        entries, order = [], []
        for i, s in slots.items():
            left = lens[i] - fed[i]
            n = 1 if (fed[i] > lens[i] // 2) else min(left, sizes[(step + i) % len(sizes)])   # portions first, single tokens later
            entries.append((s, reqs[i][fed[i]:fed[i] + n], list(range(n))))
            order.append((i, n))
        out = eng.run(entries).cpu().numpy()
        table = eng.pages.table()
        for i, sl in slots.items():
            for pg in table[sl]:
                if pg >= 0:
                    page_users.setdefault(int(pg), set()).add(i)
        r = 0
        for i, n in order:
            got[i].append(out[r:r + n])
            r += n
            fed[i] += n
        for i in [i for i in slots if fed[i] == lens[i]]:
            eng.release(slots.pop(i))
        step += 1
    assert len(used_slots) > len(set(used_slots)), "no slot was used twice: the test does not test reuse"
    assert eng.free_pages == 10 and any(len(u) > 1 for u in page_users.values()), "no page went from one request to another"
    for i in range(len(reqs)):
        e = L.logit_error(np.concatenate(got[i]), want[i])
        assert (e.max() if dtype == "float32" else np.median(e)) < (F32_MODEL if dtype == "float32" else BF16_MODEL_TYPICAL), (i, e.max())


def test_long_decoding_over_page_and_chunk_borders(tmp_path):
    cfg = L.make_config([L.layer(chunk=50), L.layer(chunk=130, mlp=L.moe(experts=7, top=1, ff=16)), L.layer(chunk=64, v_mix=False), L.layer(chunk=None)])
    w = L.random_weights(cfg, seed=8)
    toks = np.random.default_rng(4).integers(0, cfg["vocab"], size=330).tolist()
    want = _forward(cfg, w, toks)
    eng = _engine(tmp_path, cfg, w, max_tokens=384, page_len=64)
    s = eng.admit()
    outs = [_logits(eng, s, toks[:45])] + [_logits(eng, s, toks[p:p + 1]) for p in range(45, 330)]
    assert eng.graph_replays > 200
    assert L.logit_error(np.concatenate(outs), want).max() < F32_MODEL


def test_first_tokens_of_a_sequence_after_a_used_slot(tmp_path):
    """A slot and pages that held a long request serve the next one: its first tokens equal the restatement's."""
    w = L.random_weights(CFG_A, seed=9)
    rng = np.random.default_rng(10)
    eng = _engine(tmp_path, CFG_A, w, max_seqs=1, max_tokens=96)
    for n in (90, 4, 1, 2, 35):
        toks = rng.integers(0, CFG_A["vocab"], size=n).tolist()
        s = eng.admit()
        got = np.concatenate([_logits(eng, s, toks[:1]), _logits(eng, s, toks[1:])]) if n > 1 else _logits(eng, s, toks)
        eng.release(s)
        assert L.logit_error(got, _forward(CFG_A, w, toks)).max() < F32_MODEL, n


def _follows_greedy(cfg, w, prompt, produced):
    seq = list(prompt)
    for k, tok in enumerate(produced):
        lg = _forward(cfg, w, seq)[-1]
        order = np.argsort(lg)
        close = lg[order[-1]] - lg[order[-2]] <= 1e-3 * np.abs(lg).max()      # a near tie may fall either way: follow the engine
        assert tok == int(order[-1]) or (close and tok == int(order[-2])), (prompt[:4], k)
        seq.append(tok)


def test_greedy_generation_through_the_scheduler(tmp_path):
    """Requests of unequal length through ContinuousBatcher over SequenceDecoder (prompts in portions beside decoding requests, more
    requests than slots): every request's tokens are the restatement's greedy continuation of that prompt alone."""
    from simplellminference_b200.scheduler import ContinuousBatcher
    from simplellminference_b200.seqengine import SequenceDecoder
    cfg = CFG_A
    w = L.random_weights(cfg, seed=12)
    rng = np.random.default_rng(13)
    prompts = [rng.integers(0, cfg["vocab"], size=n).tolist() for n in (5, 40, 1, 23, 64, 7)]
    new = 10
    eng = _engine(tmp_path, cfg, w, max_tokens=6 * 32, max_seqs=3, page_len=32)
    cb = ContinuousBatcher(SequenceDecoder(eng, prefill_chunk=16), chunk=4)
    ids = [cb.submit(p, new) for p in prompts]
    out = cb.run()
    assert cb.stats.max_live == 3 and eng.free_pages == 6
    for rid, p in zip(ids, prompts):
        got = [int(t) for t in out[rid]]
        assert got[:len(p) - 1] == p[1:]
        _follows_greedy(cfg, w, p, got[len(p) - 1:])


def test_trace_replayer_command(tmp_path):
    """bin/trace_run end to end on a Lovulix folder: the model class comes from config.json."""
    import json
    import subprocess
    cfg = CFG_ODD
    w = L.random_weights(cfg, seed=15)
    folder = L.write_model(str(tmp_path / "model"), cfg, w)
    rng = np.random.default_rng(16)
    a, b = rng.integers(0, cfg["vocab"], size=70).tolist(), rng.integers(0, cfg["vocab"], size=9).tolist()
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[30:31], "want": [0]}, {"id": "b", "tokens": b, "want": [8]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[31:], "want": [38]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "c", "tokens": b, "want": [0, 8]}], "end": ["c"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out_dir = tmp_path / "out"
    for dtype, tol in (("float32", F32_MODEL), ("bfloat16", 1e-1)):
        r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out_dir), "--max-tokens", "128"],
                           input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
        wa, wb = _forward(cfg, w, a), _forward(cfg, w, b)
        V = cfg["vocab"]
        got = [np.fromfile(out_dir / f"{n}.f32", dtype="<f4").reshape(-1, V) for n in range(4)]
        assert L.logit_error(got[0], wa[[0, 29]]).max() < tol and L.logit_error(got[1], np.stack([wa[30], wb[8]])).max() < tol
        assert L.logit_error(got[2], wa[[69]]).max() < tol and L.logit_error(got[3], wb[[0, 8]]).max() < tol


def test_generation_command_line(tmp_path):
    """python -m simplellminference_b200.generate on a Lovulix folder: registry, engine, scheduler, device arg-max."""
    import json
    import subprocess
    cfg = CFG_TC
    w = L.random_weights(cfg, seed=21)
    folder = L.write_model(str(tmp_path / "model"), cfg, w)
    prompts = [[3, 1, 4, 1, 5, 9, 2, 6], [7]]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cmd = [sys.executable, "-m", "simplellminference_b200.generate", "--model", folder, "--dtype", "float32", "--max-new-tokens", "6", "--prefill-chunk", "3"]
    for p in prompts:
        cmd += ["--prompt", ",".join(str(t) for t in p)]
    r = subprocess.run(cmd, cwd=root, capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    lines = [json.loads(ln) for ln in r.stdout.splitlines() if ln.startswith("{")]
    assert [ln["prompt"] for ln in lines] == prompts
    for ln in lines:
        assert len(ln["tokens"]) == 6
        _follows_greedy(cfg, w, ln["prompt"], ln["tokens"])
