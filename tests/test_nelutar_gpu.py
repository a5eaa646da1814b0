"""Nelutar on the GPU against the plain float64 restatement (tests/nelutar_oracle.py): every mechanism alone, whole prompts with the
stream after every layer, decoding through the cache and the recurrent state, portions down to two tokens, unequal requests in one batch,
pages and slots that are freed and used again, keys that stand out just inside and just outside the windows (in prompts and in decoding, at
page borders) and far back, long memories of the states, other sizes (also values that happen to be equal or 1), and greedy generation
through the scheduler and the command lines. Small random models, made here; fp32 mode is compared tightly, bf16 mode within the rounding
of bf16 operands."""
import os
import sys

import numpy as np
import pytest

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import nelutar_oracle as O  # noqa: E402
import nelutar_testlib as L  # noqa: E402

pytestmark = pytest.mark.gpu

F32_TOL = 2e-5     # relative rms of a vector, fp32 mode: one mechanism
F32_MODEL = 5e-5   # logits of a whole model
BF16_TOL = 1e-1    # bf16 operands of the products: worst position of a shallow model
BF16_MIXER = 3e-2  # one mixer with bf16 operands and a bf16 cache
BF16_MODEL_TYPICAL = 8e-2
EPS = 1e-5

# every mixer and both feed-forwards, a layer without one, layers that run again with the weights of an earlier one
_A = [L.lightning_pair(), L.delta_pair(mlp=L.moe()), L.retention_layer(mlp=L.moe(experts=6, top=2, groups=3, keep=1, shared=0)),
      L.delta_pair(size=33, rheads=2, rkv=2, conv=2, mlp=None), L.lightning_pair(heads=6, kv_heads=3, size=50, conv=2, mlp=L.moe(groups=0, top=4))]
CFG_A = L.make_config(_A[:3] + [L.again(_A, 1)] + _A[3:4] + _A[4:] + [L.again(_A, 0), L.again(_A, 2)])
# values that a model may happen to make equal or 1: one head, one tap, a window of one position and none at all, one expert, one group, groups
# of one expert, no rotation, every dimension rotated, a decay of one, one bucket
CFG_ONES = L.make_config([L.delta_pair(heads=1, kv_heads=1, dim=32, vdim=32, size=1, rot_dims=32, rheads=1, rkv=1, rdim=32, rvdim=32, conv=1,
                                       mlp=L.moe(experts=1, top=1, ff=32, groups=1, keep=1, scale=1.0, shared=32, limit=1.0, shared_limit=1.0)),
                          L.lightning_pair(heads=2, kv_heads=2, dim=16, vdim=16, size=None, rot_dims=0, conv=1, softcap=0.0, rheads=1, rdim=32, rvdim=32, left=1.0, right=1.0,
                                           mlp=L.moe(experts=4, top=2, groups=4, keep=2)),
                          L.retention_layer(heads=1, dim=32, vdim=32, rot_dims=32, decay=[1.0], mlp=L.dense(32)),
                          L.retention_layer(heads=2, dim=1, vdim=1, rot_dims=0, mlp=L.moe(experts=4, top=4, groups=2, keep=2)),
                          L.delta_pair(heads=4, kv_heads=1, dim=8, vdim=8, size=4, rot_dims=2, rheads=4, rkv=4, rdim=1, rvdim=1, conv=2, mlp=None)],
                         vocab=61, width=32, buckets=1, mul_prev=1, mul_cur=1)
# head widths the tensor-core attention and products take, enough tokens in the tests for the tensor-core products
CFG_TC = L.make_config([L.lightning_pair(heads=4, kv_heads=2, dim=32, vdim=32, size=40, rot_dims=16, rheads=2, rdim=32, rvdim=64, mlp=L.moe(experts=8, top=2, ff=64, shared=64)),
                        L.delta_pair(heads=2, kv_heads=1, dim=64, vdim=64, size=None, rot_dims=64, rheads=4, rkv=2, rdim=32, rvdim=32, conv=4, mlp=L.dense(96)),
                        L.retention_layer(heads=4, dim=32, vdim=64, rot_dims=32, mlp=L.moe(experts=4, top=1, ff=64, groups=2, keep=1, shared=40))], width=64, vocab=128)
# sizes that are multiples of nothing
CFG_ODD = L.make_config([L.delta_pair(heads=10, kv_heads=5, dim=6, vdim=7, size=45, rot_dims=2, scale=0.7, rheads=9, rkv=3, rdim=35, rvdim=5, conv=5, mlp=L.moe(experts=9, top=4, ff=11, groups=3, keep=2, shared=23)),
                         L.retention_layer(heads=5, dim=70, vdim=33, rot_dims=6, base=77.0, mlp=L.dense(17)),
                         L.lightning_pair(heads=9, kv_heads=3, dim=10, vdim=13, size=17, rot_dims=6, base=77.0, conv=4, softcap=1.5, rheads=7, rdim=3, rvdim=37, mlp=None),
                         L.lightning_pair(heads=3, kv_heads=1, dim=18, vdim=5, size=70, rot_dims=18, conv=6, rheads=1, rdim=5, rvdim=700, mlp=L.moe(experts=7, top=1, ff=9, groups=0, shared=0))],
                        vocab=67, width=50, eps=1e-6, buckets=211)
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


def _forward(cfg, w, toks):
    return O.forward(toks, w, cfg)[0]


# ------------------------------------------------------------------------------------------------ mechanisms alone
# name -> (layer, the tensors' prefix inside the layer, which part of the mixer's description, the restatement)
def _mech(kind, **kw):
    if kind == "attention":
        return L.delta_pair(mlp=None, **kw), "mix.left.", lambda m: m["left"], lambda h, w, p, m: O.window_attention(h, w, p, m, EPS, False)
    if kind == "unit_attention":
        return L.lightning_pair(mlp=None, **kw), "mix.left.", lambda m: m["left"], lambda h, w, p, m: O.window_attention(h, w, p, m, EPS, True)
    if kind == "delta":
        return L.delta_pair(mlp=None, **kw), "mix.right.", lambda m: m["right"], lambda h, w, p, m: O.channel_delta_mixer(h, w, p, m, EPS)
    if kind == "lightning":
        return L.lightning_pair(mlp=None, **kw), "mix.right.", lambda m: m["right"], lambda h, w, p, m: O.lightning(h, w, p, m, EPS)
    return L.retention_layer(mlp=None, **kw), "mix.", lambda m: m, lambda h, w, p, m: O.retention(h, w, p, m, EPS)


def _mech_stub(kind, layer, w, width, dtype="float32"):
    import torch

    from simplellminference_b200 import layers
    from simplellminference_b200.config import BF16, F32, NelutarConfig
    from simplellminference_b200.seqops import Ops
    dev = torch.device("cuda")
    ops = Ops(BF16 if dtype == "bfloat16" else F32)
    wt = {k: torch.tensor(v, device=dev, dtype=torch.bfloat16 if dtype == "bfloat16" else torch.float32) for k, v in w.items()}
    lc = NelutarConfig.from_dict(L.make_config([layer], width=width)).layers[0]
    mech = {"attention": lambda: layers.ConvRotaryAttention(lc.left, wt, "l0.mix.left.", ops, dev, EPS),
            "unit_attention": lambda: layers.ConvRotaryAttention(lc.left, wt, "l0.mix.left.", ops, dev, EPS, unit_heads=True),
            "delta": lambda: layers.ChannelDeltaRule(lc.right, wt, "l0.mix.right.", ops, dev, EPS),
            "lightning": lambda: layers.DecayedAttention(lc.right, wt, "l0.mix.right.", ops, dev, EPS, silu=True, row_norm=True, sigmoid_gate=True),
            "retention": lambda: layers.DecayedAttention(lc.mixer, wt, "l0.mix.", ops, dev, EPS, kscale=lc.mixer.dim ** -0.5)}[kind]()
    group = layers.MixerGroup([("mix", mech, 1.0)], ops, dev)

    def fn(step, h, states):
        y = step.scratch("sub_out", step.T * width)
        group.forward(step, h, states[0], y)
        return [y[:step.T * width].view(step.T, width)]
    return L.Stub([group.state_spec()], fn, ops, dev)


ALONE = [("attention", {}), ("attention", dict(heads=3, kv_heads=3, dim=20, vdim=9, size=9, rot_dims=20)), ("attention", dict(heads=8, kv_heads=1, dim=8, vdim=130, size=64, rot_dims=2)),
         ("attention", dict(heads=6, kv_heads=3, dim=12, size=None, rot_dims=0)), ("unit_attention", {}), ("unit_attention", dict(heads=1, kv_heads=1, dim=7, vdim=3, size=5, rot_dims=6, conv=1)),
         ("unit_attention", dict(heads=6, kv_heads=2, dim=32, vdim=40, size=None, rot_dims=32, conv=4, softcap=0.0)), ("unit_attention", dict(conv=0, rot_dims=0, size=40)),
         ("unit_attention", dict(heads=2, kv_heads=2, dim=36, vdim=4, size=70, rot_dims=4, conv=7, softcap=0.8)), ("delta", {}), ("delta", dict(rheads=1, rkv=1, rdim=1, rvdim=1, conv=1)),
         ("delta", dict(rheads=4, rkv=4, rdim=64, rvdim=40, conv=4)), ("delta", dict(rheads=2, rkv=1, rdim=130, rvdim=33, conv=2)), ("delta", dict(rheads=2, rkv=1, rdim=35, rvdim=70, conv=6)),
         ("delta", dict(rheads=1, rkv=1, rdim=600, rvdim=8, conv=3)), ("lightning", {}), ("lightning", dict(rheads=1, rdim=1, rvdim=1)), ("lightning", dict(rheads=4, rdim=32, rvdim=64)),
         ("lightning", dict(rheads=2, rdim=17, rvdim=300)), ("lightning", dict(rheads=1, rdim=4, rvdim=2100)), ("retention", {}), ("retention", dict(heads=4, dim=64, vdim=128, rot_dims=64)),
         ("retention", dict(heads=1, dim=33, vdim=5, rot_dims=0, decay=[1.0])), ("retention", dict(heads=2, dim=130, vdim=40, rot_dims=34))]


def _check_alone(kind, kw, h, portions, dtype="float32", tol=F32_TOL, seed=11, tweak=None, **feed_kw):
    layer, pre, part, oracle = _mech(kind, **kw)
    d = h.shape[1]
    w = L.random_weights(L.make_config([layer], width=d), seed=seed)
    if tweak:
        tweak(w)
    want = oracle(h.astype(np.float64), _w64(w), "l0." + pre, part(layer["mixer"]))
    got = L.feed(_mech_stub(kind, layer, w, d, dtype), h, portions, **feed_kw)[0]
    assert _rel(got, want) < tol, (kind, kw, portions[:4], _rel(got, want))
    return want


@pytest.mark.parametrize("portions", [[75], [33, 2, 15, 16, 1, 1, 1, 1, 5], [1] * 75], ids=["whole", "portions", "tokens"])
def test_each_mixer_alone(portions):
    h = np.random.default_rng(5).standard_normal((75, 48)).astype(np.float32)
    for kind, kw in ALONE:
        _check_alone(kind, kw, h, portions)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_each_mixer_alone_in_a_long_portion(dtype):
    """Portions of more than 512 tokens (kernels that let a warp walk several tokens, more work than fits the machine at once), then more portions
    and single tokens from the state they leave."""
    h = L.bf16_round(np.random.default_rng(6).standard_normal((1215, 64))).astype(np.float32)
    for kind, kw in (("attention", {}), ("attention", dict(dim=36, vdim=20, rot_dims=36, size=None)), ("unit_attention", {}), ("unit_attention", dict(conv=2, dim=24, vdim=20, size=70)),
                     ("unit_attention", dict(conv=4, dim=32, vdim=32, rot_dims=32)), ("unit_attention", dict(conv=1)), ("unit_attention", dict(conv=6, heads=6, kv_heads=3)),
                     ("unit_attention", dict(conv=0, dim=7, vdim=5, rot_dims=2)), ("delta", {}), ("delta", dict(rheads=2, rkv=1, rdim=40, rvdim=36, conv=4)), ("lightning", {}),
                     ("retention", {})):
        for portions in ([1215], [519, 2, 690, 1, 1, 2]):
            _check_alone(kind, kw, h, portions, dtype=dtype, tol=F32_TOL if dtype == "float32" else BF16_MIXER, seed=13, max_tokens=1248)


@pytest.mark.parametrize("portions", [[80], [40, 2, 37, 1]], ids=["whole", "portions"])
def test_each_mixer_alone_bf16(portions):
    """bf16 matrices, operands and cache; portions of a prompt take the tensor-core attention where the head widths allow it."""
    h = L.bf16_round(np.random.default_rng(7).standard_normal((80, 64))).astype(np.float32)
    for kind, kw in (("attention", dict(heads=4, kv_heads=2, dim=32, vdim=32, size=30, rot_dims=16)), ("attention", dict(heads=3, kv_heads=1, dim=12, vdim=8, size=None)),
                     ("unit_attention", dict(heads=4, kv_heads=1, dim=48, vdim=64, size=50)), ("unit_attention", {}), ("delta", dict(rheads=4, rkv=2, rdim=64, rvdim=64, conv=4)),
                     ("delta", {}), ("lightning", dict(rheads=4, rdim=32, rvdim=64)), ("lightning", {}), ("retention", dict(heads=4, dim=64, vdim=128, rot_dims=64)), ("retention", {})):
        _check_alone(kind, kw, h, portions, dtype="bfloat16", tol=BF16_MIXER, seed=13)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_recurrences_over_long_portions_beside_short_ones(dtype):
    """Portions longer than the ranges and blocks that the recurrences work in, beside single tokens and short portions of another sequence, cut
    at, just before and just after their borders; the state a long portion leaves is the one the next step starts from."""
    import torch

    from simplellminference_b200.seqengine import SequenceEngine
    rng = np.random.default_rng(21)
    d, TA, TB = 48, 700, 300
    for kind, kw in (("delta", {}), ("delta", dict(rheads=4, rkv=2, rdim=64, rvdim=32, conv=4)), ("delta", dict(rheads=2, rkv=2, rdim=35, rvdim=70)), ("lightning", {}),
                     ("lightning", dict(rheads=2, rdim=32, rvdim=64)), ("retention", {}), ("retention", dict(heads=2, dim=64, vdim=32, rot_dims=64)),
                     ("unit_attention", dict(conv=4)), ("unit_attention", dict(heads=3, kv_heads=1, dim=9, vdim=7, rot_dims=4, conv=6))):
        layer, pre, part, oracle = _mech(kind, **kw)
        w = L.random_weights(L.make_config([layer], width=d), seed=17)
        stub = _mech_stub(kind, layer, w, d, dtype)
        ha, hb = L.bf16_round(rng.standard_normal((TA, d))).astype(np.float32), L.bf16_round(rng.standard_normal((TB, d))).astype(np.float32)
        eng = SequenceEngine(stub, max_tokens=1280, max_seqs=2, page_len=32, graphs=False)
        sa, sb = eng.admit(), eng.admit()
        # (tokens of a, tokens of b) per step
        steps = [(129, 1), (1, 128), (256, 1), (127, 130), (2, 1), (65, 2), (120, 37)]
        assert sum(a for a, _ in steps) == TA and sum(b for _, b in steps) == TB
        got_a, got_b, pa, pb = [], [], 0, 0
        for na, nb in steps:
            stub.h = torch.tensor(np.concatenate([ha[pa:pa + na], hb[pb:pb + nb]]), dtype=torch.float32, device=stub.device).contiguous().view(-1)
            eng.run([(sa, np.zeros(na, np.int32), []), (sb, np.zeros(nb, np.int32), [])])
            out = stub.outs[0].cpu().numpy()
            got_a.append(out[:na]); got_b.append(out[na:na + nb])
            pa, pb = pa + na, pb + nb
        tol = F32_TOL if dtype == "float32" else BF16_MIXER
        for got, h in ((got_a, ha), (got_b, hb)):
            want = oracle(h.astype(np.float64), _w64(w), "l0." + pre, part(layer["mixer"]))
            assert _rel(np.concatenate(got), want) < tol, (kind, kw, _rel(np.concatenate(got), want))


def _scan_stub(kind, H, G, dk, dv, consts, blocks):
    """Columns [q | k | v | beta logits | step logits] straight into the recurrence kernels, in blocks of tokens or token by token."""
    import torch

    from simplellminference_b200.config import BF16, RotaryConfig
    from simplellminference_b200.layers import rotary_frequencies
    from simplellminference_b200.seqops import Ops
    dev, ops = torch.device("cuda"), Ops(BF16)
    t = lambda a: torch.tensor(np.asarray(a), dtype=torch.float32, device=dev)   # noqa: E731
    steps = {"channel": H * dk, "head": H}.get(kind, 0)
    sizes = [G * dk, G * dk, H * dv, H if steps else 0, steps]
    offs, width = [4 * sum(sizes[:i]) for i in range(5)], sum(sizes)
    c = {k: t(v) for k, v in consts.items()}
    key, freq = rotary_frequencies(RotaryConfig(dk // 4 * 2, 50.0), dev) if kind == "retention" and dk >= 4 else ((), None)

    def fn(step, h, states):
        base, S = h.data_ptr(), states[0]["S"]
        q, k, v, bl, al = (base + o for o in offs)
        out = torch.empty(step.T, H * dv, device=dev)
        ws = step.chunk_scratch(H, dk, dv) if blocks else None
        assert (ws is not None) == (blocks and step.T - step.nseg + 1 >= step.chunk_min_tokens)
        if steps:
            rule = ops.channel_delta_rule if kind == "channel" else ops.delta_rule
            rule(step.b, q, width, k, width, v, width, bl, width, al, width, c["A_log"], c["dt_bias"], H, G, dk, dv, 1e-6, dk ** -0.5, S, out, H * dv, None, 0, 0, 0, None,
                 step.st, chunk_ws=ws)
        else:
            ops.decay_scan(step.b, q, width, k, width, v, width, c["decay"], c["rate"], step.angles(key, freq) if key else None, len(key), 1, kind == "lightning",
                           dk ** -0.5 if kind == "retention" else 1.0, H, dk, dv, S, out, H * dv, step.st, chunk_ws=ws)
        return [out]
    rot = {"dims": len(key) * 2, "base": 50.0}
    return L.Stub([{"pages": [], "slots": [("S", (H, dk, dv))]}], fn, ops, dev), sizes, rot


def _scan_oracle(kind, x, sizes, H, G, dk, dv, consts, rot):
    n = x.shape[0]
    q, k, v, bl, al = np.split(x.astype(np.float64), np.cumsum(sizes)[:-1], axis=1)
    q, k, v = q.reshape(n, G, dk), k.reshape(n, G, dk), v.reshape(n, H, dv)
    out = np.zeros((n, H, dv))
    if kind in ("channel", "head"):
        q, k, beta = O.unit_vectors(q) * dk ** -0.5, O.unit_vectors(k), O.sigmoid(bl)
        step = O.softplus(al + consts["dt_bias"]).reshape(n, H, -1)
        g = np.broadcast_to(np.exp(-np.exp(np.asarray(consts["A_log"], np.float64))[None, :, None] * step), (n, H, dk))
        for h in range(H):
            out[:, h] = O.channel_delta_rule(q[:, h * G // H], k[:, h * G // H], v[:, h], beta[:, h], g[:, h])
        return out.reshape(n, H * dv)
    if kind == "lightning":
        q, k, v = O.silu(q), O.silu(k), O.silu(v)
    else:
        q, k = O.rotate(q, rot, False), O.rotate(k, rot, False) * dk ** -0.5
    for h in range(H):
        out[:, h] = O.decayed_attention(q[:, h], k[:, h], v[:, h], consts["decay64"][h])
    return out.reshape(n, H * dv)


def test_recurrences_in_blocks_of_tokens_keep_fp32_accuracy():
    """The block form of the recurrences (tensor cores, operands as two bf16 terms) and the form that walks token by token, both against the
    restatement on the same fp32 inputs: weak and strong decays (a channel that forgets everything within a token), step sizes near one,
    keys that repeat, one head and shared key heads, widths that are multiples of nothing, portions that end inside a block, a state that is
    carried from portion to portion and into single tokens."""
    rng = np.random.default_rng(51)
    cases = [("channel", 2, 1, 128, 128), ("channel", 3, 3, 64, 40), ("channel", 1, 1, 1, 1), ("channel", 4, 2, 33, 130), ("channel", 2, 2, 100, 5), ("head", 4, 2, 128, 64),
             ("head", 3, 1, 20, 70), ("retention", 2, 2, 128, 128), ("retention", 3, 3, 6, 33), ("retention", 1, 1, 70, 200), ("lightning", 2, 2, 64, 64), ("lightning", 3, 3, 97, 3)]
    for kind, H, G, dk, dv in cases:
        for flavour in ("weak", "mixed", "strong"):
            n = 150
            decay = {"weak": 1.0 - 10.0 ** -np.linspace(3, 5, H), "mixed": np.linspace(0.3, 0.999, H), "strong": np.linspace(1e-4, 0.2, H)}[flavour]
            consts = {"A_log": rng.uniform(*{"weak": (-9, -6), "mixed": (-3, 1), "strong": (1, 4)}[flavour], size=H).astype(np.float32), "decay": decay.astype(np.float32),
                      "rate": -np.log(decay), "decay64": decay.astype(np.float32).astype(np.float64),
                      "dt_bias": rng.uniform(-3, 3, size=H * dk if kind == "channel" else H).astype(np.float32)}
            consts["rate"] = (-np.log(consts["decay64"])).astype(np.float32)
            results = []
            for blocks in (True, False):
                stub, sizes, rot = _scan_stub(kind, H, G, dk, dv, consts, blocks)
                if not results:
                    x = rng.standard_normal((n, sum(sizes))).astype(np.float32)
                    if sizes[3]:
                        x[:, sum(sizes[:3]):sum(sizes[:4])] += 3.0          # step sizes near one
                        x[20:60, sizes[0]:2 * sizes[0]] = x[19, sizes[0]:2 * sizes[0]] + 0.05 * x[20:60, sizes[0]:2 * sizes[0]]   # keys that nearly repeat
                    want = _scan_oracle(kind, x, sizes, H, G, dk, dv, consts, rot)
                for portions in ([n], [37, 16, 1, 40, 2, 54], [100] + [1] * 50):
                    got = L.feed(stub, x, portions)[0]
                    assert _rel(got, want) < 5e-5, (kind, H, dk, dv, flavour, blocks, portions[:3], _rel(got, want))
                    results.append(_rel(got, want))
            print(kind, H, G, dk, dv, flavour, ["%.1e" % r for r in results])


def test_state_and_rings_of_a_slot_used_again():
    """A slot that carried one sequence's state and convolution inputs serves another: its first tokens see zeros, not the old state."""
    from simplellminference_b200.seqengine import SequenceEngine
    rng = np.random.default_rng(3)
    d = 48
    for kind in ("attention", "unit_attention", "delta", "lightning", "retention"):
        layer, pre, part, oracle = _mech(kind)
        w = L.random_weights(L.make_config([layer], width=d), seed=4)
        stub = _mech_stub(kind, layer, w, d)
        eng = SequenceEngine(stub, max_tokens=128, max_seqs=1, page_len=32, graphs=False)
        for T, portions in ((50, [50]), (3, [1, 2]), (40, [2, 38]), (1, [1])):
            h = rng.standard_normal((T, d)).astype(np.float32)
            got = L.feed(stub, h, portions, engine=eng)[0]
            want = oracle(h.astype(np.float64), _w64(w), "l0." + pre, part(layer["mixer"]))
            assert _rel(got, want) < F32_TOL, (kind, T)


def _standing_out(kind, d, H, window):
    """An attention layer and weights in which the query of a position reads the first third of its input row and the key the second
    third, through the same map, with no convolution reaching back and no rotation: a query row whose first third repeats the second third of
    an earlier row gives that position (and no other, itself included) a score far above the rest."""
    t = d // 3
    kw = dict(heads=H, kv_heads=H // 2, dim=16, vdim=16, size=window, rot_dims=0)
    kw.update(dict(conv=2, scale=0.9, softcap=20.0) if kind == "unit_attention" else dict(scale=3.0))
    layer, pre, part, oracle = _mech(kind, **kw)
    w = L.random_weights(L.make_config([layer], width=d), seed=3)
    p = "l0.mix.left."
    a = w[p + "k"][:, :t].copy()
    w[p + "q"][:] = 0.0
    w[p + "k"][:] = 0.0
    # the query heads of a group read through their key head's map
    w[p + "q"][:, :t] = np.repeat(a.reshape(H // 2, 1, 16, t), 2, axis=1).reshape(H * 16, t)
    w[p + "k"][:, t:2 * t] = a
    if kind == "unit_attention":
        for n in ("q", "k"):                                    # the convolution passes the current token only
            w[f"{p}{n}.conv"][:] = 0.0
            w[f"{p}{n}.conv"][:, -1] = 1.0
    run = lambda h: oracle(h.astype(np.float64), _w64(w), p, part(layer["mixer"]))   # noqa: E731
    return _mech_stub(kind, layer, w, d), run, t


@pytest.mark.parametrize("decode", [False, True], ids=["prompt", "decoded"])
@pytest.mark.parametrize("kind", ["attention", "unit_attention"])
def test_keys_just_inside_and_outside_the_window(kind, decode):
    """The key input of an earlier position is repeated as the query input of a later one: when that position is the oldest one inside the
    window the query's output is essentially its value; one further back it is something else — the restatement says so and the engine has to
    follow it, with the key before, at and after a border of pages of 32."""
    rng = np.random.default_rng(9)
    d, T, H, window = 48, 150, 4, 37
    stub, oracle, t = _standing_out(kind, d, H, window)
    seen = []
    for query in (149, 100, 68, 69, 70):                      # oldest visible key 113 / 64 / 32 / 33 / 34
        for key, visible in ((query - window + 1, True), (query - window, False), (query - 1, True), (0, False)):
            h = rng.standard_normal((T, d)).astype(np.float32)
            h[key, t:2 * t] *= 2.0                          # a long key: no other key's chance alignment with the query comes close
            h[query, :t] = h[key, t:2 * t]
            want = oracle(h)
            got = L.feed(stub, h, [query] + [1] * (T - query) if decode else [T])[0]
            assert _rel(got, want) < F32_TOL, (query, key, _rel(got, want))
            base = h.copy()
            base[key] = rng.standard_normal(d)
            seen.append((visible, _rel(oracle(base)[query], want[query])))
    shown = sorted(r for v, r in seen if v)
    assert shown[0] > 0.05 and shown[len(shown) // 2] > 0.3, "a visible repeated position does not stand out: the test would not notice a lost key"
    # (a hidden key's successor still reads it through the value's convolution; the query's own row is two and more positions away)
    assert max(r for v, r in seen if not v) < (1e-6 if kind == "attention" else 0.2), "a hidden position changes the restatement's result"


@pytest.mark.parametrize("decode", [False, True], ids=["prompt", "decoded"])
@pytest.mark.parametrize("kind", ["attention", "unit_attention"])
def test_a_key_far_back_among_hundreds(kind, decode):
    """One position hundreds of tokens back (the first token, one at a page border, one in the middle of a page) towers over all others."""
    rng = np.random.default_rng(10)
    d, T, H = 48, 420, 4
    stub, oracle, t = _standing_out(kind, d, H, 400)
    shown = []
    for query, key in ((419, 20), (400, 64), (330, 0), (399, 31)):
        h = rng.standard_normal((T, d)).astype(np.float32)
        h[key, t:2 * t] *= 2.0
        h[query, :t] = h[key, t:2 * t]
        want = oracle(h)
        got = L.feed(stub, h, [320] + [1] * (T - 320) if decode else [200, 220])[0]
        assert _rel(got, want) < F32_TOL, (query, key, _rel(got, want))
        base = h.copy()
        base[key] = rng.standard_normal(d)
        shown.append(_rel(oracle(base)[query], want[query]))
    assert min(shown) > 0.3, "the far position does not stand out"


def test_long_memory_of_the_states():
    """Decays close to one: what a token wrote hundreds of positions back still shows in the output, in a prompt cut into portions and in
    decoding, as the restatement says."""
    rng = np.random.default_rng(14)
    d, T = 48, 400
    long = [0.9995, 0.9999, 1.0]
    for kind, kw in (("delta", dict(rheads=2, rkv=1, rdim=24)), ("retention", dict(heads=3, rot_dims=0, decay=long)), ("retention", dict(heads=3, decay=long)), ("lightning", {})):
        layer, pre, part, oracle = _mech(kind, **kw)
        if kind == "lightning":
            layer["mixer"]["right"]["decay"] = long
        w = L.random_weights(L.make_config([layer], width=d), seed=6)
        if kind == "delta":
            w["l0.mix.right.A_log"][:] = -6.0
            w["l0.mix.right.b"][:] *= 0.1
        run = lambda h: oracle(h.astype(np.float64), _w64(w), "l0." + pre, part(layer["mixer"]))   # noqa: E731
        h = rng.standard_normal((T, d)).astype(np.float32)
        h[3] *= 4.0
        want = run(h)
        for portions in ([T], [130, 2, 200, 68], [300] + [1] * 100):
            got = L.feed(_mech_stub(kind, layer, w, d), h, portions)[0]
            assert _rel(got, want) < F32_TOL, (kind, portions[:2], _rel(got, want))
        other = h.copy()
        other[3] = rng.standard_normal(d)
        # (the delta rule overwrites what later keys find: its early token fades first)
        assert _rel(run(other)[-1 if kind != "delta" else 40], want[-1 if kind != "delta" else 40]) > 1e-3, "the early token has faded: the test would not notice a lost state"


def test_delta_rule_decays_rows_of_the_state_by_channel():
    """One key channel forgets at once and the others never: the restatement differs visibly from a decay per head (the channels' mean), and the
    engine follows the decay per channel."""
    rng = np.random.default_rng(31)
    d, T = 48, 60
    layer, pre, part, oracle = _mech("delta", rheads=2, rkv=2, rdim=8, rvdim=12, conv=1)
    w = L.random_weights(L.make_config([layer], width=d), seed=9)
    p = "l0.mix.right."
    w[p + "A_log"][:] = 0.0
    w[p + "a2"][:] = 0.0
    w[p + "dt_bias"][:] = -8.0
    w[p + "dt_bias"].reshape(2, 8)[:, 3] = 3.0
    h = rng.standard_normal((T, d)).astype(np.float32)
    want = oracle(h.astype(np.float64), _w64(w), p, part(layer["mixer"]))
    for portions in ([T], [20, 2] + [1] * 38):
        assert _rel(L.feed(_mech_stub("delta", layer, w, d), h, portions)[0], want) < F32_TOL
    flat = dict(w)
    flat[p + "dt_bias"] = np.full(16, -8.0, np.float32)
    assert _rel(oracle(h.astype(np.float64), _w64(flat), p, part(layer["mixer"])), want) > 0.05


def test_branch_seam_alone():
    """The sum of up to four branches, each with a weight per channel and normed or not, then the norm; widths with and without 16-byte rows."""
    import torch

    from simplellminference_b200.config import F32
    from simplellminference_b200.seqops import Ops
    rng, dev, ops = np.random.default_rng(2), torch.device("cuda"), Ops(F32)
    st = torch.cuda.current_stream().cuda_stream
    for d, T in ((48, 5), (50, 70), (1000, 3), (1001, 2), (4096, 66), (6000, 2), (16384, 1), (9001, 1)):
        for n, normed in ((0, []), (1, [0]), (2, [1, 1]), (3, [1, 1, 0]), (4, [0, 1, 0, 1])):
            x = (3 * rng.standard_normal((T, d))).astype(np.float32)
            ys, gains = rng.standard_normal((n, T, d)).astype(np.float32) * 2, rng.standard_normal((n, d)).astype(np.float32)
            nw, eps = rng.standard_normal(d).astype(np.float32), 1e-3
            new = x.astype(np.float64)
            for y, g, k in zip(ys, gains, normed):
                new = new + g * (O.unit_rms(y, eps) if k else y.astype(np.float64))
            t = lambda a: torch.tensor(a, device=dev)   # noqa: E731
            xt, nt, yt, gt = t(x), t(nw), [t(y) for y in ys], [t(g) for g in gains]
            h, h16 = torch.empty_like(xt), torch.empty(T, d, dtype=torch.bfloat16, device=dev)
            ops.branch_seam(xt, xt, list(zip(yt, gt, normed)), eps, nt, h, T, d, st, h16=h16)
            want = O.rms_norm(new, nw, eps)
            assert _rel(xt.cpu().numpy(), new) < 1e-6 and _rel(h.cpu().numpy(), want) < 1e-6, (d, T, n)
            assert _rel(h16.float().cpu().numpy(), want) < 4e-3
            xt = t(x)
            ops.branch_seam(xt, xt, list(zip(yt, gt, normed)), eps, None, None, T, d, st)     # the sum alone
            assert _rel(xt.cpu().numpy(), new) < 1e-6


def _ff_stub(mlp, w, d, dtype="float32"):
    import torch

    from simplellminference_b200 import layers
    from simplellminference_b200.config import BF16, F32, NelutarConfig
    from simplellminference_b200.seqops import Ops
    dev, ops = torch.device("cuda"), Ops(BF16 if dtype == "bfloat16" else F32)
    wt = {k: torch.tensor(v, device=dev, dtype=torch.bfloat16 if dtype == "bfloat16" else torch.float32) for k, v in w.items()}
    c = NelutarConfig.from_dict(L.make_config([L.retention_layer(mlp=mlp)], width=d)).layers[0].mlp
    if mlp["kind"] == "dense":
        ff = layers.SiluGluFeedForward(c, wt, "l0.mlp.", ops, dev)
    else:
        ff = layers.ExpertsFeedForward(c, wt, "l0.mlp.", ops, dev, activation=3, gated=True, sigmoid_scores=True, normalise=True, in_group=True)
    group = layers.MixerGroup([("ff", ff, 1.0)], ops, dev)

    def fn(step, h, states):
        T = step.T
        y = step.scratch("sub_out", T * d)
        # as a model's seam leaves the rows: bf16 rows where the product takes them, fp32 rows where something reads those
        h16 = step.scratch("rows16", (T * d + 1) // 2) if group.proj.takes_rows16(step) else None
        if h16 is not None:
            h16[:(T * d + 1) // 2].view(torch.bfloat16)[:T * d] = h.to(torch.bfloat16)
        group.forward(step, h if h16 is None or group.reads_f32(step) else None, {}, [y], h16=h16)
        return [y[:T * d].view(T, d)]
    return L.Stub([{"pages": [], "slots": []}], fn, ops, dev), ff


def _oracle_ff(mlp, w, h):
    return O.ff(h.astype(np.float64), _w64(w), "l0.mlp.", mlp)


MOES = [L.moe(), L.moe(experts=9, top=1, ff=7, groups=3, keep=1), L.moe(experts=2, top=2, ff=16, groups=1, keep=1), L.moe(experts=40, top=8, ff=4, groups=8, keep=4),
        L.moe(experts=1, top=1, ff=5, groups=0), L.moe(experts=6, top=2, groups=6, keep=3, shared=0), L.moe(experts=64, top=6, ff=4, groups=32, keep=5, scale=0.3)]


def test_feed_forwards_alone():
    """The gated feed-forward and the mixture of clamped experts: grouped choice, corrected choice scores, normalised and scaled weights, a
    shared expert with sizes and limits of its own."""
    rng, d, T = np.random.default_rng(4), 40, 37
    for mlp in [L.dense(56)] + MOES:
        w = L.random_weights(L.make_config([L.retention_layer(mlp=mlp)], width=d), seed=2)
        stub, _ = _ff_stub(mlp, w, d)
        h = (2 * rng.standard_normal((T, d))).astype(np.float32)
        for portions in ([T], [1] * 5 + [T - 5]):
            assert _rel(L.feed(stub, h, portions)[0], _oracle_ff(mlp, w, h)) < F32_TOL, mlp


def test_routing_branches_show_in_the_result():
    """Each rule of the router left out of the restatement changes its result visibly, with the weights the engine is tested with; negative
    choice scores stay choosable inside a kept group."""
    rng, d, T = np.random.default_rng(41), 40, 60
    mlp = L.moe(experts=8, top=3, groups=4, keep=2)
    w = _w64(L.random_weights(L.make_config([L.retention_layer(mlp=mlp)], width=d), seed=5))
    h = 2 * rng.standard_normal((T, d))
    want = O.moe_ff(h, w, "l0.mlp.", mlp)
    other = lambda m, ww=w: _rel(O.moe_ff(h, ww, "l0.mlp.", m), want)   # noqa: E731
    r = mlp["router"]
    assert other(dict(mlp, router={k: v for k, v in r.items() if k != "groups"})) > 0.02
    assert other(mlp, dict(w, **{"l0.mlp.correction": np.zeros(8)})) > 0.02
    assert other(dict(mlp, expert={"ff": 12, "limit": 50.0})) > 0.02 and other(dict(mlp, shared=dict(mlp["shared"], limit=0.9))) > 0.01
    s = O.sigmoid(h @ w["l0.mlp.router"].T)
    chosen, weight = O.route(h, w, "l0.mlp.", r)
    assert (np.take_along_axis(s + w["l0.mlp.correction"], chosen, -1) < 0).any(), "no chosen expert has a negative choice score"
    np.testing.assert_allclose(weight.sum(-1), r["scale"])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_experts_with_the_tokens_gathered_per_expert(dtype, monkeypatch):
    """Steps of many tokens multiply a token only with the experts it uses, one launch for all experts' first products and one for the second
    ones: the same numbers as the form that computes every expert. Sizes the tensor-core tiles take (also an expert nobody is routed to) and
    sizes they do not."""
    from simplellminference_b200 import layers
    rng = np.random.default_rng(14)
    for d, T, mlp in ((64, 150, L.moe(experts=8, top=2, ff=64, groups=2, keep=1, shared=64)), (64, 300, L.moe(experts=12, top=1, ff=72, groups=0)), (64, 150, L.moe(experts=5, top=1, ff=24, groups=0)),
                      (128, 700, L.moe(experts=4, top=2, ff=128, groups=2, keep=2, shared=0)), (50, 90, L.moe(experts=6, top=3, ff=11, groups=3, keep=2))):
        w = L.random_weights(L.make_config([L.retention_layer(mlp=mlp)], width=d), seed=5)
        if mlp["router"]["experts"] == 12:
            w["l0.mlp.correction"][7] = -40.0                    # never chosen
        stub, ff = _ff_stub(mlp, w, d, dtype)
        h = L.bf16_round(2 * rng.standard_normal((T, d))).astype(np.float32)
        monkeypatch.setattr(layers.ExpertsFeedForward, "gather_min_tokens", 10 ** 9)
        every = L.feed(stub, h, [T])[0]
        monkeypatch.setattr(layers.ExpertsFeedForward, "gather_min_tokens", 64)
        monkeypatch.setattr(layers.ExpertsFeedForward, "gather_launch_cost", 0.0)
        assert ff._gathered_pays(T)
        gathered = L.feed(stub, h, [T])[0]
        want = _oracle_ff(mlp, w, h)
        tol = F32_TOL if dtype == "float32" else BF16_MIXER
        assert _rel(gathered, want) < tol and _rel(every, want) < tol, (mlp, _rel(gathered, want), _rel(every, want))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_experts_chosen_on_the_device_in_steps_of_few_tokens(dtype, monkeypatch):
    """Decoding steps stream only the chosen experts' matrices: the same numbers as the form that computes every expert."""
    from simplellminference_b200 import layers
    rng, d = np.random.default_rng(15), 64
    for mlp, T in ((L.moe(experts=12, top=2, ff=32, groups=3, keep=2), 3), (L.moe(experts=9, top=1, ff=24, groups=3, keep=1), 8), (L.moe(experts=8, top=3, ff=20), 2)):
        w = L.random_weights(L.make_config([L.retention_layer(mlp=mlp)], width=d), seed=6)
        stub, ff = _ff_stub(mlp, w, d, dtype)
        h = L.bf16_round(2 * rng.standard_normal((T, d))).astype(np.float32)
        monkeypatch.setattr(layers.ExpertsFeedForward, "index_launch_cost", 1e9)
        assert not ff._indexed_pays(T)
        every = L.feed(stub, h, [T])[0]
        monkeypatch.setattr(layers.ExpertsFeedForward, "index_launch_cost", 0.0)
        assert ff._indexed_pays(T)
        indexed = L.feed(stub, h, [T])[0]
        want = _oracle_ff(mlp, w, h)
        tol = F32_TOL if dtype == "float32" else BF16_MIXER
        assert _rel(indexed, want) < tol and _rel(every, want) < tol, (mlp, _rel(indexed, want), _rel(every, want))


# ------------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("cfg", ALL, ids=IDS)
def test_whole_prompt_matches_oracle_fp32_and_layers(tmp_path, cfg):
    w = L.random_weights(cfg, seed=1)
    toks = np.random.default_rng(2).integers(0, cfg["vocab"], size=140).tolist()
    want, taps_want = O.forward(toks, w, cfg)
    for streams in (True, False):                              # mechanisms side by side on streams of their own, and one after the other
        eng = _engine(tmp_path, cfg, w, branch_streams=streams)
        taps = []
        got = eng.run([(eng.admit(), toks, list(range(len(toks))))], tap=lambda i, x: taps.append(x.clone().cpu().numpy())).cpu().numpy()
        assert len(taps) == len(cfg["layers"])
        for i, (a, b) in enumerate(zip(taps, taps_want)):
            assert _rel(a, b) < F32_MODEL, (i, _rel(a, b))
        assert L.logit_error(got, want).max() < F32_MODEL


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_long_prompt_and_what_follows_it(tmp_path, dtype):
    """700 tokens in one portion, then a short portion and single tokens from the caches and states it leaves."""
    cfg = CFG_TC
    w = L.random_weights(cfg, seed=27)
    toks = np.random.default_rng(28).integers(0, cfg["vocab"], size=720).tolist()
    want = _forward(cfg, w, toks)
    eng = _engine(tmp_path, cfg, w, dtype=dtype, max_tokens=768, page_len=64)
    s = eng.admit()
    got = np.concatenate([_logits(eng, s, toks[:700]), _logits(eng, s, toks[700:709])] + [_logits(eng, s, toks[p:p + 1]) for p in range(709, 720)])
    e = L.logit_error(got, want)
    if dtype == "float32":
        assert e.max() < F32_MODEL
    else:
        assert np.median(e) < BF16_MODEL_TYPICAL and np.median(e[700:]) < BF16_MODEL_TYPICAL and (e > 0.3).mean() < 0.1


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
    # Several layers deep, rounding of the operands is multiplied by what follows it, and a choice of experts that is a near tie may fall
    # the other way: the typical position is held to the rounding, outliers are few. The mechanisms alone are held to the rounding
    # itself in test_each_mixer_alone_bf16.
    for got in (whole, cut):
        e = L.logit_error(got, want)
        assert np.median(e) < BF16_MODEL_TYPICAL and (e > 0.3).mean() < 0.1, (np.median(e), (e > 0.3).mean())
    e = L.logit_error(cut, whole)
    assert np.median(e) < BF16_MODEL_TYPICAL, np.median(e)


def test_model_whose_layers_leave_bf16_rows_only(tmp_path, monkeypatch):
    """With the tokens gathered per expert on the tensor cores nothing of a layer reads the normed rows in fp32: the seams leave bf16 rows alone,
    and the logits are those of the form that computes every expert."""
    from simplellminference_b200 import layers
    cfg = L.make_config([L.lightning_pair(heads=4, kv_heads=2, dim=32, vdim=32, rot_dims=16, rheads=2, rdim=32, rvdim=64, mlp=L.moe(experts=8, top=2, ff=64, shared=64)),
                         L.delta_pair(heads=2, kv_heads=1, dim=64, vdim=64, rot_dims=64, rheads=4, rkv=2, rdim=32, rvdim=32, mlp=L.moe(experts=4, top=1, ff=72, groups=2, keep=1))],
                        width=64, vocab=128)
    w = L.random_weights(cfg, seed=23)
    toks = np.random.default_rng(24).integers(0, cfg["vocab"], size=200).tolist()
    want, got, read = _forward(cfg, w, toks), {}, []
    for gathers in (False, True):
        monkeypatch.setattr(layers.ExpertsFeedForward, "gather_min_tokens", 64 if gathers else 10 ** 9)
        monkeypatch.setattr(layers.ExpertsFeedForward, "gather_launch_cost", 0.0)
        eng = _engine(tmp_path, cfg, w, dtype="bfloat16")
        plain = layers.MixerGroup.reads_f32
        monkeypatch.setattr(layers.MixerGroup, "reads_f32", lambda self, step, plain=plain: read.append(plain(self, step)) or read[-1])
        read.clear()
        got[gathers] = _logits(eng, eng.admit(), toks)
        monkeypatch.setattr(layers.MixerGroup, "reads_f32", plain)
        assert read and all(r != gathers for r in read)
        assert np.median(L.logit_error(got[gathers], want)) < BF16_MODEL_TYPICAL
    assert np.median(L.logit_error(got[True], got[False])) < BF16_MODEL_TYPICAL


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


@pytest.mark.parametrize("cfg", [CFG_A, CFG_ODD], ids=["mixed", "odd"])
def test_unequal_requests_in_one_batch_and_reuse_of_pages_and_slots(tmp_path, cfg):
    """Seven requests of unequal length through three slots and ten pages of 32: portions of prompts beside single tokens of others, every
    request's logits equal the restatement's of that request alone; pages and slots go from finished requests to new ones."""
    w = L.random_weights(cfg, seed=7)
    rng = np.random.default_rng(8)
    lens = [70, 33, 5, 96, 64, 1, 47]
    reqs = [rng.integers(0, cfg["vocab"], size=n).tolist() for n in lens]
    want = [_forward(cfg, w, r) for r in reqs]
    eng = _engine(tmp_path, cfg, w, max_tokens=320, max_seqs=3, page_len=32)
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
        assert L.logit_error(np.concatenate(got[i]), want[i]).max() < F32_MODEL, i


def test_long_decoding_over_page_borders_and_past_the_windows(tmp_path):
    layers = [L.lightning_pair(size=50), L.delta_pair(size=130, mlp=L.moe()), L.retention_layer()]
    cfg = L.make_config(layers + [L.again(layers, 1)])
    w = L.random_weights(cfg, seed=8)
    toks = np.random.default_rng(4).integers(0, cfg["vocab"], size=330).tolist()
    want = _forward(cfg, w, toks)
    eng = _engine(tmp_path, cfg, w, max_tokens=384, page_len=64)
    s = eng.admit()
    outs = [_logits(eng, s, toks[:60])] + [_logits(eng, s, toks[p:p + 1]) for p in range(60, 330)]
    assert eng.graph_replays > 200
    assert L.logit_error(np.concatenate(outs), want).max() < F32_MODEL


def test_several_requests_decode_together_in_captured_steps(tmp_path):
    """Four requests at different positions step together: the captured step's parallel branches give every one what it gets alone, in both
    number formats."""
    cfg = CFG_TC
    w = L.random_weights(cfg, seed=31)
    rng = np.random.default_rng(32)
    reqs = [rng.integers(0, cfg["vocab"], size=n + 30).tolist() for n in (50, 3, 31, 64)]
    for dtype, tol in (("float32", F32_MODEL), ("bfloat16", None)):
        eng = _engine(tmp_path, cfg, w, dtype=dtype)
        slots = [eng.admit() for _ in reqs]
        got = [[g] for g in (_logits(eng, s, r[:-30]) for s, r in zip(slots, reqs))]
        for k in range(30):
            out = eng.run([(s, [r[len(r) - 30 + k]], [0]) for s, r in zip(slots, reqs)]).cpu().numpy()
            for i in range(len(reqs)):
                got[i].append(out[i:i + 1])
        assert eng.graph_replays >= 28
        for r, g in zip(reqs, got):
            e = L.logit_error(np.concatenate(g), _forward(cfg, w, r))
            assert e.max() < tol if tol else np.median(e) < BF16_MODEL_TYPICAL, (dtype, e.max())


def test_first_tokens_of_a_sequence_after_a_used_slot(tmp_path):
    """A slot (recurrent states, convolution rings, the previous token) and pages that held a long request serve the next one: its first tokens
    equal the restatement's."""
    w = L.random_weights(CFG_A, seed=9)
    rng = np.random.default_rng(10)
    eng = _engine(tmp_path, CFG_A, w, max_seqs=1, max_tokens=96)
    for n in (90, 4, 1, 2, 35):
        toks = rng.integers(0, CFG_A["vocab"], size=n).tolist()
        s = eng.admit()
        got = np.concatenate([_logits(eng, s, toks[:1]), _logits(eng, s, toks[1:])]) if n > 1 else _logits(eng, s, toks)
        eng.release(s)
        assert L.logit_error(got, _forward(CFG_A, w, toks)).max() < F32_MODEL, n


def test_a_layer_with_borrowed_weights_keeps_a_state_of_its_own(tmp_path):
    """Two layers with one set of weights: the model differs from the one whose second layer is left out, and follows the restatement in
    portions and token by token; the weights are held once."""
    layers = [L.delta_pair(mlp=L.moe())]
    cfg = L.make_config(layers + [L.again(layers, 0)])
    w = L.random_weights(cfg, seed=19)
    assert not any(k.startswith("l1.") for k in w)
    toks = np.random.default_rng(20).integers(0, cfg["vocab"], size=70).tolist()
    want = _forward(cfg, w, toks)
    assert L.logit_error(_forward(L.make_config(layers), w, toks), want).max() > 0.05
    eng = _engine(tmp_path, cfg, w)
    assert eng.model.layers[0] is eng.model.layers[1] and eng.states[0]["left.k"].data_ptr() != eng.states[1]["left.k"].data_ptr()
    for portions in ([70], [40, 2, 28], [30] + [1] * 40):
        s, outs, p = eng.admit(), [], 0
        for n in portions:
            outs.append(_logits(eng, s, toks[p:p + n]))
            p += n
        eng.release(s)
        assert L.logit_error(np.concatenate(outs), want).max() < F32_MODEL, portions[:2]


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
    """bin/trace_run end to end on a Nelutar folder: the model class comes from config.json."""
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
    for dtype, tol in (("float32", F32_MODEL), ("bfloat16", BF16_TOL)):
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
    """python -m simplellminference_b200.generate on a Nelutar folder: registry, engine, scheduler, device arg-max."""
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
