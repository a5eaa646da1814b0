"""Nelutar: a decoder-only model of parallel layers, x <- x + ls1 * mixer(h) + ls2 * ff(h) with h = norm(x) (one RMS norm with a weight per
channel, one scale per channel on each result); the embedding adds a hashed table indexed by the (previous token, token) pair; a layer may
use another layer's weights with a cache and state of its own. Mixers: window attention beside the gated delta rule with a decay per key
channel, half the sum of the two results, each normed over the model's width; window attention with convolved and normed heads and capped
scores beside lightning attention, a weighted sum; and retention. Feed-forwards: gated, or a mixture of clamped experts with a grouped sigmoid
router beside an expert every token uses.

The class only DESCRIBES the model with the mechanisms of ``layers``: the mixers and the feed-forward of a layer are one ``MixerGroup`` whose
members run side by side, and what lies between two layers is one kernel. Cache, state slots, batching and the step loop belong to
``seqengine.SequenceEngine``. Tensor names: ``embed``, ``bigram``, ``l<i>.norm1`` / ``ls1`` / ``ls2``, ``l<i>.mix.*`` (``left.*`` / ``right.*``,
``left.out`` / ``right.out`` for the norms over the width), ``l<i>.mlp.*``, ``final.norm``, ``head``."""
from __future__ import annotations

from ..config import ExpertsConfig
from ..layers import ChannelDeltaRule, ConvRotaryAttention, DecayedAttention, ExpertsFeedForward, FusedLinear, MixerGroup, SiluGluFeedForward

INTERLEAVED, HALVES = 0, 1      # rotary layouts: dimension 2i pairs with 2i+1, or i with i + dims/2
BRANCH_WEIGHT = 0.5             # of each of the two normed results of a ``parallel`` mixer


class _Layer:
    """``gains``: per member of the group the weight per channel its result enters the stream with (layer scale, constant factors and the
    weight of a norm over the width in one vector); ``normed``: whether the result is divided by its root mean square first."""

    def __init__(self, group, norm, gains, normed):
        self.group, self.norm, self.gains, self.normed = group, norm, gains, normed


class NelutarModel:
    def __init__(self, cfg, w, ops, device):
        self.cfg, self.ops, self.device = cfg, ops, device
        self.vocab, self.width = cfg.vocab, cfg.width
        self.embed = w["embed"].contiguous()
        self.pairs = w["bigram"].contiguous() if cfg.pair_buckets else None
        if self.pairs is not None and int(self.pairs.shape[0]) != cfg.pair_buckets + 1:
            raise ValueError(f"bigram holds {int(self.pairs.shape[0])} rows, {cfg.pair_buckets} buckets need one more")
        self.final_w = self._vector(w, "final.norm")
        self.head = FusedLinear([(w["head"], None)], ops, device)
        own = {i: self._layer(lc, w, f"l{i}.") for i, lc in enumerate(cfg.layers) if lc.weights_of is None}
        self.layers = [own[i if lc.weights_of is None else lc.weights_of] for i, lc in enumerate(cfg.layers)]

    def _vector(self, w, name):
        v = w[name].float().contiguous()
        if tuple(v.shape) != (self.width,):
            raise ValueError(f"{name} is {tuple(v.shape)}, the model is {self.width} wide")
        return v

    def _layer(self, lc, w, pre):
        ops, device, eps = self.ops, self.device, self.cfg.norm_eps
        mix = pre + "mix."
        ls1 = self._vector(w, pre + "ls1")
        if lc.type == "parallel":
            members = [("left", ConvRotaryAttention(lc.left, w, mix + "left.", ops, device, eps, layout=INTERLEAVED)),
                       ("right", ChannelDeltaRule(lc.right, w, mix + "right.", ops, device, eps))]
            gains = [BRANCH_WEIGHT * ls1 * self._vector(w, f"{mix}{side}.out") for side in ("left", "right")]
            normed = [True, True]
        elif lc.type == "parallel_2":
            members = [("left", ConvRotaryAttention(lc.left, w, mix + "left.", ops, device, eps, layout=INTERLEAVED, unit_heads=True)),
                       ("right", DecayedAttention(lc.right, w, mix + "right.", ops, device, eps, silu=True, row_norm=True, sigmoid_gate=True))]
            gains, normed = [lc.left_scale * ls1, lc.right_scale * ls1], [False, False]
        else:
            members = [("mix", DecayedAttention(lc.mixer, w, mix, ops, device, eps, layout=HALVES, kscale=lc.mixer.dim ** -0.5))]
            gains, normed = [ls1], [False]
        if isinstance(lc.mlp, ExpertsConfig):
            members.append(("ff", ExpertsFeedForward(lc.mlp, w, pre + "mlp.", ops, device, activation=ExpertsFeedForward.CLAMPED, gated=True, sigmoid_scores=True,
                                                     normalise=True, in_group=True)))
        elif lc.mlp is not None:
            members.append(("ff", SiluGluFeedForward(lc.mlp, w, pre + "mlp.", ops, device)))
        if lc.mlp is not None:
            gains.append(self._vector(w, pre + "ls2"))
            normed.append(False)
        return _Layer(MixerGroup([(n, m, 1.0) for n, m in members], ops, device), self._vector(w, pre + "norm1"), [g.contiguous() for g in gains], normed)

    def state_specs(self):
        """One entry per layer run (a layer with another's weights has a cache and state of its own): what its mechanisms declare."""
        return [layer.group.state_spec() for layer in self.layers]

    def forward(self, step, ids, states, rows, n_rows, tap=None):
        """The step's tokens through every layer; returns logits [n_rows][vocab] (fp32) of the batch rows listed in ``rows``."""
        ops, c, T, d = self.ops, self.cfg, step.T, self.width
        x = step.scratch("stream", T * d)
        if self.pairs is not None:
            ops.embed_pair(ids, step.prev_ids, self.embed, self.pairs, self.vocab, d, c.pair_buckets, c.pair_mul_prev, c.pair_mul_cur, x, T, step.st)
        else:
            ops.embed(ids, self.embed, self.vocab, d, 1, x, T, step.st)

        # the seam in front of a layer (or of the head) adds what the layer before left, and norms: bf16 rows for tensor-core products,
        # fp32 rows where something reads those
        def seam(results, norm_w, group):
            h16 = step.scratch("rows16", (T * d + 1) // 2) if group is not None and group.proj.takes_rows16(step) else None
            h = step.scratch("normed", T * d) if h16 is None or group.reads_f32(step) else None
            ops.branch_seam(x, x, results, c.norm_eps, norm_w, h, T, d, step.st, h16=h16)
            return h, h16

        h, h16 = seam([], self.layers[0].norm, self.layers[0].group)
        for i, layer in enumerate(self.layers):
            ys = [step.scratch(f"branch_out{k}", T * d) for k in range(len(layer.gains))]
            layer.group.forward(step, h, states[i], ys, h16=h16)
            results = list(zip(ys, layer.gains, layer.normed))
            if i + 1 < len(self.layers):
                h, h16 = seam(results, self.layers[i + 1].norm, self.layers[i + 1].group)
            else:
                h, h16 = seam(results, self.final_w if n_rows else None, None)
            if tap is not None:
                tap(i, x[:T * d].view(T, d))
        if n_rows == 0:
            return None
        picked = step.scratch("picked", n_rows * d)
        ops.gather_rows(h, d, rows, n_rows, d, picked, step.st)
        logits = step.scratch("logits", n_rows * self.vocab)
        T_save = step.T
        step.T = n_rows               # the head runs over the picked rows only
        try:
            self.head(step, picked.data_ptr(), d, logits.data_ptr(), self.vocab)
        finally:
            step.T = T_save
        return logits[:n_rows * self.vocab].view(n_rows, self.vocab)
