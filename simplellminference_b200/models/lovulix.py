"""Lovulix: a decoder-only model whose sublayers read the residual stream itself and whose only norms sit on their results,
x <- x + norm1(mixer(x)), then x <- x + norm2(ff(x)) (RMS norms with a weight per channel). Mixer: chunked softmax attention with
whole-projection norms on queries and keys, rotary positions scaled by wavelength bands, scores mixed over the heads before the softmax, a
sink, values blended with those of the first such layer and a gate per channel. Feed-forward: a mixture of gated (silu) experts whose
sigmoid scores multiply what the experts read, plus an expert every token uses. The logits carry a constant factor.

The class only DESCRIBES the model with the mechanisms of ``layers``; cache, batching and the step loop belong to
``seqengine.SequenceEngine``. Tensor names: ``embed``, ``l<i>.norm1`` / ``norm2``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``."""
from __future__ import annotations

from ..layers import ExpertsFeedForward, FusedLinear, MixerGroup, ScoreMixingAttention

SILU = 2              # activation number of the feed-forward kernels
ROTARY_LAYOUT = 1     # dimension i pairs with i + dims/2


class _Layer:
    def __init__(self, mixer, ff, norm1, norm2):
        self.mixer, self.ff, self.norm1, self.norm2 = mixer, ff, norm1, norm2


class LovulixModel:
    def __init__(self, cfg, w, ops, device):
        self.cfg, self.ops, self.device = cfg, ops, device
        self.vocab, self.width = cfg.vocab, cfg.width
        self.embed = w["embed"].contiguous()
        self.final_w = self._vector(w, "final.norm")
        self.head = FusedLinear([(w["head"], None)], ops, device)
        self.layers = []
        kept = False                      # has a layer kept its values for the later ones?
        for i, lc in enumerate(cfg.layers):
            pre = f"l{i}."
            share = None
            if lc.mixer.v_mix:
                share, kept = "blend" if kept else "keep", True
            mixer = ScoreMixingAttention(lc.mixer, w, pre + "mix.", ops, device, cfg.norm_eps, ROTARY_LAYOUT, share)
            ff = None
            if lc.mlp is not None:
                ff = ExpertsFeedForward(lc.mlp, w, pre + "mlp.", ops, device, activation=SILU, gated=True, sigmoid_scores=True, scale_input=True)
            self.layers.append(_Layer(MixerGroup([("mix", mixer, 1.0)], ops, device), ff, self._vector(w, pre + "norm1"),
                                      self._vector(w, pre + "norm2") if ff is not None else None))

    def _vector(self, w, name):
        v = w[name].float().contiguous()
        if tuple(v.shape) != (self.width,):
            raise ValueError(f"{name} is {tuple(v.shape)}, the model is {self.width} wide")
        return v

    def state_specs(self):
        """One entry per layer: the pools its mixer declares."""
        return [layer.mixer.state_spec() for layer in self.layers]

    def forward(self, step, ids, states, rows, n_rows, tap=None):
        """The step's tokens through every layer; returns logits [n_rows][vocab] (fp32) of the batch rows listed in ``rows``."""
        ops, c, T, d = self.ops, self.cfg, step.T, self.width
        xa, xb = step.scratch("stream_a", T * d), step.scratch("stream_b", T * d)      # the residual sum goes from one to the other
        y = step.scratch("sub_out", T * d)
        ops.embed(ids, self.embed, self.vocab, d, 1, xa, T, step.st)
        # a seam adds the normed sublayer result to the stream and leaves the stream as the operand rows of the next sublayer's product;
        # the last one also norms it for the head (the factor on the logits rides on that norm)
        chain = [(i, body, norm) for i, layer in enumerate(self.layers) for body, norm in ((layer.mixer, layer.norm1), (layer.ff, layer.norm2)) if body is not None]
        ready = False
        for n, (i, body, norm) in enumerate(chain):
            if isinstance(body, MixerGroup):
                body.forward(step, xa, states[i], y, h16_ready=ready)
            else:
                body.forward(step, xa, y, h16_ready=ready)
            if n + 1 == len(chain):
                h = step.scratch("normed", T * d)
                ops.seam(step.b, xa, d, step.st, x_out=xb, y=y, post_w=norm, pre_g=c.logit_scale, eps=c.norm_eps, pre_w=self.final_w, h=h)
            else:
                rows16 = chain[n + 1][1].proj.operand_rows(step)
                ops.seam(step.b, xa, d, step.st, x_out=xb, y=y, post_w=norm, eps=c.norm_eps, h16=rows16)
                ready = rows16 is not None
            xa, xb = xb, xa
            if tap is not None and (n + 1 == len(chain) or chain[n + 1][0] != i):
                tap(i, xa[:T * d].view(T, d))
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
