"""Plain float64 restatement of the Lovulix design, one function per mechanism, whole sequences only (no cache, no portions, no batches).
It shares nothing with the package: the tests compare the framework's kernels, cache and scheduler against it.

Notation: x [n][width] is the residual stream of one sequence, W a dictionary name -> float64 array, positions count from 0."""
from __future__ import annotations

import math

import numpy as np


def f64(a):
    return np.asarray(a, dtype=np.float64)


def rms_norm(x, w, eps):
    x = f64(x)
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * f64(w)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def band_frequencies(dims, base, scaling):
    """Angular step of pair i: base^(-2i/dims); wavelengths short against the original context keep it, long ones are slowed down by
    the factor, those between the two bounds take a blend that is linear in (original / wavelength)."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling:
            wave = 2.0 * math.pi / f
            lo, hi, orig, factor = (float(scaling[k]) for k in ("low", "high", "original", "factor"))
            if wave < orig / hi:
                pass
            elif wave > orig / lo:
                f = f / factor
            else:
                s = (orig / wave - lo) / (hi - lo)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return out


def rotate_halves(x, dims, freq):
    """x [n][heads][dim]: of the first `dims` dimensions i turns with i + dims/2, by (position * freq[i])."""
    x = f64(x).copy()
    pos = np.arange(x.shape[0], dtype=np.float64)
    half = dims // 2
    for i in range(half):
        c, s = np.cos(pos * freq[i])[:, None], np.sin(pos * freq[i])[:, None]
        u, v = x[:, :, i].copy(), x[:, :, i + half].copy()
        x[:, :, i] = u * c - v * s
        x[:, :, i + half] = v * c + u * s
    return x


def same_chunk(n, size):
    """see[i][j]: does position i see position j? Only j <= i of its own chunk of `size` positions (None: every j <= i)."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    ok = j <= i
    if size:
        ok &= (i // size) == (j // size)
    return ok


def mixed_scores(q, k, T, scale):
    """q [n][H][dk], k [n][G][dk] -> scores [H][n][n]: every head's own q.k * scale first, then each head takes a weighted sum of all
    heads' scores, score_h = sum_g T[h][g] own_g."""
    H, G = q.shape[1], k.shape[1]
    own = np.stack([(q[:, h] @ k[:, h // (H // G)].T) * scale for h in range(H)])
    return np.einsum("hg,gij->hij", f64(T), own)


def sink_softmax(s, see, sink):
    """Softmax over the visible keys of s [n][n] with one more term exp(sink) in the denominator."""
    s = np.where(see, s, -np.inf)
    m = np.maximum(s.max(axis=1, keepdims=True), sink)
    e = np.exp(s - m)
    return e / (e.sum(axis=1, keepdims=True) + np.exp(sink - m))


def attention(h, W, pre, m, eps, v_first=None):
    """(result [n][width], the layer's own values [n][G][dv]). `v_first`: values of the first layer of the kind, blended in."""
    h = f64(h)
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    n = h.shape[0]
    q = rms_norm(h @ f64(W[pre + "q"]).T, W[pre + "q.norm"], eps).reshape(n, H, dk)      # the norm runs over all heads at once
    k = rms_norm(h @ f64(W[pre + "k"]).T, W[pre + "k.norm"], eps).reshape(n, G, dk)
    own = (h @ f64(W[pre + "v"]).T).reshape(n, G, dv)
    v = own
    if v_first is not None:
        lam = float(W[pre + "vmix"])
        v = (1.0 - lam) * own + lam * v_first
    rot = m.get("rot")
    if rot and rot["dims"]:
        freq = band_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
        q, k = rotate_halves(q, rot["dims"], freq), rotate_halves(k, rot["dims"], freq)
    see = same_chunk(n, (m.get("mask") or {}).get("size"))
    s = mixed_scores(q, k, W[pre + "talk"], m["scale"])
    out = np.zeros((n, H, dv))
    for hh in range(H):
        out[:, hh] = sink_softmax(s[hh], see, float(W[pre + "sink"][hh])) @ v[:, hh // (H // G)]
    gated = out.reshape(n, H * dv) * sigmoid(h @ f64(W[pre + "g"]).T)
    return gated @ f64(W[pre + "o"]).T, own


def glu(h, W, pre):
    return (silu(f64(h) @ f64(W[pre + "gate"]).T) * (f64(h) @ f64(W[pre + "up"]).T)) @ f64(W[pre + "down"]).T


def route(h, W, pre, top):
    """(experts chosen [n][top], their scores): sigmoid of the router's outputs, the largest first, the lower index on a tie."""
    s = sigmoid(f64(h) @ f64(W[pre + "router"]).T)
    order = np.argsort(-s, axis=1, kind="stable")[:, :top]
    return order, np.take_along_axis(s, order, axis=1)


def experts_ff(h, W, pre, mlp):
    """Every token through its `top` experts, the score on what the expert reads, plus the shared expert on the plain input."""
    h = f64(h)
    chosen, score = route(h, W, pre, mlp["router"]["top"])
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(chosen[t], score[t]):
            out[t] += glu((s * h[t])[None], W, f"{pre}e{int(e)}.")[0]
    if mlp.get("shared"):
        out += glu(h, W, pre + "shared.")
    return out


def forward(cfg: dict, W: dict, tokens, layer_outputs: list | None = None):
    """Logits [n][vocab] of one sequence; layer_outputs (if a list) receives the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = f64(W["embed"])[np.asarray(tokens)]
    v_first = None
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        mixes = bool(m.get("v_mix"))
        y, own = attention(x, W, p + "mix.", m, eps, v_first if mixes else None)
        if mixes and v_first is None:
            v_first = own
        x = x + rms_norm(y, W[p + "norm1"], eps)
        if l.get("mlp"):
            x = x + rms_norm(experts_ff(x, W, p + "mlp.", l["mlp"]), W[p + "norm2"], eps)
        if layer_outputs is not None:
            layer_outputs.append(x.copy())
    return rms_norm(x, W["final.norm"], eps) @ f64(W["head"]).T * float(cfg["logit_scale"])
