"""Plain float64 restatement of the Nelutar design, one function per mechanism, whole sequences only (no cache, no portions, no
batches). It shares nothing with the package: the tests compare the framework's kernels, cache and scheduler against it.

Notation: x [n][width] is the residual stream of one sequence, W a dictionary name -> float64 array, positions count from 0."""
from __future__ import annotations

import numpy as np

from vasosun_oracle import causal_conv, delta_rule, embed, f64, sigmoid, silu, softmax, softplus, unit_rms  # noqa: F401  (the same mathematics)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def unit_vectors(x, eps=1e-6):
    """x / sqrt(sum x^2 + eps) over the last axis."""
    return x / np.sqrt((x * x).sum(-1, keepdims=True) + eps)


def rotate(x, rot, interleaved):
    """x [n][heads][dim]: pairs of the first rot.dims dimensions turn by position * base^(-2i/dims); pair i is (2i, 2i+1), or (i, i + dims/2)."""
    x = f64(x).copy()
    dims = (rot or {}).get("dims") or 0
    if not dims:
        return x
    half = dims // 2
    ang = np.arange(x.shape[0])[:, None, None] * (float(rot["base"]) ** (-2.0 * np.arange(half) / dims))
    cs, sn = np.cos(ang), np.sin(ang)
    a, b = (slice(0, dims, 2), slice(1, dims, 2)) if interleaved else (slice(0, half), slice(half, dims))
    u, v = x[..., a].copy(), x[..., b].copy()
    x[..., a] = u * cs - v * sn
    x[..., b] = v * cs + u * sn
    return x


def window_attention(h, W, pre, m, eps, unit_heads):
    """Grouped softmax attention over the last mask.size positions; with ``unit_heads`` q, k and v pass a convolution first and q and k are
    divided by their root mean square (no weight) after the rotation; scores may be capped."""
    n = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def branch(name, heads, width):
        z = h @ W[pre + name].T
        if m.get("conv"):
            z = causal_conv(z, W[pre + name + ".conv"])
        return z.reshape(n, heads, width)
    q, k, v = branch("q", H, dk), branch("k", G, dk), branch("v", G, dv)
    q, k = rotate(q, m.get("rot"), True), rotate(k, m.get("rot"), True)
    if unit_heads:
        q, k = unit_rms(q, eps), unit_rms(k, eps)
    size = (m.get("mask") or {}).get("size") or n + 1
    dist = np.arange(n)[:, None] - np.arange(n)[None, :]
    sees = (dist >= 0) & (dist < size)
    out = np.zeros((n, H, dv))
    for hh in range(H):
        g = hh // (H // G)
        s = (q[:, hh] @ k[:, g].T) * m["scale"]
        if m.get("softcap"):
            s = m["softcap"] * np.tanh(s / m["softcap"])
        out[:, hh] = softmax(np.where(sees, s, -np.inf)) @ v[:, g]
    return out.reshape(n, H * dv) @ W[pre + "o"].T


def channel_delta_rule(q, k, v, beta, g):
    """One head with a decay per key channel: S <- diag(g) S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q. g [n][dk]."""
    n, dk = q.shape
    S = np.zeros((dk, v.shape[1]))
    o = np.zeros_like(v)
    for t in range(n):
        S = g[t][:, None] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + np.outer(k[t], u)
        o[t] = S.T @ q[t]
    return o


def channel_delta_mixer(h, W, pre, m, eps):
    n = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def branch(name, heads, width):
        return silu(causal_conv(h @ W[pre + name].T, W[pre + name + ".conv"])).reshape(n, heads, width)
    q, k, v = unit_vectors(branch("q", G, dk)) * dk ** -0.5, unit_vectors(branch("k", G, dk)), branch("v", H, dv)
    beta = sigmoid(h @ W[pre + "b"].T)
    step = softplus((h @ W[pre + "a1"].T) @ W[pre + "a2"].T + W[pre + "dt_bias"]).reshape(n, H, dk)
    g = np.exp(-np.exp(W[pre + "A_log"])[None, :, None] * step)
    gate = sigmoid((h @ W[pre + "g1"].T) @ W[pre + "g2"].T).reshape(n, H, dv)
    out = np.zeros((n, H, dv))
    for hh in range(H):
        kv = hh // (H // G)
        o = channel_delta_rule(q[:, kv], k[:, kv], v[:, hh], beta[:, hh], g[:, hh])
        out[:, hh] = unit_rms(o, eps) * W[pre + "norm"] * gate[:, hh]
    return out.reshape(n, H * dv) @ W[pre + "o"].T


def decayed_attention(q, k, v, decay):
    """One head: S <- decay S + k v^T, o = S^T q."""
    S = np.zeros((k.shape[1], v.shape[1]))
    o = np.zeros_like(v)
    for t in range(q.shape[0]):
        S = decay * S + np.outer(k[t], v[t])
        o[t] = S.T @ q[t]
    return o


def _heads(h, W, pre, m):
    n, H = h.shape[0], m["heads"]
    return tuple((h @ W[pre + name].T).reshape(n, H, m[width]) for name, width in (("q", "dim"), ("k", "dim"), ("v", "vdim")))


def retention(h, W, pre, m, eps):
    n, H, dv = h.shape[0], m["heads"], m["vdim"]
    q, k, v = _heads(h, W, pre, m)
    q, k = rotate(q, m.get("rot"), False), rotate(k, m.get("rot"), False) * m["dim"] ** -0.5
    o = np.stack([unit_rms(decayed_attention(q[:, i], k[:, i], v[:, i], m["decay"][i]), eps) for i in range(H)], axis=1)
    return (o.reshape(n, H * dv) * silu(h @ W[pre + "g"].T)) @ W[pre + "o"].T


def lightning(h, W, pre, m, eps):
    n, H, dv = h.shape[0], m["heads"], m["vdim"]
    q, k, v = (silu(z) for z in _heads(h, W, pre, m))
    o = np.stack([decayed_attention(q[:, i], k[:, i], v[:, i], m["decay"][i]) for i in range(H)], axis=1).reshape(n, H * dv)
    return (rms_norm(o, W[pre + "norm"], eps) * sigmoid(h @ W[pre + "g"].T)) @ W[pre + "o"].T


def mixer(h, W, pre, kind, m, eps):
    if kind == "parallel":
        left = window_attention(h, W, pre + "left.", m["left"], eps, False)
        right = channel_delta_mixer(h, W, pre + "right.", m["right"], eps)
        return 0.5 * (rms_norm(left, W[pre + "left.out"], eps) + rms_norm(right, W[pre + "right.out"], eps))
    if kind == "parallel_2":
        return (m["left_scale"] * window_attention(h, W, pre + "left.", m["left"], eps, True)
                + m["right_scale"] * lightning(h, W, pre + "right.", m["right"], eps))
    if kind == "retention":
        return retention(h, W, pre, m, eps)
    raise ValueError(kind)


def dense_ff(h, W, pre):
    return (silu(h @ W[pre + "gate"].T) * (h @ W[pre + "up"].T)) @ W[pre + "down"].T


def clamped_expert(h, W, pre, limit):
    g, u = np.minimum(h @ W[pre + "gate"].T, limit), np.clip(h @ W[pre + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ W[pre + "down"].T


def route(h, W, pre, r):
    """(chosen [n][top], their weights [n][top]): sigmoid scores; groups ranked by the sum of their two largest corrected scores, the best
    ``keep`` of them stay; the largest corrected scores in those are chosen; the weights are the plain scores, normalised, times scale."""
    s = sigmoid(h @ W[pre + "router"].T)
    choice = s + W[pre + "correction"]
    groups = r.get("groups")
    if groups:
        n, count = h.shape[0], groups["count"]
        per = r["experts"] // count
        top2 = -np.sort(-choice.reshape(n, count, per), axis=-1)[..., :2].sum(-1)
        best = np.argsort(-top2, axis=-1, kind="stable")[:, :groups["keep"]]
        stays = np.zeros((n, count), bool)
        np.put_along_axis(stays, best, True, axis=-1)
        choice = np.where(np.repeat(stays, per, axis=-1), choice, -np.inf)
    chosen = np.argsort(-choice, axis=-1, kind="stable")[:, :r["top"]]
    w = np.take_along_axis(s, chosen, axis=-1)
    return chosen, w / (w.sum(-1, keepdims=True) + 1e-20) * r["scale"]


def moe_ff(h, W, pre, mlp):
    chosen, weight = route(h, W, pre, mlp["router"])
    out = np.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        at, k = np.nonzero(chosen == e)
        if at.size:
            out[at] += weight[at, k][:, None] * clamped_expert(h[at], W, f"{pre}e{e}.", mlp["expert"]["limit"])
    if mlp.get("shared"):
        out += clamped_expert(h, W, pre + "shared.", mlp["shared"]["limit"])
    return out


def ff(h, W, pre, mlp):
    return dense_ff(h, W, pre) if mlp["kind"] == "dense" else moe_ff(h, W, pre, mlp)


def forward(tokens, W, cfg):
    """tokens of ONE sequence -> (logits [n][vocab], the residual stream after every layer [layers][n][width])."""
    W = {k: f64(v) for k, v in W.items()}
    eps = cfg["norm"]["eps"]
    big = cfg["embedding"]["bigram"]
    x = embed(tokens, W["embed"], W["bigram"], big["buckets"], big["mul_prev"], big["mul_cur"])
    taps = []
    for i, lc in enumerate(cfg["layers"]):
        pre = f"l{lc.get('weights_of', i)}."
        h = rms_norm(x, W[pre + "norm1"], eps)
        y = W[pre + "ls1"] * mixer(h, W, pre + "mix.", lc["type"], lc["mixer"], eps)
        if lc.get("mlp") is not None:
            y = y + W[pre + "ls2"] * ff(h, W, pre + "mlp.", lc["mlp"])
        x = x + y
        taps.append(x.copy())
    return rms_norm(x, W["final.norm"], eps) @ W["head"].T, np.stack(taps)
