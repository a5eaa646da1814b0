"""Test helpers for the Nelutar design: small configurations and random weights written as a model folder (config.json +
model.safetensors in bf16). Nothing here is used by the product package."""
from __future__ import annotations

import numpy as np

from kodezen_testlib import Stub, feed  # noqa: F401  (a stub model that feeds rows to one mechanism through the engine)
from munazen_testlib import bf16_round, logit_error, to_bf16_bits, write_model  # noqa: F401  (the file format and the measure are the same)


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def moe(experts=8, top=3, ff=12, limit=0.9, groups=4, keep=2, scale=1.5, shared=20, shared_limit=1.3):
    r = {"experts": experts, "top": top, "scale": scale}
    if groups:
        r["groups"] = {"count": groups, "keep": keep}
    m = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": r}
    if shared:
        m["shared"] = {"ff": shared, "limit": shared_limit}
    return m


def _layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": dense() if mlp == "dense" else mlp}


def _attention(heads, kv_heads, dim, vdim, size, rot_dims, base, scale, conv=0, softcap=0.0):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if size is not None:
        m["mask"] = {"size": size}
    if rot_dims:
        m["rot"] = {"dims": rot_dims, "base": base}
    if conv:
        m["conv"] = conv
    if softcap:
        m["softcap"] = softcap
    return m


def decays(heads, first=0.5, last=0.998):
    """Different in every head, from a short memory to a long one."""
    return [float(1.0 - (1.0 - first) * ((1.0 - last) / (1.0 - first)) ** (h / max(1, heads - 1))) for h in range(heads)]


def delta_pair(heads=4, kv_heads=2, dim=16, vdim=12, size=20, rot_dims=8, base=1000.0, scale=0.3, rheads=6, rkv=3, rdim=10, rvdim=14, conv=3, mlp="dense"):
    """Window attention beside the gated delta rule with a decay per key channel."""
    return _layer("parallel", {"left": _attention(heads, kv_heads, dim, vdim, size, rot_dims, base, scale),
                               "right": {"heads": rheads, "kv_heads": rkv, "dim": rdim, "vdim": rvdim, "conv": conv}}, mlp)


def lightning_pair(heads=4, kv_heads=2, dim=16, vdim=12, size=20, rot_dims=8, base=500.0, scale=0.6, conv=3, softcap=4.0, rheads=3, rdim=10, rvdim=14, left=0.7,
                   right=1.2, mlp="dense"):
    """Window attention with convolved, normed heads and capped scores beside lightning attention."""
    return _layer("parallel_2", {"left": _attention(heads, kv_heads, dim, vdim, size, rot_dims, base, scale, conv, softcap),
                                 "right": {"heads": rheads, "dim": rdim, "vdim": rvdim, "decay": decays(rheads, 0.4, 0.99)}, "left_scale": left, "right_scale": right}, mlp)


def retention_layer(heads=3, dim=12, vdim=18, rot_dims=8, base=2000.0, mlp="dense", decay=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay or decays(heads)}
    if rot_dims:
        m["rot"] = {"dims": rot_dims, "base": base}
    return _layer("retention", m, mlp)


def again(layers, j):
    """A layer that uses layer j's weights."""
    return dict(layers[j], weights_of=j)


def make_config(layers, vocab=83, width=48, eps=1e-5, buckets=53, mul_prev=29, mul_cur=11):
    return {"architecture": "Nelutar", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "embedding": {"bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}, "layers": layers}


def random_weights(cfg: dict, seed: int = 0, rank: int = 9) -> dict:
    """name -> float32 array of bf16-representable values (so that both storage types hold the same numbers)."""
    rng = np.random.default_rng(seed)
    d = cfg["width"]
    w = {}

    def mat(n_out, n_in, gain=1.0):
        return bf16_round(rng.standard_normal((n_out, n_in)) * gain / np.sqrt(n_in))

    def vec(n, mean=0.0, std=0.1):
        return bf16_round(mean + std * rng.standard_normal(n))

    def attention(p, m):
        H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for n, rows in (("q", H * dk), ("k", G * dk), ("v", G * dv)):
            w[p + n] = mat(rows, d, 1.5)
            if m.get("conv"):
                w[p + n + ".conv"] = bf16_round(0.6 * rng.standard_normal((rows, m["conv"])))
        w[p + "o"] = mat(d, H * dv)

    def decayed(p, m, norm):
        H, dk, dv = m["heads"], m["dim"], m["vdim"]
        for n, rows in (("q", H * dk), ("k", H * dk), ("v", H * dv), ("g", H * dv)):
            w[p + n] = mat(rows, d, 1.5)
        if norm:
            w[p + "norm"] = vec(H * dv, 1.0, 0.3)
        w[p + "o"] = mat(d, H * dv)

    w["embed"] = bf16_round(rng.standard_normal((cfg["vocab"], d)))
    w["bigram"] = bf16_round(0.7 * rng.standard_normal((cfg["embedding"]["bigram"]["buckets"] + 1, d)))
    w["head"] = mat(cfg["vocab"], d, 3.0)
    w["final.norm"] = vec(d, 0.8, 0.4)
    for i, l in enumerate(cfg["layers"]):
        if l.get("weights_of") is not None:
            continue
        p, m = f"l{i}.", l["mixer"]
        w[p + "norm1"], w[p + "ls1"] = vec(d, 0.9, 0.3), vec(d, 0.7, 0.3)
        if l["type"] == "parallel":
            attention(p + "mix.left.", m["left"])
            r, q = m["right"], p + "mix.right."
            H, G, dk, dv = r["heads"], r["kv_heads"], r["dim"], r["vdim"]
            for n, rows in (("q", G * dk), ("k", G * dk), ("v", H * dv)):
                w[q + n] = mat(rows, d, 1.5)
                w[q + n + ".conv"] = bf16_round(0.6 * rng.standard_normal((rows, r["conv"])))
            w[q + "b"], w[q + "a1"], w[q + "a2"], w[q + "g1"], w[q + "g2"] = mat(H, d, 2.0), mat(rank, d), mat(H * dk, rank, 2.0), mat(rank, d), mat(H * dv, rank, 2.0)
            w[q + "A_log"], w[q + "dt_bias"], w[q + "norm"] = vec(H, -1.0, 0.8), vec(H * dk, 0.0, 0.7), vec(dv, 1.0, 0.3)
            w[q + "o"] = mat(d, H * dv)
            w[p + "mix.left.out"], w[p + "mix.right.out"] = vec(d, 0.9, 0.3), vec(d, 1.1, 0.3)
        elif l["type"] == "parallel_2":
            attention(p + "mix.left.", m["left"])
            decayed(p + "mix.right.", m["right"], True)
        else:
            decayed(p + "mix.", m, False)
        mlp = l.get("mlp")
        if mlp:
            w[p + "ls2"] = vec(d, 0.6, 0.3)
            if mlp["kind"] == "dense":
                w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"] = mat(mlp["ff"], d, 2.0), mat(mlp["ff"], d), mat(d, mlp["ff"])
            else:
                r = mlp["router"]
                parts = [(f"e{e}", mlp["expert"]["ff"]) for e in range(r["experts"])] + ([("shared", mlp["shared"]["ff"])] if mlp.get("shared") else [])
                for n, f in parts:
                    w[f"{p}mlp.{n}.gate"], w[f"{p}mlp.{n}.up"], w[f"{p}mlp.{n}.down"] = mat(f, d, 1.5), mat(f, d, 1.5), mat(d, f, 1.5)
                # scores far enough apart that a close call is rare; a correction large enough to change choices and to make some negative
                w[p + "mlp.router"], w[p + "mlp.correction"] = mat(r["experts"], d, 3.0), vec(r["experts"], -0.3, 0.4)
    return {k: np.asarray(v, dtype=np.float32) for k, v in w.items()}
