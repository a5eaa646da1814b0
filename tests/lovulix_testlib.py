"""Test helpers for the Lovulix design: small configurations and random weights written as a model folder (config.json +
model.safetensors in bf16). Nothing here is used by the product package."""
from __future__ import annotations

import numpy as np

from kodezen_testlib import Stub, feed  # noqa: F401  (a stub model that feeds rows to one mechanism through the engine)
from munazen_testlib import bf16_round, logit_error, to_bf16_bits, write_model  # noqa: F401  (the file format and the measure are the same)

BANDS = {"factor": 3.0, "low": 1.0, "high": 5.0, "original": 200}


def moe(experts=5, top=2, ff=12, shared=20):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def layer(heads=4, kv_heads=2, dim=16, vdim=12, scale=0.3, chunk=20, rot_dims=8, base=1000.0, scaling=BANDS, v_mix=True, mlp="moe"):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix}
    if chunk is not None:
        m["mask"] = {"size": chunk}
    if rot_dims:
        m["rot"] = {"dims": rot_dims, "base": base, "scaling": scaling}
    return {"type": "attention", "mixer": m, "mlp": moe() if mlp == "moe" else mlp}


def make_config(layers, vocab=83, width=48, eps=1e-5, logit_scale=0.7):
    return {"architecture": "Lovulix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale, "layers": layers}


def random_weights(cfg: dict, seed: int = 0) -> dict:
    """name -> float32 array of bf16-representable values (so that both storage types hold the same numbers)."""
    rng = np.random.default_rng(seed)
    d = cfg["width"]
    w = {}

    def mat(n_out, n_in, gain=1.0):
        return bf16_round(rng.standard_normal((n_out, n_in)) * gain / np.sqrt(n_in))

    def vec(n, mean=0.0, std=0.1):
        return bf16_round(mean + std * rng.standard_normal(n))

    w["embed"] = bf16_round(rng.standard_normal((cfg["vocab"], d)))
    w["head"] = mat(cfg["vocab"], d, 3.0)
    w["final.norm"] = vec(d, 0.8, 0.4)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        w[p + "norm1"] = vec(d, 0.7, 0.3)
        w[p + "mix.q"], w[p + "mix.k"], w[p + "mix.v"] = mat(H * dk, d, 1.5), mat(G * dk, d, 1.5), mat(G * dv, d, 1.5)
        w[p + "mix.q.norm"], w[p + "mix.k.norm"] = vec(H * dk, 1.2, 0.4), vec(G * dk, 1.2, 0.4)
        w[p + "mix.vmix"] = np.float32(bf16_round(np.array([0.3 + 0.1 * i]))[0])
        w[p + "mix.talk"] = bf16_round(0.8 * np.eye(H) + 0.5 * rng.standard_normal((H, H)) / np.sqrt(H))
        w[p + "mix.sink"] = vec(H, 0.5, 1.0)
        w[p + "mix.g"], w[p + "mix.o"] = mat(H * dv, d, 1.5), mat(d, H * dv)
        mlp = l.get("mlp")
        if mlp:
            w[p + "norm2"] = vec(d, 0.7, 0.3)
            r, ff = mlp["router"], mlp["expert"]["ff"]
            parts = [(f"e{e}", ff) for e in range(r["experts"])] + ([("shared", mlp["shared"]["ff"])] if mlp.get("shared") else [])
            for n, f in parts:
                w[f"{p}mlp.{n}.gate"], w[f"{p}mlp.{n}.up"], w[f"{p}mlp.{n}.down"] = mat(f, d, 1.5), mat(f, d, 1.5), mat(d, f, 1.5)
            w[p + "mlp.router"] = mat(r["experts"], d, 4.0)      # scores far enough apart that a close call is rare
    return {k: np.asarray(v, dtype=np.float32) for k, v in w.items()}
