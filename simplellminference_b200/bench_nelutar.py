"""Throughput of the Nelutar design at layer sizes of real models (random weights), beside the closest model of the framework at equal
width and depth: Vasosun (the same sequence engine; window attention, the gated delta rule, a mixture of experts). Prompt tokens per second
of one whole prompt, and decoded tokens per second of 1 and 4 requests stepping together at a context of the prompt's length. Used by
``bench.py --nelutar``; prints one JSON object per model and size.

Timing and roofline fractions as in ``bench_hybrid`` (CUDA events on the launching stream, 3 warm-ups, medians). The algorithmic work of
a mixture-of-experts layer is that of the experts a token USES (``top`` of them and the shared one); where the implementation computes
every expert for every token the "executed" fractions show it. ``mechanisms_alone`` times the launches of one mechanism between its input
and its output product, on one layer's shapes, beside the like mechanism of an earlier design: window attention (Nelutar's two forms,
Vasosun's), the delta rule (a decay per key channel, Vasosun's decay per head) and the linear recurrences (constant decay, Kodezen's
state-space duality), each against the time its algorithmic bytes or products take at the measured peaks."""
from __future__ import annotations

import json

import numpy as np

from .bench_hybrid import _time
from .bench_vasosun import bench_vasosun

SIZES = {
    # name: width, layer pattern repeats ([parallel_2 (gated), parallel, retention, parallel_2 (experts)] each), prompt length
    "w1024": dict(width=1024, repeats=2, prompt=2048),
    "w2048": dict(width=2048, repeats=2, prompt=2048),
    "w4096": dict(width=4096, repeats=1, prompt=2048),
}
WINDOW = 1024
EXPERTS, TOP, GROUPS, KEEP = 8, 2, 4, 2
RANK = 128


def nelutar_config(width: int, repeats: int, vocab: int = 32000) -> dict:
    heads = width // 128
    ff = ((8 * width // 3) + 255) // 256 * 256
    attention = {"heads": heads, "kv_heads": max(1, heads // 4), "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": WINDOW}, "rot": {"dims": 128, "base": 500000.0}}
    decay = [1.0 - 2.0 ** (-5.0 - 3.0 * h / heads) for h in range(heads)]
    linear = {"heads": heads, "dim": 128, "vdim": 128, "decay": decay}
    dense = {"kind": "dense", "ff": ff}
    moe = {"kind": "moe", "expert": {"ff": ff // 2, "limit": 7.0}, "shared": {"ff": ff // 2, "limit": 7.0},
           "router": {"experts": EXPERTS, "top": TOP, "scale": 2.5, "groups": {"count": GROUPS, "keep": KEEP}}}
    pair2 = {"left": dict(attention, conv=4, softcap=30.0), "right": linear, "left_scale": 0.9, "right_scale": 1.05}
    layers = [{"type": "parallel_2", "mixer": pair2, "mlp": dense},
              {"type": "parallel", "mixer": {"left": attention, "right": {"heads": heads, "kv_heads": max(1, heads // 2), "dim": 128, "vdim": 128, "conv": 4}}, "mlp": moe},
              {"type": "retention", "mixer": dict(linear, rot={"dims": 128, "base": 10000.0}), "mlp": moe},
              {"type": "parallel_2", "mixer": pair2, "mlp": moe}] * repeats
    return {"architecture": "Nelutar", "vocab": vocab, "width": width, "norm": {"eps": 1e-6},
            "embedding": {"bigram": {"buckets": 65521, "mul_prev": 1000003, "mul_cur": 8191}}, "layers": layers}


def random_nelutar_weights(cfg: dict, device, seed: int = 0) -> dict:
    """Random bf16 tensors under the design's tensor names, made on the device."""
    import torch
    g = torch.Generator(device=device)
    g.manual_seed(seed)
    d = cfg["width"]

    def mat(n_out, n_in, gain=1.0):
        return (torch.randn(n_out, n_in, generator=g, device=device) * (gain / n_in ** 0.5)).to(torch.bfloat16)

    def vec(n, mean=0.0, std=0.1):
        return (mean + std * torch.randn(n, generator=g, device=device)).to(torch.bfloat16)

    def attention(p, m):
        H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for n, rows in (("q", H * dk), ("k", G * dk), ("v", G * dv)):
            w[p + n] = mat(rows, d)
            if m.get("conv"):
                w[p + n + ".conv"] = (0.5 * torch.randn(rows, m["conv"], generator=g, device=device)).to(torch.bfloat16)
        w[p + "o"] = mat(d, H * dv)

    def decayed(p, m, norm):
        H, dk, dv = m["heads"], m["dim"], m["vdim"]
        for n, rows in (("q", H * dk), ("k", H * dk), ("v", H * dv), ("g", H * dv)):
            w[p + n] = mat(rows, d)
        if norm:
            w[p + "norm"] = vec(H * dv, 1.0)
        w[p + "o"] = mat(d, H * dv)

    w = {"embed": torch.randn(cfg["vocab"], d, generator=g, device=device).to(torch.bfloat16), "head": mat(cfg["vocab"], d), "final.norm": vec(d, 1.0),
         "bigram": (0.5 * torch.randn(cfg["embedding"]["bigram"]["buckets"] + 1, d, generator=g, device=device)).to(torch.bfloat16)}
    for i, l in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", l["mixer"], l["mlp"]
        w[p + "norm1"], w[p + "ls1"], w[p + "ls2"] = vec(d, 1.0), vec(d, 0.5), vec(d, 0.5)
        if l["type"] == "parallel":
            attention(p + "mix.left.", m["left"])
            r, q = m["right"], p + "mix.right."
            H, G, dk, dv = r["heads"], r["kv_heads"], r["dim"], r["vdim"]
            for n, rows in (("q", G * dk), ("k", G * dk), ("v", H * dv)):
                w[q + n] = mat(rows, d)
                w[q + n + ".conv"] = (0.5 * torch.randn(rows, r["conv"], generator=g, device=device)).to(torch.bfloat16)
            w[q + "b"], w[q + "a1"], w[q + "a2"], w[q + "g1"], w[q + "g2"] = mat(H, d), mat(RANK, d), mat(H * dk, RANK), mat(RANK, d), mat(H * dv, RANK)
            w[q + "A_log"], w[q + "dt_bias"], w[q + "norm"], w[q + "o"] = vec(H, -1.0, 0.5), vec(H * dk), vec(dv, 1.0), mat(d, H * dv)
            w[p + "mix.left.out"], w[p + "mix.right.out"] = vec(d, 1.0), vec(d, 1.0)
        elif l["type"] == "parallel_2":
            attention(p + "mix.left.", m["left"])
            decayed(p + "mix.right.", m["right"], True)
        else:
            decayed(p + "mix.", m, False)
        if mlp["kind"] == "dense":
            w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"] = mat(mlp["ff"], d), mat(mlp["ff"], d), mat(d, mlp["ff"])
        else:
            for n, f in [(f"e{e}", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])] + [("shared", mlp["shared"]["ff"])]:
                w[f"{p}mlp.{n}.gate"], w[f"{p}mlp.{n}.up"], w[f"{p}mlp.{n}.down"] = mat(f, d), mat(f, d), mat(d, f)
            w[p + "mlp.router"], w[p + "mlp.correction"] = mat(mlp["router"]["experts"], d, 2.0), vec(mlp["router"]["experts"], 0.0, 0.05)
    return w


def _used_params(cfg: dict, w: dict) -> tuple:
    """(matrix parameters a token uses, all matrix parameters): a routed expert counts by the share of tokens it gets."""
    total = used = 0.0
    for n, t in w.items():
        if t.dim() < 2 or n in ("embed", "bigram") or n.endswith(".conv"):
            continue
        total += t.numel()
        share = 1.0
        if ".mlp.e" in n:
            r = cfg["layers"][int(n[1:n.index(".")])]["mlp"]["router"]
            share = r["top"] / r["experts"]
        used += share * t.numel()
    return used, total


def _state_bytes(cfg: dict, T: int) -> int:
    """Bytes a decoding step must read per request besides the matrices: cache rows inside the windows (bf16), recurrent states (fp32, read
    and written)."""
    n = 0
    for l in cfg["layers"]:
        m = l["mixer"]
        if "left" in m:
            a = m["left"]
            n += 2 * min(T, a["mask"]["size"]) * a["kv_heads"] * (a["dim"] + a["vdim"])
        r = m.get("right", m)
        n += 2 * 4 * r["heads"] * r["dim"] * r["vdim"]
    return n


# ------------------------------------------------------------------------------------------------ mechanisms alone
def _mechanisms(width: int, ops, dev):
    """(name, mechanism, widths of its input columns): Nelutar's and the like ones of earlier designs, at this module's layer shapes."""
    import torch

    from . import layers as M
    from .config import (ConvRotaryAttentionConfig, DecayedAttentionConfig, DeltaRuleConfig, LogDistanceAttentionConfig, RotaryConfig, StateSpaceDualityConfig, WindowMask)
    H, dk = width // 128, 128
    G, eps = max(1, H // 4), 1e-6
    K = max(1, H // 2)
    gen = torch.Generator(device=dev)
    gen.manual_seed(3)
    mat = lambda *s: (0.1 * torch.randn(*s, device=dev, generator=gen)).to(torch.bfloat16)   # noqa: E731
    att = {"m." + n: mat(rows, 8) for n, rows in (("q", H * dk), ("k", G * dk), ("v", G * dk))}
    att.update({f"m.{n}.conv": mat(rows, 4) for n, rows in (("q", H * dk), ("k", G * dk), ("v", G * dk))})
    att.update({"m.o": mat(width, H * dk), "m.r1": mat(H).abs(), "m.r2": mat(H).abs()})
    rot, mask = RotaryConfig(dk, 5e5), WindowMask(WINDOW)
    delta = {"m." + n: mat(rows, 8) for n, rows in (("q", K * dk), ("k", K * dk), ("v", H * dk), ("b", H), ("a", H), ("g", H * dk), ("a1", RANK), ("g1", RANK))}
    delta.update({f"m.{n}.conv": mat(rows, 4) for n, rows in (("q", K * dk), ("k", K * dk), ("v", H * dk))})
    delta.update({"m.a2": mat(H * dk, RANK), "m.g2": mat(H * dk, RANK), "m.A_log": mat(H) - 1, "m.norm": mat(dk), "m.o": mat(width, H * dk)})
    lin = {"m." + n: mat(H * dk, 8) for n in ("q", "k", "v", "g")}
    lin.update({"m.o": mat(width, H * dk), "m.norm": mat(H * dk)})
    decay = tuple(1.0 - 2.0 ** (-5.0 - 3.0 * h / H) for h in range(H))
    ssd_channels = (H + 2) * dk
    ssd = {"m.in": mat(H * dk + ssd_channels + H, 8), "m.conv": mat(ssd_channels, 4), "m.A_log": mat(H) - 1, "m.dt_bias": mat(H), "m.norm": mat(H * dk), "m.o": mat(width, H * dk)}
    deltac = DeltaRuleConfig(H, K, dk, dk, 4)
    return [("attention: rotary window", M.ConvRotaryAttention(ConvRotaryAttentionConfig(H, G, dk, dk, dk ** -0.5, rot, mask), att, "m.", ops, dev, eps)),
            ("attention: convolved, normed, capped", M.ConvRotaryAttention(ConvRotaryAttentionConfig(H, G, dk, dk, dk ** -0.5, rot, mask, 30.0, 4), att, "m.", ops, dev, eps, unit_heads=True)),
            ("attention: log-distance window (Vasosun)", M.LogDistanceWindowAttention(LogDistanceAttentionConfig(H, G, dk, dk, dk ** -0.5, mask, 0.1, 1024), att, "m.", ops, dev)),
            ("delta rule: decay per key channel", M.ChannelDeltaRule(deltac, dict(delta, **{"m.dt_bias": mat(H * dk)}), "m.", ops, dev, eps)),
            ("delta rule: decay per head (Vasosun)", M.GatedDeltaRule(deltac, dict(delta, **{"m.dt_bias": mat(H)}), "m.", ops, dev, eps)),
            ("linear: retention", M.DecayedAttention(DecayedAttentionConfig(H, dk, dk, decay, RotaryConfig(dk, 1e4)), lin, "m.", ops, dev, eps, kscale=dk ** -0.5)),
            ("linear: lightning", M.DecayedAttention(DecayedAttentionConfig(H, dk, dk, decay), lin, "m.", ops, dev, eps, silu=True, row_norm=True, sigmoid_gate=True)),
            ("linear: state-space duality (Kodezen)", M.StateSpaceDuality(StateSpaceDualityConfig(H, dk, dk, 1, 1, 4), ssd, "m.", ops, dev, eps))]


def _alone(mech, T: int, context: int = 0) -> float:
    """Milliseconds of the mechanism's launches (no input or output product): a prompt of ``T`` tokens, or one token behind ``context``."""
    import torch

    from .seqengine import SequenceEngine
    dev, ops = mech.out.w.device, mech.ops
    sizes = [int(p[0].shape[0]) for p in mech.inputs]
    n = sum(sizes)
    offs = [sum(sizes[:i]) for i in range(len(sizes))]
    gen = torch.Generator(device=dev)
    gen.manual_seed(1)
    cols = torch.randn(max(T, context), n, device=dev, generator=gen)

    class One:
        device = dev

        def state_specs(self):
            return [mech.state_spec()]

        def forward(self, step, ids, states, rows, n_rows, tap=None):
            c = cols[:step.T] if step.T > 1 else cols[-1:]

            def call():
                step.turned.clear()
                step.st = torch.cuda.current_stream(dev).cuda_stream
                mech.forward(step, [c.data_ptr() + 4 * o for o in offs], n, states[0], step.scratch("mix_part", step.T * mech.width))
            self.call = call
            call()

    model = One()
    model.ops = ops
    eng = SequenceEngine(model, max_tokens=T + context + 64, max_seqs=1, graphs=False)
    slot = eng.admit()
    if context:
        eng.run([(slot, np.zeros(context, np.int32), [])])
    eng.run([(slot, np.zeros(T, np.int32), [])])      # the engine keeps the step as it is: its launches can be captured and repeated
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        model.call()
    flush = torch.empty(64 * 1024 * 1024, dtype=torch.float32, device=dev)      # larger than L2
    ms = []
    for _ in range(13):
        flush.zero_()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        graph.replay()
        b.record()
        torch.cuda.synchronize()
        ms.append(a.elapsed_time(b))
    return float(np.median(ms[3:]))


def bench_mechanisms(width: int, T: int, hbm_gbs: float, tflops: float) -> dict:
    """Per mechanism: time of a prompt and of one token behind it, and how far each is from the time its bytes (inputs, result, state or
    visible cache rows) or its products take at the measured peaks."""
    import torch

    from .config import BF16
    from .seqops import Ops
    ops = Ops(BF16)
    H, dk = width // 128, 128
    G = max(1, H // 4)
    out = {}
    for name, mech in _mechanisms(width, ops, torch.device("cuda")):
        row_bytes = 4.0 * (sum(int(p[0].shape[0]) for p in mech.inputs)) + 2.0 * mech.width      # fp32 columns in, bf16 operand rows out
        keys = np.minimum(np.arange(T) + 1, WINDOW)
        if name.startswith("attention"):
            flops, token_bytes = float(keys.sum()) * H * 4 * dk, 2.0 * WINDOW * G * 2 * dk
        else:
            flops, token_bytes = float(T) * H * (6 if name.startswith("delta") else 4) * dk * dk, 2.0 * 4 * H * dk * dk
        p, t = _alone(mech, T), _alone(mech, 1, context=T)
        floor_p = max(T * row_bytes / (hbm_gbs * 1e9), flops / (tflops * 1e12)) * 1e3
        floor_t = (row_bytes + token_bytes) / (hbm_gbs * 1e9) * 1e3
        out[name] = {"prompt_ms": round(p, 4), "prompt_fraction_of_roofline": round(floor_p / p, 4), "decode_us": round(1e3 * t, 2), "decode_fraction_of_roofline": round(floor_t / t, 4)}
    return out


def bench_nelutar(name: str, hbm_gbs: float, tflops: float) -> dict:
    import torch

    from .config import BF16, NelutarConfig
    from .layers import ExpertsFeedForward
    from .models.nelutar import NelutarModel
    from .seqengine import SequenceEngine
    from .seqops import Ops
    size = SIZES[name]
    dev = torch.device("cuda")
    cfg = nelutar_config(size["width"], size["repeats"])
    w = random_nelutar_weights(cfg, dev)
    used, total = _used_params(cfg, w)
    ops = Ops(BF16)
    model = NelutarModel(NelutarConfig.from_dict(cfg), w, ops, dev)
    T = size["prompt"]
    eng = SequenceEngine(model, max_tokens=4 * (T + 128), max_seqs=4)
    rng = np.random.default_rng(1)
    prompt = rng.integers(0, cfg["vocab"], size=T).astype(np.int32)

    def prefill():
        s = eng.admit()
        eng.run([(s, prompt, [T - 1])])
        eng.release(s)

    l0 = ops.launches
    prefill_ms = _time(prefill, 5)
    out = {"model": f"nelutar-{name}", "width": size["width"], "layers": len(cfg["layers"]), "matrix_params": int(total), "matrix_params_used_per_token": int(used),
           "prompt_len": T, "prefill_ms": round(prefill_ms, 3), "prefill_tokens_per_sec": round(T / prefill_ms * 1e3, 1),
           "prefill_gemm_tflops": round(2.0 * used * T / prefill_ms / 1e9, 1), "prefill_gemm_tflops_executed": round(2.0 * total * T / prefill_ms / 1e9, 1),
           "prefill_launches": (ops.launches - l0) // 8}
    experts = [m for l in model.layers for _, m, _ in l.group.members if isinstance(m, ExpertsFeedForward)]
    gathered = bool(experts) and all(f._gathered_pays(T) for f in experts)
    if gathered:                                     # a token is multiplied with the experts it uses only
        out["prefill_gemm_tflops_executed"] = out["prefill_gemm_tflops"]
    out["prefill_fraction_of_measured_bf16_peak"] = round(out["prefill_gemm_tflops"] / tflops, 3)
    out["prefill_fraction_of_measured_bf16_peak_executed"] = round(out["prefill_gemm_tflops_executed"] / tflops, 3)
    state_bytes = _state_bytes(cfg, T)
    for n in (1, 4):
        slots = [eng.admit() for _ in range(n)]
        eng.run([(s, prompt, []) for s in slots])
        tok = [int(prompt[-1])] * n

        def step():
            eng.run([(s, [t], [0]) for s, t in zip(slots, tok)])

        ms = _time(step, 30, warmup=4)
        out[f"decode{n}_ms_per_step"] = round(ms, 4)
        out[f"decode{n}_tokens_per_sec"] = round(n / ms * 1e3, 1)
        # one request reads the experts it uses; four requests together touch most of them
        weights = used if n == 1 else total
        executed = used if (n == 1 and experts and all(f._indexed_pays(n) for f in experts)) else total
        out[f"decode{n}_fraction_of_measured_hbm"] = round((2.0 * weights + n * state_bytes) / (ms * 1e-3) / (hbm_gbs * 1e9), 3)
        out[f"decode{n}_fraction_of_measured_hbm_executed"] = round((2.0 * executed + n * state_bytes) / (ms * 1e-3) / (hbm_gbs * 1e9), 3)
        for s in slots:
            eng.release(s)
    out["graph_replays"] = eng.graph_replays
    return out


def main(sizes, hbm_gbs: float, tflops: float) -> list:
    """A size named ``<size>-alone`` runs Nelutar without the model beside it (for a launch list of one model)."""
    res = []
    for name in sizes:
        alone = name.endswith("-alone")
        name = name[:-len("-alone")] if alone else name
        arms = [("nelutar", lambda: bench_nelutar(name, hbm_gbs, tflops))]
        if not alone:
            arms.append(("vasosun", lambda: bench_vasosun(name, hbm_gbs, tflops)))
            arms.append(("mechanisms", lambda: {"mechanisms_alone": SIZES[name]["width"], **bench_mechanisms(SIZES[name]["width"], SIZES[name]["prompt"], hbm_gbs, tflops)}))
        for label, fn in arms:
            try:
                r = fn()
            except Exception as ex:   # one size that does not fit or run must not hide the others
                r = {"model": f"{label}-{name}", "error": f"{type(ex).__name__}: {ex}"[:300]}
            print(json.dumps(r), flush=True)
            res.append(r)
    return res
