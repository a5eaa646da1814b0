"""Throughput of the Lovulix design at layer sizes of real models (random weights), beside the closest model of the framework at equal
width and depth: Kodezen (the same sequence engine; attention whose heads are mixed after the softmax, the same mixture of gated experts).
Prompt tokens per second of one whole prompt, and decoded tokens per second of 1 and 4 requests stepping together at a context of the
prompt's length. Used by ``bench.py --lovulix``; prints one JSON object per model and size.

Timing and roofline fractions as in ``bench_hybrid`` (CUDA events on the launching stream, 3 warm-ups, medians). The algorithmic work of
a mixture-of-experts layer is that of the experts a token USES (``top`` of them and the shared one); where the implementation computes
every expert for every token the "executed" fractions show it. ``attention_*`` times the two mixers' attention launches alone (the
preparation kernel, the attention and, where the design has them, merge and head mix) on one layer's shapes, against the products a
score-and-value pass needs by definition: 2 (dim + vdim) per query head and visible key, plus 2 per pair of heads for the mix."""
from __future__ import annotations

import json

import numpy as np

from .bench_hybrid import _time
from .bench_kodezen import KEEP_FIRST, WINDOW, bench_kodezen

SIZES = {
    # name: width, layers, prompt length
    "w1024": dict(width=1024, layers=8, prompt=2048),
    "w2048": dict(width=2048, layers=8, prompt=2048),
    "w4096": dict(width=4096, layers=4, prompt=2048),
}
CHUNK = 1024
EXPERTS, TOP = 8, 2


def lovulix_config(width: int, layers: int, vocab: int = 32000) -> dict:
    heads = width // 128
    ff = ((4 * width // 3) + 127) // 128 * 128
    mixer = {"heads": heads, "kv_heads": max(1, heads // 4), "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": CHUNK}, "v_mix": True,
             "rot": {"dims": 128, "base": 500000.0, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}}
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": EXPERTS, "top": TOP}, "shared": {"ff": ff}}
    return {"architecture": "Lovulix", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "logit_scale": 0.25,
            "layers": [{"type": "attention", "mixer": mixer, "mlp": mlp} for _ in range(layers)]}


def random_lovulix_weights(cfg: dict, device, seed: int = 0) -> dict:
    """Random bf16 tensors under the design's tensor names, made on the device."""
    import torch
    g = torch.Generator(device=device)
    g.manual_seed(seed)
    d = cfg["width"]

    def mat(n_out, n_in, gain=1.0):
        return (torch.randn(n_out, n_in, generator=g, device=device) * (gain / n_in ** 0.5)).to(torch.bfloat16)

    def vec(n, mean=0.0, std=0.1):
        return (mean + std * torch.randn(n, generator=g, device=device)).to(torch.bfloat16)

    w = {"embed": torch.randn(cfg["vocab"], d, generator=g, device=device).to(torch.bfloat16), "head": mat(cfg["vocab"], d), "final.norm": vec(d, 1.0)}
    for i, l in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", l["mixer"], l["mlp"]
        H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        w[p + "norm1"], w[p + "norm2"] = vec(d, 0.5), vec(d, 0.5)
        w[p + "mix.q"], w[p + "mix.k"], w[p + "mix.v"], w[p + "mix.g"], w[p + "mix.o"] = mat(H * dk, d), mat(G * dk, d), mat(G * dv, d), mat(H * dv, d), mat(d, H * dv)
        w[p + "mix.q.norm"], w[p + "mix.k.norm"], w[p + "mix.sink"], w[p + "mix.vmix"] = vec(H * dk, 1.0), vec(G * dk, 1.0), vec(H), vec(1, 0.5)[0]
        w[p + "mix.talk"] = (torch.eye(H, device=device) + 0.2 * torch.randn(H, H, generator=g, device=device) / H ** 0.5).to(torch.bfloat16)
        ff, sff = mlp["expert"]["ff"], mlp["shared"]["ff"]
        for e in range(mlp["router"]["experts"]):
            w[f"{p}mlp.e{e}.gate"], w[f"{p}mlp.e{e}.up"], w[f"{p}mlp.e{e}.down"] = mat(ff, d), mat(ff, d), mat(d, ff)
        w[p + "mlp.shared.gate"], w[p + "mlp.shared.up"], w[p + "mlp.shared.down"] = mat(sff, d), mat(sff, d), mat(d, sff)
        w[p + "mlp.router"] = mat(mlp["router"]["experts"], d, 2.0)
    return w


def _used_params(cfg: dict, w: dict) -> tuple:
    """(matrix parameters a token uses, all matrix parameters): a routed expert counts by the share of tokens it gets."""
    total = used = 0.0
    for n, t in w.items():
        if t.dim() < 2 or n == "embed" or n.endswith("talk"):
            continue
        total += t.numel()
        share = 1.0
        if ".mlp.e" in n:
            r = cfg["layers"][int(n[1:n.index(".")])]["mlp"]["router"]
            share = r["top"] / r["experts"]
        used += share * t.numel()
    return used, total


def _cache_bytes(cfg: dict, pos: int) -> int:
    """Bytes of cache rows (bf16) the token at ``pos`` must read: those of its own chunk."""
    return sum(2 * (pos % l["mixer"]["mask"]["size"] + 1) * l["mixer"]["kv_heads"] * (l["mixer"]["dim"] + l["mixer"]["vdim"]) for l in cfg["layers"])


def _attention_alone(T: int, width: int, mixes_first: bool, context: int = 0):
    """(milliseconds, algorithmic FLOPs, algorithmic cache bytes) of one layer's attention launches: a prompt of ``T`` tokens, or with
    ``context`` a single token behind that many. ``mixes_first``: this design's mixer, else the one that mixes after the softmax."""
    import torch

    from .config import BF16, RotaryConfig, ScoreMixingAttentionConfig, TalkingHeadsAttentionConfig, WindowMask
    from .layers import ScoreMixingAttention, TalkingHeadsAttention
    from .seqengine import SequenceEngine
    from .seqops import Ops
    dev, ops = torch.device("cuda"), Ops(BF16)
    H, dk = width // 128, 128
    G = max(1, H // 4)
    ones = lambda *s: torch.ones(*s, device=dev, dtype=torch.bfloat16)   # noqa: E731
    w = {"m.q": ones(H * dk, 8), "m.k": ones(G * dk, 8), "m.v": ones(G * dk, 8), "m.g": ones(H * dk, 8), "m.o": ones(width, H * dk), "m.talk": ones(H, H), "m.sink": ones(H)}
    if mixes_first:
        w.update({"m.q.norm": ones(H * dk), "m.k.norm": ones(G * dk)})
        mech = ScoreMixingAttention(ScoreMixingAttentionConfig(H, G, dk, dk, dk ** -0.5, RotaryConfig(dk, 1e4), CHUNK, False), w, "m.", ops, dev, 1e-6)
        n = (2 * H + 2 * G) * dk
    else:
        w.update({"m.q.norm": ones(dk), "m.k.norm": ones(dk)})
        mech = TalkingHeadsAttention(TalkingHeadsAttentionConfig(H, G, dk, dk, dk ** -0.5, RotaryConfig(64, 1e4), WindowMask(WINDOW, KEEP_FIRST), 1), w, "m.", ops, dev, 1e-6)
        n = (H + G) * dk
    gen = torch.Generator(device=dev)
    gen.manual_seed(1)
    total = context + T
    cols = torch.randn(total, n, device=dev, generator=gen)
    offs = [0, H * dk, (H + G) * dk, (H + 2 * G) * dk]

    class One:
        ops, device = None, dev

        def state_specs(self):
            return [mech.state_spec()]

        def forward(self, step, ids, states, rows, n_rows, tap=None):
            c = cols[:step.T] if step.T > 1 else cols[-1:]

            def call():
                step.turned.clear()
                step.st = torch.cuda.current_stream(dev).cuda_stream
                mech.forward(step, [c.data_ptr() + 4 * o for o in offs[:len(mech.inputs)]], n, states[0], step.scratch("mix_part", step.T * mech.width))
            self.call = call
            call()

    model = One()
    model.ops = ops
    eng = SequenceEngine(model, max_tokens=total + 64, max_seqs=1, graphs=False)
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
    pos = np.arange(context, total)
    keys = (pos % CHUNK + 1) if mixes_first else np.minimum(pos + 1, WINDOW) + np.where(pos >= WINDOW, np.minimum(KEEP_FIRST, pos + 1 - WINDOW), 0)
    return float(np.median(ms[3:])), float(keys.sum()) * H * (2 * (dk + dk) + 2 * H), float(2 * keys[-1] * G * 2 * dk)


def bench_attention(width: int, T: int, hbm_gbs: float, tflops: float) -> dict:
    out = {}
    for name, first in (("lovulix", True), ("kodezen", False)):
        ms, flops, _ = _attention_alone(T, width, first)
        out[name] = {"prompt_ms": round(ms, 4), "prompt_algorithmic_tflops": round(flops / ms / 1e9, 1), "prompt_fraction_of_measured_bf16_peak": round(flops / ms / 1e9 / tflops, 4)}
        # the token at the end of a chunk / behind a full window
        ms, _, nbytes = _attention_alone(1, width, first, context=2 * CHUNK - 1)
        out[name].update({"decode_us": round(1e3 * ms, 2), "decode_fraction_of_measured_hbm": round(nbytes / (ms * 1e-3) / (hbm_gbs * 1e9), 4)})
    return out


def bench_lovulix(name: str, hbm_gbs: float, tflops: float) -> dict:
    import torch

    from .config import BF16, LovulixConfig
    from .layers import ExpertsFeedForward
    from .models.lovulix import LovulixModel
    from .seqengine import SequenceEngine
    from .seqops import Ops
    size = SIZES[name]
    dev = torch.device("cuda")
    cfg = lovulix_config(size["width"], size["layers"])
    w = random_lovulix_weights(cfg, dev)
    used, total = _used_params(cfg, w)
    ops = Ops(BF16)
    model = LovulixModel(LovulixConfig.from_dict(cfg), w, ops, dev)
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
    out = {"model": f"lovulix-{name}", "width": size["width"], "layers": len(cfg["layers"]), "matrix_params": int(total), "matrix_params_used_per_token": int(used),
           "prompt_len": T, "prefill_ms": round(prefill_ms, 3), "prefill_tokens_per_sec": round(T / prefill_ms * 1e3, 1),
           "prefill_gemm_tflops": round(2.0 * used * T / prefill_ms / 1e9, 1), "prefill_gemm_tflops_executed": round(2.0 * total * T / prefill_ms / 1e9, 1),
           "prefill_launches": (ops.launches - l0) // 8}
    out["prefill_fraction_of_measured_bf16_peak"] = round(out["prefill_gemm_tflops"] / tflops, 3)
    out["prefill_fraction_of_measured_bf16_peak_executed"] = round(out["prefill_gemm_tflops_executed"] / tflops, 3)
    experts = [l.ff for l in model.layers if isinstance(l.ff, ExpertsFeedForward)]
    for n in (1, 4):
        slots = [eng.admit() for _ in range(n)]
        eng.run([(s, prompt[:-40], []) for s in slots])      # the timed steps then run at the end of a chunk
        tok = [int(prompt[-1])] * n

        def step():
            eng.run([(s, [t], [0]) for s, t in zip(slots, tok)])

        ms = _time(step, 30, warmup=4)
        state_bytes = _cache_bytes(cfg, T - 20)
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
    """A size named ``<size>-alone`` runs Lovulix without the model beside it (for a launch list of one model)."""
    res = []
    for name in sizes:
        alone = name.endswith("-alone")
        name = name[:-len("-alone")] if alone else name
        arms = [("lovulix", lambda: bench_lovulix(name, hbm_gbs, tflops))]
        if not alone:
            arms.append(("kodezen", lambda: bench_kodezen(name, hbm_gbs, tflops)))
            arms.append(("attention", lambda: {"attention_alone": SIZES[name]["width"], **bench_attention(SIZES[name]["width"], SIZES[name]["prompt"], hbm_gbs, tflops)}))
        for label, fn in arms:
            try:
                r = fn()
            except Exception as ex:   # one size that does not fit or run must not hide the others
                r = {"model": f"{label}-{name}", "error": f"{type(ex).__name__}: {ex}"[:300]}
            print(json.dumps(r), flush=True)
            res.append(r)
    return res
