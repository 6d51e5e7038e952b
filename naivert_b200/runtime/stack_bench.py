"""Throughput of layer-stack models at the sizes of a real model's layers (random weights on the device).

    python bench.py --workload stack [--model tumatar-bench|tumatar-bench-dense|zuzupel-bench] [--prompt 8192] [--steps 64] [--kernels]

Prefill: one prompt through the chunk path, CUDA events around the run.  Decode: rounds of the captured graph behind that
prompt (step + sampler + tail), CUDA events around K replays.  ``--kernels`` adds tables with one row per kernel kind: time,
the bytes it must move or the FLOPs it must do, and the fraction of the copy bandwidth / dense bf16 rate (recurrences on the
CUDA cores: nominal fp32 rate) that is.  Weights of one
token or chunk exceed the 126 MB L2, so no flush is needed between iterations.
"""
from __future__ import annotations

import json
import os
from typing import Dict, List, Tuple

import torch

from ..models.registry import resolve_model
from ..models.spec import SamplingParams
from ..prefill.stack_mixers import MIXERS as CHUNK_MIXERS
from .stack_mixers import MIXERS
from .engine import Engine

FP32_TFLOPS = 148 * 128 * 2 * 1.965e-3          # CUDA cores, nominal: SMs x lanes x FMA x boost clock
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}


def peaks() -> dict:
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__)))), "MEASURED_PEAKS.json")
    if os.path.isfile(path):
        d = json.load(open(path))
        return {"hbm_gbs": float(d["hbm_gbs"]), "bf16_tflops": float(d["bf16_tflops"]), "source": "measured"}
    return FALLBACK_PEAKS


# --------------------------------------------------------------------------- work per kernel kind
class Work:
    """(tensor-core FLOPs, bytes, CUDA-core fp32 FLOPs) by stage; bytes are the operands once."""

    def __init__(self, hidden: int, es: int):
        self.W, self.es, self.stages = hidden, es, {}

    def add(self, name: str, flops: float, nbytes: float, flops32: float = 0.0) -> None:
        a = self.stages.setdefault(name, [0.0, 0.0, 0.0])
        for i, v in enumerate((flops, nbytes, flops32)):
            a[i] += v

    def add32(self, name: str, flops32: float, nbytes: float) -> None:
        self.add(name, 0.0, nbytes, flops32)

    def gemm(self, name: str, n: int, k: int, rows: int, out_bytes: int, z: int = 1, mats: int = 1) -> None:
        self.add(name, 2.0 * n * k * rows * z * mats, z * (mats * n * k * 2 + rows * k * self.es + rows * n * out_bytes))


def chunk_work(eng, pos0: int, R: int) -> Dict[str, List[float]]:
    """Work per stage over all runs of one chunk at ``pos0``."""
    spec = eng.spec
    W, es = spec.hidden, 4 if eng.target.f32 else 2
    w = Work(W, es)
    for r in eng.target.runs:
        d = r["layer"]
        m, f = d["spec"].mixer, d["spec"].mlp
        w.add("rows", 0, R * W * (4 + 4 + 4 + es))
        CHUNK_MIXERS[d["kind"]].work(w, m, d, pos0, R)
        if f is None:
            continue
        w.add("rows", 0, R * W * (4 + 4 + 4 + es))
        if f.kind == "relu2":
            w.gemm("ff_up", f.ff, W, R, es)
            w.gemm("ff_down", W, f.ff, R, 4)
        elif f.kind == "dense":
            w.gemm("dense_gate_up", f.ff, W, R, es, mats=2)
            w.gemm("dense_down", W, f.ff, R, 4)
        else:
            rt = f.routing
            P = R * rt.top_k
            used = min(rt.expert_count, P)
            w.gemm("router", rt.expert_count, W, R, 4)
            w.add("choice", 0, R * rt.expert_count * 4)
            w.add("expert_count", 0, P * 8)
            w.add("expert_gather", 0, 2 * P * W * es)
            w.add("expert_gate_up", 4.0 * P * W * f.ff, used * 2 * W * f.ff * 2 + P * (W + f.ff) * es)
            w.add("expert_down", 2.0 * P * W * f.ff, used * W * f.ff * 2 + P * (f.ff * es + W * 4))
    return w.stages


def step_work(eng, pos: int) -> List[Tuple[str, float]]:
    """(kind, bytes that must move) of every launch of the step, in launch order."""
    out: List[Tuple[str, float]] = []
    t = eng.target
    for r in t.runs:
        d = r["layer"]
        f = d["spec"].mlp
        out += MIXERS[d["kind"]].step_work(t, d["spec"].mixer, d, pos)
        if f is None:
            continue
        if f.kind == "relu2":
            out += [("ff_up", d["up"].nbytes), ("ff_down", d["down"].nbytes)]
        elif f.kind == "dense":
            out += [("dense_gate_up", 2 * d["gate"].nbytes), ("dense_down", d["down"].nbytes)]
        else:
            per = d["gate"].n * d["gate"].ld * 2
            k = f.routing.top_k
            out += [("router", d["router"].nbytes), ("expert_gate_up", 2 * k * per), ("expert_down", k * d["down"].n * d["down"].ld * 2)]
    return out + [("head", t.head.nbytes)]


# --------------------------------------------------------------------------- measurements
def chunk_table(eng, prompt: torch.Tensor, pos0: int, R: int) -> List[dict]:
    pf, pk = eng.prefill, peaks()
    pf.extend(prompt[pos0:pos0 + R], pos0)
    pf.profile = True
    reps = 3
    for _ in range(reps):
        pf.extend(prompt[pos0:pos0 + R], pos0)          # recurrent layers restart from the slot tagged pos0
    ms = pf.stage_ms()
    pf.profile = False
    work = chunk_work(eng, pos0, R)
    rows = []
    for name, (total, calls) in sorted(ms.items(), key=lambda kv: -kv[1][0]):
        t = total / reps * 1e-3
        fl, by, f32 = work.get(name, (0.0, 0.0, 0.0))
        bound = max(fl / (pk["bf16_tflops"] * 1e12), by / (pk["hbm_gbs"] * 1e9), f32 / (FP32_TFLOPS * 1e12))
        rows.append({"kernel": name, "calls": calls // reps, "ms": round(t * 1e3, 3), "tflops": round((fl + f32) / t * 1e-12, 1),
                     "gbs": round(by / t * 1e-9, 1), "roofline": round(bound / t, 3)})
    return rows


def step_table(eng, pos: int, steps: int = 4) -> List[dict]:
    """Kernel times of the step without programmatic overlap (CUPTI records), matched to the launch list in order."""
    from torch.profiler import ProfilerActivity, profile
    t, pk = eng.target, peaks()
    pdl, t.pdl = t.pdl, False
    t.set_inputs([1], pos)
    t.step()
    torch.cuda.synchronize()
    with profile(activities=[ProfilerActivity.CUDA]) as prof:
        for _ in range(steps):
            t.step()
        torch.cuda.synchronize()
    t.pdl = pdl
    ev = sorted((e for e in prof.events() if any(x in e.name for x in ("stack_", "latent_", "state_step", "group_decode"))), key=lambda e: e.time_range.start)
    work = step_work(eng, pos)
    if len(ev) != steps * len(work):
        raise RuntimeError(f"{len(ev)} kernel records for {steps} x {len(work)} launches")
    agg: Dict[str, List[float]] = {}
    for i, e in enumerate(ev):
        name, nbytes = work[i % len(work)]
        a = agg.setdefault(name, [0.0, 0.0, 0])
        a[0] += e.device_time if hasattr(e, "device_time") else e.cuda_time
        a[1] += nbytes
        a[2] += 1
    return [{"kernel": k, "calls": v[2] // steps, "us_each": round(v[0] / v[2], 2), "mb_each": round(v[1] / v[2] / 1e6, 2),
             "gbs": round(v[1] / v[0] * 1e-3, 1), "roofline": round(v[1] / v[0] * 1e-3 / pk["hbm_gbs"], 3)}
            for k, v in sorted(agg.items(), key=lambda kv: -kv[1][0])]


def closest_stack(model: str) -> str:
    """The layer-stack model of equal width, feed-forward and vocabulary that a design is measured beside ("": none)."""
    return {"zuzupel-bench": "tumatar-bench-dense"}.get(model, "")


def closest(prompt_len: int, chunk: int, layers: int, steps: int) -> dict:
    """The speculative target (W8A8, same width, heads and experts) at equal depth: chunked prefill, its eight-row step, and the
    kernels of both with the weight bytes they must read or the FLOPs they must do."""
    from torch.profiler import ProfilerActivity, profile
    spec, pk = resolve_model("naive-n0.5").with_layers(layers), peaks()
    dev = torch.device("cuda", torch.cuda.current_device())
    eng = Engine.build(spec, capacity=-(-(prompt_len + 256) // 128) * 128, device=dev, prefill_chunk=chunk)
    try:
        g = torch.Generator().manual_seed(0)
        prompt = torch.randint(0, spec.vocab - 16, (prompt_len + 1,), generator=g, dtype=torch.int32).pin_memory()
        pf, t = eng.prefill, eng.target
        pf.warm_chunks([pf.quantum, chunk])
        pf.run(prompt, 0, prompt_len)
        pre_ms = sorted((pf.run(prompt, 0, prompt_len), pf.executor_ms())[1] for _ in range(3))[1]
        pf.profile = True
        pf.run(prompt, prompt_len - chunk, prompt_len)
        stages = pf.stage_ms()
        pf.profile = False
        flops = {"qkv_gemm": sum(d["wqkv"].numel() for d in t.layers), "o_gemm": sum(d["wo"].w.numel() for d in t.layers)}
        table = [{"stage": k, "ms": v, **({"tflops": round(2.0 * flops[k] * chunk / v * 1e-9, 1),
                                          "roofline": round(2.0 * flops[k] * chunk / v * 1e-9 / pk["bf16_tflops"], 3)} if k in flops else {})}
                 for k, v in sorted(stages.items(), key=lambda kv: -kv[1])]
        pdl, t.pdl = t.pdl, False
        t.set_inputs(torch.arange(8), prompt_len)
        for _ in range(3):
            t.step()
        torch.cuda.synchronize()
        with profile(activities=[ProfilerActivity.CUDA]) as prof:
            for _ in range(steps):
                t.step()
            torch.cuda.synchronize()
        t.pdl = pdl
        by_name: Dict[str, List[float]] = {}
        for e in prof.events():
            n = e.name.replace("(anonymous namespace)::", "").split("(")[0]
            by_name.setdefault(n, []).append(e.device_time if hasattr(e, "device_time") else e.cuda_time)
        rt = spec.routing
        active = rt.expert_count * (1 - (1 - rt.top_k / rt.expert_count) ** 8)
        moe_bytes = active * 3 * rt.intermediate * spec.hidden
        mean = {"moe_layer_kernel": moe_bytes, "6": sum(d["wqkv"].numel() for d in t.layers) / layers * 2}
        rows = []
        for n, v in sorted(by_name.items(), key=lambda kv: -sum(kv[1])):
            r = {"kernel": n[-90:], "calls": len(v) // steps, "us_each": round(sum(v) / len(v), 2)}
            by = moe_bytes if "moe_layer" in n else mean["6"] if "false, false, 6" in n else None
            if by:
                r.update(mb_each=round(by / 1e6, 1), roofline=round(by / (sum(v) / len(v)) * 1e-3 / pk["hbm_gbs"], 3))
            rows.append(r)
        return {"model": spec.name, "dtype": "fp8 weights and activations", "prefill_tokens_per_s": round(prompt_len / (pre_ms * 1e-3), 1),
                "prefill_stages_last_chunk": table, "step8_kernels": rows, "step8_us_no_overlap": round(sum(sum(v) for v in by_name.values()) / steps, 1)}
    finally:
        eng.close()


def run(model: str, prompt_len: int, steps: int, warmup: int, chunk: int, kernels: bool, layers: int = 0, clocks=None) -> dict:
    spec = resolve_model(model)
    if layers:
        spec = spec.with_layers(layers)
    dev = torch.device("cuda", torch.cuda.current_device())
    capacity = prompt_len + steps + warmup + 128
    eng = Engine.build(spec, capacity=capacity, device=dev, prefill_chunk=chunk)
    try:
        g = torch.Generator().manual_seed(0)
        prompt = torch.randint(0, spec.vocab, (prompt_len,), generator=g, dtype=torch.int32).pin_memory()
        eng.prefill.warm_chunks([chunk])
        eng.prefill.run(prompt, 0, prompt_len - 1)
        torch.cuda.synchronize()
        pre = []
        for _ in range(3):
            eng.prefill.run(prompt, 0, prompt_len - 1)
            pre.append(eng.prefill.executor_ms())
        pre_ms = sorted(pre)[1]
        sp = SamplingParams(temperature=1.0, top_p=1e-6, seed=1)
        eng.open(prompt, steps + warmup + 8, sp)
        r = eng.round
        r.stop_ids.fill_(-1)
        r.launch(warmup)
        torch.cuda.synchronize()
        if clocks is not None:
            clocks.start()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        with torch.cuda.stream(r.stream):
            a.record()
        r.launch(steps)
        with torch.cuda.stream(r.stream):
            b.record()
        torch.cuda.synchronize()
        if clocks is not None:
            clocks.stop_flag.set()
            clocks.join()
        dec_ms = a.elapsed_time(b) / steps
        eng.fabric.check()
        read = sum(n for _, n in step_work(eng, prompt_len))
        out = {"metric": "layer-stack decode tokens/s (one sequence)", "value": round(1e3 / dec_ms, 2), "unit": "tokens/s", "n_gpus": 1,
               "steps": steps, "warmup": warmup, "ms_per_step": round(dec_ms, 4), "higher_is_better": True, "dtype": "bf16",
               "data": "synthetic: random weights drawn on the device, uniform random prompt ids",
               "decode_bytes_per_token": int(read), "decode_roofline": round(read / (dec_ms * 1e-3) * 1e-9 / peaks()["hbm_gbs"], 3),
               "prefill": {"tokens_per_s": round((prompt_len - 1) / (pre_ms * 1e-3), 1), "ms": round(pre_ms, 3), "chunk": chunk},
               "config": {"model": spec.name, "layers": spec.layer_count, "hidden": spec.hidden, "seq_len": prompt_len, "global_batch": 1,
                          "kernels_per_round": r.kernels_per_round, "l2": "weights of a step exceed the 126 MB L2"},
               "peaks": peaks(), "gpu_launches": int(r.kernels_per_round * steps)}
        if clocks is not None:
            out["clocks"] = clocks.summary()
        if kernels:
            n0 = min(prompt_len // 2, prompt_len - 1 - chunk) if prompt_len > chunk else 0
            eng.prefill.run(prompt, 0, n0) if n0 else None
            out["chunk_kernels"] = {"pos0": n0, "rows": chunk, "table": chunk_table(eng, prompt, n0, min(chunk, prompt_len - n0))}
            eng.prefill.run(prompt, 0, prompt_len - 1)
            out["step_kernels"] = {"pos": prompt_len - 1, "table": step_table(eng, prompt_len - 1)}
        eng.fabric.check()
        return out
    finally:
        eng.close()
