"""Measuring packed decoders: throughput through the registry's runner, and single kernels as CUDA graphs of many launches over
rotating buffers."""
from __future__ import annotations

import json
import os
from typing import Callable, Dict, List

import torch

from ..models.registry import create_decoder

FP32_CORE_TFLOPS = 148 * 128 * 2 * 1.965e-3   # nominal: SMs x lanes x 2 x GHz


def peaks() -> Dict[str, float]:
    path = os.path.join(os.path.dirname(os.path.abspath(__file__)), "..", "..", "MEASURED_PEAKS.json")
    try:
        with open(path) as f:
            d = json.load(f)
        return {"hbm_gbs": d["hbm_gbs"], "bf16_tflops": d["bf16_tflops"], "source": "measured"}
    except OSError:
        return {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}


def event_ms(fn: Callable[[], None]) -> float:
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    fn()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b)


def model_numbers(config, batch: int, prompt: int, steps: int, warmup: int) -> Dict[str, float]:
    runner = create_decoder(config, None, "bfloat16", batch=batch, max_len=prompt + steps + warmup + 8)
    ids = torch.randint(0, runner.cfg.vocab_size, (batch, prompt), generator=torch.Generator().manual_seed(1))
    for _ in range(3):
        runner.prefill(ids)
    prefill = sorted(event_ms(lambda: runner.prefill(ids)) for _ in range(5))[2]
    for _ in range(warmup):
        runner.decode_step(None)
    launches = runner.sess.last_run_launch_count()

    def loop():
        for _ in range(steps):
            runner.decode_step(None)
    start = runner.cur_len
    times = []
    for _ in range(3):
        runner.cur_len = start
        times.append(event_ms(loop) / steps)
    runner.sess.check_device_status()
    decode = sorted(times)[1]
    return {"prefill_ms": round(prefill, 3), "prefill_tokens_per_s": round(batch * prompt / prefill * 1e3, 1), "decode_ms": round(decode, 4),
            "decode_tokens_per_s": round(batch / decode * 1e3, 1), "decode_launches": launches}


def graph_us(calls: List[Callable[[], object]], rounds: int = 4) -> float:
    """Microseconds per call of ``calls`` (the same kernel over different buffers) replayed as one CUDA graph."""
    for c in calls[:3]:
        c()
    torch.cuda.synchronize()
    keep, graph = [], torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        for c in calls:
            keep.append(c())
    for _ in range(3):
        graph.replay()
    t = sorted(event_ms(graph.replay) for _ in range(rounds))[rounds // 2]
    return t * 1e3 / len(calls)


class KernelRows:
    """Rows of a kernel table: time, the time its job needs at the measured peaks, and their quotient."""

    def __init__(self):
        self.peaks, self.rows = peaks(), []

    def add(self, name: str, design: str, us: float, bytes_: float = 0, tflop: float = 0.0, core_tflop: float = 0.0) -> None:
        best = max((bytes_ / self.peaks["hbm_gbs"] * 1e-3, "hbm"), (tflop / self.peaks["bf16_tflops"] * 1e6, "bf16 tensor"),
                   (core_tflop / FP32_CORE_TFLOPS * 1e6, "fp32 cores (nominal)"))
        self.rows.append({"kernel": name, "design": design, "us": round(us, 2), "roofline_us": round(best[0], 2), "of": best[1],
                          "fraction": round(best[0] / us, 3)})


def run_pair(name: str, configs, kernel_numbers, sizes, batch: int, prompt: int, steps: int, warmup: int) -> Dict:
    """A design beside the paged Llama decoder of equal size, per width: ``configs(width)`` returns both configurations,
    ``kernel_numbers(width, batch, prompt, context)`` the kernel rows."""
    out = {"metric": f"{name}_prefill_decode_tokens_per_s", "unit": "tokens/s", "dtype": "bf16", "n_gpus": 1, "data": "synthetic, random weights",
           "config": {"layers": 8, "global_batch": batch, "seq_len": prompt, "decode_tokens": steps, "peaks": peaks(),
                      "l2": "weights larger than L2; kernels over rotating buffers"}, "sizes": {}}
    for width in sizes:
        entry = {}
        for who, c in zip((name, "llama"), configs(width)):
            entry[who] = model_numbers(c, batch, prompt, steps, max(warmup, 3))
            torch.cuda.empty_cache()
        entry["kernels"] = kernel_numbers(width, batch, prompt, prompt)
        out["sizes"][str(width)] = entry
    first = out["sizes"][str(sizes[-1])][name]
    out.update(value=first["decode_tokens_per_s"], ms_per_step=first["decode_ms"], steps=steps, warmup=max(warmup, 3), higher_is_better=True)
    return out
