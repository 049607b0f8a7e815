"""What the benchmarks of single model designs share: CUDA-event timing, measured peaks, one JSON line per measurement."""
from __future__ import annotations

import json
import os

import torch


def peaks():
    path = os.path.join(os.path.dirname(os.path.abspath(__file__)), "MEASURED_PEAKS.json")
    if os.path.exists(path):
        with open(path) as f:
            p = json.load(f)
        return p["hbm_gbs"], p["bf16_tflops"], "measured"
    return 6650.0, 1590.0, "fallback"


def timed(fn, reps, warm=3):
    for _ in range(warm):
        fn()
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for _ in range(reps):
        fn()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) / reps


def emit(**kw):
    print(json.dumps(kw), flush=True)


class KernelBench:
    """Times single calls on a cold L2 and reports them against the measured roofline."""

    FP32_TFLOPS = 148 * 128 * 2 * 1.965e9 / 1e12        # one fp32 FMA per lane and clock at the maximum clock

    def __init__(self, dev):
        self.flush = torch.empty(256 << 20, dtype=torch.uint8, device=dev)
        self.hbm, self.tf, self.src = peaks()

    def cold(self, fn, reps=8):
        """Median milliseconds of one call, every call after a write of twice the L2."""
        for _ in range(3):
            fn()
        ms = []
        for _ in range(reps):
            self.flush.add_(1)
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            fn()
            e1.record()
            torch.cuda.synchronize()
            ms.append(e0.elapsed_time(e1))
        return sorted(ms)[len(ms) // 2]

    def report(self, name, shape, ms, gbytes=0.0, tflop=0.0, fp32=0.0, like=None):
        t = {"hbm": gbytes / self.hbm * 1e3, "bf16": tflop / self.tf * 1e3, "fp32": fp32 / self.FP32_TFLOPS * 1e3}
        bound = max(t, key=t.get)
        emit(metric="kernel", kernel=name, shape=shape, us=ms * 1e3, bound=bound, roofline_us=t[bound] * 1e3, fraction=t[bound] / ms, peaks=self.src, like=like)
