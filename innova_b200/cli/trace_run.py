"""oil-trace-run: feed given token ids through a model directory step by step and write the logits asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps come on standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

Each entry continues its request (a new id starts one); ``want`` are places among its tokens; ``end`` lists the requests that
are finished after the step. ``OUT/<step>.f32`` receives the wanted logits as little-endian fp32 rows in the order of the
entries, and ``done <step>`` is printed after every step. The steps run through ``inference.Generator.step``, the call that
batched generation makes, with the same cache and kernels; nothing is sampled."""
from __future__ import annotations

import argparse
import json
import os
import sys


def main(argv=None):
    ap = argparse.ArgumentParser(prog="oil-trace-run", description=__doc__.splitlines()[0])
    ap.add_argument("--model", required=True, help="directory with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="existing directory for <step>.f32")
    ap.add_argument("--max-tokens", type=int, default=65536, help="most tokens the live requests hold at any time")
    ap.add_argument("--max-requests", type=int, default=256, help="most live requests")
    ap.add_argument("--device", default="cuda")
    a = ap.parse_args(argv)
    if a.dtype == "float32":
        os.environ["NVIDIA_TF32_OVERRIDE"] = "0"       # read by the matrix library when it starts
    import torch
    from .. import _native
    from ..formats import export
    from ..inference.generator import Generator
    from ..inference.kv_cache import PAGE
    from ..models.registry import model_class
    from ..ops import runtime as rt
    dev = torch.device(a.device)
    if dev.type == "cuda":
        if not torch.cuda.is_available():
            raise RuntimeError("no CUDA device")
        dev = torch.device("cuda", torch.cuda.current_device())
    cls = model_class(export.read_config_dir(a.model))
    _native.use_subset(cls.architecture.lower(), cls.CUDA_SOURCES, cls.HOST_SOURCES)
    model = export.load_model(a.model, dtype=getattr(torch, a.dtype), device=dev)
    rows = max(1, min(a.max_requests, a.max_tokens))
    gen = Generator(model, max_batch=rows, max_seq=a.max_tokens, num_pages=-(-a.max_tokens // PAGE) + rows)
    live, free = {}, list(range(rows - 1, -1, -1))     # request id -> [cache row, tokens so far]
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        tokens, start, at, want, base = [], [], [], [], 0
        for e in step["entries"]:
            if e["id"] not in live:
                if not free:
                    raise RuntimeError(f"more than {rows} live requests")
                live[e["id"]] = [free.pop(), 0]
            row, n = live[e["id"]]
            tokens.append(e["tokens"])
            start.append(n)
            at.append(row)
            want += [base + w for w in e["want"]]
            base += len(e["tokens"])
            live[e["id"]][1] = n + len(e["tokens"])
        if tokens:
            logits = gen.step(tokens, start, at, want)
            if want:
                logits.float().cpu().numpy().astype("<f4").tofile(os.path.join(a.out, f"{step['step']}.f32"))
            if dev.type == "cuda":
                rt.check_status(dev)
        for r in step.get("end", []):
            row, _ = live.pop(r)
            gen.cache.free(row)
            free.append(row)
        print("done", step["step"], flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
