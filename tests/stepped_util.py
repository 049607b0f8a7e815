"""What the tests of the layer-list decoders share: devices, comparison, portions, model directories, trace replay."""
import json
import os
import subprocess
import sys

import pytest
import torch

from innova_b200.inference.state_cache import StepBatch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BOTH = [("cpu", torch.float32), pytest.param(("cuda", torch.float32), marks=pytest.mark.gpu), pytest.param(("cuda", torch.bfloat16), marks=pytest.mark.gpu)]
IDS = ["cpu-f32", "cuda-f32", "cuda-bf16"]


def tokens(n, cfg, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def error(got, want):
    """Root mean square of the difference over the logits' own, worst row."""
    d = got.double().cpu() - want
    return float((d.square().mean(-1).sqrt() / want.square().mean(-1).sqrt().clamp_min(1e-6)).max())


def tol(dev):
    return 6e-2 if dev[1] == torch.bfloat16 else 3e-5


def run(model, toks, cuts, cache=None, row=0):
    """Logits of every position when the sequence arrives in portions of the given sizes (the last size repeats)."""
    cache = cache or model.make_cache(2, len(toks) + 1)
    out, pos, k = [], 0, 0
    while pos < len(toks):
        n = min(cuts[min(k, len(cuts) - 1)], len(toks) - pos)
        cache.reserve(row, pos + n)
        out.append(model.step(cache, StepBatch(cache, [toks[pos:pos + n]], [pos], [row], want=range(n), vocab=model.cfg.vocab_size)))
        pos, k = pos + n, k + 1
        cache.commit([row], [pos])
    return torch.cat(out)


def write_dir(path, cfg, w):
    path.mkdir()
    (path / "config.json").write_text(json.dumps(cfg))
    head, blob = {}, b""
    for n, t in w.items():
        raw = t.bfloat16().contiguous().view(torch.int16).numpy().tobytes()
        head[n] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [len(blob), len(blob) + len(raw)]}
        blob += raw
    js = json.dumps(head).encode()
    (path / "model.safetensors").write_bytes(len(js).to_bytes(8, "little") + js + blob)


def with_config(tmp_path, cfg):
    (tmp_path / "c").mkdir()
    (tmp_path / "c" / "config.json").write_text(json.dumps(cfg))
    return str(tmp_path / "c")


def replay(model_dir, out, steps, dtype, device):
    out.mkdir()
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(model_dir), "--dtype", dtype, "--out", str(out),
                        "--max-tokens", "512", "--device", device], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {s['step']}" for s in steps]
