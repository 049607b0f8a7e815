"""Prefill and decode throughput of Mekazen decoders (random weights) beside the closest model of the framework at equal size, and
the kernels of the design on their own. Run as ``python bench.py --design mekazen`` (optionally ``--section model`` or ``kernels``);
prints one JSON line per measurement.

Closest model: ``DenseModel`` through ``Generator`` (the other grouped-query decoder with RMS norms and a gated MLP; bf16 KV cache).
Times are CUDA events around warm, repeated calls; the model figures run over weights larger than L2, the kernel figures flush L2
before every call. Chunks are as long as the decoded contexts, so both models attend to everything there."""
from __future__ import annotations

import torch

from bench_design import KernelBench, emit, timed

SIZES = {
    # name: width, ff, heads, key heads (head size 128), vocabulary
    "1k": (1024, 2816, 8, 2, 32768),
    "2k": (2048, 5632, 16, 4, 32768),
    "4k": (4096, 11008, 32, 8, 32768),
}
CHUNK, LAYERS = 4096, 8


def mekazen_config(size):
    from innova_b200.models.mekazen import MekazenConfig
    E, F, H, G, V = SIZES[size]
    rot = {"dims": 64, "base": 500000.0, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}
    layer = {"type": "attention", "mixer": {"heads": H, "kv_heads": G, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": CHUNK}, "rot": rot},
             "mlp": {"kind": "dense", "ff": F}}
    return MekazenConfig(vocab_size=V, width=E, layers=[layer] * LAYERS, logit_softcap=30.0, max_seq_len=8192 + 64)


def model_section(sizes):
    from bench import ClockSampler
    from innova_b200.inference.generator import Generator
    from innova_b200.models import DenseModel, TransformerConfig
    from innova_b200.models.mekazen import MekazenModel
    dev = torch.device("cuda")
    for size in sizes:
        E, F, H, G, V = SIZES[size]
        clocks = ClockSampler(0)
        clocks.start()
        gen = Generator(MekazenModel(mekazen_config(size), seed=0, device=dev), max_batch=64, max_seq=8192 + 64, num_pages=64 * 160)
        dense_cfg = TransformerConfig(vocab_size=V, hidden_size=E, num_layers=LAYERS, num_heads=H, num_kv_heads=G, head_dim=128, ffn_hidden_size=F,
                                      max_seq_len=8192 + 64)
        dense = Generator(DenseModel(dense_cfg, dtype=torch.bfloat16, device=dev), kv_format="bf16", max_batch=64, max_seq=2048 + 64)
        g = torch.Generator().manual_seed(1)

        def ids(n):
            return torch.randint(0, V, (n,), generator=g).tolist()

        def fresh(gen, rows):
            for r in range(rows):
                gen.cache.free(r)
        base = dict(size=size, width=E, ff=F, heads=H, kv_heads=G, layers=LAYERS)
        for B, S in ((1, 2048), (1, 8192), (4, 2048)):
            toks = [ids(S) for _ in range(B)]

            def prefill():
                fresh(gen, B)
                gen.step(toks, [0] * B, list(range(B)))
            ms = timed(prefill, 5)
            emit(metric="prefill", model="mekazen", batch=B, prompt=S, ms=ms, tokens_per_s=B * S / ms * 1e3, **base)
            if S <= 2048:
                t = torch.tensor(toks, device=dev)

                def dprefill():
                    fresh(dense, B)
                    dense._forward(t, [0] * B)
                ms = timed(dprefill, 5)
                emit(metric="prefill", model="dense", batch=B, prompt=S, ms=ms, tokens_per_s=B * S / ms * 1e3, **base)
        for B in (1, 16, 64):
            S = 2048 if B <= 16 else 1024
            fresh(gen, 64)
            for b in range(B):
                gen.step([ids(S)], [0], [b])
            pos = [S]

            def decode():
                gen.step([[7 + b] for b in range(B)], [pos[0]] * B, list(range(B)))
                pos[0] += 1
            ms = timed(decode, 40, warm=8)
            ms_dev = timed(gen._graphs[B][0].replay, 40, warm=3)
            emit(metric="decode", model="mekazen", batch=B, context=S, ms=ms, device_ms=ms_dev, tokens_per_s=B / ms * 1e3, **base)
            fresh(dense, 64)
            for b in range(B):
                dense._forward(torch.tensor([ids(S)], device=dev), [0], slots=[b])
            dpos, t1 = [S], torch.full((B, 1), 7, device=dev)

            def ddecode():
                dense._forward(t1, [dpos[0]] * B)
                dpos[0] += 1
            ms = timed(ddecode, 20, warm=4)
            emit(metric="decode", model="dense", batch=B, context=S, ms=ms, tokens_per_s=B / ms * 1e3, **base)
        clocks.stop_flag = True
        emit(metric="clocks", **clocks.summary(), **base)
        gen = dense = None
        import gc
        gc.collect()
        torch.cuda.empty_cache()


def kernel_section(size="2k"):
    """Every kernel of the design alone, and the like kernel of the closest model: time, bytes or FLOPs, fraction of the roofline."""
    from innova_b200 import ops
    from innova_b200.inference.kv_cache import PagedKVCache
    from innova_b200.inference.state_cache import KeyValues, StepBatch, StepCache
    from innova_b200.ops import kv_attention as ka
    from innova_b200.ops import latent_attention as la
    from innova_b200.ops.hyper import gated_silu
    from innova_b200.ops.sandwich import sandwich_step, softcap_
    E, F, H, G, V = SIZES[size]
    D = 128
    dev, bf = torch.device("cuda"), torch.bfloat16
    bench = KernelBench(dev)
    cold, report = bench.cold, bench.report
    rand = lambda *s: torch.randn(*s, device=dev)
    # residual step (two norms and the residual) and, as the like kernel, the RMS norm of the dense decoder
    for T in (8192, 64):
        x, y, w = rand(T, E), rand(T, E).to(bf if T > 64 else torch.float32), rand(E)
        report("sandwich_step", f"T{T} E{E}", cold(lambda: sandwich_step(x, bf, 1e-5, 1.0, y=y, post_w=w, norm_w=w)), T * E * (8 + y.element_size() + 2) / 1e9)
        xb, wb = x.to(bf), w.to(bf)
        report("rms_norm", f"T{T} E{E}", cold(lambda: ops.rms_norm(xb, wb, 1e-5)), T * E * 4 / 1e9, like="sandwich_step")
    # norm, rotation and append; like kernels: rotation in place, append to the dense decoder's cache
    freq = ka.rope_frequencies(64, 5e5).to(dev)
    qn, kn = rand(H * D), rand(G * D)
    cos, sin = ops.rope_tables(8192, D, 5e5, dev)
    for T, B in ((8192, 1), (64, 64), (1, 1)):
        S = T // B
        c = StepCache(B, 8192, dev, kv=[KeyValues(G, D)])
        kv = PagedKVCache(1, G, D, B, 8192, dev, "bf16")
        start = 0 if S > 1 else 1000
        for i in range(B):
            c.reserve(i, start + S)
            kv.reserve(i, start + S)
        b = StepBatch(c, [[0] * S] * B, [start] * B, list(range(B)))
        dt = bf if T > 64 else torch.float32
        proj = rand(T, (2 * H + G) * D).to(dt)
        report("qkv_prep", f"T{T} H{H} G{G} D{D}",
               cold(lambda: ka.qkv_append(proj, 0, H * D, H * D, H, G, D, D, qn, kn, 1e-5, freq, c.kv[0], c.page_table, b, want_k=S > 1)),
               T * D * ((H + G) * proj.element_size() + (H + (3 if S > 1 else 2) * G) * 2) / 1e9)
        qkv = rand(B, S, (H + 2 * G) * D).to(bf)
        pos = torch.arange(start, start + S, dtype=torch.int32, device=dev).repeat(B)
        with torch.no_grad():
            report("rope", f"T{T} H{H} G{G} D{D}", cold(lambda: ops.rope_qk(qkv, cos, sin, H, G, D, pos)), T * D * (H + G) * 4 / 1e9, like="qkv_prep")
        k, v = qkv[..., H * D:(H + G) * D], qkv[..., (H + G) * D:]
        report("kv_append", f"T{T} G{G} D{D}", cold(lambda: kv.append(0, k, v, list(range(B)), [start] * B)), T * D * G * 8 / 1e9, like="qkv_prep")
    # attention, decode, against the dense decoder's paged attention (bf16 cache) at the same heads and span
    for B in (1, 16, 64):
        for n in (1024, 4096):
            c = StepCache(B, 4096, dev, kv=[KeyValues(G, D, chunk=4096)])
            kv = PagedKVCache(1, G, D, B, 4096, dev, "bf16")
            for i in range(B):
                c.reserve(i, n)
                kv.reserve(i, n)
            kv.commit(list(range(B)), [n] * B)
            c.kv[0].normal_()
            b = StepBatch(c, [[0]] * B, [n - 1] * B, list(range(B)))
            q, gate = rand(B, H * D).to(bf), rand(B, H * D)
            gb, fl = B * n * G * D * 4 / 1e9, B * H * n * D * 4 / 1e12
            report("kv_attend", f"B{B} H{H} G{G} D{D} keys {n}", cold(lambda: ka.kv_attend(q, c.kv[0], c.page_table, H, 0.09, b, chunk=4096, gate=gate)), gb, fl)
            report("paged_decode", f"B{B} H{H} G{G} D{D} keys {n}", cold(lambda: kv.decode_attention(0, q, H, 0.09)), gb, fl, like="kv_attend")
        wl, xl = rand(4096, E).to(bf), rand(B, E).to(bf)
        if B <= 32:
            report("skinny_gemm", f"M{B} N4096 K{E}", cold(lambda: ops.skinny_gemm(xl, wl)), wl.numel() * 2 / 1e9)
            wh = rand(V, E).to(bf)
            report("skinny_gemm softcap", f"M{B} N{V} K{E}", cold(lambda: ops.skinny_gemm(xl, wh, softcap=30.0)), (wh.numel() * 2 + B * V * 4) / 1e9)
        report("gemm", f"M{B} N4096 K{E}", cold(lambda: ops.gemm(xl, wl)), wl.numel() * 2 / 1e9, like="skinny_gemm")
    # attention, prompts
    for B, S in ((1, 4096), (4, 2048)):
        T = B * S
        c = StepCache(B, S, dev, kv=[KeyValues(G, D)])
        for i in range(B):
            c.reserve(i, S)
        b = StepBatch(c, [[0] * S] * B, [0] * B, list(range(B)))
        qkv, gate = rand(B, S, (H + 2 * G) * D).to(bf), rand(T, H * D).to(bf)
        flat = qkv.view(T, -1)
        q, k, v = flat[:, :H * D], flat[:, H * D:(H + G) * D], flat[:, (H + G) * D:]
        fl = lambda chunk: B * H * S * min(chunk, S) / 2 * D * 4 / 1e12
        for chunk in (4096, 1024):
            report("packed_flash", f"{B} x {S} H{H} G{G} D{D} chunk {chunk} gated",
                   cold(lambda: la.packed_flash(q, k, v, H, D, 0.09, None, b, kv_heads=G, chunk=chunk, gate=gate)), tflop=fl(chunk))
        with torch.no_grad():
            report("flash_attention", f"{B} x {S} H{H} G{G} D{D}", cold(lambda: ops.flash_attention(qkv, H, G, D)), tflop=fl(S), like="packed_flash")
            short = qkv.view(T // 1024, 1024, -1)        # the same work as chunks of 1024
            report("flash_attention", f"{T // 1024} x 1024 H{H} G{G} D{D}", cold(lambda: ops.flash_attention(short, H, G, D)), tflop=fl(1024), like="packed_flash")
    z = rand(512, V)
    report("softcap", f"512 x {V}", cold(lambda: softcap_(z, 30.0)), z.numel() * 8 / 1e9)
    gu = rand(8192, 2 * F).to(bf)
    report("gated_silu", f"8192 x {F}", cold(lambda: gated_silu(gu, F, bf)), gu.numel() * 3 / 1e9, like="softcap")


def main(section="all", sizes=None):
    if section in ("all", "kernels"):
        kernel_section()
    if section in ("all", "model"):
        model_section(sizes or list(SIZES))
    return 0
