"""Prefill and decode throughput of Vebesun decoders (random weights) beside the closest models of the framework at equal size,
and the kernels of the design on their own. Run as ``python bench.py --design vebesun`` (optionally ``--section model`` or
``kernels``); prints one JSON line per measurement.

Closest models: ``HybridEngine`` (the other gated delta-rule decoder; one sequence at a time) and ``DenseModel`` through
``Generator`` (the other batched attention decoder, bf16 KV cache). Times are CUDA events around warm, repeated calls; the
model figures run over weights larger than L2, the kernel figures flush L2 before every call."""
from __future__ import annotations

import torch

from bench_design import KernelBench, emit, timed

SIZES = {
    # name: width, ff, heads (head size 128), latent rank, vocabulary
    "1k": (1024, 2816, 8, 256, 32768),
    "2k": (2048, 5632, 16, 512, 32768),
    "4k": (4096, 11008, 32, 512, 32768),
}
WINDOW, LAYERS, STREAMS, RANK = 1024, 8, 4, 128


def vebesun_config(size):
    from innova_b200.models.vebesun import VebesunConfig
    E, F, H, R, V = SIZES[size]
    attn = {"type": "latent_attention", "mixer": {"heads": H, "dim": 128, "vdim": 128, "kv_rank": R, "scale": 128 ** -0.5, "mask": {"size": WINDOW}},
            "mlp": {"kind": "dense", "ff": F}}
    delta = {"type": "channel_delta", "mixer": {"heads": H, "kv_heads": H, "dim": 128, "vdim": 128, "conv": 4}, "mlp": {"kind": "dense", "ff": F}}
    layers = [attn if i % 4 == 3 else delta for i in range(LAYERS)]
    ranks = {str(i): (RANK, RANK) for i in range(LAYERS) if i % 4 != 3}
    return VebesunConfig(vocab_size=V, width=E, layers=layers, streams=STREAMS, embedding_scale=E ** 0.5, max_seq_len=8192 + 64, ranks=ranks)


def model_section(sizes):
    from bench import ClockSampler
    from innova_b200.inference.generator import Generator
    from innova_b200.inference.hybrid_engine import HybridConfig, HybridEngine
    from innova_b200.models import DenseModel, TransformerConfig
    from innova_b200.models.vebesun import VebesunModel
    dev = torch.device("cuda")
    for size in sizes:
        E, F, H, R, V = SIZES[size]
        clocks = ClockSampler(0)
        clocks.start()
        gen = Generator(VebesunModel(vebesun_config(size), seed=0, device=dev), max_batch=64, max_seq=8192 + 64, num_pages=64 * 160)
        dense_cfg = TransformerConfig(vocab_size=V, hidden_size=E, num_layers=LAYERS, num_heads=H, head_dim=128, ffn_hidden_size=F, max_seq_len=8192 + 64)
        dense = Generator(DenseModel(dense_cfg, dtype=torch.bfloat16, device=dev), kv_format="bf16", max_batch=64, max_seq=2048 + 64)
        hyb_cfg = HybridConfig(vocab_size=V, hidden=E, layers=LAYERS, full_every=4, ffn=F, k_heads=H, v_heads=H, d_k=128, d_v=128, heads=H, kv_heads=H,
                               head_dim=128, max_kv=8192)
        hyb = HybridEngine(hyb_cfg, device=dev, dtype=torch.bfloat16).init_random(0)
        g = torch.Generator().manual_seed(1)

        def ids(n):
            return torch.randint(0, V, (n,), generator=g).tolist()

        def fresh(gen, rows):
            for r in range(gen.cache.max_batch):
                gen.cache.free(r)
        base = dict(size=size, width=E, ff=F, heads=H, layers=LAYERS)
        for B, S in ((1, 2048), (1, 8192), (4, 2048)):
            toks = [ids(S) for _ in range(B)]

            def prefill():
                fresh(gen, B)
                gen.step(toks, [0] * B, list(range(B)))
            ms = timed(prefill, 5)
            emit(metric="prefill", model="vebesun", batch=B, prompt=S, ms=ms, tokens_per_s=B * S / ms * 1e3, **base)
            if S <= 2048:
                t = torch.tensor(toks, device=dev)

                def dprefill():
                    fresh(dense, B)
                    dense._forward(t, [0] * B)
                ms = timed(dprefill, 5)
                emit(metric="prefill", model="dense", batch=B, prompt=S, ms=ms, tokens_per_s=B * S / ms * 1e3, **base)
        hs = 128

        def hprefill():
            hyb.reset()
            hyb.prefill(ids(hs))
        ms = timed(hprefill, 1, warm=1)
        emit(metric="prefill", model="hybrid", batch=1, prompt=hs, ms=ms, tokens_per_s=hs / ms * 1e3, note="token loop: time is linear in the prompt", **base)
        for B in (1, 16, 64):
            S = 2048 if B <= 16 else 1024
            fresh(gen, B)
            for b in range(B):
                gen.step([ids(S)], [0], [b])
            pos = [S]

            def decode():
                gen.step([[7 + b] for b in range(B)], [pos[0]] * B, list(range(B)))
                pos[0] += 1
            ms = timed(decode, 40, warm=8)
            graph = gen._graphs[B][0]
            ms_dev = timed(graph.replay, 40, warm=3)
            emit(metric="decode", model="vebesun", batch=B, context=S, ms=ms, device_ms=ms_dev, tokens_per_s=B / ms * 1e3, **base)
            fresh(dense, B)
            for b in range(B):
                dense._forward(torch.tensor([ids(S)], device=dev), [0], slots=[b])
            dpos, t1 = [S], torch.full((B, 1), 7, device=dev)

            def ddecode():
                dense._forward(t1, [dpos[0]] * B)
                dpos[0] += 1
            ms = timed(ddecode, 20, warm=4)
            emit(metric="decode", model="dense", batch=B, context=S, ms=ms, tokens_per_s=B / ms * 1e3, **base)
            if B == 1:
                ms = timed(lambda: hyb.append_token(7), 10, warm=3)
                emit(metric="decode", model="hybrid", batch=1, context=hs, ms=ms, tokens_per_s=1e3 / ms, **base)
        clocks.stop_flag = True
        emit(metric="clocks", **clocks.summary(), **base)
        gen = dense = hyb = None
        import gc
        gc.collect()
        torch.cuda.empty_cache()


def kernel_section(size="2k"):
    """Every kernel of the design alone, and the like kernel of the closest model: time, bytes or FLOPs, fraction of the roofline."""
    from innova_b200 import ops
    from innova_b200.inference.kv_cache import PagedKVCache
    from innova_b200.inference.state_cache import Latents, StepBatch, StepCache
    from innova_b200.ops import delta_rule as dr
    from innova_b200.ops import latent_attention as la
    from innova_b200.ops import runtime as rt
    from innova_b200.ops.hyper import HyperIn, HyperOut, gated_silu, hyper_step
    E, F, H, R, V = SIZES[size]
    dev, bf = torch.device("cuda"), torch.bfloat16
    bench = KernelBench(dev)
    cold, report = bench.cold, bench.report
    rand = lambda *s: torch.randn(*s, device=dev)
    # residual step (streams) and, as the like kernel, the fused residual-add RMSNorm of the dense decoder
    for T in (8192, 64):
        x, y = rand(T, STREAMS, E), rand(T, E).to(bf if T > 64 else torch.float32)
        o = torch.ones(STREAMS, device=dev)
        nxt, prev = HyperIn(o, rand(E), rand(E), 1e-5), HyperOut(y, torch.eye(STREAMS, device=dev), o)
        report("hyper_step", f"T{T} S{STREAMS} E{E}", cold(lambda: hyper_step(x, bf, prev, nxt)), (2 * STREAMS * T * E * 4 + T * E * (2 + y.element_size())) / 1e9)
        xb, w = rand(T, E).to(bf), rand(E).to(bf)
        report("rms_norm", f"T{T} E{E}", cold(lambda: ops.rms_norm(xb, w, 1e-5)), T * E * 4 / 1e9, like="hyper_step")
        gu = rand(T, 2 * F).to(bf if T > 64 else torch.float32)
        report("gated_silu", f"T{T} F{F}", cold(lambda: gated_silu(gu, F, bf)), (gu.numel() * gu.element_size() + T * F * 2) / 1e9)
    # delta rule
    s = dr.DeltaShape(H, H, 128, 128, 4, RANK, RANK)
    lens = {"1x8192": [8192], "16x1024": [1024] * 16}
    for name, ls in lens.items():
        T = sum(ls)
        c = StepCache(len(ls), max(ls) + 16, dev, states=[s])
        for i, n in enumerate(ls):
            c.reserve(i, n)
        b = StepBatch(c, [[0] * n for n in ls], [0] * len(ls), list(range(len(ls))))
        proj, z, gate = rand(T, s.offsets[6]).to(bf), rand(T, H * 128) - 4, rand(T, H * 128).to(bf)
        taps, A, dt, nw, o = rand(4, s.channels), rand(H), rand(H * 128), rand(128), rand(T, H * 128)
        lib, st, arr = rt.lib(), rt.stream_ptr(), s.c_array()
        blocks, vblocks = torch.empty(b.n_chunks * H * s.block_floats, device=dev), torch.empty(b.n_chunks * H * 8 * 256, device=dev)

        def chunk():
            rt.check(lib.inv_delta_chunk(proj.data_ptr(), proj.stride(0), 0, taps.data_ptr(), c.ring[0].data_ptr(), b.chunk_seq.data_ptr(),
                                         b.cu_chunk.data_ptr(), b.cu.data_ptr(), b.start.data_ptr(), b.slots.data_ptr(), A.data_ptr(), dt.data_ptr(),
                                         z.data_ptr(), z.stride(0), blocks.data_ptr(), vblocks.data_ptr(), b.n_chunks, arr, st), "chunk")

        def scan():
            rt.check(lib.inv_delta_scan(blocks.data_ptr(), vblocks.data_ptr(), o.data_ptr(), c.state[0].data_ptr(), b.cu_chunk.data_ptr(),
                                        b.cu.data_ptr(), b.start.data_ptr(), b.slots.data_ptr(), b.n, rt.status_tensor(dev).data_ptr(), arr, st), "scan")
        moved = (blocks.numel() + vblocks.numel()) * 4 / 1e9
        report("delta_chunk", f"{name} H{H}", cold(chunk), moved + T * H * 128 * (3 * 2 + 4) / 1e9, fp32=T * H * 128 * (16 * 3 + 12) * 2 / 1e12)
        report("delta_scan", f"{name} H{H} 128x128", cold(scan), moved + T * H * 128 * 4 / 1e9, fp32=2 * T * H * (3 * 128 * 128 + 2 * 16 * 128) / 1e12)

        def hnorm():
            rt.check(lib.inv_gated_head_norm(o.data_ptr(), nw.data_ptr(), gate.data_ptr(), gate.stride(0), 0, proj.data_ptr(), proj.stride(0), 0, T, H,
                                             128, 1e-5, st), "norm")
        report("gated_head_norm", f"{name} H{H}", cold(hnorm), T * H * 128 * 8 / 1e9)
        del blocks, vblocks, o, proj, z, gate
    for B in (1, 16, 64):
        c = StepCache(B, 64, dev, states=[s])
        for i in range(B):
            c.reserve(i, 11)
        b = StepBatch(c, [[0]] * B, [10] * B, list(range(B)))
        proj, a2t, g2t = rand(B, s.offsets[6]), (rand(RANK, H * 128) * 0.1).to(bf), (rand(RANK, H * 128) * 0.1).to(bf)
        args = (rand(4, s.channels), rand(H), rand(H * 128) - 4, rand(128), 1e-5, c.ring[0], c.state[0], b)
        report("delta_decode", f"B{B} H{H} 128x128", cold(lambda: dr.delta_decode(s, proj, a2t, g2t, *args)),
               (B * H * 128 * 128 * 8 + 2 * RANK * H * 128 * 2 + B * s.offsets[6] * 4 + 3 * B * s.channels * 4) / 1e9)
    # attention, decode: latents against the dense decoder's paged KV cache (bf16) at the same heads and span
    for B in (1, 16, 64):
        c = StepCache(B, 2048, dev, latents=[Latents(R, WINDOW)])
        for i in range(B):
            c.reserve(i, 1537)
        b = StepBatch(c, [[0]] * B, [1536] * B, list(range(B)))
        c.latent[0].normal_()
        q = rand(B, H * R).to(bf)
        report("latent_attend", f"B{B} H{H} R{R} window {WINDOW}", cold(lambda: la.latent_attend(q, c.latent[0], c.page_table, H, 0.05, WINDOW, b, WINDOW)),
               (B * WINDOW * R * 2 + 2 * q.numel() * 2) / 1e9, tflop=B * H * WINDOW * R * 4 / 1e12)
        wk, qh = rand(H, R, 128).to(bf), rand(B, H * 128).to(bf)
        report("head_proj q", f"B{B} H{H} 128->{R}", cold(lambda: la.head_proj(qh, wk)), (wk.numel() + qh.numel() + q.numel()) * 2 / 1e9)
        wv = rand(H, 128, R).to(bf)
        report("head_proj o", f"B{B} H{H} {R}->128", cold(lambda: la.head_proj(q, wv)), (wv.numel() + qh.numel() + q.numel()) * 2 / 1e9)
        kv = PagedKVCache(1, H, 128, B, 2048, dev, "bf16")
        for i in range(B):
            kv.reserve(i, WINDOW)
        kv.commit(list(range(B)), [WINDOW] * B)
        report("paged_decode", f"B{B} H{H} D128 context {WINDOW}", cold(lambda: kv.decode_attention(0, qh, H, 0.09)), B * WINDOW * H * 128 * 4 / 1e9,
               tflop=B * H * WINDOW * 128 * 4 / 1e12, like="latent_attend")
        wl, xl = rand(4096, E).to(bf), rand(B, E).to(bf)
        report("skinny_gemm", f"M{B} N4096 K{E}", cold(lambda: ops.skinny_gemm(xl, wl)), wl.numel() * 2 / 1e9)
        report("gemm", f"M{B} N4096 K{E}", cold(lambda: ops.gemm(xl, wl)), wl.numel() * 2 / 1e9, like="skinny_gemm")
    # attention, prompts
    T = 8192
    c = StepCache(1, T, dev, latents=[Latents(R, WINDOW)])
    c.reserve(0, T)
    b = StepBatch(c, [[0] * T], [0], [0])
    qkv = rand(1, T, 3 * H * 128).to(bf)
    q, k, v = (qkv[0, :, i * H * 128:(i + 1) * H * 128] for i in range(3))
    fl = H * (T * WINDOW - WINDOW * WINDOW / 2) * 128 * 4 / 1e12
    report("packed_flash", f"T{T} H{H} D128 window {WINDOW}", cold(lambda: la.packed_flash(q, k, v, H, 128, 0.09, WINDOW, b)), tflop=fl)
    with torch.no_grad():
        report("flash_attention", f"T{T} H{H} D128 window {WINDOW}", cold(lambda: ops.flash_attention(qkv, H, H, 128, window=WINDOW)), tflop=fl, like="packed_flash")
    pr, nw = rand(T, H * 128 + R).to(bf), rand(R)
    report("latent_prep", f"T{T} R{R}", cold(lambda: la.latent_append(pr, H * 128, R, nw, 1e-5, c.latent[0], c.page_table, b, want_c=True)), T * R * 6 / 1e9)


def main(section="all", sizes=None):
    if section in ("all", "kernels"):
        kernel_section()
    if section in ("all", "model"):
        model_section(sizes or list(SIZES))
    return 0
