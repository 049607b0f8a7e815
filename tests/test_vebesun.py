"""Vebesun decoders against the plain statement of their equations in ``vebesun_oracle.py``.

Every test makes its own small configuration and seeded weights. The ``dev`` fixture runs a test on the CPU path and, on a GPU
box, on the CUDA kernels in 32-bit and in bf16 (``cuda-f32``, ``cuda-bf16``)."""
import json
import math

import numpy as np
import pytest
import torch

import vebesun_oracle as oracle
from innova_b200.inference.generator import Generator
from innova_b200.inference.state_cache import Latents, StepBatch, StepCache
from innova_b200.models.vebesun import VebesunConfig, VebesunModel
from innova_b200.ops import delta_rule as dr
from innova_b200.ops import latent_attention as la
from innova_b200.ops.hyper import HyperIn, HyperOut, gated_silu, hyper_step
from stepped_util import BOTH, IDS, error, replay, run, tokens, tol, with_config, write_dir


@pytest.fixture(params=BOTH, ids=IDS)
def dev(request):
    return request.param


def attn(heads, dim, vdim, rank, size, scale=None):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "scale": scale or dim ** -0.5,
                                                  "mask": {"size": size}}}


def delta(heads, kv_heads, dim, vdim, conv):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def config(layers, width=96, vocab=120, streams=3, loop=None, eps=1e-5, scale=7.5):
    return {"architecture": "Vebesun", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "layers": layers, "loop": loop}


def ff(layer, n):
    return {**layer, "mlp": None if n is None else {"kind": "dense", "ff": n}}


CONFIGS = {
    # heads shared by key heads, a window that is no multiple of a page, the loop in the middle, an MLP behind the delta rule
    "mixed": config([ff(delta(6, 2, 24, 40, 3), 88), ff(attn(3, 40, 24, 56, 21), None), ff(attn(5, 24, 32, 40, 9), 72), ff(delta(4, 4, 32, 16, 5), None)],
                    loop={"start": 1, "stop": 3, "times": 3}),
    # sizes that are no multiple of 8, one stream, one tap, window of one page
    "odd": config([ff(attn(3, 20, 12, 27, 16), 50), ff(delta(3, 1, 20, 13, 1), 31), ff(delta(5, 5, 17, 22, 2), None)], width=52, vocab=77, streams=1),
    # everything looped, four streams, values wider than keys, a window of one token
    "loop": config([ff(delta(2, 2, 64, 72, 4), None), ff(attn(2, 16, 96, 64, 1), 64), ff(attn(4, 64, 64, 48, 33), 40)], width=64, streams=4,
                   loop={"start": 0, "stop": 3, "times": 2}, eps=1e-3),
    # heads too large for the flash kernel, a state tile of the largest decode size, five streams
    # a state tile too large for the one-launch decode kernel, more streams than the unrolled residual kernels, no feed-forward
    "tile": config([ff(delta(1, 1, 256, 224, 2), None), ff(attn(3, 32, 32, 48, 12), None)], width=48, streams=7),
    "large": config([ff(attn(2, 144, 80, 160, 50), 64), ff(delta(2, 1, 160, 128, 4), 48)], width=128, streams=5),
}


def build(cfg, dev, seed=0, **kw):
    w = oracle.random_weights(cfg, seed, **kw)
    return VebesunModel.from_tensors(cfg, w, dtype=dev[1], device=dev[0]), w


# ------------------------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("S,E", [(1, 64), (2, 37), (3, 200), (4, 128), (6, 52)])
def test_hyper_step(dev, S, E):
    d, dt = dev
    g = torch.Generator().manual_seed(S * 100 + E)
    T, V = 9, 11
    ids = torch.randint(0, V, (T,), generator=g)
    table = torch.randn(V, E, generator=g).to(dt)
    mix, out, inw = torch.randn(S, S, generator=g), torch.randn(S, generator=g), torch.randn(S, generator=g)
    nw, nb, y = torch.randn(E, generator=g), torch.randn(E, generator=g), torch.randn(T, E, generator=g).to(dt)
    pad = torch.zeros(V, (E + 7) // 8 * 8, dtype=dt)
    pad[:, :E] = table
    ypad = torch.zeros(T, (E + 7) // 8 * 8, dtype=dt)
    ypad[:, :E] = y
    t = lambda a: a.to(d)
    nxt = HyperIn(t(inw), t(nw), t(nb), 1e-5)
    x = torch.empty(T, S, E, device=d)
    h0 = hyper_step(x, dt, None, nxt, t(ids.int()), t(pad), 3.0)
    xs = [table.float()[ids] * 3.0 for _ in range(S)]
    close = dict(atol=6e-2, rtol=2e-2) if dt == torch.bfloat16 else dict(atol=2e-5, rtol=1e-5)
    assert torch.allclose(h0.float().cpu(), oracle.layer_norm(oracle.hyper_in(xs, inw), nw, nb, 1e-5), **close)
    x += t(torch.randn(T, S, E, generator=g))
    xs = [x[:, s].cpu() for s in range(S)]
    want = oracle.hyper_out(xs, mix, out, y.float())
    rows = torch.tensor([7, 0, 3], dtype=torch.int32)
    prev = HyperOut(t(ypad), t(mix), t(out))
    some = hyper_step(x, dt, prev, nxt, rows=t(rows))                       # a selection leaves the streams alone
    full = oracle.layer_norm(oracle.hyper_in(want, inw), nw, nb, 1e-5)
    assert torch.allclose(some.float().cpu(), full[rows.long()], **close) and torch.equal(x[:, 0].cpu(), xs[0])
    h = hyper_step(x, dt, prev, nxt)
    assert torch.allclose(h.float().cpu(), full, **close)
    assert torch.allclose(x.cpu(), torch.stack(want, 1), atol=1e-5, rtol=1e-5)


@pytest.mark.gpu
@pytest.mark.parametrize("M", [1, 7, 16, 17, 40, 64])
@pytest.mark.parametrize("N,K", [(48, 96), (53, 52), (256, 1000), (5000, 128), (8, 20)])
def test_skinny_product(M, N, K):
    from innova_b200.ops import skinny_gemm
    pad = lambda a: torch.nn.functional.pad(a, (0, -a.shape[1] % 8), value=float("nan")).cuda().bfloat16()      # padding is never used
    x, w = pad(torch.randn(M, K))[:, :K], pad(torch.randn(2 * N, K) * K ** -0.5)[:, :K]
    want = x.double() @ w.double().t()
    assert torch.allclose(skinny_gemm(x, w[:N]).double(), want[:, :N], atol=2e-4, rtol=1e-3)
    got = skinny_gemm(x, w, n=N - 3, silu_half=N, out_dtype=torch.bfloat16).double()
    assert torch.allclose(got, oracle.silu(want[:, :N - 3]) * want[:, N:2 * N - 3], atol=3e-2, rtol=2e-2)


@pytest.mark.parametrize("F", [24, 19])
def test_gated_silu(dev, F):
    d, dt = dev
    half = (F + 7) // 8 * 8
    x = torch.zeros(6, 2 * half)
    x[:, :F], x[:, half:half + F] = torch.randn(6, F), torch.randn(6, F)
    x = x.to(dt)
    got = gated_silu(x.to(d), F, dt).float().cpu()
    want = oracle.silu(x[:, :F].float()) * x[:, half:half + F].float()
    assert got.shape == want.shape and torch.allclose(got, want, atol=3e-2 if dt == torch.bfloat16 else 1e-5)


class Rows:
    """Cache rows for a mechanism on its own: rings and states of one recurrent run, or pages of one attention run."""

    def __init__(self, d, dt, states=(), latents=(), n=4, max_seq=512):
        self.c = StepCache(n, max_seq, d, dt, latents=latents, states=states)

    def batch(self, lens, start, rows):
        for r, n, s in zip(rows, lens, start):
            self.c.reserve(r, n + s)
        return StepBatch(self.c, [[0] * n for n in lens], start, rows)


SHAPES = [dr.DeltaShape(4, 2, 16, 24, 3, 6, 9), dr.DeltaShape(3, 3, 40, 33, 1, 8, 8), dr.DeltaShape(6, 1, 64, 64, 4, 24, 24), dr.DeltaShape(2, 2, 128, 128, 5, 16, 40),
          dr.DeltaShape(2, 2, 50, 256, 2, 4, 4), dr.DeltaShape(1, 1, 200, 20, 4, 8, 8), dr.DeltaShape(4, 2, 32, 16, 9, 7, 130)]


def delta_inputs(s, n, seed, dt):
    g = torch.Generator().manual_seed(seed)
    proj = torch.zeros(n, s.offsets[6])
    for off, m in zip(s.offsets, (s.Hk * s.D, s.Hk * s.D, s.H * s.Dv, s.rank_a, s.rank_g, s.H)):
        proj[:, off:off + m] = torch.randn(n, m, generator=g)
    return proj.to(dt)


def delta_params(s, dt, seed=5):
    g = torch.Generator().manual_seed(seed)
    p = {n: torch.randn(*shape, generator=g) for n, shape in {"taps": (s.taps, s.channels), "A_log": (s.H,), "dt": (s.H * s.D,), "norm": (s.Dv,)}.items()}
    p["dt"] = p["dt"] - 3          # slow decays: the state reaches far back
    p["a2"] = (torch.randn(s.H * s.D, s.rank_a, generator=g) * s.rank_a ** -0.5).to(dt)
    p["g2"] = (torch.randn(s.H * s.Dv, s.rank_g, generator=g) * s.rank_g ** -0.5).to(dt)
    return p


def delta_oracle(s, p, proj, eps):
    """The mixer between its projections, from the oracle's functions."""
    o, n = s.offsets, proj.shape[0]
    x = proj.double()
    c = oracle.silu(oracle.short_conv(x[:, : s.channels], p["taps"].double().t()))
    head = torch.arange(s.H) // (s.H // s.Hk)
    q = (oracle.unit(c[:, o[0]:o[0] + s.Hk * s.D].view(n, s.Hk, s.D)) * s.D ** -0.5)[:, head]
    k = oracle.unit(c[:, o[1]:o[1] + s.Hk * s.D].view(n, s.Hk, s.D))[:, head]
    w = {"a1": torch.eye(s.rank_a).double(), "a2": p["a2"].double(), "dt_bias": p["dt"].double(), "A_log": p["A_log"].double()}
    g = oracle.channel_decay(w, "", s.H, s.D, x[:, o[3]:o[3] + s.rank_a])
    out, S = oracle.delta_rule(q, k, c[:, o[2]:o[2] + s.H * s.Dv].view(n, s.H, s.Dv), torch.sigmoid(x[:, o[5]:o[5] + s.H]), g)
    gate = torch.sigmoid(x[:, o[4]:o[4] + s.rank_g] @ p["g2"].double().t()).view(n, s.H, s.Dv)
    return (oracle.rms_normalise(out, eps) * p["norm"].double() * gate).reshape(n, -1), S


def delta_run(s, p, dev, projs, starts, rows, R, decode=False):
    """One call of the product's mixer core on packed sequences."""
    d, dt = dev
    proj = torch.cat(projs)
    b = R.batch([len(x) for x in projs], starts, rows)
    t = lambda a: a.to(d)
    args = (t(p["taps"]), t(p["A_log"]), t(p["dt"]), t(p["norm"]), 1e-5, R.c.ring[0], R.c.state[0], b)
    pad = lambda a: torch.nn.functional.pad(a, (0, -a.shape[1] % 8)).contiguous()
    if decode:
        return dr.delta_decode(s, t(proj), t(pad(p["a2"].t())), t(pad(p["g2"].t())), *args).float().cpu()
    o = s.offsets
    z = pad(proj[:, o[3]:o[3] + s.rank_a].float() @ p["a2"].float().t())
    gate = pad((proj[:, o[4]:o[4] + s.rank_g].float() @ p["g2"].float().t()).to(dt))
    return dr.delta_prompt(s, t(proj), t(z), t(gate), *args).float().cpu()


@pytest.mark.parametrize("s", SHAPES, ids=lambda s: f"H{s.H}k{s.Hk}D{s.D}v{s.Dv}t{s.taps}")
def test_delta_rule_prompts_portions_and_decoding(dev, s):
    d, dt = dev
    lens, p = [37, 5, 18], delta_params(s, dt)
    xs = [delta_inputs(s, n, 10 + i, dt) for i, n in enumerate(lens)]
    want = [delta_oracle(s, p, x, 1e-5) for x in xs]
    close = dict(atol=4e-2, rtol=4e-2) if dt == torch.bfloat16 else dict(atol=3e-5, rtol=3e-4)
    R = Rows(d, dt, [s])
    R.c.state[0].fill_(7.0)               # what an earlier sequence left behind
    R.c.ring[0].fill_(7.0)
    got = delta_run(s, p, dev, xs, [0, 0, 0], [2, 0, 3], R)
    assert torch.allclose(got, torch.cat([w[0] for w in want]).float(), **close)
    for row, w in zip([2, 0, 3], want):
        assert torch.allclose(R.c.state[0][R.c.slot_of(row)].cpu(), w[1].float(), atol=2e-4 if dt == torch.float32 else 2e-3)
    # the same first sequence again: a prompt portion, two tokens, then token by token, in a slot used before
    x, at = xs[0], 0
    outs = []
    for n, dec in [(20, False), (2, False)] + [(1, True)] * 9 + [(3, False)] + [(1, True)] * 3:
        outs.append(delta_run(s, p, dev, [x[at:at + n]], [at], [0], R, decode=dec))
        at += n
    assert at == 37 and torch.allclose(torch.cat(outs), want[0][0].float(), **close)
    # joint decoding of two sequences at different positions
    R2, halves = Rows(d, dt, [s]), [(xs[0], 30), (xs[2], 12)]
    for row, (x, n) in zip((1, 3), halves):
        delta_run(s, p, dev, [x[:n]], [0], [row], R2)
    R2.c.swap(1, 2)                       # a sequence that changes its row keeps its state
    for k in range(6):
        o = delta_run(s, p, dev, [x[n + k:n + k + 1] for x, n in halves], [n + k for _, n in halves], [2, 3], R2, decode=True)
        assert torch.allclose(o, torch.stack([want[0][0][30 + k], want[2][0][12 + k]]).float(), **close)


@pytest.mark.gpu
def test_delta_decode_reads_fp32_rows():
    s = SHAPES[2]
    p = delta_params(s, torch.bfloat16)
    x = delta_inputs(s, 3, 1, torch.float32)
    R = Rows("cuda", torch.bfloat16, [s])
    got = torch.cat([delta_run(s, p, ("cuda", torch.bfloat16), [x[i:i + 1]], [i], [0], R, decode=True) for i in range(3)])
    assert torch.allclose(got, delta_oracle(s, p, x, 1e-5)[0].float(), atol=2e-2, rtol=2e-2)


@pytest.mark.parametrize("window", [1, 2, 15, 16, 17, 40, 250, None])
@pytest.mark.parametrize("H,R", [(3, 32), (20, 80), (16, 512)])
def test_latent_attention_sees_exactly_its_window(dev, H, R, window):
    """A key that stands out sits just inside, just outside, at page borders and far away; reading it or not decides the output."""
    d, dt = dev
    if d == "cpu" and R == 512:
        pytest.skip("size covered on the GPU")
    n = 300
    g = torch.Generator().manual_seed(R)
    c = torch.randn(n, R, generator=g)
    dirs = torch.nn.functional.normalize(torch.randn(H, R, generator=g), dim=-1)
    far = [0, 15, 16, 31, 59, 60, 61, 127, 128, 255, 256]
    c[far] += 9.0 * dirs[torch.arange(len(far)) % H]            # the key each head looks for
    c = c.to(dt)
    rc = Rows(d, dt, latents=[Latents((R + 15) // 16 * 16, window)])
    b = rc.batch([n], [0], [1])
    nw = torch.ones(R, device=d)
    la.latent_append(c.to(d), 0, R, nw, 0.0, rc.c.latent[0], rc.c.page_table, b)
    cn = oracle.rms_normalise(c.double(), 0.0).to(dt).double()
    edge = sorted({p + k for p in far for k in ((0, window - 1, window) if window else (0, 3)) if p + k < n} | {n - 1})
    q = (dirs * 6.0).repeat(len(edge), 1, 1).to(dt)
    rows = Rows.batch(rc, [1], [edge[0]], [1])                  # a batch object to overwrite: single queries at chosen positions
    rows.tok_pos = torch.tensor(edge, dtype=torch.int32, device=d)
    rows.tok_seq = torch.zeros(len(edge), dtype=torch.int32, device=d)
    got = la.latent_attend(q.reshape(len(edge), H * R).to(d), rc.c.latent[0], rc.c.page_table, H, 1.0, window, rows, window or 512)
    see = oracle.window_visible(n, window)
    for i, p in enumerate(edge):
        s = q[i].double() @ cn.t()
        w = torch.softmax(s.masked_fill(~see[p], -math.inf), -1) @ cn
        assert torch.allclose(got[i].view(H, R).double().cpu(), w, atol=3e-2 if dt == torch.bfloat16 else 2e-5), (p, window)


@pytest.mark.gpu
@pytest.mark.parametrize("T,K,N", [(1, 64, 48), (17, 128, 512), (40, 512, 64), (130, 48, 16)])
def test_head_products(T, K, N):
    H = 5
    a, w = torch.randn(T, H * K + 8, device="cuda").bfloat16(), (torch.randn(H, N, K, device="cuda") * K ** -0.5).bfloat16()
    got = la.head_proj(a[:, : H * K], w).float().view(T, H, N)
    assert torch.allclose(got, torch.einsum("thk,hnk->thn", a[:, : H * K].float().view(T, H, K), w.float()), atol=3e-2, rtol=2e-2)


@pytest.mark.gpu
@pytest.mark.parametrize("D", [64, 128])
@pytest.mark.parametrize("window", [1, 63, 128, 200, None])
def test_packed_flash_attention(D, window):
    lens, H = [1, 300, 129, 128, 64], 3
    q, k, v = (torch.randn(sum(lens), H * D, device="cuda").bfloat16() for _ in range(3))
    rc = Rows("cuda", torch.bfloat16, latents=[Latents(16, window)], n=5)
    got = la.packed_flash(q, k, v, H, D, D ** -0.5, window, rc.batch(lens, [0] * 5, range(5))).float()
    at = 0
    for n in lens:
        s = torch.einsum("ihd,jhd->hij", *(x[at:at + n].float().view(n, H, D) for x in (q, k))) * D ** -0.5
        p = torch.softmax(s.masked_fill(~oracle.window_visible(n, window).cuda(), -math.inf), -1)
        want = torch.einsum("hij,jhd->ihd", p, v[at:at + n].float().view(n, H, D)).reshape(n, -1)
        assert torch.allclose(got[at:at + n], want, atol=2e-2, rtol=2e-2)
        at += n


# ------------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("name", CONFIGS)
def test_logits_and_residuals(dev, name):
    cfg = CONFIGS[name]
    model, w = build(cfg, dev)
    toks = tokens(75, cfg, 1)
    res = []
    want = oracle.forward(cfg, w, toks, residuals=res)
    cache, got_res = model.make_cache(1, 80), []
    cache.reserve(0, 75)
    got = model.step(cache, StepBatch(cache, [toks], [0], [0], want=range(75)), residuals=got_res)
    assert error(got, want) < tol(dev)
    assert len(got_res) == len(res) == len(model.runs)
    for a, b in zip(got_res, res):
        assert error(a, b) < tol(dev)
    assert error(model(torch.tensor([toks, toks[::-1]])).cpu()[0], want) < tol(dev)          # the whole-sequence form


@pytest.mark.parametrize("name", CONFIGS)
@pytest.mark.parametrize("cuts", [[1], [2], [3], [16], [17, 1], [40, 2, 1], [31, 1, 1, 9]], ids=str)
def test_portions_and_token_by_token(dev, name, cuts):
    cfg = CONFIGS[name]
    model, w = build(cfg, dev, 3)
    toks = tokens(58, cfg, 2)
    assert error(run(model, toks, cuts), oracle.forward(cfg, w, toks)) < tol(dev)


@pytest.mark.parametrize("name", ["mixed", "loop"])
def test_long_decoding(dev, name):
    cfg = CONFIGS[name]
    model, w = build(cfg, dev, 4)
    toks = tokens(200, cfg, 5)
    assert error(run(model, toks, [20, 1]), oracle.forward(cfg, w, toks)) < tol(dev)


def test_unequal_requests_and_reused_rows(dev):
    cfg = CONFIGS["mixed"]
    model, w = build(cfg, dev, 6)
    seqs = [tokens(n, cfg, 20 + n) for n in (1, 43, 16, 70)]
    want = [oracle.forward(cfg, w, s + tokens(12, cfg, 9)) for s in seqs]
    tail = tokens(12, cfg, 9)
    gen = Generator(model, max_batch=6, max_seq=96)
    gen.use_graphs = False
    for rows in ([0, 1, 2, 3], [5, 3, 0, 2]):                    # the second pass runs in rows and pages used before
        pos = [0] * 4
        lg = gen.step(seqs, pos, rows)
        assert error(lg, torch.stack([x[len(s) - 1] for x, s in zip(want, seqs)])) < tol(dev)
        for k in range(12):
            live = [i for i in range(4) if not (i == 1 and k >= 5)]          # one request ends early
            if k == 5:
                gen.cache.free(rows[1])
            lg = gen.step([[tail[k]]] * len(live), [len(seqs[i]) + k for i in live], [rows[i] for i in live])
            assert error(lg, torch.stack([want[i][len(seqs[i]) + k] for i in live])) < tol(dev)
        # mixed: one request goes on by one token while another one's prompt comes in
        gen.cache.free(rows[0])
        a, b = len(seqs[3]) + 12, tokens(1, cfg, 77)
        lg = gen.step([b, seqs[2]], [a, 0], [rows[3], rows[0]])
        assert error(lg, torch.stack([oracle.forward(cfg, w, seqs[3] + tail + b)[-1], want[2][len(seqs[2]) - 1]])) < tol(dev)
        for r in rows:
            gen.cache.free(r)
        assert len(gen.cache._free) == gen.cache.num_pages


@pytest.mark.gpu
@pytest.mark.parametrize("n", [20, 40, 70])
@pytest.mark.parametrize("name", ["mixed", "large", "tile"])
def test_wide_decode_batches(name, n):
    """Projections change kernels with the number of rows: up to 32, up to 64, more."""
    cfg = CONFIGS[name]
    for dt in (torch.float32, torch.bfloat16):
        model, w = build(cfg, ("cuda", dt), 14)
        seqs = [tokens(3 + i % 5, cfg, i % 7) + tokens(3, cfg, 90 + i % 3) for i in range(n)]
        known = {}
        gen = Generator(model, max_batch=n, max_seq=32)
        gen.use_graphs = False
        at = [len(s) - 3 for s in seqs]
        gen.step([s[:p] for s, p in zip(seqs, at)], [0] * n, list(range(n)))
        for k in range(3):
            lg = gen.step([[s[p + k]] for s, p in zip(seqs, at)], [p + k for p in at], list(range(n)))
            for i, s in enumerate(seqs):
                if tuple(s) not in known:
                    known[tuple(s)] = oracle.forward(cfg, w, s)
            assert error(lg, torch.stack([known[tuple(s)][p + k] for s, p in zip(seqs, at)])) < tol(("cuda", dt))


def test_pages_behind_every_window_are_given_back():
    cfg = config([ff(attn(2, 16, 16, 32, 20), 32)], streams=2)
    model, w = build(cfg, ("cpu", torch.float32))
    toks = tokens(200, cfg, 3)
    cache = model.make_cache(1, 256, num_pages=5)                # far fewer pages than the sequence has
    assert error(run(model, toks, [30, 7, 1], cache), oracle.forward(cfg, w, toks)) < 3e-5
    assert len(cache._free) >= 5 - 3
    cache.free(0)
    assert sorted(cache._free) == list(range(5))
    with pytest.raises(MemoryError):
        cache.reserve(0, 100)
    assert len(cache._free) == 5


def far_model(dev, size):
    """One attention layer whose first head looks for one marked token: the mark's latent stands out and its value is large."""
    cfg = config([ff(attn(2, 16, 16, 32, size), None)], width=64, vocab=40, streams=2, scale=1.0)
    w = oracle.random_weights(cfg, 8)
    w["embed"][39] *= 6.0
    h = torch.nn.functional.normalize(w["embed"][39] - w["embed"][39].mean(), dim=0)
    w["l0.mix.dkv"][0] = h
    w["l0.mix.uk"][:] *= 0.3
    w["l0.mix.uk"][0, 0] = 4.0
    w["l0.mix.q"][0] = 0.0
    w["l0.norm1.b"][:] = 0.5
    w["l0.mix.q"][0, :] = 0.25                                     # a constant query along the marked key
    w["l0.mix.uv"] *= 0.03
    w["l0.mix.uv"][0, 0] = 0.5                                     # head 0 carries the mark, the rest next to nothing
    w = {n: t.bfloat16().float() for n, t in w.items()}
    return cfg, w, VebesunModel.from_tensors(cfg, w, dtype=dev[1], device=dev[0])


@pytest.mark.parametrize("size", [1, 5, 16, 17, 32, 48])
@pytest.mark.parametrize("cuts", [[120], [50, 1], [13, 2]], ids=str)
def test_window_edges_of_a_model(dev, size, cuts):
    cfg, w, model = far_model(dev, size)
    for mark in (0, 3, 15, 16, 47, 48):
        toks = [t % 39 for t in tokens(120, cfg, mark)]
        toks[mark] = 39
        want = oracle.forward(cfg, w, toks)
        got = run(model, toks, cuts)
        assert error(got, want) < tol(dev)
        if mark + size < 120:      # one token further the mark is out of sight, and that shows: the test can see the edge
            wider = {**cfg, "layers": [ff(attn(2, 16, 16, 32, size + 1), None)]}
            off = oracle.forward(wider, w, toks)
            assert error(off[mark + size:mark + size + 1], want[mark + size:mark + size + 1]) > 2 * tol(dev)


@pytest.mark.parametrize("change", ["taps", "decay", "state", "loop", "streams", "gate", "scale"])
def test_each_mechanism_moves_the_logits(change):
    """The comparison above would notice: the oracle with one mechanism changed is far from the unchanged model."""
    cfg = CONFIGS["mixed"]
    model, w = build(cfg, ("cpu", torch.float32), 2)
    toks = tokens(40, cfg, 4)
    bad, bcfg = dict(w), json.loads(json.dumps(cfg))
    if change == "taps":
        bad["l0.mix.q.conv"] = w["l0.mix.q.conv"].flip(1)
    elif change == "decay":
        bad["l0.mix.A_log"] = w["l0.mix.A_log"] + 1
    elif change == "state":
        bad["l3.mix.b"] = torch.zeros_like(w["l3.mix.b"])
    elif change == "loop":
        bcfg["loop"]["times"] = 2
    elif change == "streams":
        bad["l1.hc1.mix"] = w["l1.hc1.mix"].t()
    elif change == "gate":
        bad["l0.mix.g1"] = torch.zeros_like(w["l0.mix.g1"])
    else:
        bcfg["layers"][1]["mixer"]["scale"] *= 1.5
    assert error(run(model, toks, [40]), oracle.forward(bcfg, bad, toks)) > 1e-2


# ------------------------------------------------------------------------------------------------ generation, files, command line
def greedy(cfg, w, prompt, n):
    out = list(prompt)
    for _ in range(n):
        out.append(int(oracle.forward(cfg, w, out, dtype=torch.float64)[-1].argmax()))
    return out[len(prompt):]


def test_greedy_generation_and_scheduler(dev):
    from innova_b200.inference.serving import ContinuousBatching, Request, StreamingGenerator
    cfg = CONFIGS["mixed"]
    model, w = build(cfg, dev, 11)
    prompts = [tokens(n, cfg, 40 + n) for n in (9, 3, 26, 14, 1)]
    new = [8, 12, 5, 10, 7]
    want = [greedy(cfg, w, p, n) for p, n in zip(prompts, new)]
    if dev[1] == torch.bfloat16:      # rounding may decide a close pair of tokens: compare with generation one by one
        one = Generator(model, max_batch=1, max_seq=64)
        want = [one.generate_tokens([p], n)[0] for p, n in zip(prompts, new)]
    agree = (lambda a, b: sum(x == y for x, y in zip(a, b)) >= 0.6 * len(b)) if dev[1] == torch.bfloat16 else (lambda a, b: a == b)
    gen = Generator(model, max_batch=3, max_seq=64)
    assert all(agree(a, b[:5]) for a, b in zip(gen.generate_tokens(prompts[:3], 5), want))
    cb = ContinuousBatching(gen)      # five requests through three rows: rows and pages are handed on
    for i, (p, n) in enumerate(zip(prompts, new)):
        cb.add_request(Request(id=i, tokens=p, max_tokens=n))
    out = cb.run()
    assert all(len(out[i]) == n and agree(out[i], want[i]) for i, n in enumerate(new))
    assert agree(StreamingGenerator(gen).generate(prompts[0], 6).tokens, want[0][:6])
    with pytest.raises(ValueError):
        gen.step([[cfg["vocab"]]], [0], [0])
    with pytest.raises(NotImplementedError):
        gen._forward_tree([1], [-1], 3)


@pytest.mark.gpu
def test_decode_graphs_equal_eager_steps():
    cfg = CONFIGS["loop"]
    for dt in (torch.float32, torch.bfloat16):
        model, w = build(cfg, ("cuda", dt), 12)
        toks = [tokens(60, cfg, 50 + i) for i in range(3)]
        want = torch.stack([oracle.forward(cfg, w, t) for t in toks])
        gen = Generator(model, max_batch=4, max_seq=128)
        for rows in ([0, 1, 2], [3, 0, 1]):                      # the captured step serves other rows and positions
            for r in range(4):
                gen.cache.free(r)
            gen.step([t[:20 + 5 * i] for i, t in enumerate(toks)], [0, 0, 0], rows)
            for k in range(30):
                at = [20 + 5 * i + k for i in range(3)]
                lg = gen.step([[t[p]] for t, p in zip(toks, at)], at, rows)
                assert error(lg, torch.stack([want[i, p] for i, p in enumerate(at)])) < tol(("cuda", dt))
        assert list(gen._graphs) == [3]


def test_model_directory_and_oil_file(tmp_path):
    from innova_b200.formats import export
    cfg = CONFIGS["odd"]
    w = oracle.random_weights(cfg, 21)
    write_dir(tmp_path / "m", cfg, w)
    m = export.load_model(str(tmp_path / "m"), dtype=torch.float32)
    toks = tokens(30, cfg, 1)
    want = oracle.forward(cfg, w, toks)
    assert isinstance(m, VebesunModel) and error(run(m, toks, [30]), want) < 3e-5
    export.save_model(m, str(tmp_path / "m.oil"))
    m2 = export.load_model(str(tmp_path / "m.oil"), dtype=torch.float32)
    assert isinstance(m2, VebesunModel) and error(run(m2, toks, [11, 1]), want) < 3e-5
    assert {n: tuple(t.shape) for n, t in m2.state_dict_reference().items()} == {n: tuple(t.shape) for n, t in w.items()}
    del w["l1.mix.norm"]
    write_dir(tmp_path / "bad", cfg, w)
    with pytest.raises(KeyError, match="l1.mix.norm"):
        export.load_model(str(tmp_path / "bad"))
    with pytest.raises(ValueError, match="architecture"):
        export.load_model_dir(with_config(tmp_path, {"architecture": "nothing"}))


def test_configuration():
    c = VebesunConfig.from_dict(CONFIGS["mixed"])
    assert c.order() == [0, 1, 2, 1, 2, 1, 2, 3]
    assert VebesunConfig.from_dict(c.to_dict()) == c
    assert VebesunConfig.from_dict({**CONFIGS["mixed"], "loop": None}).order() == [0, 1, 2, 3]
    with pytest.raises(ValueError):
        VebesunConfig.from_dict({**CONFIGS["mixed"], "loop": {"start": 2, "stop": 9, "times": 2}})
    with pytest.raises(ValueError):
        VebesunConfig.from_dict(config([{"type": "other", "mixer": {}, "mlp": None}]))


def test_trace_replay(dev, tmp_path):
    cfg = CONFIGS["mixed"]
    w = oracle.random_weights(cfg, 31)
    write_dir(tmp_path / "m", cfg, w)
    a, b = tokens(50, cfg, 1), tokens(33, cfg, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 21, 29]}, {"id": "b", "tokens": b[:32], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[32:], "want": [0]}, {"id": "a", "tokens": a[30:31], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[31:32], "want": []}], "end": []}]
    steps += [{"step": 3 + k, "entries": [{"id": "a", "tokens": [a[32 + k]], "want": [0]}], "end": ["a"] if k == 17 else []} for k in range(18)]
    steps.append({"step": 30, "entries": [{"id": "a", "tokens": b, "want": [32]}], "end": []})       # the name and the row again
    replay(tmp_path / "m", tmp_path / "o", steps, "bfloat16" if dev[1] == torch.bfloat16 else "float32", dev[0])
    wa, wb = oracle.forward(cfg, w, a), oracle.forward(cfg, w, b)
    read = lambda n: torch.from_numpy(np.fromfile(tmp_path / "o" / f"{n}.f32", dtype="<f4").copy()).view(-1, cfg["vocab"])
    assert error(read(0), wa[[0, 21, 29]]) < tol(dev) and error(read(1), torch.stack([wb[32], wa[30]])) < tol(dev)
    assert not (tmp_path / "o" / "2.f32").exists()
    assert error(torch.cat([read(3 + k) for k in range(18)]), wa[32:50]) < tol(dev) and error(read(30), wb[32:]) < tol(dev)


def test_command_line_generation(tmp_path, capsys):
    from innova_b200.cli.infer import main
    cfg = {**CONFIGS["odd"], "vocab": 300}       # no byte tokenizer for such a vocabulary: ids in, ids out
    w = oracle.random_weights(cfg, 41)
    write_dir(tmp_path / "m", cfg, w)
    main(["--model", str(tmp_path / "m"), "--tokens", "5,9,2", "--greedy", "--max-tokens", "6", "--device", "cpu"])
    assert json.loads(capsys.readouterr().out.splitlines()[-1])["new_tokens"] == greedy(cfg, w, [5, 9, 2], 6)
