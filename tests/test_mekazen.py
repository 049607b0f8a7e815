"""Mekazen decoders against the plain statement of their equations in ``mekazen_oracle.py``.

Every test makes its own small configuration and seeded weights. The ``dev`` fixture runs a test on the CPU path and, on a GPU
box, on the CUDA kernels in 32-bit and in bf16 (``cuda-f32``, ``cuda-bf16``)."""
import json
import math

import numpy as np
import pytest
import torch

import mekazen_oracle as oracle
from innova_b200.inference.generator import Generator
from innova_b200.inference.state_cache import KeyValues, StepBatch, StepCache
from innova_b200.models.mekazen import MekazenConfig, MekazenModel
from innova_b200.ops import kv_attention as ka
from innova_b200.ops import latent_attention as la
from innova_b200.ops.sandwich import sandwich_step, softcap_
from stepped_util import BOTH, IDS, error, replay, run, tokens, tol, with_config, write_dir


@pytest.fixture(params=BOTH, ids=IDS)
def dev(request):
    return request.param


def rot(dims, base=10000.0, scaling=None):
    return {"dims": dims, "base": base, "scaling": scaling}


SCALED = {"factor": 5.0, "low": 1.5, "high": 3.0, "original": 96}


def attn(heads, kv_heads, dim, size, r, ff, scale=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale or dim ** -0.5, "rot": r,
                                           "mask": None if size is None else {"size": size}},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(layers, width=96, vocab=120, eps=1e-5, cap=11.0):
    return {"architecture": "Mekazen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers, "logit_softcap": cap}


CONFIGS = {
    # grouped heads, chunks that are no multiple of a page, layers that differ in every size, one without a feed-forward
    "mixed": config([attn(6, 2, 24, 21, rot(12, scaling=SCALED), 88), attn(3, 3, 40, 33, rot(40, 500.0), None), attn(4, 1, 64, 16, rot(2), 72)]),
    # sizes that are no multiple of 8, no soft limit, no rotation in one layer, a chunk of one token
    "odd": config([attn(3, 1, 20, 7, rot(6, 300.0, SCALED), 50), attn(5, 5, 12, 1, None, 31), attn(2, 1, 18, 40, rot(18), 9)], width=52, vocab=77, cap=None),
    # more than eight query heads per key head, no mask, head sizes of 128 and more
    "wide": config([attn(18, 2, 128, None, rot(64, 1e6, SCALED), 64), attn(2, 1, 144, 50, rot(144), None), attn(9, 1, 200, 24, rot(100), 40)], width=128,
                   eps=1e-3, cap=2.5),
    # head sizes beyond the tensor-core kernels
    "large": config([attn(2, 1, 264, 30, rot(66), 48), attn(3, 3, 250, 64, rot(50), None)], width=64, cap=30.0),
}


def build(cfg, dev, seed=0):
    w = oracle.random_weights(cfg, seed)
    return MekazenModel.from_tensors(cfg, w, dtype=dev[1], device=dev[0]), w


# ------------------------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("E", [64, 37, 200, 1028, 5000, 9000])
@pytest.mark.parametrize("offset", [0.0, 1.0])
def test_sandwich_step(dev, E, offset):
    d, dt = dev
    g = torch.Generator().manual_seed(E)
    T, V, eps = 9, 11, 1e-3
    pad = lambda a: torch.nn.functional.pad(a, (0, -a.shape[1] % 8), value=float("nan"))              # padding is never used
    ids = torch.randint(0, V, (T,), generator=g)
    table, y = torch.randn(V, E, generator=g).to(dt), (torch.randn(T, E, generator=g) * 3).to(dt)
    post, nw = torch.randn(E, generator=g), torch.randn(E, generator=g)
    t = lambda a: a.to(d)
    norm = lambda v, w: oracle.centred_norm(v.double(), w.double() - 1 + offset, eps)
    close = dict(atol=6e-2, rtol=2e-2) if dt == torch.bfloat16 else dict(atol=2e-5, rtol=1e-5)
    x = torch.empty(T, E, device=d)
    h = sandwich_step(x, dt, eps, offset, norm_w=t(nw), ids=t(ids.int()), table=t(pad(table)), scale=2.5)
    x0 = table.float()[ids] * 2.5
    assert torch.equal(x.cpu(), x0) and torch.allclose(h.double().cpu(), norm(x0, nw), **close)
    want = x0.double() + norm(y.float(), post)
    rows = torch.tensor([7, 0, 3], dtype=torch.int32)
    some = sandwich_step(x, dt, eps, offset, y=t(pad(y)), post_w=t(post), norm_w=t(nw), rows=t(rows))          # a selection leaves x alone
    assert torch.allclose(some.double().cpu(), norm(want, nw)[rows.long()], **close) and torch.equal(x.cpu(), x0)
    assert sandwich_step(x.clone(), dt, eps, offset, y=t(pad(y)), post_w=t(post)) is None
    plain = x.clone()
    sandwich_step(plain, dt, eps, offset, y=t(pad(y)))                                                      # no norm of the output
    assert torch.allclose(plain.cpu(), x0 + y.float(), atol=1e-5)
    h = sandwich_step(x, dt, eps, offset, y=t(pad(y)), post_w=t(post), norm_w=t(nw))
    assert torch.allclose(h.double().cpu(), norm(want, nw), **close) and torch.allclose(x.double().cpu(), want, atol=1e-4, rtol=1e-5)
    many = x.repeat(40, 1).clone()                                                                         # the launch shape of prompts
    h2 = sandwich_step(many, dt, eps, offset, y=t(pad(y)).repeat(40, 1), post_w=t(post), norm_w=t(nw))
    ref = norm(x.cpu().double() + norm(y.float(), post), nw)
    assert torch.allclose(h2.double().cpu(), ref.repeat(40, 1), **close)


def test_fp32_output_of_small_products_enters_a_bf16_model(dev):
    d, dt = dev
    x, y, w = torch.randn(3, 40), torch.randn(3, 40), torch.randn(40)
    x1 = x.clone().to(d)
    h = sandwich_step(x1, dt, 1e-5, 1.0, y=y.to(d), post_w=w.to(d), norm_w=w.to(d))
    want = x + oracle.centred_norm(y, w, 1e-5)
    assert torch.allclose(x1.cpu(), want, atol=1e-5) and error(h, oracle.centred_norm(want, w, 1e-5).double()) < tol(dev)


@pytest.mark.parametrize("rows", [3, 50])
def test_softcap(dev, rows):
    for ld, n in ((300, 297), (301, 301), (5000, 4999)):
        z = torch.randn(rows, ld) * 40
        x = z.clone().to(dev[0])
        got = softcap_(x[:, :n], 30.0).cpu()
        assert torch.allclose(got, oracle.softcap(z[:, :n], 30.0), atol=1e-5) and got.abs().max() <= 30.0
        assert torch.equal(x[:, n:].cpu(), z[:, n:])


@pytest.mark.gpu
@pytest.mark.parametrize("M,N,K", [(1, 53, 52), (17, 5000, 128), (40, 256, 1000)])
def test_skinny_product_with_softcap(M, N, K):
    from innova_b200.ops import skinny_gemm
    pad = lambda a: torch.nn.functional.pad(a, (0, -a.shape[1] % 8)).cuda().bfloat16()
    x, w = pad(torch.randn(M, K))[:, :K], pad(torch.randn(N, K) * 3 * K ** -0.5)[:, :K]
    assert torch.allclose(skinny_gemm(x, w, softcap=2.0).double(), oracle.softcap(x.double() @ w.double().t(), 2.0), atol=5e-4, rtol=1e-3)


def test_frequencies():
    for r in (rot(32, 1e6, SCALED), rot(64, 500.0, SCALED), rot(10), rot(8, 100.0, {"factor": 2.0, "low": 1.0, "high": 1.0, "original": 50})):
        got = ka.rope_frequencies(r["dims"], r["base"], r["scaling"])
        assert got.dtype == torch.float32 and torch.allclose(got.double(), oracle.frequencies(r), rtol=1e-6)
    f = oracle.frequencies(rot(64, 500.0, SCALED)) / oracle.frequencies(rot(64, 500.0))          # all three ranges of the scaling occur
    assert f[0] == 1 and abs(f[-1] - 1 / SCALED["factor"]) < 1e-12 and ((f > 0.21) & (f < 0.99)).any()


class Rows:
    """A cache of one attention run on its own."""

    def __init__(self, d, dt, G, D, n=4, max_seq=512, chunk=None, window=None):
        self.c = StepCache(n, max_seq, d, dt, kv=[KeyValues(G, D, window, chunk)])
        self.c.kv[0].fill_(50.0)                   # what earlier sequences left behind

    def batch(self, lens, start, rows):
        for r, n, s in zip(rows, lens, start):
            self.c.reserve(r, n + s)
        return StepBatch(self.c, [[0] * n for n in lens], start, rows)

    def at(self, positions, row):
        """A batch of single queries at chosen positions of one row."""
        b = self.batch([1], [0], [row])
        b.tok_pos = torch.tensor(positions, dtype=torch.int32, device=self.c.device)
        b.tok_seq = torch.zeros(len(positions), dtype=torch.int32, device=self.c.device)
        return b

    def stored(self, row, n):
        """Keys and values [n, G, 2, D] of a row."""
        j = torch.arange(n)
        return self.c.kv[0].cpu()[self.c.page_table.cpu()[row, j // 16].long(), :, :, j % 16]


@pytest.mark.parametrize("H,G,D,pairs", [(6, 2, 24, 6), (3, 3, 40, 20), (4, 1, 64, 0), (24, 3, 128, 16), (2, 1, 144, 72), (40, 8, 256, 100)])
@pytest.mark.parametrize("norms,own_v", [(True, False), (False, True)])
def test_norm_rotation_and_append(dev, H, G, D, pairs, norms, own_v):
    d, dt = dev
    Dp = (D + 63) // 64 * 64
    nq, nk, lens = H * Dp, G * Dp, [19, 1, 4]
    g = torch.Generator().manual_seed(H * D)
    T = sum(lens)
    proj = torch.zeros(T, nq + 2 * nk + 8)
    cols = {"q": (0, H), "k": (nq, G), "v": (nq + nk, G)}
    for off, n in cols.values():
        proj[:, off:off + n * Dp].view(T, n, Dp)[..., :D] = torch.randn(T, n, D, generator=g) * 2
    proj = proj.to(dt)
    pad = lambda n: torch.nn.functional.pad(torch.randn(n, D, generator=g) + 1, (0, Dp - D)).reshape(-1)
    qn, kn, freq = pad(H), pad(G), torch.rand(pairs, generator=g)
    R = Rows(d, dt, G, Dp)
    start, rows = [300, 7, 40], [3, 1, 0]
    b = R.batch(lens, start, rows)
    t = lambda a: a.to(d)
    off_v = nq + nk if own_v else nq
    q, k = ka.qkv_append(t(proj), 0, nq, off_v, H, G, D, Dp, t(qn) if norms else None, t(kn) if norms else None, 1e-2, t(freq), R.c.kv[0], R.c.page_table, b,
                         want_k=True)
    pos = torch.cat([torch.arange(s, s + n) for s, n in zip(start, lens)])
    close = dict(atol=3e-2, rtol=1e-2) if dt == torch.bfloat16 else dict(atol=2e-4, rtol=1e-4)      # (fp32 angles at position 300)

    def part(off, n, norm):
        x = proj[:, off:off + n * Dp].double().view(T, n, Dp)[..., :D].reshape(T, -1)
        if norms:
            x = oracle.rms_normalise(x, 1e-2) * norm.double().view(n, Dp)[:, :D].reshape(-1)
        return oracle.rotate(x.view(T, n, D), pos, freq.double())
    assert torch.allclose(q.double().cpu().view(T, H, Dp)[..., :D], part(0, H, qn), **close)
    keys = part(nq, G, kn)
    assert torch.allclose(k.double().cpu().view(T, G, Dp)[..., :D], keys, **close) and not q.view(T, H, Dp)[..., D:].any()
    at = 0
    for n, s, r in zip(lens, start, rows):
        kv = R.stored(r, s + n)[s:].double()
        assert torch.allclose(kv[:, :, 0, :D], keys[at:at + n], **close)
        assert torch.equal(kv[:, :, 1], proj[at:at + n, off_v:off_v + nk].double().view(n, G, Dp))
        at += n
    rest = R.stored(3, 300)
    assert (rest == 50).all()                                          # nothing before the start was touched


@pytest.mark.parametrize("chunk,window", [(1, None), (2, None), (15, None), (16, None), (17, None), (40, None), (128, None), (250, None), (None, None), (None, 33)])
@pytest.mark.parametrize("H,G,D", [(3, 1, 64), (20, 2, 128), (4, 4, 192), (9, 1, 256), (2, 1, 40)])
def test_attention_sees_exactly_its_chunk(dev, H, G, D, chunk, window):
    """A key that stands out sits just inside, just outside, at page borders and far away; reading it or not decides the output."""
    d, dt = dev
    n, grp = 300, H // G
    g = torch.Generator().manual_seed(D)
    kv = torch.randn(n, G, 2, D, generator=g)
    dirs = torch.nn.functional.normalize(torch.randn(H, D, generator=g), dim=-1)
    far = [0, 14, 15, 16, 17, 31, 39, 40, 127, 128, 249, 250, 255, 256]
    for i, j in enumerate(far):
        kv[j, (i % H) // grp, 0] += 9.0 * dirs[i % H]                  # the key each head looks for
    kv = kv.to(dt)
    R = Rows(d, dt, G, D, chunk=chunk, window=window)
    R.batch([n], [0], [1])
    j = torch.arange(n)
    R.c.kv[0][R.c.page_table[1, j // 16].long(), :, :, (j % 16).to(d)] = kv.to(d)
    edge = sorted({p for q in far for p in (q, q + 1, q + (chunk or window or 3) - 1, q + (chunk or window or 3)) if p < n} | {n - 1})
    q, gate = (dirs * 6.0).repeat(len(edge), 1, 1).to(dt), torch.randn(len(edge), H * D + 5, generator=g).to(dt)
    got = {}
    for name, gt in (("gate", gate.to(d)[:, : H * D]), ("wide gate", gate.to(d).float()[:, : H * D]), ("none", None)):
        got[name] = ka.kv_attend(q.reshape(len(edge), -1).to(d), R.c.kv[0], R.c.page_table, H, 1.0, R.at(edge, 1), window, chunk, gt).double().cpu()
    see = oracle.chunk_visible(n, chunk) if not window else oracle.chunk_visible(n, None) & (j.view(n, 1) - j < window)
    close = dict(atol=3e-2, rtol=1e-2) if dt == torch.bfloat16 else dict(atol=3e-5, rtol=1e-4)
    for i, p in enumerate(edge):
        want = oracle.softmax_attention(q[i:i + 1].double().expand(n, H, D), kv[:, :, 0].double(), kv[:, :, 1].double(), 1.0, see[p].expand(n, n))[0]
        gated = want * oracle.sigmoid(gate[i, : H * D].double())
        assert torch.allclose(got["none"][i], want, **close) and torch.allclose(got["gate"][i], gated, **close), (p, chunk)
        assert torch.allclose(got["wide gate"][i], gated, **close)


@pytest.mark.gpu
@pytest.mark.parametrize("splits,warps", [(1, 4), (2, 4), (4, 8), (8, 4), (8, 8)])
@pytest.mark.parametrize("chunk", [20, 400, None])
def test_every_cluster_shape_gives_the_same(splits, warps, chunk, monkeypatch):
    H, G, D, n = 12, 2, 128, 500
    R = Rows("cuda", torch.bfloat16, G, D, chunk=chunk)
    R.batch([n], [0], [2])
    R.c.kv[0].normal_()
    pos = [0, 1, 15, 16, 19, 20, 255, 399, 400, 499]
    q = torch.randn(len(pos), H * D, device="cuda").bfloat16()
    f = lambda: ka.kv_attend(q, R.c.kv[0], R.c.page_table, H, 0.2, R.at(pos, 2), chunk=chunk).float()
    monkeypatch.setattr(ka, "cluster_shape", lambda *_: (1, 4))
    base = f()
    monkeypatch.setattr(ka, "cluster_shape", lambda *_: (splits, warps))
    assert torch.allclose(f(), base, atol=1e-2, rtol=1e-2)
    kv = R.stored(2, n).double()
    want = oracle.softmax_attention(q.double().cpu()[-1].view(1, H, D).expand(n, H, D), kv[:, :, 0], kv[:, :, 1], 0.2, oracle.chunk_visible(n, chunk)[499].expand(n, n))
    assert torch.allclose(base[-1].double().cpu(), want[0], atol=2e-2, rtol=2e-2)


@pytest.mark.gpu
@pytest.mark.parametrize("D", [64, 128])
@pytest.mark.parametrize("chunk", [1, 63, 128, 200, 256, 290, None])
def test_packed_flash_attention_in_chunks(D, chunk):
    lens, H, G = [1, 300, 129, 128, 600], 6, 2
    q, k, v = (torch.randn(sum(lens), n * D, device="cuda").bfloat16() for n in (H, G, G))
    k.view(-1, G, D)[::7] *= 4                                           # some keys stand out
    gate = torch.randn(sum(lens), H * D + 8, device="cuda").bfloat16()[:, : H * D]
    b = Rows("cuda", torch.bfloat16, 1, 16, n=5, max_seq=640).batch(lens, [0] * 5, range(5))
    got = {name: la.packed_flash(q, k, v, H, D, D ** -0.5, None, b, kv_heads=G, chunk=chunk, gate=x).double().cpu() for name, x in (("gate", gate), ("none", None))}
    at = 0
    for n in lens:
        x = [a[at:at + n].double().cpu().view(n, -1, D) for a in (q, k, v)]
        want = oracle.softmax_attention(*x, D ** -0.5, oracle.chunk_visible(n, chunk))
        assert torch.allclose(got["none"][at:at + n], want, atol=2e-2, rtol=2e-2)
        assert torch.allclose(got["gate"][at:at + n], want * oracle.sigmoid(gate[at:at + n].double().cpu()), atol=2e-2, rtol=2e-2)
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
    assert len(got_res) == len(res) == len(cfg["layers"])
    for a, b in zip(got_res, res):
        assert error(a, b) < tol(dev)
    assert error(model(torch.tensor([toks, toks[::-1]])).cpu()[0], want) < tol(dev)          # the whole-sequence form
    some = model.step(cache, StepBatch(cache, [toks], [0], [0], want=[74, 3]))
    assert error(some, want[[74, 3]]) < tol(dev) and model.step(cache, StepBatch(cache, [toks], [0], [0], want=[])) is None


@pytest.mark.parametrize("name", CONFIGS)
@pytest.mark.parametrize("cuts", [[1], [2], [3], [16], [17, 1], [40, 2, 1], [31, 1, 1, 9]], ids=str)
def test_portions_and_token_by_token(dev, name, cuts):
    cfg = CONFIGS[name]
    model, w = build(cfg, dev, 3)
    toks = tokens(58, cfg, 2)
    assert error(run(model, toks, cuts), oracle.forward(cfg, w, toks)) < tol(dev)


@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_long_decoding(dev, name):
    cfg = CONFIGS[name]
    model, w = build(cfg, dev, 4)
    toks = tokens(200, cfg, 5)
    assert error(run(model, toks, [20, 1]), oracle.forward(cfg, w, toks)) < tol(dev)


def test_long_prompt(dev):
    """Several query and key blocks, with chunks whose edges fall inside them."""
    cfg = config([attn(4, 2, 64, 150, rot(16, 1e4, SCALED), 64), attn(2, 1, 128, 333, rot(128), None), attn(2, 2, 32, None, rot(8), None)], width=64)
    model, w = build(cfg, dev, 2)
    toks = tokens(700, cfg, 6)
    assert error(run(model, toks, [700]), oracle.forward(cfg, w, toks)) < tol(dev)


def test_unequal_requests_and_reused_rows(dev):
    cfg = CONFIGS["mixed"]
    model, w = build(cfg, dev, 6)
    seqs = [tokens(n, cfg, 20 + n) for n in (1, 43, 16, 70)]
    tail = tokens(12, cfg, 9)
    want = [oracle.forward(cfg, w, s + tail) for s in seqs]
    gen = Generator(model, max_batch=6, max_seq=96)
    gen.use_graphs = False
    for rows in ([0, 1, 2, 3], [5, 3, 0, 2]):                    # the second pass runs in rows and pages used before
        lg = gen.step(seqs, [0] * 4, rows)
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
@pytest.mark.parametrize("name", ["mixed", "wide"])
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
            for s in seqs:
                if tuple(s) not in known:
                    known[tuple(s)] = oracle.forward(cfg, w, s)
            assert error(lg, torch.stack([known[tuple(s)][p + k] for s, p in zip(seqs, at)])) < tol(("cuda", dt))


def test_pages_behind_every_chunk_are_given_back():
    cfg = config([attn(2, 1, 16, 20, rot(4), 32), attn(2, 1, 16, 36, rot(4), None)])
    model, w = build(cfg, ("cpu", torch.float32))
    toks = tokens(200, cfg, 3)
    cache = model.make_cache(1, 256, num_pages=5)                # far fewer pages than the sequence has
    assert error(run(model, toks, [30, 7, 1], cache), oracle.forward(cfg, w, toks)) < 3e-5
    assert cache._released[0] * 16 <= 36 * 5 < cache._released[0] * 16 + 16          # position 200 is in the chunk that starts at 180
    with pytest.raises(RuntimeError):
        cache.truncate(0, 170)
    cache.truncate(0, 190)
    assert error(run_on(model, cache, toks, 190), oracle.forward(cfg, w, toks)[190:]) < 3e-5
    cache.free(0)
    assert sorted(cache._free) == list(range(5))
    # a layer that sees everything keeps everything
    whole = MekazenModel(MekazenConfig.from_dict(config([attn(2, 1, 16, 20, None, 32), attn(2, 1, 16, None, None, None)])), dtype=torch.float32, seed=1)
    cache = whole.make_cache(1, 256)
    run(whole, toks, [100, 1], cache)
    assert cache._released == [0] and cache.bytes_per_token() == 2 * 2 * 16 * 4


def run_on(model, cache, toks, at):
    """Token by token from a cache that holds ``at`` tokens."""
    out = []
    for i in range(at, len(toks)):
        cache.reserve(0, i + 1)
        out.append(model.step(cache, StepBatch(cache, [[toks[i]]], [i], [0])))
        cache.commit([0], [i + 1])
    return torch.cat(out)


def far_model(dev, size):
    """One attention layer whose first head looks for one marked token: its key stands out, and with it its value."""
    E, D = 64, 32
    cfg = config([attn(2, 1, D, size, rot(8, 1e4, SCALED), None)], width=E, vocab=40, cap=None)
    g = torch.Generator().manual_seed(8)
    w = oracle.random_weights(cfg, 8)
    w["embed"][:, 0], w["embed"][:, 1] = 3.0, 0.0              # a constant for the query to hold on to; the mark's own dimension
    w["embed"][39, 1] = 40.0
    w["l0.norm1"][:] = 0.0
    w["l0.mix.q"][:] = torch.randn(2 * D, E, generator=g) * 0.02
    w["l0.mix.k"][:] = torch.randn(D, E, generator=g) * 0.1
    w["l0.mix.q"][D - 1, 0], w["l0.mix.k"][D - 1, 1] = 3.0, 1.5    # head 0: the last (unrotated) dimension of query and key
    w["l0.mix.q.norm"][:], w["l0.mix.k.norm"][:] = 1.5, 1.5
    w["l0.mix.g"][:] *= 0.2
    w = {n: t.bfloat16().float() for n, t in w.items()}
    return cfg, w, MekazenModel.from_tensors(cfg, w, dtype=dev[1], device=dev[0])


@pytest.mark.parametrize("size", [1, 5, 16, 17, 32, 48])
@pytest.mark.parametrize("cuts", [[120], [50, 1], [13, 2]], ids=str)
def test_chunk_edges_of_a_model(dev, size, cuts):
    cfg, w, model = far_model(dev, size)
    for mark in (0, 3, 15, 16, 47, 48):
        toks = [t % 39 for t in tokens(120, cfg, mark)]
        toks[mark] = 39
        want = oracle.forward(cfg, w, toks)
        assert error(run(model, toks, cuts), want) < tol(dev)
        edge = (mark // size + 1) * size                       # the first position from which the mark is out of sight
        if edge < 120:                                         # ... with a larger chunk it would not be, and that shows: the test can see the edge
            wider = {**cfg, "layers": [attn(2, 1, 32, None, cfg["layers"][0]["mixer"]["rot"], None)]}
            assert error(oracle.forward(wider, w, toks)[edge:edge + 1], want[edge:edge + 1]) > 2 * tol(dev)


CHANGES = ["post norm", "q norm", "k norm", "values", "pairing", "dims", "frequencies", "scale", "chunk", "chunk start", "gate", "softcap", "groups", "offset"]


@pytest.mark.parametrize("change", CHANGES)
def test_each_mechanism_moves_the_logits(change, monkeypatch):
    """The comparisons above would notice: the oracle with one mechanism changed is far from the unchanged model."""
    cfg = CONFIGS["mixed"]
    model, w = build(cfg, ("cpu", torch.float32), 2)
    toks = tokens(50, cfg, 4)
    bad, bcfg = dict(w), json.loads(json.dumps(cfg))
    plain_norm, plain_rot, plain_attn = oracle.centred_norm, oracle.rotate, oracle.softmax_attention
    if change == "post norm":
        bad["l1.norm1b"] = w["l1.norm1b"] + 0.3
    elif change in ("q norm", "k norm"):
        bad[f"l0.mix.{change[0]}.norm"] = w[f"l0.mix.{change[0]}.norm"].flip(0)
    elif change == "values":                                   # the values taken after the norm and rotation
        monkeypatch.setattr(oracle, "softmax_attention", lambda q, k, v, *a: plain_attn(q, k, k, *a))
    elif change == "pairing":                                  # halves instead of neighbours
        def halves(x, p, f):
            r = 2 * len(f)
            i = torch.arange(r).view(2, -1).t().reshape(-1)
            y = x.clone()
            y[..., i] = plain_rot(x[..., i], p, f)
            return y
        monkeypatch.setattr(oracle, "rotate", halves)
    elif change == "dims":
        bcfg["layers"][0]["mixer"]["rot"]["dims"] = 24
    elif change == "frequencies":
        bcfg["layers"][0]["mixer"]["rot"]["scaling"] = None
    elif change == "scale":
        bcfg["layers"][1]["mixer"]["scale"] *= 1.5
    elif change == "chunk":
        bcfg["layers"][2]["mixer"]["mask"]["size"] += 1
    elif change == "chunk start":                              # a sliding window of the same size
        monkeypatch.setattr(oracle, "chunk_visible", lambda n, s: (torch.arange(n).view(n, 1) >= torch.arange(n)) & (torch.arange(n).view(n, 1) - torch.arange(n) < s))
    elif change == "gate":
        bad["l0.mix.g"] = torch.zeros_like(w["l0.mix.g"])
    elif change == "softcap":
        bcfg["logit_softcap"] = None
    elif change == "groups":
        bad["l0.mix.k"] = w["l0.mix.k"].view(2, -1, 96).flip(0).reshape(-1, 96)
    else:
        monkeypatch.setattr(oracle, "centred_norm", lambda x, v, e: plain_norm(x, v - 1, e))
    assert error(run(model, toks, [50]), oracle.forward(bcfg, bad, toks)) > 1e-2


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


def test_speculative_decoding_rewinds_the_cache(dev):
    from innova_b200.inference.speculative import EXACT, SpeculativeDecoder
    cfg = CONFIGS["mixed"]
    model, w = build(cfg, dev, 11)
    other, _ = build(cfg, dev, 12)                            # drafts that are hardly ever right, and drafts that always are
    prompt = tokens(14, cfg, 3)
    want = Generator(model, max_batch=1, max_seq=96).generate_tokens([prompt], 40)[0]
    if dev[1] == torch.float32:
        assert want == greedy(cfg, w, prompt, 40)
    for draft in (model, other):
        dec = SpeculativeDecoder(Generator(model, max_batch=1, max_seq=96), Generator(draft, max_batch=1, max_seq=96), mode=EXACT)
        got = dec.generate_tokens(prompt, 40)
        assert got == want if dev[1] == torch.float32 else got[:3] == want[:3]


@pytest.mark.gpu
def test_decode_graphs_equal_eager_steps():
    cfg = CONFIGS["mixed"]
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
    assert isinstance(m, MekazenModel) and error(run(m, toks, [30]), want) < 3e-5
    export.save_model(m, str(tmp_path / "m.oil"))
    m2 = export.load_model(str(tmp_path / "m.oil"), dtype=torch.float32)
    assert isinstance(m2, MekazenModel) and error(run(m2, toks, [11, 1]), want) < 3e-5
    back = m2.state_dict_reference()
    assert set(back) == set(w) and all(torch.equal(back[n], t) for n, t in w.items())
    half = MekazenModel.from_tensors(cfg, w).state_dict_reference()                   # bf16 weights, padded for the tensor-core kernels
    assert all(torch.equal(half[n], t) for n, t in w.items())
    del w["l1.mix.q.norm"]
    write_dir(tmp_path / "bad", cfg, w)
    with pytest.raises(KeyError, match="l1.mix.q.norm"):
        export.load_model(str(tmp_path / "bad"))
    with pytest.raises(ValueError, match="architecture"):
        export.load_model_dir(with_config(tmp_path, {"architecture": "nothing"}))


def test_configuration():
    c = MekazenConfig.from_dict(CONFIGS["mixed"])
    assert MekazenConfig.from_dict(c.to_dict()) == c and c.num_layers == 3
    bad = lambda **kw: config([{**attn(4, 2, 16, 8, rot(4), 8), "mixer": {**attn(4, 2, 16, 8, rot(4), 8)["mixer"], **kw}}])
    for kw in ({"vdim": 8}, {"kv_heads": 3}, {"rot": rot(18)}, {"rot": rot(3)}):
        with pytest.raises(ValueError):
            MekazenConfig.from_dict(bad(**kw))
    with pytest.raises(ValueError):
        MekazenConfig.from_dict(config([{"type": "other", "mixer": {}, "mlp": None}]))
    with pytest.raises(ValueError):
        MekazenConfig.from_dict(config([{**attn(4, 2, 16, 8, None, 8), "mlp": {"kind": "sparse", "ff": 8}}]))


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
