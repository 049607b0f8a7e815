"""Sequence mixers and feed-forward of the layer-list decoders, as modules with fused, padded weights.

A module is built for one set of sizes, loads its tensors by name (``load``), gives them back under the same names
(``export``), and runs on packed tokens (``run(ctx, h, cache_index)``). ``ctx`` is the step (``StepContext``): it chooses the
projections' precision and kernel. A mixer says what a run of it keeps: ``cache_kind`` (an argument of ``StepCache``) and
``cache_spec``; ``check`` refuses settings that it does not have.

Weights of the projections are kept in the model's type with rows padded to 16 bytes; everything that enters a norm, a
convolution, a decay or a residual is fp32."""
from __future__ import annotations

from typing import Dict

import torch
import torch.nn as nn
import torch.nn.functional as F

from ..inference.state_cache import KeyValues, Latents
from ..ops import delta_rule as dr
from ..ops import kv_attention as ka
from ..ops import latent_attention as la
from ..ops.gemm import EPI_ATOMIC, NUM_SMS, SKINNY_ROWS, gemm, skinny_gemm
from ..ops.hyper import gated_silu
from ..ops.sandwich import softcap_


def pad_to(n: int, m: int) -> int:
    return (n + m - 1) // m * m


def frozen(*shape, dtype) -> nn.Parameter:
    return nn.Parameter(torch.zeros(*shape, dtype=dtype), requires_grad=False)


class Proj(nn.Module):
    """A projection [n, k]; stored [n padded to 8, k padded to 8] so that rows start on 16-byte boundaries."""

    def __init__(self, n: int, k: int, dtype):
        super().__init__()
        self.n, self.k = n, k
        self.weight = frozen(pad_to(n, 8), pad_to(k, 8), dtype=dtype)


def put(p: Proj, w: torch.Tensor, row: int = 0):
    p.weight[row:row + w.shape[0], : w.shape[1]].copy_(w)


class StepContext:
    """Precision of one forward step. bf16 steps of one token per sequence, at most 64 of them, hand fp32 projections to the
    consuming kernels: up to 32 rows from the skinny product, more from the tiled tcgen05 product split over K. Larger steps run
    the tiled product and write bf16."""

    SPLIT_ROWS = 64

    def __init__(self, model, cache, batch):
        self.batch, self.cache, self.dtype = batch, cache, model.dtype
        self.bf16 = cache.device.type == "cuda" and self.dtype == torch.bfloat16
        self.small = self.bf16 and batch.single and batch.T <= self.SPLIT_ROWS
        self.skinny = self.small and batch.T <= SKINNY_ROWS

    def project(self, x: torch.Tensor, p: Proj, out_dtype=None) -> torch.Tensor:
        """[T, k] -> [T, padded n] (whole padded rows)."""
        x, w = x[:, : p.k], p.weight[:, : p.k]
        if not self.bf16:
            return F.linear(x, w).to(out_dtype or self.dtype)
        rows, n = x.shape[0], w.shape[0]
        if self.skinny or (rows <= SKINNY_ROWS and out_dtype == torch.float32):
            return skinny_gemm(x, w)
        if self.small and (n + 255) // 256 <= NUM_SMS // 2:
            out = torch.zeros(rows, n, dtype=torch.float32, device=x.device)
            return gemm(x, w, out=out, epilogue=EPI_ATOMIC, split_k=max(1, NUM_SMS // ((n + 255) // 256)))
        return gemm(x, w, out_dtype=torch.float32 if self.small else (out_dtype or torch.bfloat16))

    def gated(self, x: torch.Tensor, p: Proj, ff: int) -> torch.Tensor:
        """silu(gate x) * (up x) for a projection that holds the gate rows, then (from the middle) the up rows."""
        if self.skinny:
            return skinny_gemm(x[:, : p.k], p.weight[:, : p.k], n=ff, silu_half=p.n // 2, out_dtype=torch.bfloat16)
        return gated_silu(self.project(x, p), ff, self.dtype)


    def logits(self, h: torch.Tensor, p: Proj, vocab: int, softcap=None) -> torch.Tensor:
        """fp32 [rows, vocab] of the output head, through the soft limit softcap * tanh(z / softcap) if there is one."""
        if self.bf16 and h.shape[0] <= SKINNY_ROWS:
            return skinny_gemm(h[:, : p.k], p.weight[:, : p.k], softcap=softcap or 0.0)[:, :vocab]
        z = self.project(h, p, torch.float32)[:, :vocab]
        return softcap_(z, softcap) if softcap else z


class Mixer(nn.Module):
    @classmethod
    def check(cls, m: dict, layer: int):
        pass


class GatedAttention(Mixer):
    """Grouped-query attention whose projected keys (before norm and rotation) are the values, with RMS norms over the whole query
    and key rows, rotary positions on neighbouring pairs of the first dimensions, a mask of chunks counted from position 0, and a
    sigmoid gate on the output.

    Heads are padded with zero weights to a multiple of 64 in bf16 (the tensor-core kernels' sizes). Whole bf16 prompts run the
    tcgen05 flash kernel, everything else attends over the pages."""

    kind = "attention"
    cache_kind = "kv"

    def __init__(self, width: int, m: dict, eps: float, dtype, shapes=None):
        super().__init__()
        self.H, self.G, self.D = m["heads"], m["kv_heads"], m["dim"]
        self.scale, self.eps, self.width = float(m["scale"]), eps, width
        self.chunk = (m.get("mask") or {}).get("size")
        self.Dp = pad_to(self.D, 64 if dtype == torch.bfloat16 and self.D <= 256 else 8)
        self.nq, self.nk = self.H * self.Dp, self.G * self.Dp
        self.inp = Proj(2 * self.nq + self.nk, width, dtype)         # queries, keys, gate
        self.q_norm, self.k_norm = frozen(self.nq, dtype=torch.float32), frozen(self.nk, dtype=torch.float32)
        rot = m.get("rot")
        self.register_buffer("freq", ka.rope_frequencies(rot["dims"], rot["base"], rot.get("scaling")) if rot else torch.zeros(0), persistent=False)
        self.out = Proj(width, self.nq, dtype)

    @classmethod
    def check(cls, m: dict, layer: int):
        if m.get("vdim", m["dim"]) != m["dim"]:
            raise ValueError(f"layer {layer}: values are the keys, but vdim {m['vdim']} is not dim {m['dim']}")
        if m["heads"] % m["kv_heads"]:
            raise ValueError(f"layer {layer}: {m['heads']} heads do not share {m['kv_heads']} key heads evenly")
        rot = m.get("rot")
        if rot and (rot["dims"] % 2 or not 0 <= rot["dims"] <= m["dim"]):
            raise ValueError(f"layer {layer}: cannot rotate {rot['dims']} of {m['dim']} dimensions")

    @property
    def cache_spec(self):
        return KeyValues(self.G, self.Dp, chunk=self.chunk)

    @torch.no_grad()
    def load(self, t: Dict[str, torch.Tensor], p: str):
        H, G, D, Dp, E = self.H, self.G, self.D, self.Dp, self.width
        for name, off, n in (("q", 0, H), ("k", self.nq, G), ("g", self.nq + self.nk, H)):
            self.inp.weight.data[off:off + n * Dp].view(n, Dp, -1)[:, :D, :E].copy_(t[p + name].view(n, D, E))
        self.q_norm.data.view(H, Dp)[:, :D].copy_(t[p + "q.norm"].view(H, D))
        self.k_norm.data.view(G, Dp)[:, :D].copy_(t[p + "k.norm"].view(G, D))
        self.out.weight.data[:E, :self.nq].view(E, H, Dp)[:, :, :D].copy_(t[p + "o"].view(E, H, D))

    def export(self, p: str) -> Dict[str, torch.Tensor]:
        H, G, D, Dp, E = self.H, self.G, self.D, self.Dp, self.width
        out = {p + name: self.inp.weight[off:off + n * Dp].view(n, Dp, -1)[:, :D, :E].reshape(n * D, E)
               for name, off, n in (("q", 0, H), ("k", self.nq, G), ("g", self.nq + self.nk, H))}
        out.update({p + "q.norm": self.q_norm.view(H, Dp)[:, :D].reshape(-1), p + "k.norm": self.k_norm.view(G, Dp)[:, :D].reshape(-1),
                    p + "o": self.out.weight[:E, :self.nq].view(E, H, Dp)[:, :, :D].reshape(E, H * D)})
        return out

    @staticmethod
    def shapes(width: int, m: dict, p: str, ranks) -> Dict[str, tuple]:
        nq, nk = m["heads"] * m["dim"], m["kv_heads"] * m["dim"]
        return {p + "q": (nq, width), p + "k": (nk, width), p + "q.norm": (nq,), p + "k.norm": (nk,), p + "g": (nq, width), p + "o": (width, nq)}

    def run(self, ctx: StepContext, h: torch.Tensor, index: int) -> torch.Tensor:
        b, cache, nq, nk = ctx.batch, ctx.cache, self.nq, self.nk
        proj = ctx.project(h, self.inp)
        flash = ctx.bf16 and b.fresh and not b.single and self.Dp <= 128
        q, k = ka.qkv_append(proj, 0, nq, nq, self.H, self.G, self.D, self.Dp, self.q_norm, self.k_norm, self.eps, self.freq, cache.kv[index],
                             cache.page_table, b, want_k=flash)
        gate = proj[:, nq + nk:2 * nq + nk]
        if flash:
            o = la.packed_flash(q, k, proj[:, nq:nq + nk], self.H, self.Dp, self.scale, None, b, kv_heads=self.G, chunk=self.chunk, gate=gate)
        else:
            o = ka.kv_attend(q, cache.kv[index], cache.page_table, self.H, self.scale, b, chunk=self.chunk, gate=gate)
        return ctx.project(o, self.out)


class LatentAttention(Mixer):
    """Attention whose keys and values are linear images of one cached latent per token, optionally windowed.

    Query / value heads are padded to ``Dp`` (64 or 128 where they fit, for the tcgen05 flash kernel) and the latent to ``Rp``
    with zero weights. Whole bf16 prompts expand keys and values and run flash attention; decode steps, later portions of a
    prompt and 32-bit models attend in the latent space."""

    kind = "latent_attention"
    cache_kind = "latents"

    def __init__(self, width: int, m: dict, eps: float, dtype, shapes=None):
        super().__init__()
        self.H, self.D, self.Dv, self.R = m["heads"], m["dim"], m["vdim"], m["kv_rank"]
        self.scale, self.eps, self.width = float(m["scale"]), eps, width
        self.window = (m.get("mask") or {}).get("size")
        big = max(self.D, self.Dv)
        self.Dp = 64 if big <= 64 else 128 if big <= 128 else pad_to(big, 16)
        self.Rp = pad_to(self.R, 16)
        self.off_c = self.H * self.Dp
        self.inp = Proj(self.off_c + self.Rp, width, dtype)
        self.norm = frozen(self.R, dtype=torch.float32)
        self.uk = frozen(self.H, self.Rp, self.Dp, dtype=dtype)       # per head, latent rows: q' = uk q
        self.kv = Proj(2 * self.off_c, self.Rp, dtype)                # keys of all heads, then values: expansion of prompts
        self.out = Proj(width, self.off_c, dtype)

    @property
    def cache_spec(self):
        return Latents(self.Rp, window=self.window)

    @torch.no_grad()
    def load(self, t: Dict[str, torch.Tensor], p: str):
        H, D, Dv, Dp, R = self.H, self.D, self.Dv, self.Dp, self.R
        self.inp.weight.data[: H * Dp].view(H, Dp, -1)[:, :D, : self.width].copy_(t[p + "q"].view(H, D, self.width))
        put(self.inp, t[p + "dkv"], self.off_c)
        self.norm.copy_(t[p + "dkv.norm"])
        kv = self.kv.weight.data.view(2, H, Dp, -1)
        kv[0, :, :D, :R].copy_(t[p + "uk"].view(H, D, R))
        kv[1, :, :Dv, :R].copy_(t[p + "uv"].view(H, Dv, R))
        self.uk.copy_(kv[0].transpose(1, 2))
        self.out.weight.data[: self.width].view(self.width, H, Dp)[:, :, :Dv].copy_(t[p + "o"].view(self.width, H, Dv))

    def export(self, p: str) -> Dict[str, torch.Tensor]:
        H, D, Dv, Dp, R, E = self.H, self.D, self.Dv, self.Dp, self.R, self.width
        kv = self.kv.weight.view(2, H, Dp, -1)
        return {p + "q": self.inp.weight[: H * Dp].view(H, Dp, -1)[:, :D, :E].reshape(H * D, E),
                p + "dkv": self.inp.weight[self.off_c:self.off_c + R, :E], p + "dkv.norm": self.norm,
                p + "uk": kv[0, :, :D, :R].reshape(H * D, R), p + "uv": kv[1, :, :Dv, :R].reshape(H * Dv, R),
                p + "o": self.out.weight[:E].view(E, H, Dp)[:, :, :Dv].reshape(E, H * Dv)}

    @staticmethod
    def shapes(width: int, m: dict, p: str, ranks) -> Dict[str, tuple]:
        H, D, Dv, R = m["heads"], m["dim"], m["vdim"], m["kv_rank"]
        return {p + "q": (H * D, width), p + "dkv": (R, width), p + "dkv.norm": (R,), p + "uk": (H * D, R), p + "uv": (H * Dv, R),
                p + "o": (width, H * Dv)}

    def run(self, ctx: StepContext, h: torch.Tensor, index: int) -> torch.Tensor:
        b, cache = ctx.batch, ctx.cache
        pool, T, nq = cache.latent[index], h.shape[0], self.off_c
        qc = ctx.project(h, self.inp)
        flash = ctx.bf16 and b.fresh and not b.single and self.Dp <= 128
        c, q = la.latent_append(qc, nq, self.R, self.norm, self.eps, pool, cache.page_table, b, want_c=flash,
                                nq=nq if qc.dtype != pool.dtype else 0)
        q = qc[:, :nq] if q is None else q
        if flash:
            kv = ctx.project(c, self.kv)
            o = la.packed_flash(q, kv[:, :nq], kv[:, nq:], self.H, self.Dp, self.scale, self.window, b)
        else:
            span = min(self.window or cache.max_pages * la.PAGE, cache.max_pages * la.PAGE)
            lat = la.latent_attend(la.head_proj(q, self.uk), pool, cache.page_table, self.H, self.scale, self.window, b, span)
            o = la.head_proj(lat, self.kv.weight[nq:2 * nq].view(self.H, self.Dp, self.Rp))
        return ctx.project(o, self.out)


class ChannelDelta(Mixer):
    """Gated delta rule with short convolutions, a low-rank decay per key channel and a low-rank output gate."""

    kind = "channel_delta"
    cache_kind = "states"

    def __init__(self, width: int, m: dict, eps: float, dtype, shapes=None):
        super().__init__()
        a_rank, g_rank = shapes["a1"][0], shapes["g1"][0]
        s = self.shape = dr.DeltaShape(m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"], a_rank, g_rank)
        self.width, self.eps = width, eps
        self.inp = Proj(s.offsets[6], width, dtype)
        self.taps = frozen(s.taps, s.channels, dtype=torch.float32)
        self.a2, self.g2 = Proj(s.H * s.D, a_rank, dtype), Proj(s.H * s.Dv, g_rank, dtype)
        self.a2t, self.g2t = frozen(a_rank, pad_to(s.H * s.D, 8), dtype=dtype), frozen(g_rank, pad_to(s.H * s.Dv, 8), dtype=dtype)
        self.A_log, self.dt_bias = frozen(s.H, dtype=torch.float32), frozen(s.H * s.D, dtype=torch.float32)
        self.norm = frozen(s.Dv, dtype=torch.float32)
        self.out = Proj(width, s.H * s.Dv, dtype)

    @property
    def cache_spec(self):
        return self.shape

    @torch.no_grad()
    def load(self, t: Dict[str, torch.Tensor], p: str):
        s, o = self.shape, self.shape.offsets
        for name, off in zip(("q", "k", "v", "a1", "g1", "b"), o):
            put(self.inp, t[p + name], off)
        for name, off in zip(("q", "k", "v"), o):
            w = t[f"{p}{name}.conv"]
            self.taps[:, off:off + w.shape[0]].copy_(w.t())
        put(self.a2, t[p + "a2"])
        put(self.g2, t[p + "g2"])
        self.a2t[:, : s.H * s.D].copy_(t[p + "a2"].t())
        self.g2t[:, : s.H * s.Dv].copy_(t[p + "g2"].t())
        self.A_log.copy_(t[p + "A_log"])
        self.dt_bias.copy_(t[p + "dt_bias"])
        self.norm.copy_(t[p + "norm"])
        put(self.out, t[p + "o"])

    def export(self, p: str) -> Dict[str, torch.Tensor]:
        s, o, E = self.shape, self.shape.offsets, self.width
        rows = {"q": s.Hk * s.D, "k": s.Hk * s.D, "v": s.H * s.Dv, "a1": s.rank_a, "g1": s.rank_g, "b": s.H}
        out = {p + n: self.inp.weight[off:off + r, :E] for (n, r), off in zip(rows.items(), o)}
        for n, off in zip("qkv", o):
            out[f"{p}{n}.conv"] = self.taps[:, off:off + rows[n]].t()
        out.update({p + "a2": self.a2.weight[: s.H * s.D, : s.rank_a], p + "g2": self.g2.weight[: s.H * s.Dv, : s.rank_g], p + "A_log": self.A_log,
                    p + "dt_bias": self.dt_bias, p + "norm": self.norm, p + "o": self.out.weight[:E, : s.H * s.Dv]})
        return out

    @staticmethod
    def shapes(width: int, m: dict, p: str, ranks) -> Dict[str, tuple]:
        H, Hk, D, Dv, K, (ra, rg) = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"], ranks
        out = {p + "b": (H, width), p + "A_log": (H,), p + "norm": (Dv,), p + "a1": (ra, width), p + "a2": (H * D, ra), p + "dt_bias": (H * D,),
               p + "g1": (rg, width), p + "g2": (H * Dv, rg), p + "o": (width, H * Dv)}
        for n, ch in (("q", Hk * D), ("k", Hk * D), ("v", H * Dv)):
            out[p + n], out[f"{p}{n}.conv"] = (ch, width), (ch, K)
        return out

    def run(self, ctx: StepContext, h: torch.Tensor, index: int) -> torch.Tensor:
        s, b, cache = self.shape, ctx.batch, ctx.cache
        proj = ctx.project(h, self.inp)
        args = (self.taps, self.A_log, self.dt_bias, self.norm, self.eps, cache.ring[index], cache.state[index], b)
        if b.single and s.tile_bytes <= dr.DECODE_MAX_TILE:
            o = dr.delta_decode(s, proj, self.a2t, self.g2t, *args)
        else:
            wide = proj.to(ctx.dtype)      # (a decode step with a state tile too large for the one-launch kernel has fp32 rows)
            z = ctx.project(wide[:, s.offsets[3]:], self.a2, torch.float32)
            gate = ctx.project(wide[:, s.offsets[4]:], self.g2).to(ctx.dtype)
            o = dr.delta_prompt(s, proj, z, gate, *args)
        return ctx.project(o, self.out)


class GatedMLP(nn.Module):
    """W_down (silu(W_gate h) * (W_up h))."""

    def __init__(self, width: int, ff: int, dtype):
        super().__init__()
        self.width, self.ff, self.half = width, ff, pad_to(ff, 8)
        self.inp = Proj(2 * self.half, width, dtype)
        self.out = Proj(width, ff, dtype)

    @torch.no_grad()
    def load(self, t, p):
        put(self.inp, t[p + "gate"])
        put(self.inp, t[p + "up"], self.half)
        put(self.out, t[p + "down"])

    def export(self, p):
        return {p + "gate": self.inp.weight[: self.ff, : self.width], p + "up": self.inp.weight[self.half:self.half + self.ff, : self.width],
                p + "down": self.out.weight[: self.width, : self.ff]}

    def run(self, ctx: StepContext, h: torch.Tensor, index: int = 0) -> torch.Tensor:
        return ctx.project(ctx.gated(h, self.inp, self.ff), self.out)


MIXERS = {c.kind: c for c in (GatedAttention, LatentAttention, ChannelDelta)}
