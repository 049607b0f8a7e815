"""Attention over a paged cache of keys and values whose layers differ in head counts and sizes (``csrc/kv_attn.cu``).

``qkv_append`` is everything between a fused projection and the attention: norm of the whole query and key rows, rotation of
neighbouring pairs, append to the pages. ``kv_attend`` attends over the pages with a chunked mask, a sliding window or neither, and
an optional output gate. Whole prompts use ``latent_attention.packed_flash`` on the same arguments."""
from __future__ import annotations

import math
from typing import Optional

import torch

from .. import _native
from . import runtime as rt

_vp, _i, _f = _native.vp, _native.i32, _native.f32
_native.register_cuda_sigs({
    "inv_qkv_prep": [_vp] + [_i] * 9 + [_vp, _vp, _f, _vp, _i, _vp, _i, _vp, _i, _vp, _vp, _vp, _vp, _vp, _i, _vp],
    "inv_kv_attend": [_vp, _vp, _i, _vp, _i, _vp, _vp, _vp, _i, _i, _f, _vp, _i, _i, _vp] + [_i] * 6 + [_vp],
})

PAGE = 16


def rope_frequencies(dims: int, base: float, scaling: Optional[dict] = None) -> torch.Tensor:
    """Angle per position of every rotated pair, fp32 [dims / 2]. ``scaling`` (factor, low, high, original): pairs that turn fewer than
    ``low`` times within ``original`` positions are slowed down by ``factor``, those above ``high`` stay, the rest is interpolated."""
    out = []
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        if scaling:
            turns, low, high = scaling["original"] * f / (2.0 * math.pi), scaling["low"], scaling["high"]
            keep = 1.0 if turns > high else 0.0 if turns < low else (turns - low) / (high - low) if high > low else 1.0
            f = (1.0 - keep) * f / scaling["factor"] + keep * f
        out.append(f)
    return torch.tensor(out, dtype=torch.float32)


def _rotate_pairs(x: torch.Tensor, pos: torch.Tensor, freq: torch.Tensor) -> torch.Tensor:
    r = 2 * freq.numel()
    if r == 0:
        return x
    a = (pos.float().unsqueeze(1) * freq).unsqueeze(1)                  # [T, 1, pairs]
    u, v = x[..., 0:r:2], x[..., 1:r:2]
    y = torch.stack([u * a.cos() - v * a.sin(), v * a.cos() + u * a.sin()], -1).flatten(-2)
    return torch.cat([y, x[..., r:]], -1)


def qkv_append(proj, off_q: int, off_k: int, off_v: int, heads: int, kv_heads: int, dim: int, padded: int, q_norm, k_norm, eps: float, freq, pool,
               page_table, batch, want_k: bool = False):
    """proj [T, columns]: queries, keys and values (which may be the key columns themselves) from their offsets, heads ``padded``
    columns apart of which ``dim`` are used; pool [pages, kv_heads, 2, 16, padded]. Norm weights [heads * padded] and
    [kv_heads * padded] fp32, or None. Returns (queries [T, heads * padded], keys [T, kv_heads * padded] if ``want_k``)."""
    T, dt = proj.shape[0], pool.dtype
    nq, nk = heads * padded, kv_heads * padded
    if not proj.is_cuda:
        pos = batch.tok_pos.long()

        def part(off, n, norm, used):
            x = proj[:, off:off + n].float()
            if norm is not None:
                x = x / torch.sqrt(x.square().sum(-1, keepdim=True) / used + eps) * norm
            return _rotate_pairs(x.view(T, -1, padded), pos, freq).to(dt)
        q, k = part(off_q, nq, q_norm, heads * dim), part(off_k, nk, k_norm, kv_heads * dim)
        page = page_table[batch.rows.long()[batch.tok_seq.long()], pos // PAGE].long()
        pool[page, :, 0, pos % PAGE] = k
        pool[page, :, 1, pos % PAGE] = proj[:, off_v:off_v + nk].to(dt).view(T, kv_heads, padded)
        return q.reshape(T, nq), (k.reshape(T, nk) if want_k else None)
    q = torch.empty(T, nq, dtype=dt, device=proj.device)
    k = torch.empty(T, nk, dtype=dt, device=proj.device) if want_k else None
    rt.check(rt.lib().inv_qkv_prep(proj.data_ptr(), proj.stride(0), int(proj.dtype == torch.float32), off_q, off_k, off_v, heads, kv_heads, dim, padded,
                                   rt.ptr(q_norm), rt.ptr(k_norm), float(eps), freq.data_ptr(), freq.numel(), pool.data_ptr(),
                                   int(dt == torch.float32), page_table.data_ptr(), page_table.shape[1], batch.rows.data_ptr(),
                                   batch.tok_seq.data_ptr(), batch.tok_pos.data_ptr(), q.data_ptr(), rt.ptr(k), T, rt.stream_ptr()), "inv_qkv_prep")
    return q, k


def first_visible(pos: int, window: Optional[int], chunk: Optional[int]) -> int:
    """The first position that a token at ``pos`` sees."""
    return pos - pos % chunk if chunk else max(0, pos - window + 1) if window else 0


def cluster_shape(rows: int, groups: int, span: int):
    """(CTAs, warps per CTA) that share one (row, key head): about 1024 warps in flight altogether, at least two pages each."""
    pages, units = -(-span // PAGE), rows * groups
    if 444 < units <= 888 and pages >= 128:
        return 2, 4                  # one CTA per unit would leave the second wave of CTAs nearly empty
    warps = 4
    while warps < 32 and units * warps * 2 <= 1024 and pages >= warps * 4:
        warps *= 2
    if warps == 32 and units <= 8 and pages >= 256:
        return 8, 8
    return {4: (1, 4), 8: (1, 8), 16: (4, 4), 32: (8, 4)}[warps]


def kv_attend(q: torch.Tensor, pool, page_table, heads: int, scale: float, batch, window: Optional[int] = None, chunk: Optional[int] = None,
              gate: Optional[torch.Tensor] = None) -> torch.Tensor:
    """q [T, heads * D]; the row at position p sees the cached positions from ``first_visible(p)`` to p of its sequence, query head h
    key head h // (heads / kv_heads). ``gate`` [T, heads * D] (bf16 or fp32): the result is multiplied by its sigmoid."""
    T, G, D = q.shape[0], pool.shape[1], pool.shape[4]
    if not q.is_cuda:
        out = torch.empty(T, heads * D, dtype=q.dtype)
        rows, pos = batch.rows.long()[batch.tok_seq.long()].tolist(), batch.tok_pos.tolist()
        for t in range(T):
            j = torch.arange(first_visible(pos[t], window, chunk), pos[t] + 1)
            kv = pool[page_table[rows[t], j // PAGE].long(), :, :, j % PAGE].float()                  # [keys, G, 2, D]
            s = torch.einsum("ghd,jgd->ghj", q[t].float().view(G, heads // G, D), kv[:, :, 0]) * scale
            out[t] = torch.einsum("ghj,jgd->ghd", torch.softmax(s, -1), kv[:, :, 1]).reshape(-1).to(q.dtype)
        return out if gate is None else (out.float() * torch.sigmoid(gate.float())).to(q.dtype)
    out = torch.empty(T, heads * D, dtype=q.dtype, device=q.device)
    span = min(chunk or window or page_table.shape[1] * PAGE, page_table.shape[1] * PAGE)
    splits, warps = cluster_shape(T, G * -(-(heads // G) // 8), span)
    rt.check(rt.lib().inv_kv_attend(q.data_ptr(), pool.data_ptr(), int(pool.dtype == torch.float32), page_table.data_ptr(), page_table.shape[1],
                                    batch.rows.data_ptr(), batch.tok_seq.data_ptr(), batch.tok_pos.data_ptr(), int(window or 0), int(chunk or 0),
                                    float(scale), rt.ptr(gate), 0 if gate is None else gate.stride(0),
                                    int(gate is not None and gate.dtype == torch.float32), out.data_ptr(), T, heads, G, D, splits, warps,
                                    rt.stream_ptr()), "inv_kv_attend")
    return out
