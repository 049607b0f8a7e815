"""Attention over a paged cache of per-token latents (``csrc/latent_attn.cu``), with an optional sliding window.

``latent_append`` normalises the latent columns of a fused projection and stores them; ``latent_attend`` attends with queries
already carried into the latent space; ``head_proj`` does the per-head products around it; ``packed_flash`` is the tcgen05 flash
kernel over packed prompts whose keys and values have been expanded from the latents."""
from __future__ import annotations

from typing import Optional

import torch

from .. import _native
from . import runtime as rt

_vp, _i, _f = _native.vp, _native.i32, _native.f32
_native.register_cuda_sigs({
    "inv_latent_prep": [_vp, _i, _i, _i, _i, _i, _vp, _f, _vp, _i, _vp, _i, _vp, _vp, _vp, _vp, _i, _i, _vp, _i, _i, _vp],
    "inv_head_proj": [_vp, _i, _i, _vp, _i, _i, _i, _vp, _i, _i, _i, _vp],
    "inv_latent_attend": [_vp, _vp, _i, _i, _vp, _i, _vp, _vp, _vp, _i, _f, _vp, _vp, _i, _i, _i, _vp],
    "inv_flash_attn_packed": [_vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _i, _i, _i, _i, _f, _i, _i, _vp, _i, _vp, _vp],
})

PAGE = 16


def latent_append(proj, off_c: int, rank: int, norm_w, eps: float, pool, page_table, batch, want_c: bool = False, nq: int = 0):
    """proj [T, >= off_c + Rp]; pool [pages, 16, Rp]. Returns (c [T, Rp] or None, queries [T, nq] in the pool's type or None)."""
    T, Rp = proj.shape[0], pool.shape[2]
    if not proj.is_cuda:
        x = proj[:, off_c:off_c + rank].float()
        c = torch.zeros(T, Rp)
        c[:, :rank] = x * torch.rsqrt(x.square().mean(-1, keepdim=True) + eps) * norm_w
        c = c.to(pool.dtype)
        pos = batch.tok_pos.long()
        page = page_table[batch.rows.long()[batch.tok_seq.long()], pos // PAGE].long()
        pool[page, pos % PAGE] = c
        return (c if want_c else None), (proj[:, :nq].to(pool.dtype) if nq else None)
    c = torch.empty(T, Rp, dtype=pool.dtype, device=proj.device) if want_c else None
    q = torch.empty(T, nq, dtype=pool.dtype, device=proj.device) if nq else None
    rt.check(rt.lib().inv_latent_prep(proj.data_ptr(), proj.stride(0), int(proj.dtype == torch.float32), off_c, rank, Rp, norm_w.data_ptr(), float(eps),
                                      pool.data_ptr(), int(pool.dtype == torch.float32), page_table.data_ptr(), page_table.shape[1],
                                      batch.rows.data_ptr(), batch.tok_seq.data_ptr(), batch.tok_pos.data_ptr(), rt.ptr(c), Rp, nq, rt.ptr(q), nq, T,
                                      rt.stream_ptr()), "inv_latent_prep")
    return c, q


def head_proj(a: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """a [T, H * K] (rows may be strided), w [H, N, K] -> [T, H * N]: one product per head."""
    H, N, K = w.shape
    T = a.shape[0]
    if a.is_cuda and w.dtype == torch.bfloat16:
        out = torch.empty(T, H * N, dtype=torch.bfloat16, device=a.device)
        rt.check(rt.lib().inv_head_proj(a.data_ptr(), a.stride(0), K, w.data_ptr(), H, N, K, out.data_ptr(), H * N, N, T, rt.stream_ptr()),
                 "inv_head_proj")
        return out
    return torch.einsum("thk,hnk->thn", a[:, :H * K].reshape(T, H, K), w).reshape(T, H * N)


def key_splits(n_rows: int, heads: int, span: int) -> int:
    """How many CTAs share one row's keys: enough to fill the GPU about twice, at least 128 keys each."""
    return max(1, min(32, span // 128, (2 * 148) // max(1, n_rows * ((heads + 15) // 16))))


def latent_attend(q: torch.Tensor, pool, page_table, heads: int, scale: float, window: Optional[int], batch, span: int) -> torch.Tensor:
    """q [T, H * Rp] latent-space queries; row t sees cached positions (tok_pos[t] - window, tok_pos[t]]. ``span``: an upper bound
    of the keys a row sees (chooses the split). Returns the weighted latent sums [T, H * Rp]."""
    T, Rp = q.shape[0], pool.shape[2]
    if not q.is_cuda:
        out = torch.empty_like(q)
        rows, pos = batch.rows.long()[batch.tok_seq.long()].tolist(), batch.tok_pos.tolist()
        for t in range(T):
            lo = max(0, pos[t] - window + 1) if window else 0
            j = torch.arange(lo, pos[t] + 1)
            c = pool[page_table[rows[t], j // PAGE].long(), j % PAGE].float()
            p = torch.softmax(q[t].float().view(heads, Rp) @ c.t() * scale, -1)
            out[t] = (p @ c).reshape(-1).to(q.dtype)
        return out
    out = torch.empty_like(q)
    f32 = pool.dtype == torch.float32
    splits = 1 if f32 else key_splits(T, heads, span)
    part = torch.empty(T * heads * splits * (Rp + 2), dtype=torch.float32, device=q.device) if splits > 1 else None
    rt.check(rt.lib().inv_latent_attend(q.data_ptr(), pool.data_ptr(), int(f32), Rp, page_table.data_ptr(), page_table.shape[1], batch.rows.data_ptr(),
                                        batch.tok_seq.data_ptr(), batch.tok_pos.data_ptr(), int(window or 0), float(scale), out.data_ptr(),
                                        rt.ptr(part), splits, T, heads, rt.stream_ptr()), "inv_latent_attend")
    return out


def packed_flash(q, k, v, heads: int, head_dim: int, scale: float, window: Optional[int], batch, kv_heads: Optional[int] = None,
                 chunk: Optional[int] = None, gate: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Causal flash attention of packed whole prompts, windowed or chunked; q [T, heads * head_dim], k and v [T, kv_heads * head_dim]
    (default: as many as query heads) row views, head_dim 64 or 128. ``gate`` [T, heads * head_dim] bf16: the result is multiplied
    by its sigmoid."""
    T = q.shape[0]
    out = torch.empty(T, heads * head_dim, dtype=torch.bfloat16, device=q.device)
    rt.check(rt.lib().inv_flash_attn_packed(q.data_ptr(), k.data_ptr(), v.data_ptr(), out.data_ptr(), batch.cu.data_ptr(), batch.n, T, batch.max_len,
                                            heads, kv_heads or heads, head_dim, q.stride(0), k.stride(0), v.stride(0), out.stride(0), float(scale),
                                            int(window or 0), int(chunk or 0), rt.ptr(gate), 0 if gate is None else gate.stride(0),
                                            rt.status_tensor(q.device).data_ptr(), rt.stream_ptr()), "inv_flash_attn_packed")
    return out
