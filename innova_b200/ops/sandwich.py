"""An fp32 residual with an RMS norm on both sides of every sublayer (``csrc/sandwich.cu``), and the soft limit of logits.

``sandwich_step`` is everything between two sublayers in one launch: x <- x + RMSNorm(y) of the finished sublayer's output, then the
next sublayer's input RMSNorm(x) in the projections' type. Norms multiply by (offset + weight): offset 1 for weights stored around
zero. Without a post norm the output enters as it is. A step starts with ``ids`` (the scaled embedding rows become x)."""
from __future__ import annotations

from typing import Optional

import torch

from .. import _native
from . import runtime as rt
from .hyper import row_buffer

_vp, _i, _f = _native.vp, _native.i32, _native.f32
_native.register_cuda_sigs({
    "inv_sandwich_step": [_vp, _vp, _vp, _i, _f, _vp, _i, _i, _vp, _vp, _f, _f, _vp, _i, _i, _vp, _i, _i, _i, _vp],
    "inv_softcap": [_vp, _i, _i, _i, _f, _vp],
})


def sandwich_step(x: torch.Tensor, dtype, eps: float, offset: float, y: Optional[torch.Tensor] = None, post_w: Optional[torch.Tensor] = None,
                  norm_w: Optional[torch.Tensor] = None, ids: Optional[torch.Tensor] = None, table: Optional[torch.Tensor] = None, scale: float = 1.0,
                  rows: Optional[torch.Tensor] = None):
    """x [T, E] fp32, updated in place; y [T, >= E]. Returns the normed row [T (or len(rows)), E] in ``dtype`` if ``norm_w``. ``rows``
    (int32) restricts the result to those tokens and leaves x as it is."""
    T, E = x.shape
    if not x.is_cuda:
        return _sandwich_cpu(x, dtype, eps, offset, y, post_w, norm_w, ids, table, scale, rows)
    n = T if rows is None else rows.numel()
    h = row_buffer(n, E, dtype, x.device) if norm_w is not None else None
    rc = rt.lib().inv_sandwich_step(x.data_ptr(), rt.ptr(ids), rt.ptr(table) if ids is not None else 0, table.stride(0) if ids is not None else 0,
                                    float(scale), rt.ptr(y), 0 if y is None else y.stride(0),
                                    int(dtype == torch.float32 if y is None else y.dtype == torch.float32), rt.ptr(post_w), rt.ptr(norm_w),
                                    float(offset), float(eps), rt.ptr(h), 0 if h is None else h.stride(0), int(dtype == torch.float32),
                                    rt.ptr(rows), n, int(rows is None), E, rt.stream_ptr())
    rt.check(rc, "inv_sandwich_step")
    return h


def _sandwich_cpu(x, dtype, eps, offset, y, post_w, norm_w, ids, table, scale, rows):
    E = x.shape[1]

    def norm(v, w):
        return v / torch.sqrt(v.square().mean(-1, keepdim=True) + eps) * (offset + w)
    at = slice(None) if rows is None else rows.long()
    cur = (table[ids.long(), :E].float() * scale if ids is not None else x)[at]
    if y is not None:
        v = y[:, :E].float()[at]
        cur = cur + (norm(v, post_w) if post_w is not None else v)
    if rows is None:
        x.copy_(cur)
    return norm(cur, norm_w).to(dtype) if norm_w is not None else None


def softcap_(x: torch.Tensor, cap: float) -> torch.Tensor:
    """x <- cap * tanh(x / cap) in place; x [rows, columns] fp32."""
    if not x.is_cuda:
        return x.copy_(cap * torch.tanh(x / cap))
    rt.check(rt.lib().inv_softcap(x.data_ptr(), x.stride(0), x.shape[0], x.shape[1], float(cap), rt.stream_ptr()), "inv_softcap")
    return x
