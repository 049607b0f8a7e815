"""Hyper-connections: a residual of S parallel fp32 streams (``csrc/hyper.cu``).

``hyper_step`` is everything between two sublayers in one launch: the streams take the finished sublayer's output,
x_t <- sum_s mix[s, t] x_s + out[t] y, and the next sublayer's input LayerNorm(sum_s in[s] x_s) is written in the
projections' type. A step starts with ``ids`` (the embedding rows, scaled, fill every stream) instead of an output.
An ordinary residual connection is S = 1 with unit weights."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn.functional as F

from .. import _native
from . import runtime as rt

_vp, _i, _f = _native.vp, _native.i32, _native.f32
_native.register_cuda_sigs({
    "inv_hyper_step": [_vp, _vp, _vp, _i, _f, _vp, _i, _i, _vp, _vp, _vp, _vp, _vp, _f, _vp, _i, _i, _vp, _i, _i, _i, _i, _vp],
    "inv_gated_silu_f32": [_vp, _i, _i, _vp, _i, _i, _i, _i, _vp],
})


@dataclass
class HyperOut:
    """How a finished sublayer's output enters the streams."""
    y: torch.Tensor                          # [T, >= E] fp32 or bf16
    mix: torch.Tensor                        # [S, S] fp32, index [from, to]
    out: torch.Tensor                        # [S] fp32


@dataclass
class HyperIn:
    """What the next sublayer reads."""
    weight: torch.Tensor                     # [S] fp32
    norm_w: torch.Tensor                     # [E] fp32
    norm_b: torch.Tensor                     # [E] fp32
    eps: float


def row_buffer(T: int, n: int, dtype, device) -> torch.Tensor:
    """[T, n] view of rows padded to 16 bytes, as the tensor-map copies of the GEMMs need them."""
    return torch.empty(T, (n + 7) // 8 * 8, dtype=dtype, device=device)[:, :n]


def hyper_step(x: torch.Tensor, dtype, prev: Optional[HyperOut] = None, nxt: Optional[HyperIn] = None, ids: Optional[torch.Tensor] = None,
               table: Optional[torch.Tensor] = None, scale: float = 1.0, rows: Optional[torch.Tensor] = None, keep: bool = True):
    """x [T, S, E] fp32, updated in place when ``keep``; returns the normed input [T (or len(rows)), E] in ``dtype`` if ``nxt``.
    ``rows`` (int32) restricts the result to those tokens (the streams are then left as they are)."""
    T, S, E = x.shape
    keep = keep and rows is None
    if not x.is_cuda:
        return _hyper_step_cpu(x, dtype, prev, nxt, ids, table, scale, rows, keep)
    n = T if rows is None else rows.numel()
    h = row_buffer(n, E, dtype, x.device) if nxt is not None else None
    y = prev.y if prev is not None else None
    table_ld = table.stride(0) if ids is not None else 0
    rc = rt.lib().inv_hyper_step(
        x.data_ptr(), rt.ptr(ids), rt.ptr(table) if ids is not None else 0, table_ld, float(scale), rt.ptr(y), 0 if y is None else y.stride(0),
        int(dtype == torch.float32 if y is None else y.dtype == torch.float32),
        rt.ptr(prev.mix) if prev else 0, rt.ptr(prev.out) if prev else 0, rt.ptr(nxt.weight) if nxt else 0, rt.ptr(nxt.norm_w) if nxt else 0,
        rt.ptr(nxt.norm_b) if nxt else 0, float(nxt.eps) if nxt else 0.0, rt.ptr(h), 0 if h is None else h.stride(0), int(dtype == torch.float32),
        rt.ptr(rows), n, int(keep), S, E, rt.stream_ptr())
    rt.check(rc, "inv_hyper_step")
    return h


def _hyper_step_cpu(x, dtype, prev, nxt, ids, table, scale, rows, keep):
    cur, E = x, x.shape[2]
    if ids is not None:
        cur = (table[ids.long(), :E].float() * scale).unsqueeze(1).expand(x.shape).clone()
    if rows is not None:
        cur = cur[rows.long()]
    if prev is not None:
        y = prev.y[:, :E].float() if rows is None else prev.y[rows.long(), :E].float()
        cur = torch.einsum("nse,st->nte", cur, prev.mix) + prev.out.view(1, -1, 1) * y.unsqueeze(1)
    if keep:
        x.copy_(cur)
    if nxt is None:
        return None
    u = torch.einsum("nse,s->ne", cur, nxt.weight)
    return F.layer_norm(u, (u.shape[-1],), nxt.norm_w, nxt.norm_b, nxt.eps).to(dtype)


def gated_silu(gate_up: torch.Tensor, n: int, dtype) -> torch.Tensor:
    """silu(gate) * up from rows that hold n gate columns (padded to the row's half), then n up columns. bf16 rows take the
    training activation kernel; fp32 rows (32-bit models) the one in ``csrc/hyper.cu``."""
    T, half = gate_up.shape[0], gate_up.shape[1] // 2
    if not gate_up.is_cuda:
        return (F.silu(gate_up[:, :n].float()) * gate_up[:, half:half + n].float()).to(dtype)
    if gate_up.dtype == torch.bfloat16:
        out = torch.empty(T, half, dtype=torch.bfloat16, device=gate_up.device)
        rt.check(rt.lib().inv_act(gate_up.data_ptr(), 0, out.data_ptr(), T, half, 2, rt.stream_ptr()), "inv_act")
        return out[:, :n]
    out = row_buffer(T, n, dtype, gate_up.device)
    rt.check(rt.lib().inv_gated_silu_f32(gate_up.data_ptr(), gate_up.stride(0), half, out.data_ptr(), out.stride(0), int(dtype == torch.float32), T,
                                         n, rt.stream_ptr()), "inv_gated_silu_f32")
    return out
