"""Gated delta rule with a decay per head and key channel, its short convolutions and its gated output norm
(``csrc/delta_rule.cu``); everything between the projections and the output projection of such a mixer.

    S <- diag(g) S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q

``DeltaShape`` describes one mixer. A projection row holds [q | k | v | a | g | b], each part starting at a multiple of 8
columns: queries and keys of ``Hk`` heads, values of ``H`` heads, the two low-rank factors and one step size per head. The
state of a sequence is S ([H, D, Dv] fp32) and a ring of ``taps`` projection rows indexed by position modulo ``taps``."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Tuple

import torch
import torch.nn.functional as F

from .. import _native
from . import runtime as rt

_vp, _i, _f = _native.vp, _native.i32, _native.f32
_native.register_cuda_sigs({
    "inv_delta_chunk": [_vp, _i, _i] + [_vp] * 10 + [_i, _vp, _vp, _i, _vp, _vp],
    "inv_conv_tail": [_vp, _i, _i, _vp, _vp, _vp, _vp, _i, _vp, _vp],
    "inv_delta_scan": [_vp] * 8 + [_i, _vp, _vp, _vp],
    "inv_gated_head_norm": [_vp, _vp, _vp, _i, _i, _vp, _i, _i, _i, _i, _i, _f, _vp],
    "inv_delta_decode": [_vp, _i, _i] + [_vp] * 8 + [_i, _vp, _i, _i, _vp, _f, _vp, _i, _i, _vp, _vp, _vp],
})

DECODE_MAX_TILE = 192 * 1024      # largest [D, Dv] fp32 state tile the one-launch decode kernel keeps in shared memory

CHUNK = 16                         # tokens the prompt path advances per step of the recurrence


def _pad8(n: int) -> int:
    return (n + 7) // 8 * 8


@dataclass(frozen=True)
class DeltaShape:
    H: int          # value heads
    Hk: int         # query / key heads; value head h uses h // (H // Hk)
    D: int          # query / key size
    Dv: int         # value size
    taps: int       # convolution taps, the current token's included
    rank_a: int     # inner size of the decay's low-rank product
    rank_g: int     # inner size of the output gate's

    def __post_init__(self):
        if self.H % self.Hk or self.D > 256 or self.Dv > 256:
            raise ValueError(f"delta rule: {self} needs heads divisible by key heads and head sizes up to 256")

    @property
    def offsets(self) -> Tuple[int, ...]:
        """Start of q, k, v, a, g, b in a projection row, and the row's width."""
        out = [0]
        for n in (self.Hk * self.D, self.Hk * self.D, self.H * self.Dv, self.rank_a, self.rank_g, self.H):
            out.append(out[-1] + _pad8(n))
        return tuple(out)

    @property
    def channels(self) -> int:
        return self.offsets[3]

    @property
    def tile_bytes(self) -> int:
        return self.D * self.Dv * 4

    @property
    def block_floats(self) -> int:
        """Size of one (chunk, head) block between the chunk kernel and the scan (csrc/delta_rule.cu)."""
        d4 = (self.D + 3) // 4 * 4
        return 32 * d4 + CHUNK * d4 + CHUNK * 32 + d4

    def c_array(self):
        o = self.offsets
        return (C.c_int * 14)(self.H, self.Hk, self.D, self.Dv, self.taps, o[0], o[1], o[2], o[3], o[4], o[5], o[3], self.rank_a, self.rank_g)


def delta_prompt(s: DeltaShape, proj, z, gate, taps_w, A_log, dt_bias, norm_w, eps, ring, state, batch) -> torch.Tensor:
    """Packed tokens of several sequences -> normed, gated outputs [T, H * Dv] (type of ``gate``). ``z`` [T, >= H * D] fp32 is the
    low-rank product of the decay, ``gate`` [T, >= H * Dv] that of the output gate. Advances ``ring`` and ``state``."""
    T = proj.shape[0]
    if not proj.is_cuda:
        return _delta_prompt_cpu(s, proj, z, gate, taps_w, A_log, dt_bias, norm_w, eps, ring, state, batch)
    dev, lib, st, arr = proj.device, rt.lib(), rt.stream_ptr(), s.c_array()
    pf = int(proj.dtype == torch.float32)
    blocks = torch.empty(batch.n_chunks * s.H * s.block_floats, dtype=torch.float32, device=dev)
    vblocks = torch.empty(batch.n_chunks * s.H * ((s.Dv + 15) // 16) * 256, dtype=torch.float32, device=dev)
    rt.check(lib.inv_delta_chunk(proj.data_ptr(), proj.stride(0), pf, taps_w.data_ptr(), ring.data_ptr(), batch.chunk_seq.data_ptr(),
                                 batch.cu_chunk.data_ptr(), batch.cu.data_ptr(), batch.start.data_ptr(), batch.slots.data_ptr(), A_log.data_ptr(),
                                 dt_bias.data_ptr(), z.data_ptr(), z.stride(0), blocks.data_ptr(), vblocks.data_ptr(), batch.n_chunks, arr, st),
             "inv_delta_chunk")
    rt.check(lib.inv_conv_tail(proj.data_ptr(), proj.stride(0), pf, ring.data_ptr(), batch.cu.data_ptr(), batch.start.data_ptr(),
                               batch.slots.data_ptr(), batch.n, arr, st), "inv_conv_tail")
    o = torch.empty(T, s.H * s.Dv, dtype=torch.float32, device=dev)
    rt.check(lib.inv_delta_scan(blocks.data_ptr(), vblocks.data_ptr(), o.data_ptr(), state.data_ptr(), batch.cu_chunk.data_ptr(), batch.cu.data_ptr(),
                                batch.start.data_ptr(), batch.slots.data_ptr(), batch.n, rt.status_tensor(dev).data_ptr(), arr, st), "inv_delta_scan")
    from .hyper import row_buffer
    out = row_buffer(T, s.H * s.Dv, gate.dtype, dev)
    f32 = int(gate.dtype == torch.float32)
    rt.check(lib.inv_gated_head_norm(o.data_ptr(), norm_w.data_ptr(), gate.data_ptr(), gate.stride(0), f32, out.data_ptr(), out.stride(0), f32, T, s.H,
                                     s.Dv, float(eps), st), "inv_gated_head_norm")
    return out


def delta_decode(s: DeltaShape, proj, a2t, g2t, taps_w, A_log, dt_bias, norm_w, eps, ring, state, batch) -> torch.Tensor:
    """One token per sequence in one launch: ``proj`` [B, width] (type of the weights, or fp32) -> [B, H * Dv] in the
    type of ``a2t`` [rank_a, H * D] / ``g2t`` [rank_g, H * Dv], the transposed second factors of the low-rank products."""
    B = proj.shape[0]
    if not proj.is_cuda:
        z = proj[:, s.offsets[3]:s.offsets[3] + s.rank_a].to(a2t.dtype) @ a2t
        gate = proj[:, s.offsets[4]:s.offsets[4] + s.rank_g].to(g2t.dtype) @ g2t
        return _delta_prompt_cpu(s, proj, z.float(), gate, taps_w, A_log, dt_bias, norm_w, eps, ring, state, batch)
    from .hyper import row_buffer
    out = row_buffer(B, s.H * s.Dv, a2t.dtype, proj.device)
    rt.check(rt.lib().inv_delta_decode(proj.data_ptr(), proj.stride(0), int(proj.dtype == torch.float32), taps_w.data_ptr(), ring.data_ptr(),
                                       state.data_ptr(), batch.start.data_ptr(), batch.slots.data_ptr(), A_log.data_ptr(), dt_bias.data_ptr(),
                                       a2t.data_ptr(), a2t.stride(0), g2t.data_ptr(), g2t.stride(0), int(a2t.dtype == torch.float32),
                                       norm_w.data_ptr(), float(eps), out.data_ptr(), out.stride(0), B, rt.status_tensor(proj.device).data_ptr(),
                                       s.c_array(), rt.stream_ptr()), "inv_delta_decode")
    return out


def _delta_prompt_cpu(s, proj, z, gate, taps_w, A_log, dt_bias, norm_w, eps, ring, state, batch):
    o_q, o_k, o_v, o_a, o_g, o_b, _ = s.offsets
    outs = []
    cu = batch.cu.tolist()
    for i, (slot, st) in enumerate(zip(batch.slots.tolist(), batch.start.tolist())):
        rows = slice(cu[i], cu[i + 1])
        x, n = proj[rows].float(), cu[i + 1] - cu[i]
        C_ = s.channels
        past = torch.zeros(s.taps - 1, C_)
        for j in range(1, s.taps):
            if st - j >= 0:
                past[s.taps - 1 - j] = ring[slot, (st - j) % s.taps]
        seq = torch.cat([past, x[:, :C_]])
        for p in range(max(0, n - (s.taps - 1)), n):
            ring[slot, (st + p) % s.taps] = x[p, :C_]
        c = F.silu(sum(seq[t:t + n] * taps_w[t] for t in range(s.taps)))
        q = c[:, o_q:o_q + s.Hk * s.D].view(n, s.Hk, s.D)
        k = c[:, o_k:o_k + s.Hk * s.D].view(n, s.Hk, s.D)
        v = c[:, o_v:o_v + s.H * s.Dv].view(n, s.H, s.Dv)
        q = (q * torch.rsqrt(q.square().sum(-1, keepdim=True) + 1e-6) * s.D ** -0.5).repeat_interleave(s.H // s.Hk, 1)
        k = (k * torch.rsqrt(k.square().sum(-1, keepdim=True) + 1e-6)).repeat_interleave(s.H // s.Hk, 1)
        beta = torch.sigmoid(x[:, o_b:o_b + s.H])
        g = torch.exp(-torch.exp(A_log).view(1, s.H, 1) * F.softplus(z[rows, :s.H * s.D] + dt_bias).view(n, s.H, s.D))
        S = state[slot] if st > 0 else torch.zeros_like(state[slot])
        o = []
        for t in range(n):
            S = S * g[t].unsqueeze(-1)
            u = beta[t].unsqueeze(-1) * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
            S = S + k[t].unsqueeze(-1) * u.unsqueeze(1)
            o.append(torch.einsum("hdv,hd->hv", S, q[t]))
        state[slot] = S
        o = torch.stack(o)
        o = o * torch.rsqrt(o.square().mean(-1, keepdim=True) + eps) * norm_w
        outs.append((o.reshape(n, -1) * torch.sigmoid(gate[rows, :s.H * s.Dv].float())).to(gate.dtype))
    return torch.cat(outs)
