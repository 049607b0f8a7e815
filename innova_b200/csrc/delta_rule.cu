// Gated delta rule with one decay per head and key channel, fp32 throughout:
//   S <- diag(g) S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q          (S: [D, Dv] per head and sequence)
// with short causal convolutions in front of q, k, v and a gated per-head RMS norm behind o.
//
// Prompt path, over packed tokens of several sequences:
//   delta_prep        one warp per (token, head part): convolution + SiLU, unit norms, decays exp(-exp(A) softplus(z + dt)), beta
//   conv_tail         keeps the last taps - 1 projection rows of every sequence (a ring of `taps` rows indexed by position)
//   delta_scan        the recurrence. The rows of a sequence follow one another, so the work of a step is latency: a CTA owns
//                     a few value columns of one head, LP lanes share a column and keep their D / LP state entries in
//                     registers, tokens are staged through shared memory 16 at a time with cp.async (double buffered), and
//                     the arithmetic uses the packed fp32 pair instructions (two products per issue slot).
//   gated_head_norm   o / rms(o) * w * sigmoid(gate), cast to the projections' type
// Decode path: delta_decode does all of it for one token per sequence in one launch, one CTA per (sequence, head): the state
// tile is read once into shared memory and written once, which bounds the kernel at 8 D Dv bytes per head.
#include "sm100_common.cuh"
#include "inv_api.h"

namespace inv {

typedef unsigned long long u64;

__device__ __forceinline__ float dr_ld(const float* p) { return *p; }
__device__ __forceinline__ float dr_ld(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void dr_st(float* p, float v) { *p = v; }
__device__ __forceinline__ void dr_st(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ float dr_warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float dr_silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float dr_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float dr_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

__device__ __forceinline__ u64 f2_pack(float lo, float hi) {
  u64 d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ float f2_sum(u64 v) {
  float lo, hi;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v));
  return lo + hi;
}
__device__ __forceinline__ u64 f2_mul(u64 a, u64 b) {
  u64 d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ u64 f2_fma(u64 a, u64 b, u64 c) {
  u64 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ u64 f2_add(u64 a, u64 b) {
  u64 d;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}

// Shapes and column offsets of one mixer. Projection rows hold [q | k | v | low-rank decay | low-rank gate | beta].
struct DeltaShape {
  int H, Hk, D, Dv, taps;
  int off_q, off_k, off_v, off_a, off_g, off_b;  // columns of a projection row
  int channels;                                  // off_v + H * Dv: the convolved columns, [0, channels)
  int rank_a, rank_g;
};

// Value of convolved channel c (a column of the projection) at the token with packed row t and absolute position pos.
template <typename T>
__device__ __forceinline__ float conv_at(const T* proj, int ld, const float* taps_w, const float* ring, const DeltaShape& s, int t, int pos,
                                         int start, int c) {
  float a = 0.f;
  for (int j = 0; j < s.taps; ++j) {
    const int i = pos - j;
    if (i < 0) break;
    const float x = i >= start ? dr_ld(proj + (size_t)(t - j) * ld + c) : ring[(size_t)(i % s.taps) * s.channels + c];
    a = fmaf(x, taps_w[(size_t)(s.taps - 1 - j) * s.channels + c], a);
  }
  return a;
}

// ------------------------------------------------------------------------------------------------ prompt: prep
// Warp roles per token: [0, Hk) q heads, [Hk, 2 Hk) k heads, then H value heads (which also do the decay and beta of the head).
template <typename T>
__global__ void __launch_bounds__(128) delta_prep_kernel(const T* __restrict__ proj, int ld, const float* __restrict__ taps_w,
                                                         const float* __restrict__ ring0, const int* __restrict__ tok_seq,
                                                         const int* __restrict__ tok_pos, const int* __restrict__ start,
                                                         const int* __restrict__ slots, const float* __restrict__ A_log,
                                                         const float* __restrict__ dt_bias, float* __restrict__ qn, float* __restrict__ kn,
                                                         float* __restrict__ vv, float* __restrict__ g, int g_ld, float* __restrict__ beta,
                                                         const DeltaShape s) {
  const int lane = threadIdx.x & 31, unit = blockIdx.y * 4 + (threadIdx.x >> 5), t = blockIdx.x;
  if (unit >= 2 * s.Hk + s.H) return;
  const int seq = tok_seq[t], pos = tok_pos[t], st = start[seq];
  const float* ring = ring0 + (size_t)slots[seq] * s.taps * s.channels;
  if (unit < 2 * s.Hk) {
    const bool is_q = unit < s.Hk;
    const int h = is_q ? unit : unit - s.Hk;
    const int c0 = (is_q ? s.off_q : s.off_k) + h * s.D;
    float* dst = (is_q ? qn : kn) + ((size_t)t * s.Hk + h) * s.D;
    float v[8], ss = 0.f;
#pragma unroll
    for (int m = 0; m < 8; ++m) {
      const int d = lane + m * 32;
      v[m] = d < s.D ? dr_silu(conv_at(proj, ld, taps_w, ring, s, t, pos, st, c0 + d)) : 0.f;
      ss = fmaf(v[m], v[m], ss);
    }
    float r = 1.0f / sqrtf(dr_warp_sum(ss) + 1e-6f);
    if (is_q) r *= 1.0f / sqrtf((float)s.D);
#pragma unroll
    for (int m = 0; m < 8; ++m) {
      const int d = lane + m * 32;
      if (d < s.D) dst[d] = v[m] * r;
    }
    return;
  }
  const int h = unit - 2 * s.Hk;
  for (int d = lane; d < s.Dv; d += 32)
    vv[((size_t)t * s.H + h) * s.Dv + d] = dr_silu(conv_at(proj, ld, taps_w, ring, s, t, pos, st, s.off_v + h * s.Dv + d));
  const float ea = expf(A_log[h]);
  for (int d = lane; d < s.D; d += 32) {
    const size_t i = (size_t)t * g_ld + h * s.D + d;
    g[i] = expf(-ea * dr_softplus(g[i] + dt_bias[h * s.D + d]));  // in place: the low-rank projection becomes the decay
  }
  if (lane == 0) beta[(size_t)t * s.H + h] = dr_sigmoid(dr_ld(proj + (size_t)t * ld + s.off_b + h));
}

template <typename T>
__global__ void __launch_bounds__(256) conv_tail_kernel(const T* __restrict__ proj, int ld, float* __restrict__ ring0, const int* __restrict__ cu,
                                                        const int* __restrict__ start, const int* __restrict__ slots, const DeltaShape s) {
  const int seq = blockIdx.x, c = blockIdx.y * 256 + threadIdx.x;
  if (c >= s.channels) return;
  float* ring = ring0 + (size_t)slots[seq] * s.taps * s.channels;
  const int n = cu[seq + 1] - cu[seq], st = start[seq];
  for (int i = max(0, n - (s.taps - 1)); i < n; ++i)
    ring[(size_t)((st + i) % s.taps) * s.channels + c] = dr_ld(proj + (size_t)(cu[seq] + i) * ld + c);
}

// ------------------------------------------------------------------------------------------------ prompt: scan
constexpr int SCAN_CT = 16;  // tokens per staged chunk

template <int DP, int LP, int THREADS>
struct ScanSmem {
  static constexpr int COLS = THREADS / LP;
  static constexpr int ROW = 3 * DP;                                     // q | k | g of one token
  static constexpr int BUF = SCAN_CT * (ROW + COLS + 4);                 // + values and (padded) beta
  static constexpr int BYTES = (2 * BUF + SCAN_CT * COLS) * 4;           // two buffers and the outputs of a chunk
};

// 16-byte (vec) or 4-byte asynchronous copy into shared memory.
__device__ __forceinline__ void cp16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp4(float* dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}

template <int DP, int LP, int THREADS>
__global__ void __launch_bounds__(THREADS) delta_scan_kernel(const float* __restrict__ qn, const float* __restrict__ kn,
                                                             const float* __restrict__ vv, const float* __restrict__ g, int g_ld,
                                                             const float* __restrict__ beta, float* __restrict__ o, float* __restrict__ state0,
                                                             const int* __restrict__ cu, const int* __restrict__ start,
                                                             const int* __restrict__ slots, int H, int Hk, int D, int Dv) {
  using L = ScanSmem<DP, LP, THREADS>;
  constexpr int COLS = L::COLS, NP = DP / LP / 2;  // packed pairs of state per lane
  extern __shared__ __align__(16) float sm[];
  float* o_s = sm + 2 * L::BUF;
  const int tid = threadIdx.x, part = tid % LP, cl = tid / LP;
  const int h = blockIdx.y, seq = blockIdx.z, hk = h / (H / Hk);
  const int col0 = blockIdx.x * COLS, col = col0 + cl;
  const bool live = col < Dv;
  const int t0 = cu[seq], n = cu[seq + 1] - t0;
  float* state = state0 + ((size_t)slots[seq] * H + h) * (size_t)D * Dv;
  // entry of pair j of this lane: d = 4 (part + LP (j / 2)) + 2 (j % 2) + {0, 1}
  u64 S[NP];
#pragma unroll
  for (int j = 0; j < NP; ++j) {
    const int d = 4 * (part + LP * (j / 2)) + 2 * (j % 2);
    float a = 0.f, b = 0.f;
    if (live && start[seq] > 0) {
      if (d < D) a = state[(size_t)d * Dv + col];
      if (d + 1 < D) b = state[(size_t)(d + 1) * Dv + col];
    }
    S[j] = f2_pack(a, b);
  }
  for (int i = tid; i < 2 * L::BUF; i += THREADS) sm[i] = 0.f;  // channels beyond D and columns beyond Dv stay zero
  __syncthreads();
  const bool vec = D % 4 == 0;
  auto stage = [&](int c, int buf) {
    float* b = sm + buf * L::BUF;
    const int m = min(SCAN_CT, n - c * SCAN_CT);
    const size_t tb = (size_t)t0 + (size_t)c * SCAN_CT;
    if (vec) {
      const int per = D / 4, tot = m * per;
      for (int i = tid; i < tot; i += THREADS) {
        const int r = i / per, d = (i % per) * 4;
        const size_t t = tb + r;
        cp16(b + r * L::ROW + d, qn + (t * Hk + hk) * D + d);
        cp16(b + r * L::ROW + DP + d, kn + (t * Hk + hk) * D + d);
        cp16(b + r * L::ROW + 2 * DP + d, g + t * g_ld + (size_t)h * D + d);
      }
    } else {
      for (int i = tid; i < m * D; i += THREADS) {
        const int r = i / D, d = i % D;
        const size_t t = tb + r;
        cp4(b + r * L::ROW + d, qn + (t * Hk + hk) * D + d);
        cp4(b + r * L::ROW + DP + d, kn + (t * Hk + hk) * D + d);
        cp4(b + r * L::ROW + 2 * DP + d, g + t * g_ld + (size_t)h * D + d);
      }
    }
    float* vb = b + SCAN_CT * L::ROW;
    for (int i = tid; i < m * COLS; i += THREADS) {
      const int r = i / COLS, c2 = i % COLS;
      if (col0 + c2 < Dv) cp4(vb + r * COLS + c2, vv + ((tb + r) * H + h) * Dv + col0 + c2);
    }
    if (tid < m) cp4(vb + SCAN_CT * COLS + tid, beta + (tb + tid) * H + h);
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  const int nc = (n + SCAN_CT - 1) / SCAN_CT;
  if (nc > 0) stage(0, 0);
  for (int c = 0; c < nc; ++c) {
    if (c + 1 < nc) {
      stage(c + 1, (c + 1) & 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const float* b = sm + (c & 1) * L::BUF;
    const float* vb = b + SCAN_CT * L::ROW;
    const int m = min(SCAN_CT, n - c * SCAN_CT);
    for (int r = 0; r < m; ++r) {
      const ulonglong2* q2 = reinterpret_cast<const ulonglong2*>(b + r * L::ROW);
      const ulonglong2* k2 = reinterpret_cast<const ulonglong2*>(b + r * L::ROW + DP);
      const ulonglong2* g2 = reinterpret_cast<const ulonglong2*>(b + r * L::ROW + 2 * DP);
      u64 kk[NP], acc[4] = {0, 0, 0, 0};
#pragma unroll
      for (int j = 0; j < NP / 2; ++j) {
        const ulonglong2 gg = g2[part + LP * j], kv = k2[part + LP * j];
        kk[2 * j] = kv.x;
        kk[2 * j + 1] = kv.y;
        S[2 * j] = f2_mul(S[2 * j], gg.x);
        S[2 * j + 1] = f2_mul(S[2 * j + 1], gg.y);
        acc[(2 * j) & 3] = f2_fma(S[2 * j], kv.x, acc[(2 * j) & 3]);
        acc[(2 * j + 1) & 3] = f2_fma(S[2 * j + 1], kv.y, acc[(2 * j + 1) & 3]);
      }
      float rk = f2_sum(f2_add(f2_add(acc[0], acc[1]), f2_add(acc[2], acc[3])));
#pragma unroll
      for (int w = 1; w < LP; w <<= 1) rk += __shfl_xor_sync(0xffffffffu, rk, w);
      const float u = vb[SCAN_CT * COLS + r] * (vb[r * COLS + cl] - rk);
      const u64 uu = f2_pack(u, u);
      acc[0] = acc[1] = acc[2] = acc[3] = 0;
#pragma unroll
      for (int j = 0; j < NP / 2; ++j) {
        const ulonglong2 qv = q2[part + LP * j];
        S[2 * j] = f2_fma(kk[2 * j], uu, S[2 * j]);
        S[2 * j + 1] = f2_fma(kk[2 * j + 1], uu, S[2 * j + 1]);
        acc[(2 * j) & 3] = f2_fma(S[2 * j], qv.x, acc[(2 * j) & 3]);
        acc[(2 * j + 1) & 3] = f2_fma(S[2 * j + 1], qv.y, acc[(2 * j + 1) & 3]);
      }
      float ov = f2_sum(f2_add(f2_add(acc[0], acc[1]), f2_add(acc[2], acc[3])));
#pragma unroll
      for (int w = 1; w < LP; w <<= 1) ov += __shfl_xor_sync(0xffffffffu, ov, w);
      if (part == 0) o_s[r * COLS + cl] = ov;
    }
    __syncthreads();  // everyone is done with this buffer, and the outputs are complete
    for (int i = tid; i < m * COLS; i += THREADS) {
      const int r = i / COLS, c2 = i % COLS;
      if (col0 + c2 < Dv) o[(((size_t)t0 + (size_t)c * SCAN_CT + r) * H + h) * Dv + col0 + c2] = o_s[i];
    }
  }
  if (live) {
#pragma unroll
    for (int j = 0; j < NP; ++j) {
      const int d = 4 * (part + LP * (j / 2)) + 2 * (j % 2);
      float a, bb;
      asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(bb) : "l"(S[j]));
      if (d < D) state[(size_t)d * Dv + col] = a;
      if (d + 1 < D) state[(size_t)(d + 1) * Dv + col] = bb;
    }
  }
}

// ------------------------------------------------------------------------------------------------ prompt: output norm
template <typename TG, typename TO>
__global__ void __launch_bounds__(128) gated_head_norm_kernel(const float* __restrict__ o, const float* __restrict__ w, const TG* __restrict__ gate,
                                                              int gate_ld, TO* __restrict__ out, int out_ld, int H, int Dv, float eps) {
  const int lane = threadIdx.x & 31, h = blockIdx.y * 4 + (threadIdx.x >> 5);
  const size_t t = blockIdx.x;
  if (h >= H) return;
  const float* r = o + (t * H + h) * Dv;
  float ss = 0.f;
  for (int d = lane; d < Dv; d += 32) ss = fmaf(r[d], r[d], ss);
  const float inv = 1.0f / sqrtf(dr_warp_sum(ss) / (float)Dv + eps);
  for (int d = lane; d < Dv; d += 32)
    dr_st(out + t * out_ld + h * Dv + d, r[d] * inv * w[d] * dr_sigmoid(dr_ld(gate + t * gate_ld + h * Dv + d)));
}

// ------------------------------------------------------------------------------------------------ decode, one launch
// One CTA per (head, sequence). The head's state tile is one contiguous range: a single bulk copy brings it into shared
// memory while the convolutions, norms and low-rank products run, it is updated in place and a bulk copy writes it back.
// Row groups of threads walk the tile (VEC value columns per thread); three tiles of 128 x 128 share an SM.
constexpr int DD_THREADS = 256;
constexpr int DD_MAX_TILE = 200 * 1024;

template <typename T, typename TW, typename TO, int VEC>
__global__ void __launch_bounds__(DD_THREADS) delta_decode_kernel(const T* __restrict__ proj, int ld, const float* __restrict__ taps_w,
                                                                  float* __restrict__ ring0, float* __restrict__ state0,
                                                                  const int* __restrict__ pos_, const int* __restrict__ slots,
                                                                  const float* __restrict__ A_log, const float* __restrict__ dt_bias,
                                                                  const TW* __restrict__ a2t, int a2_ld, const TW* __restrict__ g2t, int g2_ld,
                                                                  const float* __restrict__ norm_w, float eps, TO* __restrict__ out, int out_ld,
                                                                  int* status, const DeltaShape s) {
  extern __shared__ __align__(16) float dsm[];
  __shared__ uint64_t bar;
  __shared__ int abort_flag;
  constexpr int NW = DD_THREADS / 32;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.x, b = blockIdx.y;
  const int D = s.D, Dv = s.Dv, cpr = Dv / VEC;         // threads per state row
  const int lanes_per_row = (cpr + 31) & ~31, groups = DD_THREADS / lanes_per_row;
  float* S = dsm;                        // [D, Dv]
  float* q_s = S + ((D * Dv + 3) & ~3);  // [D]
  float* k_s = q_s + D;                  // [D]
  float* g_s = k_s + D;                  // [D]
  float* v_s = g_s + D;                  // [Dv] values, then beta (v - r)
  float* gate_s = v_s + Dv;              // [Dv]
  float* lr = gate_s + Dv;               // [rank_a + rank_g]
  float* ws = lr + s.rank_a + s.rank_g;  // [2 * NW]
  float* red = ws + 2 * NW;              // [groups * Dv]
  const int pos = pos_[b], slot = slots[b], hk = h / (s.H / s.Hk);
  const T* row = proj + (size_t)b * ld;
  float* ring = ring0 + (size_t)slot * s.taps * s.channels;
  float* state = state0 + ((size_t)slot * s.H + h) * (size_t)D * Dv;
  const uint32_t tile_bytes = (uint32_t)(D * Dv) * 4u;
  const bool bulk = tile_bytes % 16 == 0;  // then every tile starts on a 16-byte boundary too
  if (tid == 0) {
    abort_flag = 0;
    mbar_init(&bar, 1);
    fence_barrier_init();
    if (bulk && pos > 0) {
      mbar_expect_tx(&bar, tile_bytes);
      asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(smem_u32(S)), "l"(state),
                   "r"(tile_bytes), "r"(smem_u32(&bar))
                   : "memory");
    }
  }
  if (pos == 0)
    for (int i = tid; i < D * Dv; i += DD_THREADS) S[i] = 0.f;
  else if (!bulk)
    for (int i = tid; i < D * Dv; i += DD_THREADS) S[i] = state[i];
  // convolutions; the current row goes into the ring slot of this position, which nobody reads in this launch
  const int nq = 2 * D + Dv;
  const bool own_qk = h % (s.H / s.Hk) == 0;
  float ssq = 0.f, ssk = 0.f;
  for (int i = tid; i < nq; i += DD_THREADS) {
    const int c = i < D ? s.off_q + hk * D + i : i < 2 * D ? s.off_k + hk * D + (i - D) : s.off_v + h * Dv + (i - 2 * D);
    const float cur = dr_ld(row + c);
    float a = cur * taps_w[(size_t)(s.taps - 1) * s.channels + c];
    for (int j = 1; j < s.taps; ++j)
      if (pos - j >= 0) a = fmaf(ring[(size_t)((pos - j) % s.taps) * s.channels + c], taps_w[(size_t)(s.taps - 1 - j) * s.channels + c], a);
    if (i >= 2 * D || own_qk) ring[(size_t)(pos % s.taps) * s.channels + c] = cur;
    a = dr_silu(a);
    if (i < D) { q_s[i] = a; ssq = fmaf(a, a, ssq); }
    else if (i < 2 * D) { k_s[i - D] = a; ssk = fmaf(a, a, ssk); }
    else v_s[i - 2 * D] = a;
  }
  for (int i = tid; i < s.rank_a + s.rank_g; i += DD_THREADS) lr[i] = dr_ld(row + (i < s.rank_a ? s.off_a + i : s.off_g + i - s.rank_a));
  ssq = dr_warp_sum(ssq);
  ssk = dr_warp_sum(ssk);
  if (lane == 0) { ws[warp] = ssq; ws[NW + warp] = ssk; }
  __syncthreads();
  float nq2 = 0.f, nk2 = 0.f;
  for (int i = 0; i < NW; ++i) { nq2 += ws[i]; nk2 += ws[NW + i]; }
  const float rq = 1.0f / sqrtf(nq2 + 1e-6f) * (1.0f / sqrtf((float)D)), rk = 1.0f / sqrtf(nk2 + 1e-6f);
  // low-rank decay and output gate (their second matrices are stored transposed: [rank, heads * channels])
  const float ea = expf(A_log[h]);
  for (int d = tid; d < D + Dv; d += DD_THREADS) {
    float a = 0.f;
    if (d < D) {
      const TW* w = a2t + h * D + d;
#pragma unroll 8
      for (int r = 0; r < s.rank_a; ++r) a = fmaf(dr_ld(w + (size_t)r * a2_ld), lr[r], a);
      g_s[d] = expf(-ea * dr_softplus(a + dt_bias[h * D + d]));
      q_s[d] *= rq;
      k_s[d] *= rk;
    } else {
      const TW* w = g2t + h * Dv + (d - D);
#pragma unroll 8
      for (int r = 0; r < s.rank_g; ++r) a = fmaf(dr_ld(w + (size_t)r * g2_ld), lr[s.rank_a + r], a);
      gate_s[d - D] = dr_sigmoid(a);
    }
  }
  const float beta = dr_sigmoid(dr_ld(row + s.off_b + h));
  bool ok = true;
  if (bulk && pos > 0) ok = mbar_wait(&bar, 0, &abort_flag, status, ERR_WAIT_FULL);
  if (!__syncthreads_and(ok)) {  // the copy never arrived: leave it a bounded time before the shared memory goes away
    const uint64_t t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 2000000ull) __nanosleep(1000);
    return;
  }
  const int grp = tid / lanes_per_row, cv = tid % lanes_per_row;
  const bool live = grp < groups && cv < cpr;
  float acc[VEC];
#pragma unroll
  for (int j = 0; j < VEC; ++j) acc[j] = 0.f;
  if (live)
#pragma unroll 4
    for (int d = grp; d < D; d += groups) {
      const float gk = g_s[d] * k_s[d];
      const float* p = S + d * Dv + cv * VEC;
      if (VEC == 4) {
        const float4 x = *reinterpret_cast<const float4*>(p);
        acc[0] = fmaf(x.x, gk, acc[0]); acc[1 % VEC] = fmaf(x.y, gk, acc[1 % VEC]);
        acc[2 % VEC] = fmaf(x.z, gk, acc[2 % VEC]); acc[3 % VEC] = fmaf(x.w, gk, acc[3 % VEC]);
      } else {
        acc[0] = fmaf(p[0], gk, acc[0]);
      }
    }
  if (live)
#pragma unroll
    for (int j = 0; j < VEC; ++j) red[grp * Dv + cv * VEC + j] = acc[j];
  __syncthreads();
  for (int v = tid; v < Dv; v += DD_THREADS) {
    float r = 0.f;
    for (int i = 0; i < groups; ++i) r += red[i * Dv + v];
    v_s[v] = beta * (v_s[v] - r);
  }
  __syncthreads();
  float u[VEC];
#pragma unroll
  for (int j = 0; j < VEC; ++j) {
    u[j] = live ? v_s[cv * VEC + j] : 0.f;
    acc[j] = 0.f;
  }
  if (live)
#pragma unroll 4
    for (int d = grp; d < D; d += groups) {
      const float gg = g_s[d], kk = k_s[d], qq = q_s[d];
      float* p = S + d * Dv + cv * VEC;
      if (VEC == 4) {
        float4 x = *reinterpret_cast<const float4*>(p);
        x.x = fmaf(kk, u[0], x.x * gg); x.y = fmaf(kk, u[1 % VEC], x.y * gg);
        x.z = fmaf(kk, u[2 % VEC], x.z * gg); x.w = fmaf(kk, u[3 % VEC], x.w * gg);
        acc[0] = fmaf(x.x, qq, acc[0]); acc[1 % VEC] = fmaf(x.y, qq, acc[1 % VEC]);
        acc[2 % VEC] = fmaf(x.z, qq, acc[2 % VEC]); acc[3 % VEC] = fmaf(x.w, qq, acc[3 % VEC]);
        *reinterpret_cast<float4*>(p) = x;
      } else {
        const float x = fmaf(kk, u[0], p[0] * gg);
        acc[0] = fmaf(x, qq, acc[0]);
        p[0] = x;
      }
    }
  if (live)
#pragma unroll
    for (int j = 0; j < VEC; ++j) red[grp * Dv + cv * VEC + j] = acc[j];
  fence_proxy_async_smem();
  __syncthreads();
  if (bulk) {
    if (tid == 0) {
      asm volatile("cp.async.bulk.global.shared::cta.bulk_group [%0], [%1], %2;" ::"l"(state), "r"(smem_u32(S)), "r"(tile_bytes) : "memory");
      asm volatile("cp.async.bulk.commit_group;" ::: "memory");
    }
  } else {
    for (int i = tid; i < D * Dv; i += DD_THREADS) state[i] = S[i];
  }
  float ov = 0.f;
  if (tid < Dv)
    for (int i = 0; i < groups; ++i) ov += red[i * Dv + tid];
  const float sq = dr_warp_sum(tid < Dv ? ov * ov : 0.f);
  if (lane == 0) ws[warp] = sq;
  __syncthreads();
  if (tid < Dv) {
    float tot = 0.f;
    for (int i = 0; i < NW; ++i) tot += ws[i];
    dr_st(out + (size_t)b * out_ld + h * Dv + tid, ov * (1.0f / sqrtf(tot / (float)Dv + eps)) * norm_w[tid] * gate_s[tid]);
  }
  if (bulk && tid == 0) asm volatile("cp.async.bulk.wait_group.read 0;" ::: "memory");
}

template <typename T, typename TW, typename TO, int VEC>
static int launch_delta_decode(const void* proj, int ld, const float* taps_w, float* ring, float* state, const int* pos, const int* slots,
                               const float* A_log, const float* dt_bias, const void* a2t, int a2_ld, const void* g2t, int g2_ld,
                               const float* norm_w, float eps, void* out, int out_ld, int B, int* status, const DeltaShape& s, cudaStream_t st) {
  const int lanes_per_row = (s.Dv / VEC + 31) & ~31, groups = DD_THREADS / lanes_per_row;
  const size_t smem = (size_t)(((s.D * s.Dv + 3) & ~3) + 3 * s.D + 2 * s.Dv + s.rank_a + s.rank_g + 2 * (DD_THREADS / 32) + groups * s.Dv) * 4;
  if (s.D * s.Dv * 4 > DD_MAX_TILE || smem > 226 * 1024) return -ERR_BAD_ARG;
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(delta_decode_kernel<T, TW, TO, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, 226 * 1024);
    if (e != cudaSuccess) return -(int)e;
    configured = true;
  }
  delta_decode_kernel<T, TW, TO, VEC><<<dim3(s.H, B), DD_THREADS, smem, st>>>(
      (const T*)proj, ld, taps_w, ring, state, pos, slots, A_log, dt_bias, (const TW*)a2t, a2_ld, (const TW*)g2t, g2_ld, norm_w, eps, (TO*)out,
      out_ld, status, s);
  const cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}

template <int DP, int LP, int THREADS>
static int launch_scan(const float* qn, const float* kn, const float* vv, const float* g, int g_ld, const float* beta, float* o, float* state,
                       const int* cu, const int* start, const int* slots, int n_seq, const DeltaShape& s, cudaStream_t st) {
  using L = ScanSmem<DP, LP, THREADS>;
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(delta_scan_kernel<DP, LP, THREADS>, cudaFuncAttributeMaxDynamicSharedMemorySize, L::BYTES);
    if (e != cudaSuccess) return -(int)e;
    configured = true;
  }
  const dim3 grid((s.Dv + L::COLS - 1) / L::COLS, s.H, n_seq);
  delta_scan_kernel<DP, LP, THREADS><<<grid, THREADS, L::BYTES, st>>>(qn, kn, vv, g, g_ld, beta, o, state, cu, start, slots, s.H, s.Hk, s.D, s.Dv);
  const cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}

static bool delta_shape_ok(const DeltaShape& s) {
  return s.H > 0 && s.Hk > 0 && s.H % s.Hk == 0 && s.D > 0 && s.D <= 256 && s.Dv > 0 && s.Dv <= 256 && s.taps > 0;
}

}  // namespace inv

using namespace inv;

// `shape`: the 14 ints of DeltaShape. proj_f32: projection rows are fp32, else bf16.
extern "C" int inv_delta_prep(const void* proj, int ld, int proj_f32, const float* taps_w, const float* ring, const int* tok_seq, const int* tok_pos,
                              const int* start, const int* slots, const float* A_log, const float* dt_bias, float* qn, float* kn, float* vv,
                              float* g, int g_ld, float* beta, int T, const int* shape, void* stream) {
  const DeltaShape s = *reinterpret_cast<const DeltaShape*>(shape);
  if (!delta_shape_ok(s)) return -ERR_BAD_ARG;
  if (T <= 0) return 0;
  const dim3 grid(T, (2 * s.Hk + s.H + 3) / 4);
  cudaStream_t st = (cudaStream_t)stream;
  if (proj_f32)
    delta_prep_kernel<float><<<grid, 128, 0, st>>>((const float*)proj, ld, taps_w, ring, tok_seq, tok_pos, start, slots, A_log, dt_bias, qn, kn, vv, g,
                                                   g_ld, beta, s);
  else
    delta_prep_kernel<__nv_bfloat16><<<grid, 128, 0, st>>>((const __nv_bfloat16*)proj, ld, taps_w, ring, tok_seq, tok_pos, start, slots, A_log,
                                                           dt_bias, qn, kn, vv, g, g_ld, beta, s);
  const cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}

extern "C" int inv_conv_tail(const void* proj, int ld, int proj_f32, float* ring, const int* cu, const int* start, const int* slots, int n_seq,
                             const int* shape, void* stream) {
  const DeltaShape s = *reinterpret_cast<const DeltaShape*>(shape);
  if (!delta_shape_ok(s)) return -ERR_BAD_ARG;
  if (n_seq <= 0) return 0;
  const dim3 grid(n_seq, (s.channels + 255) / 256);
  cudaStream_t st = (cudaStream_t)stream;
  if (proj_f32) conv_tail_kernel<float><<<grid, 256, 0, st>>>((const float*)proj, ld, ring, cu, start, slots, s);
  else conv_tail_kernel<__nv_bfloat16><<<grid, 256, 0, st>>>((const __nv_bfloat16*)proj, ld, ring, cu, start, slots, s);
  const cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}

// The recurrence over packed tokens: qn, kn [T, Hk, D], vv [T, H, Dv], g [T, g_ld], beta [T, H] -> o [T, H, Dv]; the state
// [slots, H, D, Dv] is taken as zero for sequences with start = 0. g_ld and D are multiples of 4 or D is not.
extern "C" int inv_delta_scan(const float* qn, const float* kn, const float* vv, const float* g, int g_ld, const float* beta, float* o, float* state,
                              const int* cu, const int* start, const int* slots, int n_seq, const int* shape, void* stream) {
  const DeltaShape s = *reinterpret_cast<const DeltaShape*>(shape);
  if (!delta_shape_ok(s) || (s.D % 4 == 0 && g_ld % 4)) return -ERR_BAD_ARG;
  if (n_seq <= 0) return 0;
  cudaStream_t st = (cudaStream_t)stream;
#define INV_SCAN(DP, LP, TH) launch_scan<DP, LP, TH>(qn, kn, vv, g, g_ld, beta, o, state, cu, start, slots, n_seq, s, st)
  if (s.D <= 16) return INV_SCAN(16, 4, 64);
  if (s.D <= 32) return INV_SCAN(32, 4, 64);
  if (s.D <= 64) return INV_SCAN(64, 4, 64);
  if (s.D <= 128) return INV_SCAN(128, 4, 64);
  return INV_SCAN(256, 8, 64);
#undef INV_SCAN
}

extern "C" int inv_gated_head_norm(const float* o, const float* w, const void* gate, int gate_ld, int gate_f32, void* out, int out_ld, int out_f32,
                                   int T, int H, int Dv, float eps, void* stream) {
  if (T <= 0) return 0;
  const dim3 grid(T, (H + 3) / 4);
  cudaStream_t st = (cudaStream_t)stream;
  if (gate_f32 && out_f32)
    gated_head_norm_kernel<float, float><<<grid, 128, 0, st>>>(o, w, (const float*)gate, gate_ld, (float*)out, out_ld, H, Dv, eps);
  else if (gate_f32)
    gated_head_norm_kernel<float, __nv_bfloat16><<<grid, 128, 0, st>>>(o, w, (const float*)gate, gate_ld, (__nv_bfloat16*)out, out_ld, H, Dv, eps);
  else if (!out_f32)
    gated_head_norm_kernel<__nv_bfloat16, __nv_bfloat16><<<grid, 128, 0, st>>>(o, w, (const __nv_bfloat16*)gate, gate_ld, (__nv_bfloat16*)out, out_ld,
                                                                               H, Dv, eps);
  else return -ERR_BAD_ARG;
  const cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}

// One token per sequence. Weights a2t [rank_a, a2_ld], g2t [rank_g, g2_ld] and out are bf16 (act_f32 = 0) or fp32; proj may be
// fp32 with bf16 weights (split-K accumulators). A state tile larger than DD_MAX_TILE is refused (use the prompt path).
extern "C" int inv_delta_decode(const void* proj, int ld, int proj_f32, const float* taps_w, float* ring, float* state, const int* pos,
                                const int* slots, const float* A_log, const float* dt_bias, const void* a2t, int a2_ld, const void* g2t, int g2_ld,
                                int act_f32, const float* norm_w, float eps, void* out, int out_ld, int B, int* status, const int* shape,
                                void* stream) {
  const DeltaShape s = *reinterpret_cast<const DeltaShape*>(shape);
  if (!delta_shape_ok(s)) return -ERR_BAD_ARG;
  if (B <= 0) return 0;
  cudaStream_t st = (cudaStream_t)stream;
#define INV_PD(T, TW, V)                                                                                                                          \
  launch_delta_decode<T, TW, TW, V>(proj, ld, taps_w, ring, state, pos, slots, A_log, dt_bias, a2t, a2_ld, g2t, g2_ld, norm_w, eps, out, out_ld, B, \
                                    status, s, st)
  const bool v4 = s.Dv % 4 == 0;
  if (proj_f32 && act_f32) return v4 ? INV_PD(float, float, 4) : INV_PD(float, float, 1);
  if (proj_f32) return v4 ? INV_PD(float, __nv_bfloat16, 4) : INV_PD(float, __nv_bfloat16, 1);
  if (!act_f32) return v4 ? INV_PD(__nv_bfloat16, __nv_bfloat16, 4) : INV_PD(__nv_bfloat16, __nv_bfloat16, 1);
#undef INV_PD
  return -ERR_BAD_ARG;
}
