// Gated delta rule with one decay per head and key channel, fp32 throughout:
//   S <- diag(g) S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q          (S: [D, Dv] per head and sequence)
// with short causal convolutions in front of q, k, v and a gated per-head RMS norm behind o.
//
// Prompt path, over packed tokens of several sequences, in chunks of 16 tokens. Inside a chunk that starts from state S0, with
// G_t the product of the chunk's decays up to token t,
//   u_t = beta_t (v_t - S0^T (G_t k_t) - sum_{s<t} kap[t, s] u_s)      kap[t, s] = sum_d k_t k_s G_t / G_s   (s < t)
//   o_t = S0^T (G_t q_t) + sum_{s<=t} P[t, s] u_s                      P[t, s] the same with q_t
//   S_16 = G_16 S0 + sum_t (G_16 / G_t) k_t u_t^T
// so the recurrence advances 16 tokens per step and everything that does not involve S0 is computed for all chunks at once:
//   delta_chunk       one CTA per (chunk, head): convolutions + SiLU, unit norms, decays exp(-exp(A) softplus(z + dt)), the decayed
//                     keys and queries, kap and P, and with T = (I + diag(beta) kap)^-1 diag(beta) the 16 x 16 maps T and P T.
//                     Ratios G_t / G_s are running products of decays (never quotients), so strong decays underflow to zero
//                     and nothing overflows.
//   conv_tail         keeps the last taps - 1 projection rows of every sequence (a ring of `taps` rows indexed by position)
//   delta_scan        the sequential part, fp32 FMAs: a CTA owns 16 value columns of one head with the state in shared memory; a
//                     chunk is two register-tiled products with S0, the two 16 x 16 maps and the update. Chunk blocks arrive by
//                     bulk copies, double buffered.
//   gated_head_norm   o / rms(o) * w * sigmoid(gate), cast to the projections' type
// Decode path: delta_decode does all of it for one token per sequence in one launch, one CTA per (sequence, head): the state
// tile is read once into shared memory and written once, which bounds the kernel at 8 D Dv bytes per head.
#include "sm100_common.cuh"
#include "inv_api.h"

namespace inv {

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

// Shapes and column offsets of one mixer. Projection rows hold [q | k | v | low-rank decay | low-rank gate | beta].
struct DeltaShape {
  int H, Hk, D, Dv, taps;
  int off_q, off_k, off_v, off_a, off_g, off_b;  // columns of a projection row
  int channels;                                  // off_v + H * Dv: the convolved columns, [0, channels)
  int rank_a, rank_g;
};

constexpr int CH = 16;         // tokens per chunk
constexpr int CK_THREADS = 128;

// One (chunk, head) block of floats: decayed keys and queries [D4][16 k | 16 q], keys for the update [16][D4], the maps
// [16 s][16 T | 16 PT], the chunk's decay [D4]; D4 = D rounded up to 4.
__host__ __device__ __forceinline__ int block_floats(int D4) { return 32 * D4 + CH * D4 + CH * 32 + D4; }

// Projection value of channel c at absolute position i (i < 0: before the start).
template <typename T>
__device__ __forceinline__ float conv_in(const T* proj, int ld, const float* ring, const DeltaShape& s, long row0, int start, int i, int c) {
  if (i < 0) return 0.f;
  return i >= start ? dr_ld(proj + (row0 + (i - start)) * ld + c) : ring[(size_t)(i % s.taps) * s.channels + c];
}

// ------------------------------------------------------------------------------------------------ prompt: chunks
// One exchange of the sums over 16 lanes: 2 M values per lane become M, and so on down to two.
template <int M>
__device__ __forceinline__ void fold_lanes(float* v, int l) {
  const bool up = (l & (M / 2)) != 0;
#pragma unroll
  for (int j = 0; j < M; ++j) {
    const float give = up ? v[j] : v[j + M], keep = up ? v[j + M] : v[j];
    v[j] = keep + __shfl_xor_sync(0xffffffffu, give, M / 2);
  }
  if constexpr (M > 2) fold_lanes<M / 2>(v, l);
}

// TAPS: longest convolution a thread keeps in registers while it walks down the chunk (longer ones re-read their inputs).
template <typename T, int TAPS>
__global__ void __launch_bounds__(CK_THREADS, 6) delta_chunk_kernel(const T* __restrict__ proj, int ld, const float* __restrict__ taps_w,
                                                                    const float* __restrict__ ring0, const int* __restrict__ chunk_seq,
                                                                    const int* __restrict__ cu_chunk, const int* __restrict__ cu,
                                                                    const int* __restrict__ start_, const int* __restrict__ slots,
                                                                    const float* __restrict__ A_log, const float* __restrict__ dt_bias,
                                                                    const float* __restrict__ z, int z_ld, float* __restrict__ blocks,
                                                                    float* __restrict__ vblocks, const DeltaShape s) {
  extern __shared__ __align__(16) float csm[];
  __shared__ float kap[CH][CH + 4], P[CH][CH + 4], Tm[CH][CH + 4], beta[CH];
  const int D = s.D, Dv = s.Dv, D4 = (D + 3) & ~3, cgs = (Dv + 15) / 16;
  float* q_s = csm;             // [16][D]
  float* k_s = q_s + CH * D;    // [16][D]
  float* g_s = k_s + CH * D;    // [16][D]
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, ch = blockIdx.x, h = blockIdx.y;
  const int seq = chunk_seq[ch], c0 = (ch - cu_chunk[seq]) * CH, start = start_[seq];
  const long row0 = cu[seq];                       // packed row of the portion's first token (position `start`)
  const int n = min(CH, cu[seq + 1] - (int)row0 - c0), pos0 = start + c0, hk = h / (s.H / s.Hk);
  const float* ring = ring0 + (size_t)slots[seq] * s.taps * s.channels;
  float* blk = blocks + ((size_t)ch * s.H + h) * block_floats(D4);
  float* vb = vblocks + ((size_t)ch * s.H + h) * cgs * (CH * 16);
  // a thread convolves one channel over half the chunk
  constexpr int HALF = CH / 2;
  const int n_ch = 2 * D + cgs * 16;
  for (int j = tid; j < 2 * n_ch; j += CK_THREADS) {
    const int half = j >= n_ch, i = half ? j - n_ch : j, v = i - 2 * D, tb = half * HALF;
    float* dst = i < D ? q_s + i : i < 2 * D ? k_s + (i - D) : vb + (size_t)(v >> 4) * (CH * 16) + (v & 15);
    const int step = i < 2 * D ? D : 16;
    if (v >= Dv) {                                 // padding columns of the last group
      for (int t = tb; t < tb + HALF; ++t) dst[t * step] = 0.f;
      continue;
    }
    const int c = i < D ? s.off_q + hk * D + i : i < 2 * D ? s.off_k + hk * D + (i - D) : s.off_v + h * Dv + v;
    const T* col = proj + (row0 + c0) * ld + c;
    if (s.taps <= TAPS) {
      float in[HALF + TAPS - 1], w[TAPS];          // inputs tb - (TAPS - 1) .. tb + HALF - 1
#pragma unroll
      for (int k = 0; k < TAPS; ++k) w[k] = k < s.taps ? taps_w[(size_t)(s.taps - 1 - k) * s.channels + c] : 0.f;
#pragma unroll
      for (int k = 0; k < TAPS - 1; ++k) {
        const int t = tb + k - (TAPS - 1);
        in[k] = TAPS - 1 - k < s.taps && t < n ? conv_in(proj, ld, ring, s, row0, start, pos0 + t, c) : 0.f;  // (the second half of a short chunk has no rows)
      }
#pragma unroll
      for (int k = 0; k < HALF; ++k) in[TAPS - 1 + k] = tb + k < n ? dr_ld(col + (long)(tb + k) * ld) : 0.f;
#pragma unroll
      for (int k = 0; k < HALF; ++k) {
        float a = 0.f;
#pragma unroll
        for (int m = 0; m < TAPS; ++m) a = fmaf(in[TAPS - 1 + k - m], w[m], a);
        dst[(tb + k) * step] = tb + k < n ? dr_silu(a) : 0.f;
      }
    } else {
      for (int t = tb; t < tb + HALF; ++t) {
        float a = 0.f;
        if (t < n)
          for (int m = 0; m < s.taps; ++m)
            a = fmaf(conv_in(proj, ld, ring, s, row0, start, pos0 + t - m, c), taps_w[(size_t)(s.taps - 1 - m) * s.channels + c], a);
        dst[t * step] = dr_silu(a);
      }
    }
  }
  const float ea = expf(A_log[h]);
  for (int d = tid; d < D; d += CK_THREADS) {
    const float bias = dt_bias[h * D + d];
    const float* zp = z + (row0 + c0) * z_ld + h * D + d;
#pragma unroll
    for (int t0 = 0; t0 < CH; t0 += 8) {
      float x[8];
#pragma unroll
      for (int t = 0; t < 8; ++t) x[t] = t0 + t < n ? zp[(long)(t0 + t) * z_ld] : 0.f;
#pragma unroll
      for (int t = 0; t < 8; ++t) g_s[(t0 + t) * D + d] = t0 + t < n ? expf(-ea * dr_softplus(x[t] + bias)) : 1.f;
    }
  }
  if (tid < CH) beta[tid] = tid < n ? dr_sigmoid(dr_ld(proj + (row0 + c0 + tid) * ld + s.off_b + h)) : 0.f;
  __syncthreads();
  for (int t = warp; t < CH; t += CK_THREADS / 32) {   // unit vectors; the query also carries D^-1/2
    float sq = 0.f, sk = 0.f;
    for (int d = lane; d < D; d += 32) {
      sq = fmaf(q_s[t * D + d], q_s[t * D + d], sq);
      sk = fmaf(k_s[t * D + d], k_s[t * D + d], sk);
    }
    const float rq = 1.0f / sqrtf(dr_warp_sum(sq) + 1e-6f) * (1.0f / sqrtf((float)D)), rk = 1.0f / sqrtf(dr_warp_sum(sk) + 1e-6f);
    for (int d = lane; d < D; d += 32) {
      q_s[t * D + d] *= rq;
      k_s[t * D + d] *= rk;
    }
  }
  __syncthreads();
  // decayed keys and queries, and the keys of the update: a running product down the chunk and one up
  for (int d = tid; d < D4; d += CK_THREADS) {
    const bool in = d < D;
    float G = 1.f;
#pragma unroll
    for (int t = 0; t < CH; t += 4) {
      float kk[4], qq[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        if (in) G *= g_s[(t + j) * D + d];
        kk[j] = in ? k_s[(t + j) * D + d] * G : 0.f;
        qq[j] = in ? q_s[(t + j) * D + d] * G : 0.f;
      }
      *reinterpret_cast<float4*>(blk + (size_t)d * 32 + t) = make_float4(kk[0], kk[1], kk[2], kk[3]);
      *reinterpret_cast<float4*>(blk + (size_t)d * 32 + CH + t) = make_float4(qq[0], qq[1], qq[2], qq[3]);
    }
    blk[32 * D4 + CH * D4 + CH * 32 + d] = G;
    float R = 1.f;
#pragma unroll
    for (int t = CH - 1; t >= 0; --t) {
      blk[32 * D4 + t * D4 + d] = in ? k_s[t * D + d] * R : 0.f;
      if (in) R *= g_s[t * D + d];
    }
  }
  // kap and P: 16 lanes per source token share the channels and walk upwards with w = k_src * (decays of src + 1 .. t). A warp
  // takes sources 2 m and 2 m + 1 (about the same length) for m = warp and 7 - warp, which evens out the warps.
  {
    const int l = lane & 15;
#pragma unroll
    for (int pass = 0; pass < 2; ++pass) {
      const int src = 2 * (pass ? 7 - warp : warp) + (lane >> 4), steps = CH - src;
      float v[2 * CH];                             // [j] kap, [16 + j] P for t = src + j
#pragma unroll
      for (int j = 0; j < 2 * CH; ++j) v[j] = 0.f;
      for (int d = l; d < D; d += 16) {
        const float* kp = k_s + src * D + d;
        const float* qp = q_s + src * D + d;
        const float* gp = g_s + src * D + d;
        float w = kp[0];
#pragma unroll
        for (int j = 0; j < CH; ++j) {
          if (j < steps) {
            if (j > 0) w *= gp[j * D];
            v[j] = fmaf(kp[j * D], w, v[j]);
            v[CH + j] = fmaf(qp[j * D], w, v[CH + j]);
          }
        }
      }
      // sums over the 16 lanes: each exchange halves the values a lane is responsible for; lane l ends with v[2 l'], v[2 l' + 1]
      fold_lanes<CH>(v, l);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int j = 2 * (l & 7) + e, t = src + j;
        if (t < CH) {
          if (l < 8) kap[t][src] = j > 0 ? v[e] : 0.f;
          else P[t][src] = v[e];
        }
        if (j < src) {                             // targets before the source
          if (l < 8) kap[j][src] = 0.f;
          else P[j][src] = 0.f;
        }
      }
    }
  }
  __syncthreads();
  if (tid < CH) {                                  // column tid of T by forward substitution
    float x[CH];
#pragma unroll
    for (int t = 0; t < CH; ++t) {
      float a = t == tid ? 1.f : 0.f, a2 = 0.f;
#pragma unroll
      for (int r = 0; r < CH; r += 2) {
        if (r < t) a = fmaf(-kap[t][r], x[r], a);
        if (r + 1 < t) a2 = fmaf(-kap[t][r + 1], x[r + 1], a2);
      }
      x[t] = beta[t] * (a + a2);
      Tm[t][tid] = x[t];
    }
  }
  __syncthreads();
  for (int i = tid; i < CH * CH; i += CK_THREADS) {
    const int t = i & 15, c = i >> 4;              // entry (t, c) of T and of P T
    float a = 0.f;
#pragma unroll
    for (int r = 0; r < CH; ++r) a = fmaf(P[t][r], Tm[r][c], a);
    float* tw = blk + 32 * D4 + CH * D4 + c * 32;
    tw[t] = Tm[t][c];
    tw[CH + t] = a;
  }
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
constexpr int SC_THREADS = 128;
constexpr int SC_COLS = 16;

__global__ void __launch_bounds__(SC_THREADS) delta_scan_kernel(const float* __restrict__ blocks, const float* __restrict__ vblocks,
                                                                float* __restrict__ o, float* __restrict__ state0,
                                                                const int* __restrict__ cu_chunk, const int* __restrict__ cu,
                                                                const int* __restrict__ start, const int* __restrict__ slots, int H, int D, int Dv,
                                                                int* status) {
  extern __shared__ __align__(16) float sm[];
  __shared__ uint64_t full[2];
  __shared__ int abort_flag;
  const int D4 = (D + 3) & ~3, bf = block_floats(D4), cgs = gridDim.x;
  const int stage_floats = bf + CH * SC_COLS;
  float* S = sm;                              // [D4][16]
  float* part = S + D4 * SC_COLS;             // [4 warps][32][16]
  float* R = part + 4 * 32 * SC_COLS;         // [16][16]
  float* U = R + CH * SC_COLS;                // [16][16]
  float* buf = U + CH * SC_COLS;              // [2][block | values]
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int cg = blockIdx.x, h = blockIdx.y, seq = blockIdx.z, col0 = cg * SC_COLS;
  const int ch0 = cu_chunk[seq], nc = cu_chunk[seq + 1] - ch0, row0 = cu[seq], len = cu[seq + 1] - row0;
  float* state = state0 + ((size_t)slots[seq] * H + h) * (size_t)D * Dv;
  auto stage = [&](int c) {                   // thread 0
    float* b = buf + (c & 1) * stage_floats;
    const size_t id = (size_t)(ch0 + c) * H + h;
    mbar_expect_tx(&full[c & 1], (uint32_t)stage_floats * 4u);
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(smem_u32(b)),
                 "l"(blocks + id * bf), "r"((uint32_t)bf * 4u), "r"(smem_u32(&full[c & 1]))
                 : "memory");
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(smem_u32(b + bf)),
                 "l"(vblocks + (id * cgs + cg) * (CH * SC_COLS)), "r"((uint32_t)(CH * SC_COLS) * 4u), "r"(smem_u32(&full[c & 1]))
                 : "memory");
  };
  if (tid == 0) {
    abort_flag = 0;
    mbar_init(&full[0], 1);
    mbar_init(&full[1], 1);
    fence_barrier_init();
    if (nc > 0) stage(0);
  }
  for (int i = tid; i < D4 * SC_COLS; i += SC_THREADS) {
    const int d = i / SC_COLS, c = col0 + i % SC_COLS;
    S[i] = (start[seq] > 0 && d < D && c < Dv) ? state[(size_t)d * Dv + c] : 0.f;
  }
  __syncthreads();
  const int r = tid >> 2, c4 = (tid & 3) * 4;       // phases 2 and 3: row of [16 T | 16 PT] and four columns
  const int tg = lane >> 2;                         // phase 1: four of the 32 rows, columns c4
  bool ok = true;
  for (int c = 0; c < nc; ++c) {
    if (tid == 0 && c + 1 < nc) stage(c + 1);       // its buffer was last read before the barrier that ended chunk c - 1
    ok = mbar_wait(&full[c & 1], (c >> 1) & 1, &abort_flag, status, ERR_WAIT_FULL);
    const float* b = buf + (c & 1) * stage_floats;
    // 1. [keys; queries] x S0, channels split over the warps
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
#pragma unroll 8
    for (int d = warp; d < D4; d += 4) {
      const float4 a = *reinterpret_cast<const float4*>(b + d * 32 + tg * 4);
      const float4 x = *reinterpret_cast<const float4*>(S + d * SC_COLS + c4);
      const float av[4] = {a.x, a.y, a.z, a.w}, xv[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], xv[j], acc[i][j]);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
      *reinterpret_cast<float4*>(part + (warp * 32 + tg * 4 + i) * SC_COLS + c4) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
    if (!__syncthreads_and(ok)) break;
    // 2. sum over the warps; rows 0..15 become v - S0^T k, rows 16..31 stay here for the outputs
    float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float4 x = *reinterpret_cast<const float4*>(part + (w * 32 + r) * SC_COLS + c4);
      y.x += x.x; y.y += x.y; y.z += x.z; y.w += x.w;
    }
    if (r < CH) {
      const float4 v = *reinterpret_cast<const float4*>(b + bf + r * SC_COLS + c4);
      *reinterpret_cast<float4*>(R + r * SC_COLS + c4) = make_float4(v.x - y.x, v.y - y.y, v.z - y.z, v.w - y.w);
      y = make_float4(0.f, 0.f, 0.f, 0.f);
    }
    __syncthreads();
    // 3. U = T R (rows 0..15), O = S0^T q + P T R (rows 16..31)
    const float* tw = b + 32 * D4 + CH * D4 + r;
#pragma unroll
    for (int k = 0; k < CH; ++k) {
      const float w = tw[k * 32];
      const float4 x = *reinterpret_cast<const float4*>(R + k * SC_COLS + c4);
      y.x = fmaf(w, x.x, y.x); y.y = fmaf(w, x.y, y.y); y.z = fmaf(w, x.z, y.z); y.w = fmaf(w, x.w, y.w);
    }
    if (r < CH) {
      *reinterpret_cast<float4*>(U + r * SC_COLS + c4) = y;
    } else {
      const int t = c * CH + r - CH;
      if (t < len) {
        float* dst = o + ((size_t)(row0 + t) * H + h) * Dv + col0 + c4;
        const float yv[4] = {y.x, y.y, y.z, y.w};
        if (Dv % 4 == 0 && col0 + c4 < Dv) *reinterpret_cast<float4*>(dst) = y;
        else if (Dv % 4)
#pragma unroll
          for (int j = 0; j < 4; ++j)
            if (col0 + c4 + j < Dv) dst[j] = yv[j];
      }
    }
    __syncthreads();
    // 4. S <- G S + K^T U, four channels by four columns per thread
    const float* kout = b + 32 * D4;
    const float* gend = kout + CH * D4 + CH * 32;
    for (int d = (tid >> 2) * 4; d < D4; d += SC_THREADS) {
      float a4[4][4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float g = gend[d + i];
        const float4 x = *reinterpret_cast<const float4*>(S + (d + i) * SC_COLS + c4);
        a4[i][0] = g * x.x; a4[i][1] = g * x.y; a4[i][2] = g * x.z; a4[i][3] = g * x.w;
      }
#pragma unroll
      for (int t = 0; t < CH; ++t) {
        const float4 a = *reinterpret_cast<const float4*>(kout + t * D4 + d);
        const float4 x = *reinterpret_cast<const float4*>(U + t * SC_COLS + c4);
        const float av[4] = {a.x, a.y, a.z, a.w}, xv[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) a4[i][j] = fmaf(av[i], xv[j], a4[i][j]);
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) *reinterpret_cast<float4*>(S + (d + i) * SC_COLS + c4) = make_float4(a4[i][0], a4[i][1], a4[i][2], a4[i][3]);
    }
    __syncthreads();
  }
  if (!__syncthreads_and(ok)) {  // a copy never arrived: leave the ones in flight a bounded time before the shared memory goes away
    const uint64_t t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 2000000ull) __nanosleep(1000);
    return;
  }
  for (int i = tid; i < D4 * SC_COLS; i += SC_THREADS) {
    const int d = i / SC_COLS, c = col0 + i % SC_COLS;
    if (d < D && c < Dv) state[(size_t)d * Dv + c] = S[i];
  }
}

// ------------------------------------------------------------------------------------------------ prompt: output norm
__device__ __forceinline__ void dr_ld4(const float* p, float* f) {
  const float4 v = *reinterpret_cast<const float4*>(p);
  f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
}
__device__ __forceinline__ void dr_ld4(const __nv_bfloat16* p, float* f) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  f[0] = __uint_as_float(v.x << 16); f[1] = __uint_as_float(v.x & 0xffff0000u);
  f[2] = __uint_as_float(v.y << 16); f[3] = __uint_as_float(v.y & 0xffff0000u);
}
__device__ __forceinline__ void dr_st4(float* p, const float* f) { *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]); }
__device__ __forceinline__ void dr_st4(__nv_bfloat16* p, const float* f) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]));
}

// One warp per (token, head). V = 4: the row stays in registers (Dv <= 256, Dv % 4 == 0); V = 1: any Dv.
template <typename TG, typename TO, int V>
__global__ void __launch_bounds__(256) gated_head_norm_kernel(const float* __restrict__ o, const float* __restrict__ w, const TG* __restrict__ gate,
                                                              int gate_ld, TO* __restrict__ out, int out_ld, int H, int Dv, float eps, long n_rows) {
  const int lane = threadIdx.x & 31;
  const long i = (long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (i >= n_rows) return;
  const size_t t = i / H;
  const int h = (int)(i % H);
  const float* r = o + (size_t)i * Dv;
  const TG* gp = gate + t * gate_ld + h * Dv;
  TO* op = out + t * out_ld + h * Dv;
  float ss = 0.f;
  if (V == 4) {
    float x[2][4], g[2][4];
#pragma unroll
    for (int m = 0; m < 2; ++m) {
      const int d = (lane + m * 32) * 4;
      if (d < Dv) {
        dr_ld4(r + d, x[m]);
        dr_ld4(gp + d, g[m]);
#pragma unroll
        for (int j = 0; j < 4; ++j) ss = fmaf(x[m][j], x[m][j], ss);
      }
    }
    const float inv = 1.0f / sqrtf(dr_warp_sum(ss) / (float)Dv + eps);
#pragma unroll
    for (int m = 0; m < 2; ++m) {
      const int d = (lane + m * 32) * 4;
      if (d < Dv) {
        float y[4];
        dr_ld4(w + d, y);
#pragma unroll
        for (int j = 0; j < 4; ++j) y[j] = x[m][j] * inv * y[j] * dr_sigmoid(g[m][j]);
        dr_st4(op + d, y);
      }
    }
  } else {
    for (int d = lane; d < Dv; d += 32) ss = fmaf(r[d], r[d], ss);
    const float inv = 1.0f / sqrtf(dr_warp_sum(ss) / (float)Dv + eps);
    for (int d = lane; d < Dv; d += 32) dr_st(op + d, r[d] * inv * w[d] * dr_sigmoid(dr_ld(gp + d)));
  }
}

// ------------------------------------------------------------------------------------------------ decode, one launch
// One CTA per (head, sequence). The head's state tile is one contiguous range: a single bulk copy brings it into shared
// memory while the convolutions, norms and low-rank products run, it is updated in place and a bulk copy writes it back.
// Row groups of threads walk the tile (VEC value columns per thread); three tiles of 128 x 128 share an SM.
constexpr int DD_THREADS = 256;

// a[j] += f * (element j of a 16-byte piece)
__device__ __forceinline__ void fma_row(const uint4& p, float f, float* a, __nv_bfloat16) {
  const uint32_t u[4] = {p.x, p.y, p.z, p.w};
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    a[2 * j] = fmaf(__uint_as_float(u[j] << 16), f, a[2 * j]);
    a[2 * j + 1] = fmaf(__uint_as_float(u[j] & 0xffff0000u), f, a[2 * j + 1]);
  }
}
__device__ __forceinline__ void fma_row(const uint4& p, float f, float* a, float) {
  a[0] = fmaf(__uint_as_float(p.x), f, a[0]); a[1] = fmaf(__uint_as_float(p.y), f, a[1]);
  a[2] = fmaf(__uint_as_float(p.z), f, a[2]); a[3] = fmaf(__uint_as_float(p.w), f, a[3]);
}

constexpr int DD_MAX_TILE = 192 * 1024;

template <typename T, typename TW, typename TO, int VEC>
__global__ void __launch_bounds__(DD_THREADS, 3) delta_decode_kernel(const T* __restrict__ proj, int ld, const float* __restrict__ taps_w,
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
  float* low = red;                      // [NW / 2][D + Dv], before red is used
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
  // everything later phases read from global memory is requested here, so that the waits overlap: small vectors, and this
  // thread's first rows of the low-rank matrices
  // Low-rank products: warps 0..3 work on the decay's second matrix, 4..7 on the gate's (both stored transposed: [rank, heads *
  // channels]); a lane adds VW neighbouring channels over the rows of its group.
  constexpr int VW = 16 / sizeof(TW), PRE = 4, LW = NW / 2;
  const bool is_a = warp < LW;
  const int lw = is_a ? D : Dv, lrank = is_a ? s.rank_a : s.rank_g, lld = is_a ? a2_ld : g2_ld;
  const int pieces = (lw + VW - 1) / VW, lpr = pieces <= 16 ? 16 : 32, lrows = LW * (32 / lpr);   // rows per step of the four warps
  const int lrow0 = (warp % LW) * (32 / lpr) + lane / lpr, lp0 = lane % lpr;
  const TW* lmat = is_a ? a2t + h * D : g2t + h * Dv;
  const bool vec = D % VW == 0 && Dv % VW == 0;   // rows are 16-byte multiples, so every piece is aligned
  uint4 pre[PRE];
#pragma unroll
  for (int i = 0; i < PRE; ++i) {
    const int r = lrow0 + i * lrows;
    pre[i] = (vec && lp0 < pieces && r < lrank) ? *reinterpret_cast<const uint4*>(lmat + (size_t)r * lld + lp0 * VW) : make_uint4(0, 0, 0, 0);
  }
  const float a_log = A_log[h], b_in = dr_ld(row + s.off_b + h), bias0 = tid < D ? dt_bias[h * D + tid] : 0.f, nw0 = tid < Dv ? norm_w[tid] : 0.f;
  if (pos == 0)
    for (int i = tid; i < D * Dv; i += DD_THREADS) S[i] = 0.f;
  else if (!bulk)
    for (int i = tid; i < D * Dv; i += DD_THREADS) S[i] = state[i];
  // convolutions; the current row goes into the ring slot of this position, which nobody reads in this launch
  const int nq = 2 * D + Dv;
  const bool own_qk = h % (s.H / s.Hk) == 0;
  float ssq = 0.f, ssk = 0.f;
#pragma unroll 2
  for (int i = tid; i < nq; i += DD_THREADS) {
    const int c = i < D ? s.off_q + hk * D + i : i < 2 * D ? s.off_k + hk * D + (i - D) : s.off_v + h * Dv + (i - 2 * D);
    const float cur = dr_ld(row + c);
    float a = cur * taps_w[(size_t)(s.taps - 1) * s.channels + c];
    if (s.taps <= 4) {
      float x[3], w[3];
#pragma unroll
      for (int j = 1; j < 4; ++j) {
        const bool in = j < s.taps && pos - j >= 0;
        x[j - 1] = in ? ring[(size_t)((pos - j) % s.taps) * s.channels + c] : 0.f;
        w[j - 1] = in ? taps_w[(size_t)(s.taps - 1 - j) * s.channels + c] : 0.f;
      }
#pragma unroll
      for (int j = 0; j < 3; ++j) a = fmaf(x[j], w[j], a);
    } else {
      for (int j = 1; j < s.taps; ++j)
        if (pos - j >= 0) a = fmaf(ring[(size_t)((pos - j) % s.taps) * s.channels + c], taps_w[(size_t)(s.taps - 1 - j) * s.channels + c], a);
    }
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
  const float ea = expf(a_log);
  const float* lf = lr + (is_a ? 0 : s.rank_a);
  for (int p = lp0; p < (pieces + lpr - 1) / lpr * lpr; p += lpr) {   // the same number of turns for every lane
    const int c = p * VW;
    float a[VW];
#pragma unroll
    for (int j = 0; j < VW; ++j) a[j] = 0.f;
    int r0 = lrow0;
    if (vec && p < pieces) {
      if (p == lp0) {                              // the rows requested at the start
#pragma unroll
        for (int i = 0; i < PRE; ++i) fma_row(pre[i], lrow0 + i * lrows < lrank ? lf[lrow0 + i * lrows] : 0.f, a, TW());
        r0 += PRE * lrows;
      }
#pragma unroll 8
      for (int r = r0; r < lrank; r += lrows) {
        const uint4 raw = *reinterpret_cast<const uint4*>(lmat + (size_t)r * lld + c);
        fma_row(raw, lf[r], a, TW());
      }
    } else if (p < pieces) {
      for (int r = r0; r < lrank; r += lrows)
#pragma unroll
        for (int j = 0; j < VW; ++j)
          if (c + j < lw) a[j] = fmaf(dr_ld(lmat + (size_t)r * lld + c + j), lf[r], a[j]);
    }
    if (lpr == 16)
#pragma unroll
      for (int j = 0; j < VW; ++j) a[j] += __shfl_xor_sync(0xffffffffu, a[j], 16);
    if (lane < lpr)
#pragma unroll
      for (int j = 0; j < VW; ++j)
        if (c + j < lw) low[(warp % LW) * (D + Dv) + (is_a ? 0 : D) + c + j] = a[j];
  }
  __syncthreads();
  for (int d = tid; d < D + Dv; d += DD_THREADS) {
    float a = 0.f;
#pragma unroll
    for (int i = 0; i < LW; ++i) a += low[i * (D + Dv) + d];
    if (d < D) {
      g_s[d] = expf(-ea * dr_softplus(a + (d == tid ? bias0 : dt_bias[h * D + d])));
      q_s[d] *= rq;
      k_s[d] *= rk;
    } else {
      gate_s[d - D] = dr_sigmoid(a);
    }
  }
  const float beta = dr_sigmoid(b_in);
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
    dr_st(out + (size_t)b * out_ld + h * Dv + tid, ov * (1.0f / sqrtf(tot / (float)Dv + eps)) * nw0 * gate_s[tid]);
  }
  if (bulk && tid == 0) asm volatile("cp.async.bulk.wait_group.read 0;" ::: "memory");
}

template <typename T, typename TW, typename TO, int VEC>
static int launch_delta_decode(const void* proj, int ld, const float* taps_w, float* ring, float* state, const int* pos, const int* slots,
                               const float* A_log, const float* dt_bias, const void* a2t, int a2_ld, const void* g2t, int g2_ld,
                               const float* norm_w, float eps, void* out, int out_ld, int B, int* status, const DeltaShape& s, cudaStream_t st) {
  const int lanes_per_row = (s.Dv / VEC + 31) & ~31, groups = DD_THREADS / lanes_per_row;
  const size_t smem = (size_t)(((s.D * s.Dv + 3) & ~3) + 3 * s.D + 2 * s.Dv + s.rank_a + s.rank_g + 2 * (DD_THREADS / 32) +
                                max(groups * s.Dv, DD_THREADS / 64 * (s.D + s.Dv))) * 4;
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

static bool delta_shape_ok(const DeltaShape& s) {
  return s.H > 0 && s.Hk > 0 && s.H % s.Hk == 0 && s.D > 0 && s.D <= 256 && s.Dv > 0 && s.Dv <= 256 && s.taps > 0;
}

}  // namespace inv

using namespace inv;

// `shape`: the 14 ints of DeltaShape. proj_f32: projection rows are fp32, else bf16.
extern "C" int inv_delta_chunk(const void* proj, int ld, int proj_f32, const float* taps_w, const float* ring, const int* chunk_seq,
                               const int* cu_chunk, const int* cu, const int* start, const int* slots, const float* A_log, const float* dt_bias,
                               const float* z, int z_ld, float* blocks, float* vblocks, int n_chunks, const int* shape, void* stream) {
  const DeltaShape s = *reinterpret_cast<const DeltaShape*>(shape);
  if (!delta_shape_ok(s)) return -ERR_BAD_ARG;
  if (n_chunks <= 0) return 0;
  const dim3 grid(n_chunks, s.H);
  const int smem = 3 * CH * s.D * 4;   // at most 48 KB
  cudaStream_t st = (cudaStream_t)stream;
  // channels above 192 need more than the default 48 KB with the static arrays
#define INV_CK(T, TAPS)                                                                                                                              \
  do {                                                                                                                                               \
    static bool configured = false;                                                                                                                  \
    if (!configured) {                                                                                                                               \
      const cudaError_t e = cudaFuncSetAttribute(delta_chunk_kernel<T, TAPS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 3 * CH * 256 * 4);         \
      if (e != cudaSuccess) return -(int)e;                                                                                                          \
      configured = true;                                                                                                                             \
    }                                                                                                                                                \
    delta_chunk_kernel<T, TAPS><<<grid, CK_THREADS, smem, st>>>((const T*)proj, ld, taps_w, ring, chunk_seq, cu_chunk, cu, start, slots, A_log, dt_bias, \
                                                                z, z_ld, blocks, vblocks, s);                                                        \
  } while (0)
  if (proj_f32) {
    if (s.taps <= 4) INV_CK(float, 4);
    else INV_CK(float, 8);
  } else {
    if (s.taps <= 4) INV_CK(__nv_bfloat16, 4);
    else INV_CK(__nv_bfloat16, 8);
  }
#undef INV_CK
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

// The recurrence over the chunks of n_seq sequences (blocks and vblocks of inv_delta_chunk) -> o [T, H, Dv]; the state
// [slots, H, D, Dv] is taken as zero for sequences with start = 0.
extern "C" int inv_delta_scan(const float* blocks, const float* vblocks, float* o, float* state, const int* cu_chunk, const int* cu, const int* start,
                              const int* slots, int n_seq, int* status, const int* shape, void* stream) {
  const DeltaShape s = *reinterpret_cast<const DeltaShape*>(shape);
  if (!delta_shape_ok(s)) return -ERR_BAD_ARG;
  if (n_seq <= 0) return 0;
  const int D4 = (s.D + 3) & ~3;
  const int smem = (D4 * SC_COLS + 4 * 32 * SC_COLS + 2 * CH * SC_COLS + 2 * (block_floats(D4) + CH * SC_COLS)) * 4;
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(delta_scan_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024);
    if (e != cudaSuccess) return -(int)e;
    configured = true;
  }
  delta_scan_kernel<<<dim3((s.Dv + SC_COLS - 1) / SC_COLS, s.H, n_seq), SC_THREADS, smem, (cudaStream_t)stream>>>(blocks, vblocks, o, state, cu_chunk, cu,
                                                                                                           start, slots, s.H, s.D, s.Dv, status);
  const cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}

extern "C" int inv_gated_head_norm(const float* o, const float* w, const void* gate, int gate_ld, int gate_f32, void* out, int out_ld, int out_f32,
                                   int T, int H, int Dv, float eps, void* stream) {
  if (T <= 0) return 0;
  const long n_rows = (long)T * H;
  const int grid = (int)((n_rows + 7) / 8);
  const bool v4 = Dv % 4 == 0 && Dv <= 256 && gate_ld % 4 == 0 && out_ld % 4 == 0;
  cudaStream_t st = (cudaStream_t)stream;
#define INV_HN(TG, TO)                                                                                                                          \
  do {                                                                                                                                          \
    if (v4) gated_head_norm_kernel<TG, TO, 4><<<grid, 256, 0, st>>>(o, w, (const TG*)gate, gate_ld, (TO*)out, out_ld, H, Dv, eps, n_rows);       \
    else gated_head_norm_kernel<TG, TO, 1><<<grid, 256, 0, st>>>(o, w, (const TG*)gate, gate_ld, (TO*)out, out_ld, H, Dv, eps, n_rows);          \
  } while (0)
  if (gate_f32 && out_f32) INV_HN(float, float);
  else if (!gate_f32 && !out_f32) INV_HN(__nv_bfloat16, __nv_bfloat16);
  else return -ERR_BAD_ARG;
#undef INV_HN
  const cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}

// One token per sequence. Weights a2t [rank_a, a2_ld], g2t [rank_g, g2_ld] and out are bf16 (act_f32 = 0) or fp32; proj may be
// fp32 with bf16 weights. A state tile larger than DD_MAX_TILE is refused (use the prompt path).
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
