// Attention over a paged cache of latents (one RMS-normed vector of `kv_rank` numbers per token, shared by all heads).
//
// A head's key is W_uk c and its value W_uv c. Neither is stored: the query is carried into the latent space once per token
// (q' = W_uk^T q, `head_proj`), scores and the weighted sum run on the latents themselves, and W_uv is applied to the sum.
//   latent_prep        normalises the latent columns of the fused projection, appends them to the pages, casts the queries
//   head_proj          per-head products of small batches (mma.sync, K split over the warps of a CTA)
//   latent_attend      fp32 and any size: one warp per (token, head)
//   latent_attend_mma  bf16: one CTA per (token, 16 heads, key split); latent tiles arrive through cp.async, scores and sums on
//                      the tensor cores with fp32 softmax (the 16-row warp-level MMA fits the 16 queries of a tile: a
//                      128-row tcgen05 tile would be seven eighths padding, and the kernel is bound by the latent bytes)
// A window keeps the keys j with pos - window < j <= pos; pages wholly before it are never touched.
#include "sm100_common.cuh"
#include "inv_api.h"

namespace inv {

constexpr int LA_PAGE = 16;

__device__ __forceinline__ float la_ld(const float* p) { return *p; }
__device__ __forceinline__ float la_ld(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void la_st(float* p, float v) { *p = v; }
__device__ __forceinline__ void la_st(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ float la_warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// ------------------------------------------------------------------------------------------------ prep
// in: [T, in_ld], queries in columns [0, nq), latents in [off_c, off_c + Rp). The mean square is over the true rank R; columns
// R..Rp are padding (zero weights). c_out and q_out are optional contiguous copies.
template <typename TI, typename TC>
__global__ void __launch_bounds__(128) latent_prep_kernel(const TI* __restrict__ in, int in_ld, int off_c, int R, int Rp, const float* __restrict__ w,
                                                          float eps, TC* __restrict__ pool, const int* __restrict__ page_table, int max_pages,
                                                          const int* __restrict__ rows, const int* __restrict__ tok_seq,
                                                          const int* __restrict__ tok_pos, TC* __restrict__ c_out, int c_ld, int nq,
                                                          TC* __restrict__ q_out, int q_ld) {
  __shared__ float red[4];
  const int tid = threadIdx.x;
  const size_t t = blockIdx.x;
  const TI* r = in + t * in_ld + off_c;
  float ss = 0.f;
  for (int i = tid; i < R; i += 128) {
    const float x = la_ld(r + i);
    ss = fmaf(x, x, ss);
  }
  ss = la_warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  const float inv = 1.0f / sqrtf((red[0] + red[1] + red[2] + red[3]) / (float)R + eps);
  const int pos = tok_pos[t];
  const int page = page_table[(size_t)rows[tok_seq[t]] * max_pages + pos / LA_PAGE];
  TC* dst = pool + ((size_t)page * LA_PAGE + pos % LA_PAGE) * Rp;
  for (int i = tid; i < Rp; i += 128) {
    const float x = i < R ? la_ld(r + i) * inv * w[i] : 0.f;
    la_st(dst + i, x);
    if (c_out) la_st(c_out + t * c_ld + i, x);
  }
  if (q_out)
    for (int i = tid; i < nq; i += 128) la_st(q_out + t * q_ld + i, la_ld(in + t * in_ld + i));
}

// ------------------------------------------------------------------------------------------------ mma helpers
__device__ __forceinline__ void mma_bf16_16816(float* d, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm_x4(uint32_t* r, const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(smem_u32(p)));
}
__device__ __forceinline__ void ldsm_x2(uint32_t* r, const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0, %1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void ldsm_x2_t(uint32_t* r, const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0, %1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(smem_u32(p)));
}

// ------------------------------------------------------------------------------------------------ per-head products
// out[t, h, n] = sum_k a[t, h, k] W[h, n, k]; a and out rows are [T, ld] with heads `stride` apart; W [H, N, K] dense.
// One CTA: one head, 16 columns n, MT * 16 tokens; the four warps take every fourth 16-wide k step. K % 16 == 0, N % 16 == 0.
template <int MT>
__global__ void __launch_bounds__(128) head_proj_kernel(const __nv_bfloat16* __restrict__ a, int a_ld, int a_stride, const __nv_bfloat16* __restrict__ W,
                                                        int N, int K, __nv_bfloat16* __restrict__ out, int out_ld, int out_stride, int T) {
  __shared__ float part[4][MT * 16][17];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int n0 = blockIdx.x * 16, h = blockIdx.y, t0 = blockIdx.z * MT * 16;
  const int g = lane >> 2, c2 = (lane & 3) * 2;
  float acc[MT][2][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[m][n][i] = 0.f;
  const __nv_bfloat16* wp = W + ((size_t)h * N + n0 + g) * K + c2;
  const __nv_bfloat16* ap = a + (size_t)h * a_stride + c2;
#pragma unroll 2
  for (int k = warp * 16; k < K; k += 64) {
    uint32_t b[2][2];
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      b[n][0] = *reinterpret_cast<const uint32_t*>(wp + (size_t)n * 8 * K + k);
      b[n][1] = *reinterpret_cast<const uint32_t*>(wp + (size_t)n * 8 * K + k + 8);
    }
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const int r0 = t0 + m * 16 + g, r1 = r0 + 8;
      uint32_t f[4] = {0, 0, 0, 0};
      if (r0 < T) {
        f[0] = *reinterpret_cast<const uint32_t*>(ap + (size_t)r0 * a_ld + k);
        f[2] = *reinterpret_cast<const uint32_t*>(ap + (size_t)r0 * a_ld + k + 8);
      }
      if (r1 < T) {
        f[1] = *reinterpret_cast<const uint32_t*>(ap + (size_t)r1 * a_ld + k);
        f[3] = *reinterpret_cast<const uint32_t*>(ap + (size_t)r1 * a_ld + k + 8);
      }
#pragma unroll
      for (int n = 0; n < 2; ++n) mma_bf16_16816(acc[m][n], f, b[n][0], b[n][1]);
    }
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      part[warp][m * 16 + g][n * 8 + c2] = acc[m][n][0];
      part[warp][m * 16 + g][n * 8 + c2 + 1] = acc[m][n][1];
      part[warp][m * 16 + g + 8][n * 8 + c2] = acc[m][n][2];
      part[warp][m * 16 + g + 8][n * 8 + c2 + 1] = acc[m][n][3];
    }
  __syncthreads();
  for (int i = threadIdx.x; i < MT * 16 * 16; i += 128) {
    const int r = i / 16, n = i % 16;
    if (t0 + r < T)
      out[(size_t)(t0 + r) * out_ld + (size_t)h * out_stride + n0 + n] =
          __float2bfloat16_rn(part[0][r][n] + part[1][r][n] + part[2][r][n] + part[3][r][n]);
  }
}

// ------------------------------------------------------------------------------------------------ generic attention
// q [T, H, Rp] (ld = H * Rp), out the same shape. NR * 32 >= Rp.
template <typename T, int NR>
__global__ void __launch_bounds__(128) latent_attend_kernel(const T* __restrict__ q, const T* __restrict__ pool, int Rp,
                                                            const int* __restrict__ page_table, int max_pages, const int* __restrict__ rows,
                                                            const int* __restrict__ tok_seq, const int* __restrict__ tok_pos, int window, float scale,
                                                            T* __restrict__ out, int H) {
  const int lane = threadIdx.x & 31, h = blockIdx.y * 4 + (threadIdx.x >> 5);
  const size_t t = blockIdx.x;
  if (h >= H) return;
  const int pos = tok_pos[t];
  const int* pages = page_table + (size_t)rows[tok_seq[t]] * max_pages;
  const int lo = window > 0 ? max(0, pos - window + 1) : 0;
  float qr[NR], acc[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int d = lane + i * 32;
    qr[i] = d < Rp ? la_ld(q + (t * H + h) * Rp + d) : 0.f;
    acc[i] = 0.f;
  }
  float m = -INFINITY, l = 0.f;
  for (int j0 = lo; j0 <= pos; j0 += 4) {
    float s[4];
    const T* c[4];
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const int j = min(j0 + k, pos);
      c[k] = pool + ((size_t)pages[j / LA_PAGE] * LA_PAGE + j % LA_PAGE) * Rp;
      float a = 0.f;
#pragma unroll
      for (int i = 0; i < NR; ++i) {
        const int d = lane + i * 32;
        if (d < Rp) a = fmaf(qr[i], la_ld(c[k] + d), a);
      }
      s[k] = la_warp_sum(a) * scale;
      if (j0 + k > pos) s[k] = -INFINITY;
    }
    const float mn = fmaxf(m, fmaxf(fmaxf(s[0], s[1]), fmaxf(s[2], s[3])));
    const float al = expf(m - mn);
    m = mn;
    l *= al;
#pragma unroll
    for (int i = 0; i < NR; ++i) acc[i] *= al;
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const float p = expf(s[k] - m);
      l += p;
#pragma unroll
      for (int i = 0; i < NR; ++i) {
        const int d = lane + i * 32;
        if (d < Rp) acc[i] = fmaf(p, la_ld(c[k] + d), acc[i]);
      }
    }
  }
  const float inv = 1.0f / l;
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int d = lane + i * 32;
    if (d < Rp) la_st(out + (t * H + h) * Rp + d, acc[i] * inv);
  }
}

// ------------------------------------------------------------------------------------------------ tensor-core attention
// CTA: token t, heads [16 hb, 16 hb + 16), keys of split z. Four warps. A stage is KT latents (rows padded by 8 elements).
// NT: n8 column tiles of the sum per warp, 4 * 8 * NT >= Rp; warp w owns columns [w * 8 * NT, (w + 1) * 8 * NT).
constexpr int LM_KT = 32;
template <int NT>
__global__ void __launch_bounds__(128) latent_attend_mma_kernel(const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ pool, int Rp,
                                                                const int* __restrict__ page_table, int max_pages, const int* __restrict__ rows,
                                                                const int* __restrict__ tok_seq, const int* __restrict__ tok_pos, int window,
                                                                float scale, __nv_bfloat16* __restrict__ out, float* __restrict__ part, int H,
                                                                int stages) {
  extern __shared__ __align__(16) uint8_t lsm[];
  const int ldr = Rp + 8;                                            // row stride in elements
  __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(lsm);        // [16][ldr]
  __nv_bfloat16* c_s = q_s + 16 * ldr;                               // [stages][LM_KT][ldr]
  __nv_bfloat16* p_s = c_s + (size_t)stages * LM_KT * ldr;           // [16][LM_KT + 8]
  float* mx_s = reinterpret_cast<float*>(p_s + 16 * (LM_KT + 8));    // [4][16]
  float* sum_s = mx_s + 64;                                          // [4][16]
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int hb = blockIdx.y, split = blockIdx.z, splits = gridDim.z;
  const size_t t = blockIdx.x;
  const int pos = tok_pos[t];
  const int* pages = page_table + (size_t)rows[tok_seq[t]] * max_pages;
  const int lo_all = window > 0 ? max(0, pos - window + 1) : 0;
  // whole pages per split, counted from the page of the first visible key
  const int page_lo = lo_all / LA_PAGE, n_pages = pos / LA_PAGE + 1 - page_lo;
  const int per = (n_pages + splits - 1) / splits;
  const int j_begin = (page_lo + split * per) * LA_PAGE;
  const int j_end = min((page_lo + min((split + 1) * per, n_pages)) * LA_PAGE, pos + 1);
  const int n_tiles = j_end > j_begin ? (j_end - j_begin + LM_KT - 1) / LM_KT : 0;
  const int chunks = Rp / 8;                                         // 16-byte pieces of a row
  for (int i = tid; i < 16 * chunks; i += 128) {
    const int r = i / chunks, c = i % chunks, h = hb * 16 + r;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (h < H) v = *reinterpret_cast<const uint4*>(q + (t * H + h) * (size_t)Rp + c * 8);
    *reinterpret_cast<uint4*>(q_s + r * ldr + c * 8) = v;
  }
  auto stage = [&](int tile) {
    __nv_bfloat16* dst = c_s + (size_t)(tile % stages) * LM_KT * ldr;
    const int j0 = j_begin + tile * LM_KT;
    for (int i = tid; i < LM_KT * chunks; i += 128) {
      const int r = i / chunks, c = i % chunks, j = min(j0 + r, j_end - 1);  // rows past the end repeat the last key: finite, masked
      const __nv_bfloat16* src = pool + ((size_t)pages[j / LA_PAGE] * LA_PAGE + j % LA_PAGE) * Rp + c * 8;
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst + r * ldr + c * 8)), "l"(src) : "memory");
    }
  };
  for (int i = 0; i < stages - 1; ++i) {
    if (i < n_tiles) stage(i);
    asm volatile("cp.async.commit_group;" ::: "memory");
  }
  float acc[NT][4];
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int i = 0; i < 4; ++i) acc[n][i] = 0.f;
  const int g = lane >> 2, c2 = (lane & 3) * 2;
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;          // rows g and g + 8 (identical in all warps)
  const float cs = scale * 1.4426950408889634f;
  for (int tile = 0; tile < n_tiles; ++tile) {
    if (stages == 3) asm volatile("cp.async.wait_group 1;" ::: "memory");
    else asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();  // the tile has landed for every thread, and the slot refilled below is no longer read
    if (tile + stages - 1 < n_tiles) stage(tile + stages - 1);
    asm volatile("cp.async.commit_group;" ::: "memory");
    const __nv_bfloat16* c = c_s + (size_t)(tile % stages) * LM_KT * ldr;
    // scores of this warp's 8 keys
    float s[4] = {0.f, 0.f, 0.f, 0.f}, s2[4] = {0.f, 0.f, 0.f, 0.f};
    const __nv_bfloat16* qa = q_s + (lane & 15) * ldr + (lane >> 4) * 8;
    const __nv_bfloat16* cb = c + (warp * 8 + (lane & 7)) * ldr + ((lane >> 3) & 1) * 8;
    int k = 0;
    for (; k + 32 <= Rp; k += 32) {
      uint32_t a[4], b[2], a2[4], b2[2];
      ldsm_x4(a, qa + k);
      ldsm_x2(b, cb + k);
      ldsm_x4(a2, qa + k + 16);
      ldsm_x2(b2, cb + k + 16);
      mma_bf16_16816(s, a, b[0], b[1]);
      mma_bf16_16816(s2, a2, b2[0], b2[1]);
    }
    if (k < Rp) {
      uint32_t a[4], b[2];
      ldsm_x4(a, qa + k);
      ldsm_x2(b, cb + k);
      mma_bf16_16816(s, a, b[0], b[1]);
    }
    const int j = j_begin + tile * LM_KT + warp * 8 + c2;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int jj = j + (i & 1);
      s[i] = (jj >= lo_all && jj < j_end) ? (s[i] + s2[i]) * cs : -INFINITY;
    }
    float a0 = fmaxf(s[0], s[1]), a1 = fmaxf(s[2], s[3]);
    a0 = fmaxf(a0, __shfl_xor_sync(0xffffffffu, a0, 1));
    a1 = fmaxf(a1, __shfl_xor_sync(0xffffffffu, a1, 1));
    a0 = fmaxf(a0, __shfl_xor_sync(0xffffffffu, a0, 2));
    a1 = fmaxf(a1, __shfl_xor_sync(0xffffffffu, a1, 2));
    if ((lane & 3) == 0) {
      mx_s[warp * 16 + g] = a0;
      mx_s[warp * 16 + g + 8] = a1;
    }
    __syncthreads();
    a0 = fmaxf(fmaxf(mx_s[g], mx_s[16 + g]), fmaxf(mx_s[32 + g], mx_s[48 + g]));
    a1 = fmaxf(fmaxf(mx_s[g + 8], mx_s[24 + g]), fmaxf(mx_s[40 + g], mx_s[56 + g]));
    const float n0 = fmaxf(m0, a0), n1 = fmaxf(m1, a1);
    const float b0 = n0 == -INFINITY ? 0.f : n0, b1 = n1 == -INFINITY ? 0.f : n1;  // no visible key yet: all weights are 0
    const float al0 = exp2f(m0 - b0), al1 = exp2f(m1 - b1);
    m0 = n0;
    m1 = n1;
    const float e0 = exp2f(s[0] - b0), e1 = exp2f(s[1] - b0), e2 = exp2f(s[2] - b1), e3 = exp2f(s[3] - b1);
    l0 = l0 * al0 + (e0 + e1);  // this thread's share; folded over the row at the end
    l1 = l1 * al1 + (e2 + e3);
    *reinterpret_cast<uint32_t*>(p_s + g * (LM_KT + 8) + warp * 8 + c2) = pack_bf16x2(e0, e1);
    *reinterpret_cast<uint32_t*>(p_s + (g + 8) * (LM_KT + 8) + warp * 8 + c2) = pack_bf16x2(e2, e3);
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      acc[n][0] *= al0; acc[n][1] *= al0; acc[n][2] *= al1; acc[n][3] *= al1;
    }
    __syncthreads();
#pragma unroll
    for (int ks = 0; ks < LM_KT / 16; ++ks) {
      uint32_t a[4];
      ldsm_x4(a, p_s + (lane & 15) * (LM_KT + 8) + ks * 16 + (lane >> 4) * 8);
      const __nv_bfloat16* vb = c + (ks * 16 + (lane & 15)) * ldr + warp * 8 * NT;
#pragma unroll
      for (int n = 0; n < NT; ++n)
        if ((warp * NT + n) * 8 < Rp) {
          uint32_t b[2];
          ldsm_x2_t(b, vb + n * 8);
          mma_bf16_16816(acc[n], a, b[0], b[1]);
        }
    }
  }
  l0 += __shfl_xor_sync(0xffffffffu, l0, 1);
  l1 += __shfl_xor_sync(0xffffffffu, l1, 1);
  l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
  l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
  if ((lane & 3) == 0) {
    sum_s[warp * 16 + g] = l0;
    sum_s[warp * 16 + g + 8] = l1;
  }
  __syncthreads();
  l0 = sum_s[g] + sum_s[16 + g] + sum_s[32 + g] + sum_s[48 + g];
  l1 = sum_s[g + 8] + sum_s[24 + g] + sum_s[40 + g] + sum_s[56 + g];
#pragma unroll
  for (int rr = 0; rr < 2; ++rr) {
    const int h = hb * 16 + g + rr * 8;
    if (h >= H) continue;
    const float l = rr ? l1 : l0, m = rr ? m1 : m0;
    if (splits == 1) {
      const float inv = 1.0f / l;
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        const int col = (warp * NT + n) * 8 + c2;
        if (col < Rp)
          *reinterpret_cast<uint32_t*>(out + (t * H + h) * (size_t)Rp + col) = pack_bf16x2(acc[n][rr * 2] * inv, acc[n][rr * 2 + 1] * inv);
      }
    } else {
      float* dst = part + ((t * H + h) * splits + split) * (size_t)(Rp + 2);
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        const int col = (warp * NT + n) * 8 + c2;
        if (col < Rp) *reinterpret_cast<float2*>(dst + col) = make_float2(acc[n][rr * 2], acc[n][rr * 2 + 1]);
      }
      if (warp == 0 && (lane & 3) == 0) {
        dst[Rp] = m;
        dst[Rp + 1] = l;
      }
    }
  }
}

constexpr int LA_MAX_SPLITS = 32;
__global__ void __launch_bounds__(128) latent_combine_kernel(const float* __restrict__ part, __nv_bfloat16* __restrict__ out, int Rp, int splits) {
  __shared__ float wt[LA_MAX_SPLITS];
  const size_t th = blockIdx.x;
  const float* p = part + th * splits * (size_t)(Rp + 2);
  if (threadIdx.x < 32) {
    const bool in = (int)threadIdx.x < splits;
    const float m = in ? p[(size_t)threadIdx.x * (Rp + 2) + Rp] : -INFINITY, l = in ? p[(size_t)threadIdx.x * (Rp + 2) + Rp + 1] : 0.f;
    float mx = m;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    const float e = exp2f(m - mx);
    wt[threadIdx.x] = e / la_warp_sum(l * e);
  }
  __syncthreads();
  for (int c = threadIdx.x; c < Rp; c += 128) {
    float a = 0.f;
#pragma unroll 8
    for (int i = 0; i < splits; ++i) a = fmaf(p[(size_t)i * (Rp + 2) + c], wt[i], a);
    out[th * Rp + c] = __float2bfloat16_rn(a);
  }
}

template <typename TI, typename TC>
static void launch_prep(const void* in, int in_ld, int off_c, int R, int Rp, const float* w, float eps, void* pool, const int* page_table,
                        int max_pages, const int* rows, const int* tok_seq, const int* tok_pos, void* c_out, int c_ld, int nq, void* q_out, int q_ld,
                        int T, cudaStream_t st) {
  latent_prep_kernel<TI, TC><<<T, 128, 0, st>>>((const TI*)in, in_ld, off_c, R, Rp, w, eps, (TC*)pool, page_table, max_pages, rows, tok_seq, tok_pos,
                                                (TC*)c_out, c_ld, nq, (TC*)q_out, q_ld);
}

template <typename T>
static int launch_attend(const void* q, const void* pool, int Rp, const int* page_table, int max_pages, const int* rows, const int* tok_seq,
                         const int* tok_pos, int window, float scale, void* out, int n_tok, int H, cudaStream_t st) {
  const dim3 grid(n_tok, (H + 3) / 4);
#define INV_LA(NR)                                                                                                                              \
  latent_attend_kernel<T, NR><<<grid, 128, 0, st>>>((const T*)q, (const T*)pool, Rp, page_table, max_pages, rows, tok_seq, tok_pos, window, scale, \
                                                    (T*)out, H)
  if (Rp <= 64) INV_LA(2);
  else if (Rp <= 128) INV_LA(4);
  else if (Rp <= 256) INV_LA(8);
  else if (Rp <= 512) INV_LA(16);
  else if (Rp <= 1024) INV_LA(32);
  else return -ERR_BAD_ARG;
#undef INV_LA
  return 0;
}

template <int NT>
static int launch_mma(const void* q, const void* pool, int Rp, const int* page_table, int max_pages, const int* rows, const int* tok_seq,
                      const int* tok_pos, int window, float scale, void* out, float* part, int splits, int n_tok, int H, cudaStream_t st) {
  const int ldr = Rp + 8;
  auto bytes = [&](int stages) { return (16 * ldr + stages * LM_KT * ldr + 16 * (LM_KT + 8)) * 2 + 128 * 4; };
  const int stages = bytes(3) <= 113 * 1024 ? 3 : 2;
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(latent_attend_mma_kernel<NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e != cudaSuccess) return -(int)e;
    configured = true;
  }
  latent_attend_mma_kernel<NT><<<dim3(n_tok, (H + 15) / 16, splits), 128, bytes(stages), st>>>(
      (const __nv_bfloat16*)q, (const __nv_bfloat16*)pool, Rp, page_table, max_pages, rows, tok_seq, tok_pos, window, scale, (__nv_bfloat16*)out, part, H,
      stages);
  return 0;
}

}  // namespace inv

using namespace inv;

// in_f32 / c_f32: types of the projection rows and of the pages (and copies); bf16 rows need bf16 pages.
extern "C" int inv_latent_prep(const void* in, int in_ld, int in_f32, int off_c, int R, int Rp, const float* w, float eps, void* pool, int c_f32,
                               const int* page_table, int max_pages, const int* rows, const int* tok_seq, const int* tok_pos, void* c_out, int c_ld,
                               int nq, void* q_out, int q_ld, int T, void* stream) {
  if (R < 1 || Rp < R) return -ERR_BAD_ARG;
  if (T <= 0) return 0;
  cudaStream_t st = (cudaStream_t)stream;
#define INV_LP(TI, TC) \
  launch_prep<TI, TC>(in, in_ld, off_c, R, Rp, w, eps, pool, page_table, max_pages, rows, tok_seq, tok_pos, c_out, c_ld, nq, q_out, q_ld, T, st)
  if (in_f32 && c_f32) INV_LP(float, float);
  else if (in_f32) INV_LP(float, __nv_bfloat16);
  else if (!c_f32) INV_LP(__nv_bfloat16, __nv_bfloat16);
  else return -ERR_BAD_ARG;
#undef INV_LP
  const cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}

extern "C" int inv_head_proj(const void* a, int a_ld, int a_stride, const void* W, int H, int N, int K, void* out, int out_ld, int out_stride, int T,
                             void* stream) {
  if (N % 16 || K % 16 || a_ld % 2 || a_stride % 2) return -ERR_BAD_ARG;
  if (T <= 0) return 0;
  cudaStream_t st = (cudaStream_t)stream;
#define INV_HP(MT)                                                                                                                                    \
  head_proj_kernel<MT><<<dim3(N / 16, H, (T + MT * 16 - 1) / (MT * 16)), 128, 0, st>>>((const __nv_bfloat16*)a, a_ld, a_stride, (const __nv_bfloat16*)W, \
                                                                                      N, K, (__nv_bfloat16*)out, out_ld, out_stride, T)
  if (T <= 16) INV_HP(1);
  else if (T <= 32) INV_HP(2);
  else INV_HP(4);
#undef INV_HP
  const cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}

// Attention of T query rows over the pages. fp32: the warp-per-head kernel. bf16: the tensor-core kernel, with `part`
// (fp32 [T, H, splits, Rp + 2]) when splits > 1; Rp % 16 == 0.
extern "C" int inv_latent_attend(const void* q, const void* pool, int f32, int Rp, const int* page_table, int max_pages, const int* rows,
                                 const int* tok_seq, const int* tok_pos, int window, float scale, void* out, float* part, int splits, int T, int H,
                                 void* stream) {
  if (T <= 0) return 0;
  cudaStream_t st = (cudaStream_t)stream;
  int rc;
  if (f32) {
    rc = launch_attend<float>(q, pool, Rp, page_table, max_pages, rows, tok_seq, tok_pos, window, scale, out, T, H, st);
  } else {
    if (Rp % 16 || splits < 1 || splits > LA_MAX_SPLITS || (splits > 1 && !part)) return -ERR_BAD_ARG;
#define INV_LM(NT) launch_mma<NT>(q, pool, Rp, page_table, max_pages, rows, tok_seq, tok_pos, window, scale, out, part, splits, T, H, st)
    if (Rp <= 64) rc = INV_LM(2);
    else if (Rp <= 128) rc = INV_LM(4);
    else if (Rp <= 256) rc = INV_LM(8);
    else if (Rp <= 512) rc = INV_LM(16);
    else if (Rp <= 1024) rc = INV_LM(32);
    else return -ERR_BAD_ARG;
#undef INV_LM
    if (!rc && splits > 1) latent_combine_kernel<<<T * H, 128, 0, st>>>(part, (__nv_bfloat16*)out, Rp, splits);
  }
  if (rc) return rc;
  const cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}
