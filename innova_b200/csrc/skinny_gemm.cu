// Projections of decode steps: out[M, N] = x[M, K] W[N, K]^T for M <= 64 rows, bf16 in, fp32 accumulation.
//
// Such a product reads every weight once and does almost no arithmetic, so it is bound by weight bytes and, for the sizes of
// one layer, by latency: the kernel is launched wide and keeps many 16-byte weight loads in flight per thread. A CTA owns
// NT * 8 columns; its eight warps take every eighth 32-wide slice of K and meet in shared memory. Weights and activations go
// straight from global memory into warp-level MMA fragments: a lane loads eight consecutive k of a row and both operands read
// them in the same permuted order, which a dot product does not notice. (A 128-row tcgen05 tile would be mostly padding here,
// and its tensor-memory set-up and drain cost more than the whole product.)
//
// SILU: W holds gate rows [0, N) and up rows [half, half + N); the output is silu(gate) * up.
// cap > 0 (plain form): the output is cap * tanh(out / cap), the soft limit of logits.
#include "sm100_common.cuh"
#include "inv_api.h"

namespace inv {

constexpr int SG_WARPS = 8, SG_THREADS = 32 * SG_WARPS;

__device__ __forceinline__ void sg_mma(float* d, uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint4 sg_load_stream(const __nv_bfloat16* p) {  // weights: used once, keep them out of L1
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0, %1, %2, %3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
  return v;
}
// Eight values of a row of which only the first `n` exist (n <= 0: none); used for the last slice of K.
__device__ __forceinline__ uint4 sg_mask(uint4 v, int n) {
  uint32_t u[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
  for (int j = 0; j < 4; ++j) u[j] = n >= 2 * j + 2 ? u[j] : n == 2 * j + 1 ? (u[j] & 0xffffu) : 0u;
  return make_uint4(u[0], u[1], u[2], u[3]);
}

// MT: 16-row tiles of x; NT: 8-column tiles of the CTA (gate tiles when SILU, with as many up tiles behind them).
template <int MT, int NT, bool SILU>
__global__ void __launch_bounds__(SG_THREADS) skinny_gemm_kernel(const __nv_bfloat16* __restrict__ x, int ldx, const __nv_bfloat16* __restrict__ W, int ldw,
                                                                 int M, int N, int K, int half, void* __restrict__ out, int ldo, int out_f32, float cap) {
  constexpr int WT = SILU ? 2 * NT : NT;     // weight tiles
  extern __shared__ float sg_part[];         // [SG_WARPS][MT * 16][WT * 8 + 4]
  constexpr int PL = WT * 8 + 4;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tig = lane & 3;
  const int n0 = blockIdx.x * NT * 8;
  const __nv_bfloat16* wp[WT];
#pragma unroll
  for (int t = 0; t < WT; ++t) {
    const int col = n0 + (t % NT) * 8 + g;   // columns past N read the last row and are not stored
    wp[t] = W + (size_t)(min(col, N - 1) + (t >= NT ? half : 0)) * ldw + tig * 8;
  }
  const __nv_bfloat16* xp[2 * MT];
#pragma unroll
  for (int m = 0; m < 2 * MT; ++m) xp[m] = x + (size_t)min(m * 8 + g, M - 1) * ldx + tig * 8;
  float acc[MT][WT][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int t = 0; t < WT; ++t)
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[m][t][i] = 0.f;
  auto step = [&](const uint4* w, const uint4* a) {
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int t = 0; t < WT; ++t) {
        sg_mma(acc[m][t], a[2 * m].x, a[2 * m + 1].x, a[2 * m].y, a[2 * m + 1].y, w[t].x, w[t].y);
        sg_mma(acc[m][t], a[2 * m].z, a[2 * m + 1].z, a[2 * m].w, a[2 * m + 1].w, w[t].z, w[t].w);
      }
  };
  const int full = K / 32;
  constexpr int UN = WT <= 2 ? 4 : 2;        // slices whose weights are in flight together
  int s = warp;
  for (; s + (UN - 1) * SG_WARPS < full; s += UN * SG_WARPS) {
    uint4 w[UN][WT];
#pragma unroll
    for (int u = 0; u < UN; ++u)
#pragma unroll
      for (int t = 0; t < WT; ++t) w[u][t] = sg_load_stream(wp[t] + (s + u * SG_WARPS) * 32);
#pragma unroll
    for (int u = 0; u < UN; ++u) {
      uint4 a[2 * MT];
#pragma unroll
      for (int m = 0; m < 2 * MT; ++m) a[m] = *reinterpret_cast<const uint4*>(xp[m] + (s + u * SG_WARPS) * 32);
      step(w[u], a);
    }
  }
  for (; s * 32 < K; s += SG_WARPS) {        // the rest, the last slice possibly short
    const int left = K - s * 32 - tig * 8;   // elements of this lane's eight that exist
    uint4 w[WT], a[2 * MT];
#pragma unroll
    for (int t = 0; t < WT; ++t) w[t] = left > 0 ? sg_load_stream(wp[t] + s * 32) : make_uint4(0, 0, 0, 0);
#pragma unroll
    for (int m = 0; m < 2 * MT; ++m) a[m] = left > 0 ? *reinterpret_cast<const uint4*>(xp[m] + s * 32) : make_uint4(0, 0, 0, 0);
    if (left < 8) {
#pragma unroll
      for (int t = 0; t < WT; ++t) w[t] = sg_mask(w[t], left);
#pragma unroll
      for (int m = 0; m < 2 * MT; ++m) a[m] = sg_mask(a[m], left);
    }
    step(w, a);
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int t = 0; t < WT; ++t) {
      float* p = sg_part + (size_t)(warp * MT * 16 + m * 16 + g) * PL + t * 8 + 2 * tig;
      *reinterpret_cast<float2*>(p) = make_float2(acc[m][t][0], acc[m][t][1]);
      *reinterpret_cast<float2*>(p + 8 * PL) = make_float2(acc[m][t][2], acc[m][t][3]);
    }
  __syncthreads();
  for (int i = tid; i < MT * 16 * NT * 8; i += SG_THREADS) {
    const int r = i / (NT * 8), c = i % (NT * 8);
    if (r >= M || n0 + c >= N) continue;
    float a = 0.f, b = 0.f;
#pragma unroll
    for (int w = 0; w < SG_WARPS; ++w) {
      a += sg_part[(size_t)(w * MT * 16 + r) * PL + c];
      if (SILU) b += sg_part[(size_t)(w * MT * 16 + r) * PL + NT * 8 + c];
    }
    if (SILU) a = a / (1.0f + expf(-a)) * b;
    else if (cap > 0.f) a = cap * tanhf(a / cap);
    if (out_f32) static_cast<float*>(out)[(size_t)r * ldo + n0 + c] = a;
    else static_cast<__nv_bfloat16*>(out)[(size_t)r * ldo + n0 + c] = __float2bfloat16_rn(a);
  }
}

template <int MT, int NT, bool SILU>
static int launch_skinny(const void* x, int ldx, const void* W, int ldw, int M, int N, int K, int half, void* out, int ldo, int out_f32, float cap,
                         cudaStream_t st) {
  constexpr int bytes = SG_WARPS * MT * 16 * ((SILU ? 2 : 1) * NT * 8 + 4) * 4;
  static bool configured = false;
  if (!configured && bytes > 48 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(skinny_gemm_kernel<MT, NT, SILU>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
    if (e != cudaSuccess) return -(int)e;
  }
  configured = true;
  skinny_gemm_kernel<MT, NT, SILU><<<(N + NT * 8 - 1) / (NT * 8), SG_THREADS, bytes, st>>>((const __nv_bfloat16*)x, ldx, (const __nv_bfloat16*)W, ldw, M, N,
                                                                                        K, half, out, ldo, out_f32, cap);
  const cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}

}  // namespace inv

using namespace inv;

// ldx and ldw are multiples of 8 and at least K rounded up to 8; M <= 64. silu_half > 0: the gated form above.
extern "C" int inv_skinny_gemm(const void* x, int ldx, const void* W, int ldw, int M, int N, int K, int silu_half, void* out, int ldo, int out_f32,
                               float cap, void* stream) {
  const int k8 = (K + 7) & ~7;
  if (M > 64 || (ldx % 8) || (ldw % 8) || ldx < k8 || ldw < k8 || (reinterpret_cast<uintptr_t>(x) & 15) || (reinterpret_cast<uintptr_t>(W) & 15))
    return -ERR_BAD_ARG;
  if (M <= 0 || N <= 0 || K <= 0) return 0;
  cudaStream_t st = (cudaStream_t)stream;
  const bool wide = N > 148 * 2 * 16;   // enough columns to fill the GPU with 32-column CTAs
#define INV_SG(MT)                                                                                                                          \
  (silu_half > 0 ? launch_skinny<MT, 2, true>(x, ldx, W, ldw, M, N, K, silu_half, out, ldo, out_f32, cap, st)                                   \
   : wide        ? launch_skinny<MT, 4, false>(x, ldx, W, ldw, M, N, K, 0, out, ldo, out_f32, cap, st)                                          \
                 : launch_skinny<MT, 2, false>(x, ldx, W, ldw, M, N, K, 0, out, ldo, out_f32, cap, st))
  if (M <= 16) return INV_SG(1);
  if (M <= 32) return INV_SG(2);
  return INV_SG(4);
#undef INV_SG
}
