// Hyper-connections: a residual made of S parallel streams, and the step between two sublayers in one kernel.
//
// Per token the residual is S rows of E floats (fp32, [T, S, E]). A sublayer with output y updates every stream from
// the old ones, x_t <- sum_s mix[s, t] x_s + out[t] y, and the next sublayer reads LayerNorm(sum_s in[s] x_s). One launch
// does: (first call of a step) embedding lookup and scaling into the streams, or the update with y; then the weighted
// sum, the LayerNorm, and the cast to the projections' type. A plain pre-norm residual is S = 1 with unit weights.
//
// One CTA per token; the row lives in registers (streams) and shared memory (the weighted sum), so the streams are read
// once and written once: 2 S E 4 bytes per token, the bound of this kernel.
#include "sm100_common.cuh"
#include "inv_api.h"

namespace inv {

constexpr int HC_MAX_STREAMS = 16;
constexpr int HC_MAX_WIDTH = 11776;  // the weighted sum of a row stays in 46 KB of shared memory

struct HyperParams {
  float* x;                 // [T, S, E]
  const int* ids;           // embedding rows (start of a step), or null
  const void* table;        // [V, table_ld], type of h
  int table_ld;
  float scale;
  const void* y;            // [T, y_ld] sublayer output, or null
  int y_ld;
  const float* mix;         // [S, S], index [from, to]
  const float* out_w;       // [S]
  const float* in_w;        // [S]; null: no normed output is wanted
  const float* norm_w;      // [E]
  const float* norm_b;      // [E]
  float eps;
  void* h;                  // [grid, h_ld]
  int h_ld;
  const int* rows;          // token of each output row, or null (identity)
  int write_x;
  int S, E;
};

template <typename T, int V> struct Vec;
template <> struct Vec<float, 1> {
  static __device__ __forceinline__ void ld(const void* p, size_t i, float* f) { f[0] = static_cast<const float*>(p)[i]; }
  static __device__ __forceinline__ void st(void* p, size_t i, const float* f) { static_cast<float*>(p)[i] = f[0]; }
};
template <> struct Vec<float, 4> {
  static __device__ __forceinline__ void ld(const void* p, size_t i, float* f) {
    const float4 v = *reinterpret_cast<const float4*>(static_cast<const float*>(p) + i);
    f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
  }
  static __device__ __forceinline__ void st(void* p, size_t i, const float* f) {
    *reinterpret_cast<float4*>(static_cast<float*>(p) + i) = make_float4(f[0], f[1], f[2], f[3]);
  }
};
template <> struct Vec<__nv_bfloat16, 1> {
  static __device__ __forceinline__ void ld(const void* p, size_t i, float* f) { f[0] = __bfloat162float(static_cast<const __nv_bfloat16*>(p)[i]); }
  static __device__ __forceinline__ void st(void* p, size_t i, const float* f) { static_cast<__nv_bfloat16*>(p)[i] = __float2bfloat16_rn(f[0]); }
};
template <> struct Vec<__nv_bfloat16, 4> {
  static __device__ __forceinline__ void ld(const void* p, size_t i, float* f) {
    const uint2 v = *reinterpret_cast<const uint2*>(static_cast<const __nv_bfloat16*>(p) + i);
    f[0] = __uint_as_float(v.x << 16); f[1] = __uint_as_float(v.x & 0xffff0000u);
    f[2] = __uint_as_float(v.y << 16); f[3] = __uint_as_float(v.y & 0xffff0000u);
  }
  static __device__ __forceinline__ void st(void* p, size_t i, const float* f) {
    *reinterpret_cast<uint2*>(static_cast<__nv_bfloat16*>(p) + i) = make_uint2(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]));
  }
};

__device__ __forceinline__ float hc_block_sum(float v, float* red) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  __syncthreads();  // red may still be read from the previous reduction
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
  for (int i = 0; i < (int)(blockDim.x >> 5); ++i) t += red[i];
  return t;
}

// NS: number of streams at compile time, 0 = read from the parameters.
template <int NS, typename YT, typename HT, int V>
__global__ void __launch_bounds__(NS > 0 ? 512 : 256) hyper_step_kernel(const HyperParams p) {
  extern __shared__ float hc_u[];  // [E]
  __shared__ float red[16];
  __shared__ float s_mix[HC_MAX_STREAMS * HC_MAX_STREAMS], s_out[HC_MAX_STREAMS], s_in[HC_MAX_STREAMS];
  constexpr int CAP = NS > 0 ? NS : HC_MAX_STREAMS;
  const int S = NS > 0 ? NS : p.S;
  const int E = p.E, tid = threadIdx.x;
  const size_t row = p.rows ? (size_t)p.rows[blockIdx.x] : (size_t)blockIdx.x;
  if (p.y)
    for (int i = tid; i < S * S; i += blockDim.x) s_mix[i] = p.mix[i];
  if (tid < S) {
    if (p.y) s_out[tid] = p.out_w[tid];
    if (p.in_w) s_in[tid] = p.in_w[tid];
  }
  __syncthreads();
  float* x = p.x + row * (size_t)S * E;
  const size_t tok = p.ids ? (size_t)p.ids[row] * p.table_ld : 0;
  float sum = 0.f;
  for (int e = tid * V; e < E; e += blockDim.x * V) {
    float xs[CAP][V];
    if (p.ids) {
      float t[V];
      Vec<HT, V>::ld(p.table, tok + e, t);
#pragma unroll
      for (int s = 0; s < CAP; ++s)
        if (s < S)
#pragma unroll
          for (int j = 0; j < V; ++j) xs[s][j] = t[j] * p.scale;
    } else {
#pragma unroll
      for (int s = 0; s < CAP; ++s)
        if (s < S) Vec<float, V>::ld(x, (size_t)s * E + e, xs[s]);
    }
    if (p.y) {
      float y[V], nx[CAP][V];
      Vec<YT, V>::ld(p.y, row * (size_t)p.y_ld + e, y);
#pragma unroll
      for (int t = 0; t < CAP; ++t)
        if (t < S)
#pragma unroll
          for (int j = 0; j < V; ++j) {
            float a = s_out[t] * y[j];
#pragma unroll
            for (int s = 0; s < CAP; ++s)
              if (s < S) a = fmaf(s_mix[s * S + t], xs[s][j], a);
            nx[t][j] = a;
          }
#pragma unroll
      for (int t = 0; t < CAP; ++t)
        if (t < S)
#pragma unroll
          for (int j = 0; j < V; ++j) xs[t][j] = nx[t][j];
    }
    if (p.write_x)
#pragma unroll
      for (int s = 0; s < CAP; ++s)
        if (s < S) Vec<float, V>::st(x, (size_t)s * E + e, xs[s]);
    if (p.in_w) {
      float u[V];
#pragma unroll
      for (int j = 0; j < V; ++j) {
        float a = 0.f;
#pragma unroll
        for (int s = 0; s < CAP; ++s)
          if (s < S) a = fmaf(s_in[s], xs[s][j], a);
        u[j] = a;
        sum += a;
      }
      Vec<float, V>::st(hc_u, e, u);
    }
  }
  if (!p.in_w) return;
  const float mean = hc_block_sum(sum, red) / (float)E;
  float sq = 0.f;
  for (int e = tid * V; e < E; e += blockDim.x * V) {  // each thread re-reads what it wrote
    float u[V];
    Vec<float, V>::ld(hc_u, e, u);
#pragma unroll
    for (int j = 0; j < V; ++j) {
      const float d = u[j] - mean;
      sq = fmaf(d, d, sq);
    }
  }
  const float rstd = 1.0f / sqrtf(hc_block_sum(sq, red) / (float)E + p.eps);
  for (int e = tid * V; e < E; e += blockDim.x * V) {
    float u[V], w[V], b[V];
    Vec<float, V>::ld(hc_u, e, u);
    Vec<float, V>::ld(p.norm_w, e, w);
    Vec<float, V>::ld(p.norm_b, e, b);
#pragma unroll
    for (int j = 0; j < V; ++j) u[j] = fmaf((u[j] - mean) * rstd, w[j], b[j]);
    Vec<HT, V>::st(p.h, (size_t)blockIdx.x * p.h_ld + e, u);
  }
}

template <typename YT, typename HT, int V>
static int hyper_launch(const HyperParams& p, int n, cudaStream_t st) {
  int threads = ((p.E + V - 1) / V + 31) / 32 * 32;
  const int cap = n <= 148 ? 512 : 256;  // few rows: one pass over a row, its latency is all there is
  if (threads > cap) threads = cap;
  const size_t smem = (size_t)p.E * 4;
  switch (p.S) {
    case 1: hyper_step_kernel<1, YT, HT, V><<<n, threads, smem, st>>>(p); break;
    case 2: hyper_step_kernel<2, YT, HT, V><<<n, threads, smem, st>>>(p); break;
    case 3: hyper_step_kernel<3, YT, HT, V><<<n, threads, smem, st>>>(p); break;
    case 4: hyper_step_kernel<4, YT, HT, V><<<n, threads, smem, st>>>(p); break;
    default: hyper_step_kernel<0, YT, HT, 1><<<n, 256, smem, st>>>(p); break;  // many streams: one element per thread keeps them in registers
  }
  const cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}

// silu(gate) * up over [T, 2 F] rows (gate columns first, `half` columns each), fp32 in.
template <typename OT>
__global__ void __launch_bounds__(256) gated_silu_kernel(const float* __restrict__ in, int in_ld, int half, OT* __restrict__ out, int out_ld, int F) {
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= F) return;
  const float* r = in + (size_t)blockIdx.x * in_ld;
  const float g = r[c], v = g / (1.0f + expf(-g)) * r[half + c];
  Vec<OT, 1>::st(out, (size_t)blockIdx.x * out_ld + c, &v);
}

}  // namespace inv

using namespace inv;

// Types: y_f32 / h_f32 say whether y and h (and the embedding table) are fp32, otherwise bf16 (h fp32 needs y fp32).
extern "C" int inv_hyper_step(float* x, const int* ids, const void* table, int table_ld, float scale, const void* y, int y_ld, int y_f32,
                              const float* mix, const float* out_w, const float* in_w, const float* norm_w, const float* norm_b,
                              float eps, void* h, int h_ld, int h_f32, const int* rows, int n, int write_x, int S, int E, void* stream) {
  if (S < 1 || S > HC_MAX_STREAMS || E < 1 || E > HC_MAX_WIDTH) return -ERR_BAD_ARG;
  if (h_f32 && !y_f32) return -ERR_BAD_ARG;
  if (n <= 0) return 0;
  HyperParams p{x, ids, table, table_ld, scale, y, y_ld, mix, out_w, in_w, norm_w, norm_b, eps, h, h_ld, rows, write_x, S, E};
  cudaStream_t st = (cudaStream_t)stream;
  const bool vec = E % 4 == 0 && (!y || y_ld % 4 == 0) && (!in_w || h_ld % 4 == 0) && (!ids || table_ld % 4 == 0);
  if (h_f32) return vec ? hyper_launch<float, float, 4>(p, n, st) : hyper_launch<float, float, 1>(p, n, st);
  if (y_f32) return vec ? hyper_launch<float, __nv_bfloat16, 4>(p, n, st) : hyper_launch<float, __nv_bfloat16, 1>(p, n, st);
  return vec ? hyper_launch<__nv_bfloat16, __nv_bfloat16, 4>(p, n, st) : hyper_launch<__nv_bfloat16, __nv_bfloat16, 1>(p, n, st);
}

extern "C" int inv_gated_silu_f32(const float* in, int in_ld, int half, void* out, int out_ld, int out_f32, int T, int F, void* stream) {
  if (T <= 0 || F <= 0) return 0;
  const dim3 grid(T, (F + 255) / 256);
  if (out_f32) gated_silu_kernel<float><<<grid, 256, 0, (cudaStream_t)stream>>>(in, in_ld, half, (float*)out, out_ld, F);
  else gated_silu_kernel<__nv_bfloat16><<<grid, 256, 0, (cudaStream_t)stream>>>(in, in_ld, half, (__nv_bfloat16*)out, out_ld, F);
  const cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}
