// Residual with a norm on both sides of every sublayer, in one kernel between two sublayers.
//
// The residual is one fp32 row per token. A sublayer's output y enters as x <- x + RMSNorm(y) and the next sublayer reads
// RMSNorm(x) in the projections' type; a norm multiplies by (offset + weight), so weights may be stored around one (offset 0) or
// around zero (offset 1). A step starts with the embedding rows instead of an output. One CTA per token, the row in registers: x is
// read once and written once, 4 E + 4 E + 2 E (y) + 2 E (h) bytes per token in bf16, the bound of this kernel.
#include "sm100_common.cuh"
#include "inv_api.h"

namespace inv {

struct SandwichParams {
  float* x;              // [T, E]
  const int* ids;        // embedding rows (start of a step), or null
  const void* table;     // [V, table_ld], type of h
  int table_ld;
  float scale;
  const void* y;         // [T, y_ld] sublayer output, or null
  int y_ld;
  const float* post_w;   // [E] norm of y, or null: y enters as it is
  const float* norm_w;   // [E] norm of x, or null: no normed output is wanted
  float offset, eps;
  void* h;               // [grid, h_ld]
  int h_ld;
  const int* rows;       // token of each output row, or null (identity)
  int write_x;
  int E;
};

template <typename T> struct Four;
template <> struct Four<float> {
  static __device__ __forceinline__ float4 ld(const void* p, size_t i) { return *reinterpret_cast<const float4*>(static_cast<const float*>(p) + i); }
  static __device__ __forceinline__ void st(void* p, size_t i, float4 v) { *reinterpret_cast<float4*>(static_cast<float*>(p) + i) = v; }
  static __device__ __forceinline__ float ld1(const void* p, size_t i) { return static_cast<const float*>(p)[i]; }
  static __device__ __forceinline__ void st1(void* p, size_t i, float v) { static_cast<float*>(p)[i] = v; }
};
template <> struct Four<__nv_bfloat16> {
  static __device__ __forceinline__ float4 ld(const void* p, size_t i) {
    const uint2 v = *reinterpret_cast<const uint2*>(static_cast<const __nv_bfloat16*>(p) + i);
    return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xffff0000u), __uint_as_float(v.y << 16), __uint_as_float(v.y & 0xffff0000u));
  }
  static __device__ __forceinline__ void st(void* p, size_t i, float4 v) {
    *reinterpret_cast<uint2*>(static_cast<__nv_bfloat16*>(p) + i) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
  }
  static __device__ __forceinline__ float ld1(const void* p, size_t i) { return __bfloat162float(static_cast<const __nv_bfloat16*>(p)[i]); }
  static __device__ __forceinline__ void st1(void* p, size_t i, float v) { static_cast<__nv_bfloat16*>(p)[i] = __float2bfloat16_rn(v); }
};
__device__ __forceinline__ float sw_dot(float4 a) { return fmaf(a.x, a.x, fmaf(a.y, a.y, fmaf(a.z, a.z, a.w * a.w))); }

// Every call of a block uses another `red`, so one barrier each is enough.
__device__ __forceinline__ float sw_block_sum(float v, float* red) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
  for (int i = 0; i < (int)(blockDim.x >> 5); ++i) t += red[i];
  return t;
}

// NV: groups of four values per thread, E % 4 == 0 and E <= 4 * NV * threads.
template <typename YT, typename HT, int NV>
__global__ void __launch_bounds__(512) sandwich_kernel(const SandwichParams p) {
  __shared__ float red[2][16];
  const int tid = threadIdx.x, nt = blockDim.x, E4 = p.E / 4;
  const size_t row = p.rows ? (size_t)p.rows[blockIdx.x] : (size_t)blockIdx.x;
  float* x = p.x + row * (size_t)p.E;
  float4 xr[NV], yr[NV];
  if (p.ids) {
    const size_t tok = (size_t)p.ids[row] * p.table_ld;
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (tid + i * nt < E4) {
        xr[i] = Four<HT>::ld(p.table, tok + 4 * (tid + i * nt));
        xr[i].x *= p.scale; xr[i].y *= p.scale; xr[i].z *= p.scale; xr[i].w *= p.scale;
      }
  } else {
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (tid + i * nt < E4) xr[i] = reinterpret_cast<const float4*>(x)[tid + i * nt];
  }
  if (p.y) {
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (tid + i * nt < E4) {
        yr[i] = Four<YT>::ld(p.y, row * (size_t)p.y_ld + 4 * (tid + i * nt));
        s += sw_dot(yr[i]);
      }
    if (p.post_w) {
      const float r = 1.0f / sqrtf(sw_block_sum(s, red[0]) / (float)p.E + p.eps);
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (tid + i * nt < E4) {
          const float4 w = reinterpret_cast<const float4*>(p.post_w)[tid + i * nt];
          yr[i].x *= r * (p.offset + w.x); yr[i].y *= r * (p.offset + w.y); yr[i].z *= r * (p.offset + w.z); yr[i].w *= r * (p.offset + w.w);
        }
    }
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (tid + i * nt < E4) {
        xr[i].x += yr[i].x; xr[i].y += yr[i].y; xr[i].z += yr[i].z; xr[i].w += yr[i].w;
      }
  }
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (tid + i * nt < E4) {
      if (p.write_x) reinterpret_cast<float4*>(x)[tid + i * nt] = xr[i];
      s += sw_dot(xr[i]);
    }
  if (!p.norm_w) return;
  const float r = 1.0f / sqrtf(sw_block_sum(s, red[1]) / (float)p.E + p.eps);
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (tid + i * nt < E4) {
      const float4 w = reinterpret_cast<const float4*>(p.norm_w)[tid + i * nt];
      Four<HT>::st(p.h, (size_t)blockIdx.x * p.h_ld + 4 * (tid + i * nt),
                   make_float4(xr[i].x * r * (p.offset + w.x), xr[i].y * r * (p.offset + w.y), xr[i].z * r * (p.offset + w.z), xr[i].w * r * (p.offset + w.w)));
    }
}

// Any width: every pass reads the row again.
template <typename YT, typename HT>
__global__ void __launch_bounds__(512) sandwich_any_kernel(const SandwichParams p) {
  __shared__ float red[2][16];
  const int tid = threadIdx.x, nt = blockDim.x, E = p.E;
  const size_t row = p.rows ? (size_t)p.rows[blockIdx.x] : (size_t)blockIdx.x;
  float* x = p.x + row * (size_t)E;
  const size_t tok = p.ids ? (size_t)p.ids[row] * p.table_ld : 0, yo = row * (size_t)p.y_ld;
  float ry = 1.0f;
  if (p.y && p.post_w) {
    float s = 0.f;
    for (int e = tid; e < E; e += nt) {
      const float v = Four<YT>::ld1(p.y, yo + e);
      s = fmaf(v, v, s);
    }
    ry = 1.0f / sqrtf(sw_block_sum(s, red[0]) / (float)E + p.eps);
  }
  auto value = [&](int e) {
    float v = p.ids ? Four<HT>::ld1(p.table, tok + e) * p.scale : x[e];
    if (p.y) v += Four<YT>::ld1(p.y, yo + e) * (p.post_w ? ry * (p.offset + p.post_w[e]) : 1.0f);
    return v;
  };
  float s = 0.f;
  for (int e = tid; e < E; e += nt) {
    const float v = value(e);
    s = fmaf(v, v, s);
  }
  const float r = p.norm_w ? 1.0f / sqrtf(sw_block_sum(s, red[1]) / (float)E + p.eps) : 0.f;
  for (int e = tid; e < E; e += nt) {  // an element is read and rewritten by the same thread
    const float v = value(e);
    if (p.write_x) x[e] = v;
    if (p.norm_w) Four<HT>::st1(p.h, (size_t)blockIdx.x * p.h_ld + e, v * r * (p.offset + p.norm_w[e]));
  }
}

template <typename YT, typename HT>
static int sandwich_launch(const SandwichParams& p, int n, bool vec, cudaStream_t st) {
  // few rows: one short pass over a row, its latency is all there is; many: enough values per thread to pay for the two block sums
  const int e4 = p.E / 4, few = (e4 + 511) / 512;
  const int want = n <= 148 || e4 < 256 ? 1 : e4 < 512 ? 2 : 4, rounds = few > want ? few : want;
  const int threads = ((e4 + rounds - 1) / rounds + 31) / 32 * 32;
  if (!vec || rounds > 12) sandwich_any_kernel<YT, HT><<<n, 256, 0, st>>>(p);
  else if (rounds <= 1) sandwich_kernel<YT, HT, 1><<<n, threads, 0, st>>>(p);
  else if (rounds <= 2) sandwich_kernel<YT, HT, 2><<<n, threads, 0, st>>>(p);
  else if (rounds <= 4) sandwich_kernel<YT, HT, 4><<<n, threads, 0, st>>>(p);
  else if (rounds <= 8) sandwich_kernel<YT, HT, 8><<<n, threads, 0, st>>>(p);
  else sandwich_kernel<YT, HT, 12><<<n, threads, 0, st>>>(p);
  const cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}

// x <- cap * tanh(x / cap), rows of `cols` values `ld` apart; V values per access
template <int V>
__global__ void __launch_bounds__(256) softcap_kernel(float* x, int ld, int cols, float cap, float inv_cap) {
  float* r = x + (size_t)blockIdx.x * ld;
  for (int c = (blockIdx.y * 256 + threadIdx.x) * V; c < cols; c += gridDim.y * 256 * V) {
    if (V == 4 && c + 4 <= cols) {
      float4 v = *reinterpret_cast<float4*>(r + c);
      v.x = cap * tanhf(v.x * inv_cap); v.y = cap * tanhf(v.y * inv_cap); v.z = cap * tanhf(v.z * inv_cap); v.w = cap * tanhf(v.w * inv_cap);
      *reinterpret_cast<float4*>(r + c) = v;
    } else {
      for (int i = c; i < min(c + V, cols); ++i) r[i] = cap * tanhf(r[i] * inv_cap);
    }
  }
}

}  // namespace inv

using namespace inv;

// Types: y_f32 / h_f32 say whether y and h (and the embedding table) are fp32, otherwise bf16 (h fp32 needs y fp32).
extern "C" int inv_sandwich_step(float* x, const int* ids, const void* table, int table_ld, float scale, const void* y, int y_ld, int y_f32,
                                 const float* post_w, const float* norm_w, float offset, float eps, void* h, int h_ld, int h_f32, const int* rows, int n,
                                 int write_x, int E, void* stream) {
  if (E < 1 || (h_f32 && !y_f32)) return -ERR_BAD_ARG;
  if (n <= 0) return 0;
  const SandwichParams p{x, ids, table, table_ld, scale, y, y_ld, post_w, norm_w, offset, eps, h, h_ld, rows, write_x, E};
  cudaStream_t st = (cudaStream_t)stream;
  const bool vec = E % 4 == 0 && (!y || y_ld % 4 == 0) && (!norm_w || h_ld % 4 == 0) && (!ids || table_ld % 4 == 0);
  if (h_f32) return sandwich_launch<float, float>(p, n, vec, st);
  if (y_f32) return sandwich_launch<float, __nv_bfloat16>(p, n, vec, st);
  return sandwich_launch<__nv_bfloat16, __nv_bfloat16>(p, n, vec, st);
}

extern "C" int inv_softcap(float* x, int ld, int rows, int cols, float cap, void* stream) {
  if (!(cap > 0.f)) return -ERR_BAD_ARG;
  if (rows <= 0 || cols <= 0) return 0;
  cudaStream_t st = (cudaStream_t)stream;
  if (ld % 4 == 0 && (reinterpret_cast<uintptr_t>(x) & 15) == 0)
    softcap_kernel<4><<<dim3(rows, (cols + 2047) / 2048), 256, 0, st>>>(x, ld, cols, cap, 1.0f / cap);
  else
    softcap_kernel<1><<<dim3(rows, (cols + 1023) / 1024), 256, 0, st>>>(x, ld, cols, cap, 1.0f / cap);
  const cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}
