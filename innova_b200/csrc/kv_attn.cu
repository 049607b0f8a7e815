// Attention over a paged cache of keys and values whose layers differ in head counts and sizes, with a chunked or windowed mask.
//
//   qkv_prep        one launch between the fused projection and the attention: RMS norm of the whole query row and of the whole key
//                   row (all heads at once), rotation of neighbouring pairs on the first dimensions of every head, append to the
//                   pages, queries (and, for prompts, keys) in the attention's type
//   kv_attend       any head size and fp32: one warp per (token, query head)
//   kv_attend_mma   bf16: a cluster of CTAs per (token, key head, eight query heads); the warps of the cluster take the 16-token
//                   pages of the visible range in turn and meet through distributed shared memory. Keys and values go straight
//                   from the pages into warp-level MMA fragments (a group of query heads fills at most eight rows; a 128-row
//                   tcgen05 tile would be nearly all padding, and the kernel is bound by the bytes of the keys and values)
//
// A row at position p sees [p - p % chunk, p] (chunk > 0), (p - window, p] (window > 0) or [0, p]. Pages wholly before that are
// never touched: their entries may belong to another sequence. A pool is [pages, kv heads, 2 (keys, values), 16, D].
// An output gate (pre-sigmoid, same columns as the output) is applied where the output is written.
#include "sm100_common.cuh"
#include "inv_api.h"

#include <cooperative_groups.h>

namespace inv {
namespace cg = cooperative_groups;

constexpr int KV_PAGE = 16;

__device__ __forceinline__ float kv_ld(const float* p) { return *p; }
__device__ __forceinline__ float kv_ld(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void kv_st(float* p, float v) { *p = v; }
__device__ __forceinline__ void kv_st(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ float kv_warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ int kv_first(int pos, int window, int chunk) {
  return chunk > 0 ? pos - pos % chunk : window > 0 ? max(0, pos - window + 1) : 0;
}
// Eight neighbouring values.
template <typename T> struct Eight;
template <> struct Eight<float> {
  float4 a, b;
  __device__ __forceinline__ void load(const float* p) { a = reinterpret_cast<const float4*>(p)[0]; b = reinterpret_cast<const float4*>(p)[1]; }
  __device__ __forceinline__ void get(float* f) const {
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
  }
  __device__ __forceinline__ void set(const float* f) { a = make_float4(f[0], f[1], f[2], f[3]); b = make_float4(f[4], f[5], f[6], f[7]); }
  __device__ __forceinline__ void store(float* p) const { reinterpret_cast<float4*>(p)[0] = a; reinterpret_cast<float4*>(p)[1] = b; }
};
template <> struct Eight<__nv_bfloat16> {
  uint4 v;
  __device__ __forceinline__ void load(const __nv_bfloat16* p) { v = *reinterpret_cast<const uint4*>(p); }
  __device__ __forceinline__ void get(float* f) const {
    const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      f[2 * i] = __uint_as_float(w[i] << 16);
      f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
    }
  }
  __device__ __forceinline__ void set(const float* f) {
    v = make_uint4(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]), pack_bf16x2(f[4], f[5]), pack_bf16x2(f[6], f[7]));
  }
  __device__ __forceinline__ void store(__nv_bfloat16* p) const { *reinterpret_cast<uint4*>(p) = v; }
};

// ------------------------------------------------------------------------------------------------ prep
struct QkvPrep {
  const void* in;         // [T, in_ld]
  int in_ld, off_q, off_k, off_v;
  int H, G, D, Dp;        // D: true head size (counts in the norms); heads are Dp columns apart, the padding is zero
  const float* q_norm;    // [H * Dp] or null: no norm of the queries
  const float* k_norm;    // [G * Dp] or null
  float eps;
  const float* freq;      // [pairs] angle per position
  int pairs;
  void* pool;
  const int* page_table;
  int max_pages;
  const int* rows;
  const int* tok_seq;
  const int* tok_pos;
  void* q_out;            // [T, H * Dp]
  void* k_out;            // [T, G * Dp] or null
};
constexpr int KV_MAX_PAIRS = 512;

// NCH: pieces of eight values that a thread keeps in registers between the two passes; 0: the second pass reads them again.
template <typename TI, typename TC, int NCH>
__global__ void __launch_bounds__(512) qkv_prep_kernel(const QkvPrep p) {
  __shared__ float red[2][16];
  __shared__ __align__(16) float2 turn[KV_MAX_PAIRS];
  const int tid = threadIdx.x, nt = blockDim.x;
  const size_t t = blockIdx.x;
  const TI* row = static_cast<const TI*>(p.in) + t * p.in_ld;
  const int per = p.Dp / 8, nq = p.H * per, n = (p.H + p.G) * per;
  const int pos = p.tok_pos[t];
  const int page = p.page_table[(size_t)p.rows[p.tok_seq[t]] * p.max_pages + pos / KV_PAGE];
  auto source = [&](int c) { return c < nq ? row + p.off_q + c * 8 : row + p.off_k + (c - nq) * 8; };
  Eight<TI> keep[NCH > 0 ? NCH : 1];
  float sq = 0.f, sk = 0.f;
  auto add = [&](const Eight<TI>& e, int c) {
    float f[8], s = 0.f;
    e.get(f);
#pragma unroll
    for (int i = 0; i < 8; ++i) s = fmaf(f[i], f[i], s);
    if (c < nq) sq += s;
    else sk += s;
  };
  if (NCH > 0) {
#pragma unroll
    for (int i = 0; i < (NCH > 0 ? NCH : 1); ++i)
      if (tid + i * nt < n) keep[i].load(source(tid + i * nt));
  }
  for (int i = tid; i < (p.pairs + 3) / 4 * 4; i += nt) {
    float s = 0.f, c = 1.f;
    if (i < p.pairs) sincosf((float)pos * p.freq[i], &s, &c);
    turn[i] = make_float2(c, s);
  }
  if (NCH > 0) {
#pragma unroll
    for (int i = 0; i < (NCH > 0 ? NCH : 1); ++i)
      if (tid + i * nt < n) add(keep[i], tid + i * nt);
  } else {
    for (int c = tid; c < n; c += nt) {
      keep[0].load(source(c));
      add(keep[0], c);
    }
  }
  sq = kv_warp_sum(sq);
  sk = kv_warp_sum(sk);
  if ((tid & 31) == 0) {
    red[0][tid >> 5] = sq;
    red[1][tid >> 5] = sk;
  }
  __syncthreads();
  sq = sk = 0.f;
  for (int i = 0; i < (nt >> 5); ++i) {
    sq += red[0][i];
    sk += red[1][i];
  }
  const float rq = p.q_norm ? 1.0f / sqrtf(sq / (float)(p.H * p.D) + p.eps) : 1.0f;
  const float rk = p.k_norm ? 1.0f / sqrtf(sk / (float)(p.G * p.D) + p.eps) : 1.0f;
  TC* pool = static_cast<TC*>(p.pool) + (size_t)page * p.G * 2 * KV_PAGE * p.Dp + (size_t)(pos % KV_PAGE) * p.Dp;
  const float inv_per = 1.0f / (float)per;
  auto write = [&](const Eight<TI>& e, int c) {
    const bool is_q = c < nq;
    const int piece = is_q ? c : c - nq, col = piece * 8;
    const int head = (int)(((float)piece + 0.5f) * inv_per), d0 = (piece - head * per) * 8;  // far below the fp32 range of exact integers
    TC* slot = pool + (size_t)head * (2 * KV_PAGE) * p.Dp + d0;                                // (key heads)
    float f[8];
    e.get(f);
    Eight<TC> o;
    if (!is_q) {  // the value: as projected
      if (p.off_v == p.off_k) {
        o.set(f);
      } else {
        float v[8];
        Eight<TI> ve;
        ve.load(row + p.off_v + col);
        ve.get(v);
        o.set(v);
      }
      o.store(slot + KV_PAGE * p.Dp);
    }
    const float* w = is_q ? p.q_norm : p.k_norm;
    if (w) {
      const float r = is_q ? rq : rk;
      float wv[8];
      Eight<float> we;
      we.load(w + col);
      we.get(wv);
#pragma unroll
      for (int i = 0; i < 8; ++i) f[i] = f[i] * r * wv[i];
    }
    if (d0 < 2 * p.pairs) {
      // entries past the last pair turn by nothing
      const float4* tp = reinterpret_cast<const float4*>(turn + d0 / 2);
      const float4 ta = tp[0], tb = tp[1];
      const float tc[4] = {ta.x, ta.z, tb.x, tb.z}, ts[4] = {ta.y, ta.w, tb.y, tb.w};
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float u = f[2 * i], v = f[2 * i + 1];
        f[2 * i] = u * tc[i] - v * ts[i];
        f[2 * i + 1] = v * tc[i] + u * ts[i];
      }
    }
    o.set(f);
    if (is_q) {
      o.store(static_cast<TC*>(p.q_out) + t * (size_t)(p.H * p.Dp) + col);
    } else {
      o.store(slot);
      if (p.k_out) o.store(static_cast<TC*>(p.k_out) + t * (size_t)(p.G * p.Dp) + col);
    }
  };
  if (NCH > 0) {
#pragma unroll
    for (int i = 0; i < (NCH > 0 ? NCH : 1); ++i)
      if (tid + i * nt < n) write(keep[i], tid + i * nt);
  } else {
    for (int c = tid; c < n; c += nt) {
      keep[0].load(source(c));
      write(keep[0], c);
    }
  }
}

// ------------------------------------------------------------------------------------------------ attention
struct KvAttend {
  const void* q;          // [T, H * D]
  const void* pool;
  const int* page_table;
  int max_pages;
  const int* rows;
  const int* tok_seq;
  const int* tok_pos;
  int window, chunk;
  float scale;
  const void* gate;       // [T, gate_ld] at the first gate column, or null
  int gate_ld, gate_f32;
  void* out;              // [T, H * D]
  int H, G, D;
};
__device__ __forceinline__ float kv_gate(const KvAttend& p, size_t t, int col) {
  if (!p.gate) return 1.0f;
  const size_t i = t * p.gate_ld + col;
  const float g = p.gate_f32 ? static_cast<const float*>(p.gate)[i] : __bfloat162float(static_cast<const __nv_bfloat16*>(p.gate)[i]);
  return 1.0f / (1.0f + expf(-g));
}

// One warp per (token, query head); NR * 32 >= D.
template <typename T, int NR>
__global__ void __launch_bounds__(128) kv_attend_kernel(const KvAttend p) {
  const int lane = threadIdx.x & 31, h = blockIdx.y * 4 + (threadIdx.x >> 5);
  const size_t t = blockIdx.x;
  if (h >= p.H) return;
  const int pos = p.tok_pos[t], g = h / (p.H / p.G), D = p.D;
  const int* pages = p.page_table + (size_t)p.rows[p.tok_seq[t]] * p.max_pages;
  const T* pool = static_cast<const T*>(p.pool) + (size_t)g * 2 * KV_PAGE * D;
  const size_t page_elems = (size_t)p.G * 2 * KV_PAGE * D;
  float qr[NR], acc[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int d = lane + i * 32;
    qr[i] = d < D ? kv_ld(static_cast<const T*>(p.q) + (t * p.H + h) * D + d) : 0.f;
    acc[i] = 0.f;
  }
  float m = -INFINITY, l = 0.f;
  for (int j0 = kv_first(pos, p.window, p.chunk); j0 <= pos; j0 += 4) {
    float s[4];
    const T* c[4];
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const int j = min(j0 + k, pos);
      c[k] = pool + pages[j / KV_PAGE] * page_elems + (size_t)(j % KV_PAGE) * D;
      float a = 0.f;
#pragma unroll
      for (int i = 0; i < NR; ++i) {
        const int d = lane + i * 32;
        if (d < D) a = fmaf(qr[i], kv_ld(c[k] + d), a);
      }
      s[k] = kv_warp_sum(a) * p.scale;
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
      const float e = expf(s[k] - m);
      l += e;
#pragma unroll
      for (int i = 0; i < NR; ++i) {
        const int d = lane + i * 32;
        if (d < D) acc[i] = fmaf(e, kv_ld(c[k] + KV_PAGE * D + d), acc[i]);
      }
    }
  }
  const float inv = 1.0f / l;
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int d = lane + i * 32;
    if (d < D) kv_st(static_cast<T*>(p.out) + (t * p.H + h) * D + d, acc[i] * inv * kv_gate(p, t, h * D + d));
  }
}

__device__ __forceinline__ void kv_mma(float* d, uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// grid (splits, G * ceil(group / 8), T), cluster (splits, 1, 1), NW warps. Warp w of split z takes pages z * NW + w, + splits * NW, ...
// of the visible range.
//   scores  S[head, token] = Q K^T: A = Q (rows 8..15 zero), B = K; a lane holds 8 consecutive dimensions of tokens lane / 4 and
//           lane / 4 + 8 per step of 32, and both operands use that order inside the MMA
//   softmax on the accumulator: a lane has head lane / 4, tokens 2 (lane % 4), + 1, + 8, + 9
//   values  O^T[d, head] = V^T P^T: B is the score fragment as it stands; A pairs neighbouring tokens of the lane's dimensions
// The next page's keys are requested when the scores have used up this page's, its values after this page's sum.
template <int D, int NW>
__global__ void __launch_bounds__(NW * 32) kv_attend_mma_kernel(const KvAttend p) {
  constexpr int KS = D / 32;       // 16-byte pieces of a key row per lane
  constexpr int VU = D / 64;       // 16-byte pieces of a value row per lane
  constexpr int OS = D + 4;        // row stride of the shared partial sums
  extern __shared__ float kvs[];   // sums [NW][8][OS], then max [NW][8] and denominator [NW][8]
  float* w_m = kvs + NW * 8 * OS;
  float* w_l = w_m + NW * 8;
  const cg::cluster_group cluster = cg::this_cluster();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, gid = lane >> 2, tig = lane & 3;
  const int splits = gridDim.x, split = blockIdx.x;
  const size_t t = blockIdx.z;
  const int group = p.H / p.G, blocks = (group + 7) / 8, g = blockIdx.y / blocks;
  const int h0 = g * group + (blockIdx.y % blocks) * 8, nh = min(8, (g + 1) * group - h0);
  const int pos = p.tok_pos[t], first = kv_first(pos, p.window, p.chunk);
  const int page0 = first / KV_PAGE, n_pages = pos / KV_PAGE + 1 - page0;
  const int* pages = p.page_table + (size_t)p.rows[p.tok_seq[t]] * p.max_pages + page0;
  const __nv_bfloat16* pool = static_cast<const __nv_bfloat16*>(p.pool) + (size_t)g * 2 * KV_PAGE * D;
  const size_t page_elems = (size_t)p.G * 2 * KV_PAGE * D;
  const float cs = p.scale * 1.4426950408889634f;
  uint4 kr[2][KS], vr[4][VU];
  auto load_k = [&](int i) {
    const __nv_bfloat16* base = pool + pages[i] * page_elems;
#pragma unroll
    for (int x = 0; x < 2; ++x)
#pragma unroll
      for (int s = 0; s < KS; ++s) kr[x][s] = *reinterpret_cast<const uint4*>(base + (gid + 8 * x) * D + s * 32 + tig * 8);
  };
  auto token = [&](int i, int x) { return (page0 + i) * KV_PAGE + 2 * tig + (x & 1) + 8 * (x >> 1); };
  auto load_v = [&](int i) {  // tokens that are not seen contribute nothing, whatever their slots hold
    const __nv_bfloat16* base = pool + pages[i] * page_elems + KV_PAGE * D;
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const int j = token(i, x);
      const bool seen = j >= first && j <= pos;
#pragma unroll
      for (int u = 0; u < VU; ++u)
        vr[x][u] = seen ? *reinterpret_cast<const uint4*>(base + (j % KV_PAGE) * D + u * 64 + gid * 8) : make_uint4(0, 0, 0, 0);
    }
  };
  uint4 qf[KS];
  {
    const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(p.q) + (t * p.H + h0 + gid) * D + tig * 8;
#pragma unroll
    for (int s = 0; s < KS; ++s) qf[s] = gid < nh ? *reinterpret_cast<const uint4*>(q + s * 32) : make_uint4(0, 0, 0, 0);
  }
  float acc[VU * 4][4];
#pragma unroll
  for (int i = 0; i < VU * 4; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
  float m = -INFINITY, l = 0.f;  // of head gid; l is this lane's share
  const int step = splits * NW;
  int i = split * NW + warp;
  if (i < n_pages) {
    load_k(i);
    load_v(i);
  }
  for (; i < n_pages; i += step) {
    float s[2][4];
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      s[x][0] = s[x][1] = s[x][2] = s[x][3] = 0.f;
#pragma unroll
      for (int k = 0; k < KS; ++k) {
        kv_mma(s[x], qf[k].x, 0u, qf[k].y, 0u, kr[x][k].x, kr[x][k].y);
        kv_mma(s[x], qf[k].z, 0u, qf[k].w, 0u, kr[x][k].z, kr[x][k].w);
      }
    }
    if (i + step < n_pages) load_k(i + step);
    float e[4], mx = -INFINITY;
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const int j = token(i, x);
      e[x] = j >= first && j <= pos ? s[x >> 1][x & 1] * cs : -INFINITY;
      mx = fmaxf(mx, e[x]);
    }
    mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
    mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
    const float mn = fmaxf(m, mx);   // a page of the range holds at least one visible token: finite
    const float al = exp2f(m - mn);
    m = mn;
#pragma unroll
    for (int x = 0; x < 4; ++x) e[x] = exp2f(e[x] - mn);
    l = l * al + ((e[0] + e[1]) + (e[2] + e[3]));
    const uint32_t b0 = pack_bf16x2(e[0], e[1]), b1 = pack_bf16x2(e[2], e[3]);
    if (__any_sync(0xffffffffu, al != 1.f)) {  // this lane's columns are heads 2 tig and 2 tig + 1
      const float a0 = __shfl_sync(0xffffffffu, al, 8 * tig), a1 = __shfl_sync(0xffffffffu, al, 8 * tig + 4);
#pragma unroll
      for (int k = 0; k < VU * 4; ++k) {
        acc[k][0] *= a0; acc[k][1] *= a1; acc[k][2] *= a0; acc[k][3] *= a1;
      }
    }
#pragma unroll
    for (int u = 0; u < VU; ++u) {
      const uint32_t v0[4] = {vr[0][u].x, vr[0][u].y, vr[0][u].z, vr[0][u].w}, v1[4] = {vr[1][u].x, vr[1][u].y, vr[1][u].z, vr[1][u].w};
      const uint32_t v2[4] = {vr[2][u].x, vr[2][u].y, vr[2][u].z, vr[2][u].w}, v3[4] = {vr[3][u].x, vr[3][u].y, vr[3][u].z, vr[3][u].w};
#pragma unroll
      for (int k = 0; k < 4; ++k)  // dimensions u * 64 + gid * 8 + 2 k (row gid) and + 1 (row gid + 8)
        kv_mma(acc[u * 4 + k], __byte_perm(v0[k], v1[k], 0x5410), __byte_perm(v0[k], v1[k], 0x7632), __byte_perm(v2[k], v3[k], 0x5410),
               __byte_perm(v2[k], v3[k], 0x7632), b0, b1);
    }
    if (i + step < n_pages) load_v(i + step);
  }
  l += __shfl_xor_sync(0xffffffffu, l, 1);
  l += __shfl_xor_sync(0xffffffffu, l, 2);
  if (tig == 0) {
    w_m[warp * 8 + gid] = m;
    w_l[warp * 8 + gid] = l;
  }
#pragma unroll
  for (int k = 0; k < VU * 4; ++k) {
    const int d = (k >> 2) * 64 + gid * 8 + 2 * (k & 3);
    *reinterpret_cast<float2*>(&kvs[(warp * 8 + 2 * tig) * OS + d]) = make_float2(acc[k][0], acc[k][2]);
    *reinterpret_cast<float2*>(&kvs[(warp * 8 + 2 * tig + 1) * OS + d]) = make_float2(acc[k][1], acc[k][3]);
  }
  // every warp of the cluster has left its sums; a CTA writes every splits-th piece of the output
  if (splits > 1) cluster.sync();
  else __syncthreads();
  const int pieces = nh * (D / 4);
  for (int x = split * NW * 32 + threadIdx.x; x < pieces; x += splits * NW * 32) {
    const int h = x / (D / 4), d = (x % (D / 4)) * 4;
    float mx = -INFINITY;
    for (int z = 0; z < splits; ++z) {
      const float* pm = splits > 1 ? cluster.map_shared_rank(w_m, z) : w_m;
#pragma unroll
      for (int w = 0; w < NW; ++w) mx = fmaxf(mx, pm[w * 8 + h]);
    }
    float den = 0.f;
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int z = 0; z < splits; ++z) {
      const float* pm = splits > 1 ? cluster.map_shared_rank(w_m, z) : w_m;
      const float* pl = splits > 1 ? cluster.map_shared_rank(w_l, z) : w_l;
      const float* po = splits > 1 ? cluster.map_shared_rank(kvs, z) : kvs;
#pragma unroll
      for (int w = 0; w < NW; ++w) {
        const float f = exp2f(pm[w * 8 + h] - mx);  // 0 for a warp without pages
        const float4 v = *reinterpret_cast<const float4*>(po + (w * 8 + h) * OS + d);
        den = fmaf(pl[w * 8 + h], f, den);
        o.x = fmaf(v.x, f, o.x); o.y = fmaf(v.y, f, o.y); o.z = fmaf(v.z, f, o.z); o.w = fmaf(v.w, f, o.w);
      }
    }
    const float inv = 1.0f / den;
    const int col = (h0 + h) * D + d;
    *reinterpret_cast<uint2*>(static_cast<__nv_bfloat16*>(p.out) + t * (size_t)(p.H * D) + col) =
        make_uint2(pack_bf16x2(o.x * inv * kv_gate(p, t, col), o.y * inv * kv_gate(p, t, col + 1)),
                   pack_bf16x2(o.z * inv * kv_gate(p, t, col + 2), o.w * inv * kv_gate(p, t, col + 3)));
  }
  if (splits > 1) cluster.sync();  // no CTA leaves while another one reads its sums
}

template <typename TI, typename TC>
static int launch_prep(const QkvPrep& p, int T, cudaStream_t st) {
  const int n = (p.H + p.G) * (p.Dp / 8);
  const int cap = T <= 148 ? 512 : 256;            // few rows: their latency is all there is
  const int rounds = (n + cap - 1) / cap;
  const int threads = ((n + rounds - 1) / rounds + 31) / 32 * 32;
  switch (rounds) {
    case 1: qkv_prep_kernel<TI, TC, 1><<<T, threads, 0, st>>>(p); break;
    case 2: qkv_prep_kernel<TI, TC, 2><<<T, threads, 0, st>>>(p); break;
    case 3: qkv_prep_kernel<TI, TC, 3><<<T, threads, 0, st>>>(p); break;
    case 4: qkv_prep_kernel<TI, TC, 4><<<T, threads, 0, st>>>(p); break;
    default: qkv_prep_kernel<TI, TC, 0><<<T, 512, 0, st>>>(p); break;
  }
  const cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}

template <typename T>
static int launch_attend(const KvAttend& p, int n_tok, cudaStream_t st) {
  const dim3 grid(n_tok, (p.H + 3) / 4);
  if (p.D <= 32) kv_attend_kernel<T, 1><<<grid, 128, 0, st>>>(p);
  else if (p.D <= 64) kv_attend_kernel<T, 2><<<grid, 128, 0, st>>>(p);
  else if (p.D <= 128) kv_attend_kernel<T, 4><<<grid, 128, 0, st>>>(p);
  else if (p.D <= 256) kv_attend_kernel<T, 8><<<grid, 128, 0, st>>>(p);
  else if (p.D <= 512) kv_attend_kernel<T, 16><<<grid, 128, 0, st>>>(p);
  else if (p.D <= 1024) kv_attend_kernel<T, 32><<<grid, 128, 0, st>>>(p);
  else return -ERR_BAD_ARG;
  const cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}

template <int D, int NW>
static int launch_mma(const KvAttend& p, int splits, int n_tok, cudaStream_t st) {
  constexpr int bytes = (NW * 8 * (D + 4) + 2 * NW * 8) * 4;
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(kv_attend_mma_kernel<D, NW>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
    if (e != cudaSuccess) return -(int)e;
    configured = true;
  }
  const int group = p.H / p.G;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(splits, p.G * ((group + 7) / 8), n_tok);
  cfg.blockDim = dim3(NW * 32);
  cfg.dynamicSmemBytes = bytes;
  cfg.stream = st;
  cudaLaunchAttribute attr;
  attr.id = cudaLaunchAttributeClusterDimension;
  attr.val.clusterDim.x = splits;
  attr.val.clusterDim.y = attr.val.clusterDim.z = 1;
  cfg.attrs = &attr;
  cfg.numAttrs = 1;
  const cudaError_t e = cudaLaunchKernelEx(&cfg, kv_attend_mma_kernel<D, NW>, p);
  return e == cudaSuccess ? 0 : -(int)e;
}

}  // namespace inv

using namespace inv;

// in_f32 / c_f32: types of the projection rows and of the pages (and outputs); bf16 rows need bf16 pages. Rows start on 16-byte
// boundaries, offsets and Dp are multiples of 8. pairs <= Dp / 2.
extern "C" int inv_qkv_prep(const void* in, int in_ld, int in_f32, int off_q, int off_k, int off_v, int H, int G, int D, int Dp, const float* q_norm,
                            const float* k_norm, float eps, const float* freq, int pairs, void* pool, int c_f32, const int* page_table, int max_pages,
                            const int* rows, const int* tok_seq, const int* tok_pos, void* q_out, void* k_out, int T, void* stream) {
  if (H < 1 || G < 1 || D < 1 || Dp < D || Dp % 8 || in_ld % 8 || off_q % 8 || off_k % 8 || off_v % 8 || pairs < 0 || 2 * pairs > Dp ||
      pairs > KV_MAX_PAIRS)
    return -ERR_BAD_ARG;
  if (T <= 0) return 0;
  const QkvPrep p{in, in_ld, off_q, off_k, off_v, H, G, D, Dp, q_norm, k_norm, eps, freq, pairs, pool, page_table, max_pages, rows, tok_seq, tok_pos, q_out, k_out};
  cudaStream_t st = (cudaStream_t)stream;
  if (in_f32 && c_f32) return launch_prep<float, float>(p, T, st);
  if (in_f32) return launch_prep<float, __nv_bfloat16>(p, T, st);
  if (!c_f32) return launch_prep<__nv_bfloat16, __nv_bfloat16>(p, T, st);
  return -ERR_BAD_ARG;
}

// Attention of T query rows over the pages. fp32, or bf16 with a head size the tensor-core kernel does not have: the warp-per-head
// kernel (D <= 1024). bf16 with D = 64, 128, 192 or 256: the tensor-core kernel on clusters of `splits` (1, 2, 4 or 8) CTAs of
// `warps` (4 or 8) warps.
extern "C" int inv_kv_attend(const void* q, const void* pool, int f32, const int* page_table, int max_pages, const int* rows, const int* tok_seq,
                             const int* tok_pos, int window, int chunk, float scale, const void* gate, int gate_ld, int gate_f32, void* out, int T,
                             int H, int G, int D, int splits, int warps, void* stream) {
  if (H < 1 || G < 1 || H % G || D < 1 || window < 0 || chunk < 0 || (window > 0 && chunk > 0)) return -ERR_BAD_ARG;
  if (T <= 0) return 0;
  cudaStream_t st = (cudaStream_t)stream;
  KvAttend p{q, pool, page_table, max_pages, rows, tok_seq, tok_pos, window, chunk, scale, gate, gate_ld, gate_f32, out, H, G, D};
  if (f32) return launch_attend<float>(p, T, st);
  if (D % 64 || D > 256) return launch_attend<__nv_bfloat16>(p, T, st);
  if ((splits != 1 && splits != 2 && splits != 4 && splits != 8) || (warps != 4 && warps != 8)) return -ERR_BAD_ARG;
  // the grid's third dimension ends at 65535: more rows go in several launches
  for (int t0 = 0; t0 < T; t0 += 65535) {
    KvAttend c = p;
    const int n = T - t0 < 65535 ? T - t0 : 65535;
    c.q = static_cast<const __nv_bfloat16*>(q) + (size_t)t0 * H * D;
    c.out = static_cast<__nv_bfloat16*>(out) + (size_t)t0 * H * D;
    if (gate) c.gate = static_cast<const char*>(gate) + (size_t)t0 * gate_ld * (gate_f32 ? 4 : 2);
    c.tok_seq += t0;
    c.tok_pos += t0;
    int rc;
#define INV_KV(DD) rc = warps == 8 ? launch_mma<DD, 8>(c, splits, n, st) : launch_mma<DD, 4>(c, splits, n, st)
    if (D == 64) INV_KV(64);
    else if (D == 128) INV_KV(128);
    else if (D == 192) INV_KV(192);
    else INV_KV(256);
#undef INV_KV
    if (rc) return rc;
  }
  return 0;
}
