// Attention over a paged cache in plain fp32 arithmetic, for 32-bit models and for head sizes the tensor-core kernels cannot address: the
// same op as attention_mixed.cu (keys and values of different widths, window or own-run masks, soft-capped scores, sinks, gates, several maps
// per head), and the merge of differential attention.
// One CTA = (query token, query head); 32 keys at a time: a warp per key for the scores, then every thread its columns of the values.
// Built without fast-math.
#include "common.cuh"
#include "kernels.h"

namespace ogb {

template <typename T> __device__ __forceinline__ float as_f32(T v);
template <> __device__ __forceinline__ float as_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ float as_f32<__nv_bfloat16>(__nv_bfloat16 v) { return bf2f(v); }
template <typename T> __device__ __forceinline__ T of_f32(float v);
template <> __device__ __forceinline__ float of_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 of_f32<__nv_bfloat16>(float v) { return f2bf(v); }

constexpr int ASM_THREADS = 128, ASM_KEYS = 32;

// COLS: value columns per thread (dv <= COLS * ASM_THREADS).
template <typename T, int COLS>
__global__ void __launch_bounds__(ASM_THREADS) attention_simt_kernel(OgbAttnLayer a, const T* __restrict__ q, int q_stride, const T* __restrict__ k_cache,
                                                                     const T* __restrict__ v_cache, const int32_t* __restrict__ cu,
                                                                     const int32_t* __restrict__ past_lens, const int32_t* __restrict__ tables,
                                                                     int table_cols, int block_size, T* __restrict__ out, int out_stride, int B,
                                                                     float* __restrict__ part_o, float* __restrict__ part_ml) {
  extern __shared__ float sq[];                  // [dk] the query
  __shared__ float ssc[ASM_KEYS];
  __shared__ long long sslot[ASM_KEYS];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, h = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  int rlo = 0, rhi = B - 1;
  while (rlo < rhi) {
    const int mid = (rlo + rhi + 1) >> 1;
    if (cu[mid] <= t) rlo = mid; else rhi = mid - 1;
  }
  const int b = rlo;
  if (t < cu[b] || t >= cu[b + 1]) return;
  const int pos = past_lens[b] + t - cu[b], g = h / (a.Hq / a.Hkv);
  const int lo = a.window > 0 ? max(0, pos - a.window + 1) : (a.chunk > 0 ? pos / a.chunk * a.chunk : 0);
  const int32_t* table = tables + size_t(b) * table_cols;
  const int kh = a.joint ? 1 : a.Hkv, kg = a.joint ? 0 : g;  // key heads of a cache row, the one this query meets
  const int dm = a.dk / a.maps, c0 = (h % a.maps) * dm;      // this query vector's columns of a key
  for (int i = threadIdx.x; i < dm; i += ASM_THREADS) sq[i] = as_f32(q[size_t(t) * q_stride + size_t(h) * dm + i]);
  float acc[COLS];
#pragma unroll
  for (int c = 0; c < COLS; ++c) acc[c] = 0.f;
  // the sink takes part in the maximum and the sum from the start
  float m = a.sinks ? a.sinks[h] : -INFINITY, l = a.sinks ? 1.f : 0.f;
  for (int j0 = lo; j0 <= pos; j0 += ASM_KEYS) {
    const int nk = min(ASM_KEYS, pos + 1 - j0);
    __syncthreads();
    if (threadIdx.x < nk) {
      const int j = j0 + threadIdx.x;
      sslot[threadIdx.x] = (long long)(table[j / block_size]) * block_size + j % block_size;
    }
    __syncthreads();
    for (int k = warp; k < nk; k += ASM_THREADS / 32) {
      const T* row = k_cache + (size_t(sslot[k]) * kh + kg) * a.dk + c0;
      float d = 0.f;
      for (int i = lane; i < dm; i += 32) d = fmaf(sq[i], as_f32(row[i]), d);
      d = warp_sum(d) * a.scale;
      if (lane == 0) ssc[k] = a.softcap > 0.f ? a.softcap * tanhf(d / a.softcap) : d;
    }
    __syncthreads();
    float mn = m;
    for (int k = 0; k < nk; ++k) mn = fmaxf(mn, ssc[k]);
    const float al = m == -INFINITY ? 0.f : expf(m - mn);
    l *= al;
#pragma unroll
    for (int c = 0; c < COLS; ++c) acc[c] *= al;
    for (int k = 0; k < nk; ++k) {
      const float pr = expf(ssc[k] - mn);
      l += pr;
      const T* row = v_cache + (size_t(sslot[k]) * a.Hkv + g) * a.dv;
#pragma unroll
      for (int c = 0; c < COLS; ++c) {
        const int i = c * ASM_THREADS + threadIdx.x;
        if (i < a.dv) acc[c] = fmaf(pr, as_f32(row[i]), acc[c]);
      }
    }
    m = mn;
  }
  float inv = 1.f / l;
  if (part_o) {                                  // one finished part: maximum 0, sum 1
    const size_t row = size_t(t) * a.Hq + h;
#pragma unroll
    for (int c = 0; c < COLS; ++c) {
      const int i = c * ASM_THREADS + threadIdx.x;
      if (i < a.dv) part_o[row * a.dv + i] = acc[c] * inv;
    }
    if (threadIdx.x == 0) { part_ml[row * 2] = 0.f; part_ml[row * 2 + 1] = 1.f; }
    return;
  }
  inv *= a.out_scale;
  const T* gate = static_cast<const T*>(a.gate);
  if (gate && !a.gate_wide) inv *= 1.f / (1.f + expf(-as_f32(gate[size_t(t) * a.gate_stride + h])));
#pragma unroll
  for (int c = 0; c < COLS; ++c) {
    const int i = c * ASM_THREADS + threadIdx.x;
    if (i >= a.dv) continue;
    float v = acc[c] * inv;
    if (gate && a.gate_wide) v /= 1.f + expf(-as_f32(gate[size_t(t) * a.gate_stride + size_t(h) * a.dv + i]));
    out[size_t(t) * out_stride + size_t(h) * a.dv + i] = of_f32<T>(v);
  }
}

// ------------------------------------------------------------------------------------ differential merge
template <typename T> __device__ __forceinline__ void load4(const T* p, float (&v)[4]);
template <> __device__ __forceinline__ void load4<float>(const float* p, float (&v)[4]) {
  const float4 a = *reinterpret_cast<const float4*>(p);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
}
template <> __device__ __forceinline__ void load4<__nv_bfloat16>(const __nv_bfloat16* p, float (&v)[4]) {
  const uint2 q = *reinterpret_cast<const uint2*>(p);
  const float2 a = unpack_bf16x2(q.x), b = unpack_bf16x2(q.y);
  v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
}
__device__ __forceinline__ void store4(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float (&v)[4]) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
}

struct DiffMerge {
  const float *part_o, *part_ml;
  int splits, rows_all, T, H, dv, vdim;
  float lambda, post, eps;
  int gate_stride, out_stride;
};

// Both maps' (maximum, sum) of a head in split s.
__device__ __forceinline__ float4 diff_stats(const DiffMerge& p, size_t row, int s) {
  const float2* ml = reinterpret_cast<const float2*>(p.part_ml) + size_t(s) * p.rows_all + row;
  const float2 a = ml[0], b = ml[1];
  return make_float4(a.x, a.y, b.x, b.y);
}

// The weights of up to 32 splits (from s0 on) of the two rows of a head in the difference a1 - lambda * a2, one split per lane.
__device__ __forceinline__ float2 diff_weights(const DiffMerge& p, size_t row, int s0, const float (&top)[2], const float (&inv)[2], int lane) {
  float2 w = make_float2(0.f, 0.f);
  if (s0 + lane < p.splits) {
    const float4 ml = diff_stats(p, row, s0 + lane);
    if (ml.x != -INFINITY) w.x = exp2f(ml.x - top[0]) * inv[0];
    if (ml.z != -INFINITY) w.y = -exp2f(ml.z - top[1]) * inv[1];
  }
  return w;
}

// One split (prompts): a1 / l1 - lambda * a2 / l2, everything loaded before anything is used.
template <typename T, int KEEP>
__global__ void __launch_bounds__(128) attention_diff_single_kernel(DiffMerge p, const T* __restrict__ gate, T* __restrict__ out) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const long item = long(blockIdx.x) * 4 + (threadIdx.x >> 5);
  if (item >= long(p.T) * p.H) return;
  const int t = int(item / p.H), h = int(item - long(t) * p.H);
  const size_t row = size_t(t) * 2 * p.H + 2 * h;
  const float* r = p.part_o + row * p.dv;
  const T* pg = gate ? gate + size_t(t) * p.gate_stride + size_t(h) * p.dv : nullptr;
  float a[KEEP][4], b[KEEP][4], g[KEEP][4];
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int d = k * 128 + lane * 4;
    if (d >= p.dv) continue;
    load4(r + d, a[k]);
    load4(r + p.dv + d, b[k]);
    if (pg) load4(pg + d, g[k]);
  }
  const float4 ml = diff_stats(p, row, 0);
  const float f1 = ml.y > 0.f ? 1.f / ml.y : 0.f, f2 = ml.w > 0.f ? p.lambda / ml.w : 0.f;
  float sq = 0.f;
#pragma unroll
  for (int k = 0; k < KEEP; ++k)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      a[k][e] = k * 128 + lane * 4 + e < p.vdim ? a[k][e] * f1 - b[k][e] * f2 : 0.f;
      sq = fmaf(a[k][e], a[k][e], sq);
    }
  const float f = p.post / sqrtf(warp_sum(sq) / p.vdim + p.eps);
  T* dst = out + size_t(t) * p.out_stride + size_t(h) * p.dv;
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int d = k * 128 + lane * 4;
    if (d >= p.dv) continue;
#pragma unroll
    for (int e = 0; e < 4; ++e) a[k][e] = pg ? a[k][e] * f / (1.f + expf(-g[k][e])) : a[k][e] * f;
    store4(dst + d, a[k]);
  }
}

// KEEP > 0: dv <= 128 * KEEP, a lane owns columns 4 lane .. 4 lane + 3 of every 128 (dv a multiple of 4); 0: any dv, recomputed where it is
// needed twice.  WARPS: warps of a head, the splits are divided over them (1: four heads per CTA).
template <typename T, int KEEP, int WARPS>
__global__ void __launch_bounds__(128) attention_diff_merge_kernel(DiffMerge p, const T* __restrict__ gate, T* __restrict__ out) {
  __shared__ float part[WARPS > 1 ? WARPS : 1][KEEP > 0 ? KEEP * 128 : 1];
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = WARPS > 1 ? threadIdx.x >> 5 : 0;
  const long item = WARPS > 1 ? long(blockIdx.x) : long(blockIdx.x) * 4 + (threadIdx.x >> 5);
  if (item >= long(p.T) * p.H) return;
  const int t = int(item / p.H), h = int(item % p.H);
  const size_t row = size_t(t) * 2 * p.H + 2 * h;
  float top[2] = {-INFINITY, -INFINITY}, inv[2] = {0.f, 0.f};
  for (int s = lane; s < p.splits; s += 32) {
    const float4 ml = diff_stats(p, row, s);
    top[0] = fmaxf(top[0], ml.x);
    top[1] = fmaxf(top[1], ml.z);
  }
  top[0] = warp_max(top[0]);
  top[1] = warp_max(top[1]);
  for (int s = lane; s < p.splits; s += 32) {
    const float4 ml = diff_stats(p, row, s);
    if (ml.x != -INFINITY) inv[0] += exp2f(ml.x - top[0]) * ml.y;
    if (ml.z != -INFINITY) inv[1] += exp2f(ml.z - top[1]) * ml.w;
  }
  inv[0] = warp_sum(inv[0]);
  inv[1] = warp_sum(inv[1]);
  inv[0] = inv[0] > 0.f ? 1.f / inv[0] : 0.f;
  inv[1] = inv[1] > 0.f ? p.lambda / inv[1] : 0.f;
  T* dst = out + size_t(t) * p.out_stride + size_t(h) * p.dv;
  const T* pg = gate ? gate + size_t(t) * p.gate_stride + size_t(h) * p.dv : nullptr;
  if constexpr (KEEP > 0) {
    float o[KEEP][4] = {};
    for (int s0 = 0; s0 < p.splits; s0 += 32) {
      const float2 w = diff_weights(p, row, s0, top, inv, lane);
      const int n = min(32, p.splits - s0);
#pragma unroll 4
      for (int s = warp; s < n; s += WARPS) {
        const float w1 = __shfl_sync(0xffffffffu, w.x, s), w2 = __shfl_sync(0xffffffffu, w.y, s);
        const float* r = p.part_o + (size_t(s0 + s) * p.rows_all + row) * p.dv;
#pragma unroll
        for (int k = 0; k < KEEP; ++k) {
          const int d = k * 128 + lane * 4;
          if (d >= p.dv) continue;
          float a[4], b[4];
          load4(r + d, a);
          load4(r + p.dv + d, b);
          // (an empty split's values are not defined)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            if (w1 != 0.f) o[k][e] = fmaf(w1, a[e], o[k][e]);
            if (w2 != 0.f) o[k][e] = fmaf(w2, b[e], o[k][e]);
          }
        }
      }
    }
    if constexpr (WARPS > 1) {
#pragma unroll
      for (int k = 0; k < KEEP; ++k) store4(&part[warp][k * 128 + lane * 4], o[k]);
      __syncthreads();
      if (warp != 0) return;
#pragma unroll
      for (int k = 0; k < KEEP; ++k)
        for (int q = 1; q < WARPS; ++q) {
          float a[4];
          load4(&part[q][k * 128 + lane * 4], a);
#pragma unroll
          for (int e = 0; e < 4; ++e) o[k][e] += a[e];
        }
    }
    float sq = 0.f;
#pragma unroll
    for (int k = 0; k < KEEP; ++k)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        if (k * 128 + lane * 4 + e >= p.vdim) o[k][e] = 0.f;
        sq = fmaf(o[k][e], o[k][e], sq);
      }
    const float f = p.post / sqrtf(warp_sum(sq) / p.vdim + p.eps);
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int d = k * 128 + lane * 4;
      if (d >= p.dv) continue;
      float g[4];
      if (pg) load4(pg + d, g);
#pragma unroll
      for (int e = 0; e < 4; ++e) o[k][e] = pg ? o[k][e] * f / (1.f + expf(-g[e])) : o[k][e] * f;
      store4(dst + d, o[k]);
    }
  } else {
    auto column = [&](int d) {
      float v = 0.f;
      for (int s = 0; s < p.splits; ++s) {
        const size_t r = size_t(s) * p.rows_all + row;
        const float m1 = p.part_ml[r * 2], m2 = p.part_ml[r * 2 + 2];
        if (m1 != -INFINITY) v += exp2f(m1 - top[0]) * inv[0] * p.part_o[r * p.dv + d];
        if (m2 != -INFINITY) v -= exp2f(m2 - top[1]) * inv[1] * p.part_o[(r + 1) * p.dv + d];
      }
      return v;
    };
    float sq = 0.f;
    for (int d = lane; d < p.vdim; d += 32) { const float v = column(d); sq = fmaf(v, v, sq); }
    const float f = p.post / sqrtf(warp_sum(sq) / p.vdim + p.eps);
    for (int d = lane; d < p.dv; d += 32) {
      const float v = d < p.vdim ? column(d) * f : 0.f;
      dst[d] = of_f32<T>(pg ? v / (1.f + expf(-as_f32(pg[d]))) : v);
    }
  }
}

template <typename T>
static int LaunchDiffMerge(const DiffMerge& p, const void* gate, void* out, cudaStream_t s) {
  const long items = long(p.T) * p.H;
  const bool vec = p.dv % 4 == 0 && p.dv <= 256 && p.gate_stride % 4 == 0 && p.out_stride % 4 == 0 &&
                   ((reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(out)) & (4 * sizeof(T) - 1)) == 0;
  const bool spread = p.splits > 4 && items < (1l << 30);      // several warps per head
  const dim3 grid(unsigned(spread && vec ? items : (items + 3) / 4));
#define OGB_DIFF(K, W) launch_pdl(attention_diff_merge_kernel<T, K, W>, grid, dim3(128), 0, s, p, static_cast<const T*>(gate), static_cast<T*>(out))
#define OGB_DIFF1(K) launch_pdl(attention_diff_single_kernel<T, K>, grid, dim3(128), 0, s, p, static_cast<const T*>(gate), static_cast<T*>(out))
  bool ok;
  if (!vec) ok = OGB_DIFF(0, 1);
  else if (p.splits == 1) ok = p.dv <= 128 ? OGB_DIFF1(1) : OGB_DIFF1(2);
  else if (p.dv <= 128) ok = spread ? OGB_DIFF(1, 4) : OGB_DIFF(1, 1);
  else ok = spread ? OGB_DIFF(2, 4) : OGB_DIFF(2, 1);
#undef OGB_DIFF
#undef OGB_DIFF1
  return ok ? 0 : -4;
}

template <typename T>
static int LaunchSimt(const OgbAttnLayer& a, const void* q, int q_stride, const void* k, const void* v, const int32_t* cu, const int32_t* past,
                      const int32_t* table, int table_cols, int block_size, void* out, int out_stride, int B, int T_, float* part_o, float* part_ml,
                      cudaStream_t s) {
  const dim3 grid(T_, a.Hq);
  const size_t smem = size_t(a.dk) * 4;
#define OGB_ASM(C) launch_pdl(attention_simt_kernel<T, C>, grid, dim3(ASM_THREADS), smem, s, a, static_cast<const T*>(q), q_stride, static_cast<const T*>(k), \
                              static_cast<const T*>(v), cu, past, table, table_cols, block_size, static_cast<T*>(out), out_stride, B, part_o, part_ml)
  const bool ok = a.dv <= ASM_THREADS ? OGB_ASM(1) : (a.dv <= 4 * ASM_THREADS ? OGB_ASM(4) : OGB_ASM(16));
#undef OGB_ASM
  return ok ? 0 : -4;
}

}  // namespace ogb

using namespace ogb;

OGB_API int ogb_attention_simt(const OgbAttnLayer* a, const void* q, int q_stride, const void* k_cache, const void* v_cache, const int32_t* cu_seqlens,
                               const int32_t* past_lens, const int32_t* block_table, int table_cols, int block_size, void* out, int out_stride, int B,
                               int T, void* scratch, long long scratch_bytes, int fp32, void* stream_) {
  if (B <= 0 || T <= 0) return 0;
  if (a->dv > 16 * ASM_THREADS || a->dk > 8192 || a->Hq > 65535) return -5;
  OgbAttnLayer l = *a;
  if (l.maps < 1) l.maps = 1;
  if ((l.joint && l.maps > 1) || l.Hkv <= 0 || l.Hq % l.Hkv || l.dk % l.maps || block_size <= 0 || (l.raw && l.sinks)) return -1;
  if (l.raw && (long long)T * l.Hq * (l.dv + 2) * 4 > scratch_bytes) return -2;
  float* po = l.raw ? static_cast<float*>(scratch) : nullptr;
  float* ml = po ? po + size_t(T) * l.Hq * l.dv : nullptr;
  cudaStream_t s = static_cast<cudaStream_t>(stream_);
  return fp32 ? LaunchSimt<float>(l, q, q_stride, k_cache, v_cache, cu_seqlens, past_lens, block_table, table_cols, block_size, out, out_stride, B, T, po, ml, s)
              : LaunchSimt<__nv_bfloat16>(l, q, q_stride, k_cache, v_cache, cu_seqlens, past_lens, block_table, table_cols, block_size, out, out_stride, B, T,
                                          po, ml, s);
}

// part: the scratch of a raw attention call over part_tokens tokens with the given splits; its first T tokens are merged.
OGB_API int ogb_attention_diff_merge(const float* part, int splits, int T, int part_tokens, int H, int dv, int vdim, float lambda, float post, float eps,
                                     const void* gate, int gate_stride, void* out, int out_stride, int fp32, void* stream_) {
  if (T <= 0 || H <= 0) return 0;
  if (!part || splits < 1 || T > part_tokens || vdim <= 0 || vdim > dv) return -1;
  const int rows = part_tokens * 2 * H;
  const DiffMerge p{part, part + size_t(splits) * rows * dv, splits, rows, T, H, dv, vdim, lambda, post, eps, gate ? gate_stride : 0, out_stride};
  cudaStream_t s = static_cast<cudaStream_t>(stream_);
  return fp32 ? LaunchDiffMerge<float>(p, gate, out, s) : LaunchDiffMerge<__nv_bfloat16>(p, gate, out, s);
}
