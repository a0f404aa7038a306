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
      const T* row = k_cache + (size_t(sslot[k]) * a.Hkv + g) * a.dk + c0;
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

// Differential attention on partial results: one warp per (token, head).  KEEP > 0: a lane keeps its columns (dv <= 32 * KEEP) in registers.
template <typename T, int KEEP>
__global__ void __launch_bounds__(128) attention_diff_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml, int splits,
                                                                   int rows_all, int T_, int H, int dv, int vdim, float lambda, float post, float eps,
                                                                   const T* __restrict__ gate, int gate_stride, T* __restrict__ out, int out_stride) {
  pdl_launch_dependents();
  pdl_wait();
  const long item = long(blockIdx.x) * 4 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (item >= long(T_) * H) return;
  const int t = int(item / H), h = int(item % H);
  const size_t row = size_t(t) * 2 * H + 2 * h;
  float top[2] = {-INFINITY, -INFINITY}, sum[2] = {0.f, 0.f};
  for (int s = 0; s < splits; ++s)
#pragma unroll
    for (int m = 0; m < 2; ++m) top[m] = fmaxf(top[m], part_ml[(size_t(s) * rows_all + row + m) * 2]);
  for (int s = 0; s < splits; ++s)
#pragma unroll
    for (int m = 0; m < 2; ++m) {
      const float* ml = part_ml + (size_t(s) * rows_all + row + m) * 2;
      if (ml[0] != -INFINITY) sum[m] += exp2f(ml[0] - top[m]) * ml[1];
    }
  const float inv1 = sum[0] > 0.f ? 1.f / sum[0] : 0.f, inv2 = sum[1] > 0.f ? lambda / sum[1] : 0.f;
  auto column = [&](int d) {
    float a = 0.f, b = 0.f;
    for (int s = 0; s < splits; ++s) {
      const size_t r = size_t(s) * rows_all + row;
      const float m1 = part_ml[r * 2], m2 = part_ml[r * 2 + 2];
      if (m1 != -INFINITY) a += exp2f(m1 - top[0]) * part_o[r * dv + d];
      if (m2 != -INFINITY) b += exp2f(m2 - top[1]) * part_o[(r + 1) * dv + d];
    }
    return a * inv1 - b * inv2;
  };
  float keep[KEEP > 0 ? KEEP : 1], sq = 0.f;
  if constexpr (KEEP > 0) {
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int d = lane + 32 * i;
      keep[i] = d < vdim ? column(d) : 0.f;
      sq = fmaf(keep[i], keep[i], sq);
    }
  } else {
    for (int d = lane; d < vdim; d += 32) { const float v = column(d); sq = fmaf(v, v, sq); }
  }
  const float f = post / sqrtf(warp_sum(sq) / vdim + eps);
  T* dst = out + size_t(t) * out_stride + size_t(h) * dv;
  const T* pg = gate ? gate + size_t(t) * gate_stride + size_t(h) * dv : nullptr;
  auto store = [&](int d, float v) { dst[d] = of_f32<T>(pg ? v * f / (1.f + expf(-as_f32(pg[d]))) : v * f); };
  if constexpr (KEEP > 0) {
#pragma unroll
    for (int i = 0; i < KEEP; ++i) if (lane + 32 * i < dv) store(lane + 32 * i, keep[i]);
  } else {
    for (int d = lane; d < dv; d += 32) store(d, d < vdim ? column(d) : 0.f);
  }
}

template <typename T>
static int LaunchDiffMerge(const float* po, const float* ml, int splits, int rows_all, int T_, int H, int dv, int vdim, float lambda, float post, float eps,
                           const void* gate, int gate_stride, void* out, int out_stride, cudaStream_t s) {
  const dim3 grid(unsigned((long(T_) * H + 3) / 4));
#define OGB_DIFF(K) launch_pdl(attention_diff_merge_kernel<T, K>, grid, dim3(128), 0, s, po, ml, splits, rows_all, T_, H, dv, vdim, lambda, post, eps, \
                               static_cast<const T*>(gate), gate_stride, static_cast<T*>(out), out_stride)
  const bool ok = dv <= 128 ? OGB_DIFF(4) : (dv <= 256 ? OGB_DIFF(8) : OGB_DIFF(0));
#undef OGB_DIFF
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
  if (l.Hkv <= 0 || l.Hq % l.Hkv || l.dk % l.maps || block_size <= 0 || (l.raw && l.sinks)) return -1;
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
  const float* ml = part + size_t(splits) * rows * dv;
  cudaStream_t s = static_cast<cudaStream_t>(stream_);
  return fp32 ? LaunchDiffMerge<float>(part, ml, splits, rows, T, H, dv, vdim, lambda, post, eps, gate, gate_stride, out, out_stride, s)
              : LaunchDiffMerge<__nv_bfloat16>(part, ml, splits, rows, T, H, dv, vdim, lambda, post, eps, gate, gate_stride, out, out_stride, s);
}
