// Attention over a paged cache in plain fp32 arithmetic, for 32-bit models and for head sizes the tensor-core kernels cannot address: the
// same op as attention_mixed.cu (keys and values of different widths, window or own-run masks, sinks, a gate per head).
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
                                                                     int table_cols, int block_size, T* __restrict__ out, int out_stride, int B) {
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
  for (int i = threadIdx.x; i < a.dk; i += ASM_THREADS) sq[i] = as_f32(q[size_t(t) * q_stride + size_t(h) * a.dk + i]);
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
      const T* row = k_cache + (size_t(sslot[k]) * a.Hkv + g) * a.dk;
      float d = 0.f;
      for (int i = lane; i < a.dk; i += 32) d = fmaf(sq[i], as_f32(row[i]), d);
      d = warp_sum(d);
      if (lane == 0) ssc[k] = d * a.scale;
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
  if (a.gate) inv *= 1.f / (1.f + expf(-as_f32(static_cast<const T*>(a.gate)[size_t(t) * a.gate_stride + h])));
#pragma unroll
  for (int c = 0; c < COLS; ++c) {
    const int i = c * ASM_THREADS + threadIdx.x;
    if (i < a.dv) out[size_t(t) * out_stride + size_t(h) * a.dv + i] = of_f32<T>(acc[c] * inv);
  }
}

template <typename T>
static int LaunchSimt(const OgbAttnLayer& a, const void* q, int q_stride, const void* k, const void* v, const int32_t* cu, const int32_t* past,
                      const int32_t* table, int table_cols, int block_size, void* out, int out_stride, int B, int T_, cudaStream_t s) {
  const dim3 grid(T_, a.Hq);
  const size_t smem = size_t(a.dk) * 4;
#define OGB_ASM(C) launch_pdl(attention_simt_kernel<T, C>, grid, dim3(ASM_THREADS), smem, s, a, static_cast<const T*>(q), q_stride, static_cast<const T*>(k), \
                              static_cast<const T*>(v), cu, past, table, table_cols, block_size, static_cast<T*>(out), out_stride, B)
  const bool ok = a.dv <= ASM_THREADS ? OGB_ASM(1) : (a.dv <= 4 * ASM_THREADS ? OGB_ASM(4) : OGB_ASM(16));
#undef OGB_ASM
  return ok ? 0 : -4;
}

}  // namespace ogb

using namespace ogb;

OGB_API int ogb_attention_simt(const OgbAttnLayer* a, const void* q, int q_stride, const void* k_cache, const void* v_cache, const int32_t* cu_seqlens,
                               const int32_t* past_lens, const int32_t* block_table, int table_cols, int block_size, void* out, int out_stride, int B,
                               int T, int fp32, void* stream_) {
  if (B <= 0 || T <= 0) return 0;
  if (a->dv > 16 * ASM_THREADS || a->dk > 8192 || a->Hq > 65535) return -5;
  if (a->Hkv <= 0 || a->Hq % a->Hkv || block_size <= 0) return -1;
  cudaStream_t s = static_cast<cudaStream_t>(stream_);
  return fp32 ? LaunchSimt<float>(*a, q, q_stride, k_cache, v_cache, cu_seqlens, past_lens, block_table, table_cols, block_size, out, out_stride, B, T, s)
              : LaunchSimt<__nv_bfloat16>(*a, q, q_stride, k_cache, v_cache, cu_seqlens, past_lens, block_table, table_cols, block_size, out, out_stride, B, T, s);
}
