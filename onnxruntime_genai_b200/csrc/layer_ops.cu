// Per-token kernels of the models that keep their residual stream in fp32, for bf16 and fp32 activations and any width:
//   embedding rows into the fp32 stream; RMS / layer norm of stream rows (optionally of selected rows only: the rows whose logits
//   are wanted); the gated activation act(gate) * up between two strided matrices; the causal depthwise convolution over the paged
//   window of earlier inputs.  Built without fast-math: the fp32 models are the exact form of the same code.
#include "common.cuh"
#include "kernels.h"

namespace ogb {

template <typename T> __device__ __forceinline__ float to_f32(T v);
template <> __device__ __forceinline__ float to_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f32<__nv_bfloat16>(__nv_bfloat16 v) { return bf2f(v); }
template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return f2bf(v); }

// ------------------------------------------------------------------------------------ embedding into the fp32 stream
template <typename T>
__global__ void embedding_stream_kernel(const int32_t* __restrict__ ids, const T* __restrict__ table, float* __restrict__ out, int H, int vocab,
                                        float scale) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  const int id = min(max(ids[t], 0), vocab - 1);
  for (int i = threadIdx.x; i < H; i += blockDim.x) out[size_t(t) * H + i] = to_f32(table[size_t(id) * H + i]) * scale;
}

// ------------------------------------------------------------------------------------ norm of the fp32 stream
// One CTA per output row; the row is kept in shared memory, the variance is taken from the deviations (a second pass over them).
template <typename T>
__global__ void __launch_bounds__(256) norm_stream_kernel(const float* __restrict__ x, const int32_t* __restrict__ rows, const float* __restrict__ w,
                                                          const float* __restrict__ b, T* __restrict__ out, int H, float eps, int layernorm) {
  extern __shared__ float row[];
  __shared__ float part[2][8];
  pdl_launch_dependents();
  pdl_wait();
  const float* src = x + size_t(rows ? rows[blockIdx.x] : blockIdx.x) * H;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  const bool vec = (H & 3) == 0;
  float sum = 0.f;
  if (vec) {
    for (int i = threadIdx.x; i < H / 4; i += blockDim.x) {
      const float4 v = reinterpret_cast<const float4*>(src)[i];
      reinterpret_cast<float4*>(row)[i] = v;
      sum += (v.x + v.y) + (v.z + v.w);
    }
  } else {
    for (int i = threadIdx.x; i < H; i += blockDim.x) { const float v = src[i]; row[i] = v; sum += v; }
  }
  float mean = 0.f;
  if (layernorm) {
    sum = warp_sum(sum);
    if (lane == 0) part[0][warp] = sum;
    __syncthreads();
    float t = 0.f;
    for (int i = 0; i < nw; ++i) t += part[0][i];
    mean = t / H;
  }
  float sq = 0.f;
  for (int i = threadIdx.x; i < (vec ? H / 4 : H); i += blockDim.x) {      // a thread re-reads what it stored itself
    if (vec) {
      const float4 v = reinterpret_cast<const float4*>(row)[i];
      const float a = v.x - mean, c = v.y - mean, d = v.z - mean, e = v.w - mean;
      sq += (a * a + c * c) + (d * d + e * e);
    } else {
      const float d = row[i] - mean;
      sq += d * d;
    }
  }
  sq = warp_sum(sq);
  if (lane == 0) part[1][warp] = sq;
  __syncthreads();
  float t = 0.f;
  for (int i = 0; i < nw; ++i) t += part[1][i];
  const float inv = 1.f / sqrtf(t / H + eps);
  T* dst = out + size_t(blockIdx.x) * H;
  if (vec) {
    for (int i = threadIdx.x; i < H / 4; i += blockDim.x) {
      const float4 v = reinterpret_cast<const float4*>(row)[i], g = reinterpret_cast<const float4*>(w)[i];
      float4 o = make_float4((v.x - mean) * inv * g.x, (v.y - mean) * inv * g.y, (v.z - mean) * inv * g.z, (v.w - mean) * inv * g.w);
      if (b) {
        const float4 c = reinterpret_cast<const float4*>(b)[i];
        o.x += c.x; o.y += c.y; o.z += c.z; o.w += c.w;
      }
      if constexpr (sizeof(T) == 4) reinterpret_cast<float4*>(dst)[i] = o;
      else reinterpret_cast<uint2*>(dst)[i] = make_uint2(pack_bf16x2(o.x, o.y), pack_bf16x2(o.z, o.w));
    }
  } else {
    for (int i = threadIdx.x; i < H; i += blockDim.x) dst[i] = from_f32<T>((row[i] - mean) * inv * w[i] + (b ? b[i] : 0.f));
  }
}

// ------------------------------------------------------------------------------------ act(gate) * up
// x row t: gate in columns [0, I), up in [I, 2I); out row t has I columns.  act: 0 SiLU, 1 GELU(tanh), 2 ReLU, 3 GELU(erf), 4 ReLU^2.
template <typename T>
__global__ void act_mul_rows_kernel(const T* __restrict__ x, int ldx, T* __restrict__ out, int ldo, int T_, int I, int act) {
  pdl_launch_dependents();
  pdl_wait();
  const long n = long(T_) * I;
  for (long idx = long(blockIdx.x) * blockDim.x + threadIdx.x; idx < n; idx += long(gridDim.x) * blockDim.x) {
    const long t = idx / I, i = idx % I;
    const float g = to_f32(x[t * ldx + i]), u = to_f32(x[t * ldx + I + i]);
    float a;
    if (act == 0) a = g / (1.f + expf(-g));
    else if (act == 1) a = 0.5f * g * (1.f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g)));
    else if (act == 2) a = fmaxf(g, 0.f);
    else if (act == 3) a = 0.5f * g * (1.f + erff(g * 0.7071067811865476f));
    else { const float r = fmaxf(g, 0.f); a = r * r; }
    out[t * ldo + i] = from_f32<T>(a * u);
  }
}

// ------------------------------------------------------------------------------------ causal depthwise convolution
// The gate-free form of short_conv_kernel (elementwise.cu) for any element type, channel count and alignment: one thread per
// (token, channel).  Inputs of earlier steps come from the paged cache [slots, row stride], this step's from x; x is appended.
template <typename T>
__global__ void causal_conv_rows_kernel(const T* __restrict__ x, int ldx, const T* __restrict__ w, const T* __restrict__ bias, T* __restrict__ cache,
                                        int ldcache, const int32_t* __restrict__ slots, const int32_t* __restrict__ positions,
                                        const int32_t* __restrict__ cu, const int32_t* __restrict__ past_lens, const int32_t* __restrict__ table,
                                        int table_cols, int block_size, T* __restrict__ out, int B, int C, int L, int silu) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  int lo = 0, hi = B - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (cu[mid] <= t) lo = mid; else hi = mid - 1;
  }
  const int r = lo, pos = positions[t], past = past_lens[r], t0 = cu[r], slot = slots[t];
  for (int c = threadIdx.x; c < C; c += blockDim.x) {
    float acc = bias ? to_f32(bias[c]) : 0.f;
    for (int k = 0; k < L; ++k) {
      const int q = pos - k;
      if (q < 0) break;
      float e;
      if (q >= past) e = to_f32(x[size_t(t0 + (q - past)) * ldx + c]);
      else e = to_f32(cache[(size_t(table[size_t(r) * table_cols + q / block_size]) * block_size + q % block_size) * ldcache + c]);
      acc = fmaf(to_f32(w[size_t(c) * L + (L - 1 - k)]), e, acc);
    }
    if (slot >= 0) cache[size_t(slot) * ldcache + c] = x[size_t(t) * ldx + c];
    out[size_t(t) * C + c] = from_f32<T>(silu ? acc / (1.f + expf(-acc)) : acc);
  }
}

}  // namespace ogb

using namespace ogb;

OGB_API int ogb_embedding_stream(const int32_t* ids, const void* table, int table_fp32, float* out, int T, int H, int vocab, float scale, void* stream) {
  if (T <= 0) return 0;
  auto s = static_cast<cudaStream_t>(stream);
  const dim3 block(H >= 256 ? 256 : 64);
  const bool ok = table_fp32 ? launch_pdl(embedding_stream_kernel<float>, dim3(T), block, 0, s, ids, static_cast<const float*>(table), out, H, vocab, scale)
                             : launch_pdl(embedding_stream_kernel<__nv_bfloat16>, dim3(T), block, 0, s, ids, static_cast<const __nv_bfloat16*>(table), out,
                                          H, vocab, scale);
  return ok ? 0 : -4;
}

// rows (may be null): out row i is the norm of x row rows[i].  w, b fp32 [H] (b may be null).
OGB_API int ogb_norm_stream(const float* x, const int32_t* rows, const float* w, const float* b, void* out, int out_fp32, int n_rows, int H, float eps,
                            int layernorm, void* stream) {
  if (n_rows <= 0) return 0;
  if (H <= 0 || H > 48 * 1024 / 4 - 64) return -1;
  auto s = static_cast<cudaStream_t>(stream);
  const dim3 block(H >= 1024 ? 256 : 128);
  const bool ok = out_fp32 ? launch_pdl(norm_stream_kernel<float>, dim3(n_rows), block, size_t(H) * 4, s, x, rows, w, b, static_cast<float*>(out), H, eps, layernorm)
                           : launch_pdl(norm_stream_kernel<__nv_bfloat16>, dim3(n_rows), block, size_t(H) * 4, s, x, rows, w, b,
                                        static_cast<__nv_bfloat16*>(out), H, eps, layernorm);
  return ok ? 0 : -4;
}

OGB_API int ogb_act_mul_rows(const void* x, int ldx, void* out, int ldo, int T, int I, int act, int fp32, void* stream) {
  if (T <= 0 || I <= 0) return 0;
  auto s = static_cast<cudaStream_t>(stream);
  const long nb = (long(T) * I + 255) / 256;
  const dim3 grid(unsigned(nb < 148 * 16 ? nb : 148 * 16));
  const bool ok = fp32 ? launch_pdl(act_mul_rows_kernel<float>, grid, dim3(256), 0, s, static_cast<const float*>(x), ldx, static_cast<float*>(out), ldo, T, I, act)
                       : launch_pdl(act_mul_rows_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, static_cast<const __nv_bfloat16*>(x), ldx,
                                    static_cast<__nv_bfloat16*>(out), ldo, T, I, act);
  return ok ? 0 : -4;
}

OGB_API int ogb_causal_conv_rows(const void* x, int ldx, const void* w, const void* bias, void* cache, int ldcache, const int32_t* slots,
                                 const int32_t* positions, const int32_t* cu_seqlens, const int32_t* past_lens, const int32_t* block_table,
                                 int table_cols, int block_size, void* out, int T, int B, int C, int L, int silu, int fp32, void* stream) {
  if (T <= 0) return 0;
  if (B <= 0 || C <= 0 || L < 1 || block_size <= 0) return -1;
  auto s = static_cast<cudaStream_t>(stream);
  const dim3 block(C >= 256 ? 256 : 64);
#define OGB_CONV_ARGS(TY) static_cast<const TY*>(x), ldx, static_cast<const TY*>(w), static_cast<const TY*>(bias), static_cast<TY*>(cache), ldcache, slots, \
                          positions, cu_seqlens, past_lens, block_table, table_cols, block_size, static_cast<TY*>(out), B, C, L, silu
  const bool ok = fp32 ? launch_pdl(causal_conv_rows_kernel<float>, dim3(T), block, 0, s, OGB_CONV_ARGS(float))
                       : launch_pdl(causal_conv_rows_kernel<__nv_bfloat16>, dim3(T), block, 0, s, OGB_CONV_ARGS(__nv_bfloat16));
#undef OGB_CONV_ARGS
  return ok ? 0 : -4;
}
