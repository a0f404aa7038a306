// Per-token kernels of the models that keep their residual stream in fp32, for bf16 and fp32 activations and any width:
//   embedding rows into the fp32 stream, alone or with a row hashed from the previous token and this one; sums into the stream with a tanh norm
//   of the result; RMS / layer norm of stream rows (optionally of selected rows only: the rows whose logits
//   are wanted); the norm of a sub-layer's output added to the stream (with the weighted sum of routed experts folded in); head norms,
//   rotation and cache append of attention projections; the gated activation act(gate) * up between two strided matrices and the experts'
//   form of it; the causal depthwise convolution over the paged window of earlier inputs.  Built without fast-math: the fp32 models are the exact form of the same code.
#include "common.cuh"
#include "kernels.h"

namespace ogb {

template <typename T> __device__ __forceinline__ float to_f32(T v);
template <> __device__ __forceinline__ float to_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f32<__nv_bfloat16>(__nv_bfloat16 v) { return bf2f(v); }
template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return f2bf(v); }

template <typename T> __device__ __forceinline__ void load8(const T* p, float (&v)[8]);
template <> __device__ __forceinline__ void load8<float>(const float* p, float (&v)[8]) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
template <> __device__ __forceinline__ void load8<__nv_bfloat16>(const __nv_bfloat16* p, float (&v)[8]) {
  const uint4 q = *reinterpret_cast<const uint4*>(p);
  const float2 a = unpack_bf16x2(q.x), b = unpack_bf16x2(q.y), c = unpack_bf16x2(q.z), d = unpack_bf16x2(q.w);
  v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y; v[4] = c.x; v[5] = c.y; v[6] = d.x; v[7] = d.y;
}

// ------------------------------------------------------------------------------------ embedding into the fp32 stream
template <typename T>
__global__ void embedding_stream_kernel(const int32_t* __restrict__ ids, const T* __restrict__ table, float* __restrict__ out,
                                        __nv_bfloat16* __restrict__ copy, int H, int vocab, float scale) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  const int id = min(max(ids[t], 0), vocab - 1);
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    const float v = to_f32(table[size_t(id) * H + i]) * scale;
    out[size_t(t) * H + i] = v;
    if (copy) copy[size_t(t) * H + i] = f2bf(v);
  }
}

// ------------------------------------------------------------------------------------ embedding with hashed pairs
// One CTA per token (see OgbBigram).  The request of a token is found by all threads at once: a decode step is a chain of dependent loads.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) embedding_bigram_kernel(OgbBigram p, const T* __restrict__ table, const T* __restrict__ bigram,
                                                               float* __restrict__ out) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  const int id = p.ids[t], before = p.positions[t], slot = p.slots[t];
  const int prev_id = t > 0 ? p.ids[t - 1] : 0;
  int n = 0;                                           // requests that start at or before the token
  for (int i0 = 0; i0 < p.B; i0 += blockDim.x) {
    const int i = i0 + threadIdx.x;
    const int c = __syncthreads_count(i < p.B && p.cu_seqlens[i] <= t);
    n += c;
    if (c < int(blockDim.x)) break;
  }
  const int r = n - 1;
  long long row = p.buckets;
  if (before > 0) {
    int prev = prev_id;
    if (p.cu_seqlens[r] == t) {
      const int q = before - 1, block = p.block_table[size_t(r) * p.table_cols + q / p.block_size];
      prev = block >= 0 ? p.tokens[size_t(block) * p.block_size + q % p.block_size] : 0;
    }
    row = (prev * p.mul_prev + id * p.mul_cur) % p.buckets;
    if (row < 0) row += p.buckets;
  }
  if (threadIdx.x == 0 && slot >= 0) p.tokens[slot] = id;
  const T* a = table + size_t(min(max(id, 0), p.vocab - 1)) * p.H;
  const T* b = bigram + size_t(row) * p.H;
  float* dst = out + size_t(t) * p.H;
  for (int i = threadIdx.x * VEC; i < p.H; i += blockDim.x * VEC) {
    if constexpr (VEC == 8) {
      float x[8], y[8];
      load8(a + i, x);
      load8(b + i, y);
#pragma unroll
      for (int e = 0; e < 8; ++e) x[e] = fmaf(x[e], p.scale, y[e]);
      reinterpret_cast<float4*>(dst + i)[0] = make_float4(x[0], x[1], x[2], x[3]);
      reinterpret_cast<float4*>(dst + i)[1] = make_float4(x[4], x[5], x[6], x[7]);
    } else {
      dst[i] = fmaf(to_f32(a[i]), p.scale, to_f32(b[i]));
    }
  }
}

// ------------------------------------------------------------------------------------ norm of the fp32 stream
// (See OgbNormStream.)  One CTA per output row; the row is kept in shared memory, the variance is taken from the deviations (a second pass over
// them).  ADD: rows in T are added to the stream's row first.
template <typename T>
__device__ __forceinline__ float4 added4(const OgbNormStream& p, int t, int i, float4 v) {
  auto one = [&](const T* y, float w) {
    float2 a, c;
    if constexpr (sizeof(T) == 4) {
      const float4 q = *reinterpret_cast<const float4*>(y);
      a = make_float2(q.x, q.y); c = make_float2(q.z, q.w);
    } else {
      const uint2 q = *reinterpret_cast<const uint2*>(y);
      a = unpack_bf16x2(q.x); c = unpack_bf16x2(q.y);
    }
    v.x = fmaf(w, a.x, v.x); v.y = fmaf(w, a.y, v.y); v.z = fmaf(w, c.x, v.z); v.w = fmaf(w, c.y, v.w);
  };
  const T* y = static_cast<const T*>(p.y) + i;
  if (!p.inv_pos) {
    one(y + size_t(t) * p.ldy, 1.f);
    return v;
  }
#pragma unroll 4
  for (int j = 0; j < p.k; ++j) {
    const int r = p.inv_pos[size_t(t) * p.k + j];
    if (r >= 0) one(y + size_t(r) * p.ldy, p.topk_w[size_t(t) * p.k + j]);
  }
  return v;
}

template <typename T, bool ADD>
__global__ void __launch_bounds__(256) norm_stream_kernel(OgbNormStream p) {
  extern __shared__ float row[];
  __shared__ float part[2][8];
  pdl_launch_dependents();
  pdl_wait();
  const int H = p.H, t0 = p.rows ? p.rows[blockIdx.x] : blockIdx.x;
  float* src = p.x + size_t(t0) * H;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  const bool vec = (H & 3) == 0 && (!ADD || (p.ldy & 3) == 0);
  const float eps = p.eps;
  const int layernorm = p.layernorm;
  float sum = 0.f;
  if (vec) {
    for (int i = threadIdx.x; i < H / 4; i += blockDim.x) {
      float4 v = reinterpret_cast<const float4*>(src)[i];
      if constexpr (ADD) {
        v = added4<T>(p, t0, i * 4, v);
        if (!p.rows) reinterpret_cast<float4*>(src)[i] = v;
      }
      reinterpret_cast<float4*>(row)[i] = v;
      sum += (v.x + v.y) + (v.z + v.w);
    }
  } else {
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
      float v = src[i];
      if constexpr (ADD) {
        const T* y = static_cast<const T*>(p.y) + i;
        if (!p.inv_pos) v += to_f32(y[size_t(t0) * p.ldy]);
        else
          for (int j = 0; j < p.k; ++j) {
            const int r = p.inv_pos[size_t(t0) * p.k + j];
            if (r >= 0) v = fmaf(p.topk_w[size_t(t0) * p.k + j], to_f32(y[size_t(r) * p.ldy]), v);
          }
        if (!p.rows) src[i] = v;
      }
      row[i] = v;
      sum += v;
    }
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
  T* dst = static_cast<T*>(p.out) + size_t(blockIdx.x) * H;
  T* dst2 = p.w2 ? static_cast<T*>(p.out2) + size_t(blockIdx.x) * H : nullptr;
  if (vec) {
    auto put = [&](T* d, int i, float4 o) {
      if constexpr (sizeof(T) == 4) reinterpret_cast<float4*>(d)[i] = o;
      else reinterpret_cast<uint2*>(d)[i] = make_uint2(pack_bf16x2(o.x, o.y), pack_bf16x2(o.z, o.w));
    };
    for (int i = threadIdx.x; i < H / 4; i += blockDim.x) {
      const float4 v = reinterpret_cast<const float4*>(row)[i], g = reinterpret_cast<const float4*>(p.w)[i];
      const float4 u = make_float4((v.x - mean) * inv, (v.y - mean) * inv, (v.z - mean) * inv, (v.w - mean) * inv);
      float4 o = make_float4(u.x * g.x, u.y * g.y, u.z * g.z, u.w * g.w);
      if (p.b) {
        const float4 c = reinterpret_cast<const float4*>(p.b)[i];
        o.x += c.x; o.y += c.y; o.z += c.z; o.w += c.w;
      }
      put(dst, i, o);
      if (dst2) {
        const float4 e = reinterpret_cast<const float4*>(p.w2)[i];
        put(dst2, i, make_float4(u.x * e.x, u.y * e.y, u.z * e.z, u.w * e.w));
      }
    }
  } else {
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
      const float u = (row[i] - mean) * inv;
      dst[i] = from_f32<T>(u * p.w[i] + (p.b ? p.b[i] : 0.f));
      if (dst2) dst2[i] = from_f32<T>(u * p.w2[i]);
    }
  }
}

// ------------------------------------------------------------------------------------ normed output of a sub-layer, added to the stream
// One CTA per token.  The sub-layer's row v is y[t], or the weighted sum of the experts' rows that served the token (inv_pos: their rows in
// y, topk_w: their weights, in the order of the choice).  h[t] += w * v / sqrt(mean(v^2) + eps); x[t]: the new row as bf16 (may be null).
constexpr int ADN_VEC = 8, ADN_KEEP = 4;      // columns per piece, pieces a thread keeps in registers
struct AddNormed {
  float* h; const float* w; __nv_bfloat16* x;
  const int32_t* inv_pos; const float* topk_w;
  int k, ldy, H;
  float eps;
};

template <typename T>
__device__ __forceinline__ float add_normed_col(const AddNormed& p, const T* y, int t, int i) {
  if (!p.inv_pos) return to_f32(y[size_t(t) * p.ldy + i]);
  float v = 0.f;
  for (int j = 0; j < p.k; ++j) {
    const int r = p.inv_pos[size_t(t) * p.k + j];
    if (r >= 0) v = fmaf(p.topk_w[size_t(t) * p.k + j], to_f32(y[size_t(r) * p.ldy + i]), v);
  }
  return v;
}

template <typename T, bool VEC>
__global__ void __launch_bounds__(256) add_normed_kernel(const T* __restrict__ y, AddNormed p) {
  __shared__ float part[8];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  float sq = 0.f;
  auto inv_rms = [&]() {
    sq = warp_sum(sq);
    if (lane == 0) part[warp] = sq;
    __syncthreads();
    float s = 0.f;
    for (int i = 0; i < nw; ++i) s += part[i];
    return 1.f / sqrtf(s / p.H + p.eps);
  };
  if constexpr (VEC) {
    const int nv = p.H / ADN_VEC;
    float v[ADN_KEEP][ADN_VEC];
#pragma unroll
    for (int c = 0; c < ADN_KEEP; ++c) {
      const int i = c * blockDim.x + threadIdx.x;
      if (i >= nv) break;
      if (!p.inv_pos) {
        load8(y + size_t(t) * p.ldy + i * ADN_VEC, v[c]);
      } else {
#pragma unroll
        for (int e = 0; e < ADN_VEC; ++e) v[c][e] = 0.f;
        for (int j = 0; j < p.k; ++j) {
          const int r = p.inv_pos[size_t(t) * p.k + j];
          if (r < 0) continue;
          const float wj = p.topk_w[size_t(t) * p.k + j];
          float u[ADN_VEC];
          load8(y + size_t(r) * p.ldy + i * ADN_VEC, u);
#pragma unroll
          for (int e = 0; e < ADN_VEC; ++e) v[c][e] = fmaf(wj, u[e], v[c][e]);
        }
      }
#pragma unroll
      for (int e = 0; e < ADN_VEC; ++e) sq = fmaf(v[c][e], v[c][e], sq);
    }
    const float inv = inv_rms();
#pragma unroll
    for (int c = 0; c < ADN_KEEP; ++c) {
      const int i = c * blockDim.x + threadIdx.x;
      if (i >= nv) break;
      float hv[ADN_VEC], wv[ADN_VEC];
      float* hp = p.h + size_t(t) * p.H + i * ADN_VEC;
      load8<float>(hp, hv);
      load8<float>(p.w + i * ADN_VEC, wv);
#pragma unroll
      for (int e = 0; e < ADN_VEC; ++e) hv[e] = fmaf(v[c][e] * inv, wv[e], hv[e]);
      reinterpret_cast<float4*>(hp)[0] = make_float4(hv[0], hv[1], hv[2], hv[3]);
      reinterpret_cast<float4*>(hp)[1] = make_float4(hv[4], hv[5], hv[6], hv[7]);
      if (p.x)
        *reinterpret_cast<uint4*>(p.x + size_t(t) * p.H + i * ADN_VEC) =
            make_uint4(pack_bf16x2(hv[0], hv[1]), pack_bf16x2(hv[2], hv[3]), pack_bf16x2(hv[4], hv[5]), pack_bf16x2(hv[6], hv[7]));
    }
  } else {
    for (int i = threadIdx.x; i < p.H; i += blockDim.x) {
      const float v = add_normed_col(p, y, t, i);
      sq = fmaf(v, v, sq);
    }
    const float inv = inv_rms();
    for (int i = threadIdx.x; i < p.H; i += blockDim.x) {
      const size_t at = size_t(t) * p.H + i;
      const float n = fmaf(add_normed_col(p, y, t, i) * inv, p.w[i], p.h[at]);
      p.h[at] = n;
      if (p.x) p.x[at] = f2bf(n);
    }
  }
}

// ------------------------------------------------------------------------------------ sums into the stream, tanh norm of the result
// (See OgbTanhNorm.)  Every column is on its own: blockIdx.y walks pieces of a row, VEC columns per thread.
template <typename T, int VEC>
__global__ void __launch_bounds__(128) add_tanh_norm_kernel(OgbTanhNorm p) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = p.rows ? p.rows[blockIdx.x] : blockIdx.x, i = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
  if (i >= p.H) return;
  auto load = [&](const auto* src, float (&v)[VEC]) {
    if constexpr (VEC == 8) load8(src, v); else v[0] = to_f32(*src);
  };
  const size_t at = size_t(t) * p.H + i;
  float n[VEC], u[VEC];
  load(p.h_in + at, n);
  auto add = [&](float w) {
#pragma unroll
    for (int e = 0; e < VEC; ++e) n[e] = fmaf(w, u[e], n[e]);
  };
  const T* y = static_cast<const T*>(p.y);
  if (p.inv_pos) {
    for (int j = 0; j < p.k; ++j) {
      const int r = p.inv_pos[size_t(t) * p.k + j];
      if (r < 0) continue;
      load(y + size_t(r) * p.ldy + i, u);
      add(p.topk_w[size_t(t) * p.k + j]);
    }
  } else if (y) {
    load(y + size_t(t) * p.ldy + i, u);
    add(1.f);
  }
  if (p.y2) { load(static_cast<const T*>(p.y2) + size_t(t) * p.ldy2 + i, u); add(1.f); }
  if (p.first) { load(p.first + at, u); add(1.f); }
  if (p.step) { load(p.step + i, u); add(1.f); }
  float w[VEC], b[VEC];
  load(p.w + i, w);
  load(p.b + i, b);
  if constexpr (VEC == 8) {
    if (p.h_out) {
      reinterpret_cast<float4*>(p.h_out + at)[0] = make_float4(n[0], n[1], n[2], n[3]);
      reinterpret_cast<float4*>(p.h_out + at)[1] = make_float4(n[4], n[5], n[6], n[7]);
    }
  } else {
    if (p.h_out) p.h_out[at] = n[0];
  }
#pragma unroll
  for (int e = 0; e < VEC; ++e) n[e] = fmaf(tanhf(p.alpha * n[e]), w[e], b[e]);
  T* dst = static_cast<T*>(p.x) + size_t(blockIdx.x) * p.H + i;
  if constexpr (VEC == 1) dst[0] = from_f32<T>(n[0]);
  else if constexpr (sizeof(T) == 4) {
    reinterpret_cast<float4*>(dst)[0] = make_float4(n[0], n[1], n[2], n[3]);
    reinterpret_cast<float4*>(dst)[1] = make_float4(n[4], n[5], n[6], n[7]);
  } else {
    *reinterpret_cast<uint4*>(dst) = make_uint4(pack_bf16x2(n[0], n[1]), pack_bf16x2(n[2], n[3]), pack_bf16x2(n[4], n[5]), pack_bf16x2(n[6], n[7]));
  }
}

// ------------------------------------------------------------------------------------ head norms, rotation, cache append
// One warp per (token, head).  Query heads are replaced in place; key heads go to the token's cache row; value heads are copied there.
// A lane handles pairs of columns (i, i + rot / 2) of the rotated part and single columns of the rest, V at a time.
struct QkvPrep {
  int ldp, Hq, Hkv, Hv, dim, key_row, value_row, rot, max_pos, T;
  const float *q_norm, *k_norm, *cos, *sin;
  const int32_t *positions, *slots;
  float eps;
};

template <typename T, int V> __device__ __forceinline__ void ld_cols(const T* p, float (&f)[V]) {
  if constexpr (V == 1) f[0] = to_f32(p[0]);
  else if constexpr (sizeof(T) == 4) { const float2 a = *reinterpret_cast<const float2*>(p); f[0] = a.x; f[1] = a.y; }
  else { const float2 a = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(p)); f[0] = a.x; f[1] = a.y; }
}
template <typename T, int V> __device__ __forceinline__ void st_cols(T* p, const float (&f)[V]) {
  if constexpr (V == 1) p[0] = from_f32<T>(f[0]);
  else if constexpr (sizeof(T) == 4) *reinterpret_cast<float2*>(p) = make_float2(f[0], f[1]);
  else *reinterpret_cast<uint32_t*>(p) = pack_bf16x2(f[0], f[1]);
}

// V = 2: two neighbouring columns at a time (dim and rot / 2 even, rows on even addresses), 1: any size.
template <typename T, int V>
__global__ void __launch_bounds__(256) qkv_prep_kernel(T* __restrict__ proj, T* __restrict__ k_cache, T* __restrict__ v_cache, QkvPrep p) {
  pdl_launch_dependents();
  pdl_wait();
  const int per = p.Hq + p.Hkv + p.Hv;
  const long item = long(blockIdx.x) * 8 + (threadIdx.x >> 5);
  if (item >= long(p.T) * per) return;
  const int t = int(item / per), head = int(item % per), lane = threadIdx.x & 31;
  T* row = proj + size_t(t) * p.ldp;
  const int slot = p.slots[t];
  if (head >= p.Hq + p.Hkv) {
    const int g = head - p.Hq - p.Hkv;
    if (slot < 0) return;
    const T* src = row + size_t(p.Hq + p.Hkv) * p.key_row + size_t(g) * p.value_row;
    T* dst = v_cache + (size_t(slot) * p.Hv + g) * p.value_row;
    for (int i = lane * V; i < p.value_row; i += 32 * V) {
      float f[V];
      ld_cols<T, V>(src + i, f);
      st_cols<T, V>(dst + i, f);
    }
    return;
  }
  const bool is_q = head < p.Hq;
  if (!is_q && slot < 0) return;
  T* src = row + size_t(head) * p.key_row;
  T* dst = is_q ? src : k_cache + (size_t(slot) * p.Hkv + (head - p.Hq)) * p.key_row;
  const float* w = is_q ? p.q_norm : p.k_norm;
  float inv = 1.f;
  if (w) {
    float sq = 0.f;
    for (int i = lane * V; i < p.dim; i += 32 * V) {
      float f[V];
      ld_cols<T, V>(src + i, f);
#pragma unroll
      for (int e = 0; e < V; ++e) sq = fmaf(f[e], f[e], sq);
    }
    inv = 1.f / sqrtf(warp_sum(sq) / p.dim + p.eps);
  }
  const int half = p.rot >> 1;
  const int pos = min(max(p.positions[t], 0), p.max_pos - 1);
  auto normed = [&](int i, float (&f)[V]) {
    ld_cols<T, V>(src + i, f);
    if (w) {
#pragma unroll
      for (int e = 0; e < V; ++e) f[e] = f[e] * inv * w[i + e];
    }
  };
  for (int i = lane * V; i < half; i += 32 * V) {
    float a[V], b[V], u[V], v[V];
    normed(i, a);
    normed(i + half, b);
#pragma unroll
    for (int e = 0; e < V; ++e) {
      const float c = p.cos[size_t(pos) * half + i + e], s = p.sin[size_t(pos) * half + i + e];
      u[e] = a[e] * c - b[e] * s;
      v[e] = b[e] * c + a[e] * s;
    }
    st_cols<T, V>(dst + i, u);
    st_cols<T, V>(dst + i + half, v);
  }
  for (int i = p.rot + lane * V; i < p.dim; i += 32 * V) {
    float f[V];
    normed(i, f);
    st_cols<T, V>(dst + i, f);
  }
  for (int i = p.dim + lane; i < p.key_row; i += 32) dst[i] = from_f32<T>(0.f);
}

// The same without norms, where every part is whole pieces of 8 columns (dim, rot / 2, value_row): one thread per piece, a rotated piece with its
// partner half a rotation away.
template <typename T>
__global__ void __launch_bounds__(256) qkv_prep_pieces_kernel(T* __restrict__ proj, T* __restrict__ k_cache, T* __restrict__ v_cache, QkvPrep p) {
  pdl_launch_dependents();
  pdl_wait();
  const int half = p.rot >> 1, turn = half / 8, kp = p.key_row / 8 - turn, vp = p.value_row / 8;      // pieces of a query or key head, of a value head
  const int t = blockIdx.x, n_qk = (p.Hq + p.Hkv) * kp, n = n_qk + p.Hv * vp;
  T* row = proj + size_t(t) * p.ldp;
  const int slot = p.slots[t];
  const size_t at = size_t(min(max(p.positions[t], 0), p.max_pos - 1)) * half;
  for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < n; i += gridDim.y * blockDim.x) {
    float a[8], b[8];
    auto st8 = [](T* dst, const float (&v)[8]) {
      if constexpr (sizeof(T) == 4) {
        reinterpret_cast<float4*>(dst)[0] = make_float4(v[0], v[1], v[2], v[3]);
        reinterpret_cast<float4*>(dst)[1] = make_float4(v[4], v[5], v[6], v[7]);
      } else {
        *reinterpret_cast<uint4*>(dst) = make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
      }
    };
    if (i >= n_qk) {
      if (slot < 0) continue;
      const int j = (i - n_qk) * 8;
      load8(row + size_t(p.Hq + p.Hkv) * p.key_row + j, a);
      st8(v_cache + size_t(slot) * p.Hv * p.value_row + j, a);
      continue;
    }
    const int head = i / kp, c = i - head * kp;
    const bool is_q = head < p.Hq;
    if (!is_q && slot < 0) continue;
    T* src = row + size_t(head) * p.key_row;
    T* dst = is_q ? src : k_cache + (size_t(slot) * p.Hkv + (head - p.Hq)) * p.key_row;
    if (c < turn) {
      float cs[8], sn[8], u[8], v[8];
      load8(src + c * 8, a);
      load8(src + half + c * 8, b);
      load8(p.cos + at + c * 8, cs);
      load8(p.sin + at + c * 8, sn);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        u[e] = a[e] * cs[e] - b[e] * sn[e];
        v[e] = b[e] * cs[e] + a[e] * sn[e];
      }
      st8(dst + c * 8, u);
      st8(dst + half + c * 8, v);
    } else if (!is_q) {                                // (unrotated columns of a query stay where they are)
      const int j = p.rot + (c - turn) * 8;
      load8(src + j, a);
      st8(dst + j, a);
    }
  }
}

// The same for heads whose scores are mixed: head h's scores are sum_g talk[h, g] * (scores of g), so with the queries of a key head's group G_c mixed
// into one query part, m[h, c] = sum over g in G_c of talk[h, g] q_g, they are the product of [m[h, 0] | m[h, 1] | ...] with the keys of all key
// heads side by side.  The parts are summed in fp32 from the normed and rotated queries and rounded once.  One CTA per token: its warps prepare heads
// (queries into shared memory, keys and values to the cache), then every thread mixes columns; rows of `mixed` are [Hq][Hkv][key_row].
template <typename T>
__global__ void __launch_bounds__(256) qkv_prep_mixed_kernel(const T* __restrict__ proj, T* __restrict__ k_cache, T* __restrict__ v_cache, QkvPrep p,
                                                             const float* __restrict__ talk, T* __restrict__ mixed) {
  extern __shared__ float sm[];
  float* st = sm;                            // [Hq][Hq]
  float* sq = sm + (p.Hq * p.Hq + 1) / 2 * 2;      // [Hq][key_row]
  pdl_launch_dependents();
  for (int i = threadIdx.x; i < p.Hq * p.Hq; i += blockDim.x) st[i] = talk[i];
  pdl_wait();
  const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  const T* row = proj + size_t(t) * p.ldp;
  const int slot = p.slots[t], half = p.rot >> 1;
  const size_t at = size_t(min(max(p.positions[t], 0), p.max_pos - 1)) * half;
  for (int head = warp; head < p.Hq + p.Hkv; head += nw) {
    const bool is_q = head < p.Hq;
    const T* src = row + size_t(head) * p.key_row;
    const float* w = is_q ? p.q_norm : p.k_norm;
    float inv = 1.f;
    if (w) {
      float sq2 = 0.f;
      for (int i = lane; i < p.dim; i += 32) { const float f = to_f32(src[i]); sq2 = fmaf(f, f, sq2); }
      inv = 1.f / sqrtf(warp_sum(sq2) / p.dim + p.eps);
    }
    auto normed = [&](int i) { const float f = to_f32(src[i]); return w ? f * inv * w[i] : f; };
    T* dst = is_q || slot < 0 ? nullptr : k_cache + (size_t(slot) * p.Hkv + (head - p.Hq)) * p.key_row;
    auto put = [&](int i, float f) {
      if (is_q) sq[head * p.key_row + i] = f;
      else if (dst) dst[i] = from_f32<T>(f);
    };
    for (int i = lane; i < half; i += 32) {
      const float a = normed(i), b = normed(i + half), c = p.cos[at + i], s = p.sin[at + i];
      put(i, a * c - b * s);
      put(i + half, b * c + a * s);
    }
    for (int i = p.rot + lane; i < p.key_row; i += 32) put(i, i < p.dim ? normed(i) : 0.f);
  }
  if (slot >= 0) {
    const T* src = row + size_t(p.Hq + p.Hkv) * p.key_row;
    T* dst = v_cache + size_t(slot) * p.Hv * p.value_row;
    for (int i = threadIdx.x; i < p.Hv * p.value_row; i += blockDim.x) dst[i] = src[i];
  }
  __syncthreads();
  const int G = p.Hq / p.Hkv, cols = p.Hkv * p.key_row;
  T* out = mixed + size_t(t) * p.Hq * cols;
  for (int i = threadIdx.x * 2; i < p.Hq * cols; i += blockDim.x * 2) {      // (key_row is a multiple of 8)
    const int h = i / cols, c = (i - h * cols) / p.key_row, d = i % p.key_row;
    const float* q = sq + c * G * p.key_row + d;
    const float* m = st + h * p.Hq + c * G;
    float f[2] = {0.f, 0.f};
    for (int g = 0; g < G; ++g) {
      const float2 v = *reinterpret_cast<const float2*>(q + g * p.key_row);
      f[0] = fmaf(m[g], v.x, f[0]);
      f[1] = fmaf(m[g], v.y, f[1]);
    }
    st_cols<T, 2>(out + i, f);
  }
}

// The same where every part is whole pieces of 8 columns (dim = key_row, rot / 2, value_row) and a head at most 32 pieces: LPH lanes per head (a power of two),
// one piece each, norms and the partners of a rotation by shuffles; then a thread mixes a piece of a key head's queries into four heads at a time.  Steps of few
// tokens: the CTAs (t, y) of a token have `per_cta` key heads each, with their queries and values.
template <typename T> __device__ __forceinline__ void store8(T* dst, const float (&v)[8]) {
  if constexpr (sizeof(T) == 4) {
    reinterpret_cast<float4*>(dst)[0] = make_float4(v[0], v[1], v[2], v[3]);
    reinterpret_cast<float4*>(dst)[1] = make_float4(v[4], v[5], v[6], v[7]);
  } else {
    *reinterpret_cast<uint4*>(dst) = make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
  }
}

template <typename T>
__global__ void __launch_bounds__(256) qkv_prep_mixed_pieces_kernel(const T* __restrict__ proj, T* __restrict__ k_cache, T* __restrict__ v_cache, QkvPrep p,
                                                                    const float* __restrict__ talk, T* __restrict__ mixed, int LPH,
                                                                    int per_cta) {
  extern __shared__ __align__(16) float sm[];
  const int G = p.Hq / p.Hkv, c0 = blockIdx.y * per_cta, nc = min(per_cta, p.Hkv - c0), q0 = c0 * G, nq = nc * G;      // key heads and queries of this CTA
  float* sq = sm;                            // [nq][dim]
  float* st = sm + nq * p.dim;               // [Hq][nq]
  pdl_launch_dependents();
  if (nq == p.Hq)
    for (int i = threadIdx.x; i < p.Hq * nq; i += blockDim.x) st[i] = talk[i];
  else
    for (int i = threadIdx.x; i < p.Hq * nq; i += blockDim.x) st[i] = talk[i / nq * p.Hq + q0 + i % nq];
  pdl_wait();
  const int t = blockIdx.x, tid = threadIdx.x, dim = p.dim, half = p.rot >> 1, turn = half / 8;
  const T* row = proj + size_t(t) * p.ldp;
  const int slot = p.slots[t], heads = nq + nc;
  const size_t at = size_t(min(max(p.positions[t], 0), p.max_pos - 1)) * half;
  const int l = tid % LPH, per = blockDim.x / LPH;
  for (int h0 = 0; h0 < heads; h0 += per) {
    const int head = h0 + tid / LPH;
    const bool is_q = head < nq, live = head < heads && l * 8 < dim;
    float f[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (live) load8(row + size_t(is_q ? q0 + head : p.Hq + c0 + head - nq) * dim + l * 8, f);
    const float* w = is_q ? p.q_norm : p.k_norm;
    if (p.q_norm || p.k_norm) {
      float ss = 0.f;
#pragma unroll
      for (int e = 0; e < 8; ++e) ss = fmaf(f[e], f[e], ss);
      for (int o = LPH >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      if (w && live) {
        const float inv = 1.f / sqrtf(ss / dim + p.eps);
        float g[8];
        load8(w + l * 8, g);
#pragma unroll
        for (int e = 0; e < 8; ++e) f[e] = f[e] * inv * g[e];
      }
    }
    if (turn > 0) {
      // lanes [0, turn) hold the first halves, [turn, 2 turn) the second ones
      const bool first = l < turn, turns = l < 2 * turn;
      const int lane = tid & 31, from = turns ? (first ? lane + turn : lane - turn) : lane;
      float cs[8], sn[8], o[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) o[e] = __shfl_sync(0xffffffffu, f[e], from);
      if (turns) {
        load8(p.cos + at + (first ? l : l - turn) * 8, cs);
        load8(p.sin + at + (first ? l : l - turn) * 8, sn);
#pragma unroll
        for (int e = 0; e < 8; ++e) f[e] = first ? f[e] * cs[e] - o[e] * sn[e] : f[e] * cs[e] + o[e] * sn[e];
      }
    }
    if (live) {
      if (is_q) store8(sq + head * dim + l * 8, f);
      else if (slot >= 0) store8(k_cache + (size_t(slot) * p.Hkv + c0 + head - nq) * dim + l * 8, f);
    }
  }
  if (slot >= 0)
    for (int i = blockIdx.y * blockDim.x + tid; i < p.Hv * p.value_row / 8; i += gridDim.y * blockDim.x) {
      float f[8];
      load8(row + size_t(p.Hq + p.Hkv) * dim + i * 8, f);
      store8(v_cache + size_t(slot) * p.Hv * p.value_row + i * 8, f);
    }
  __syncthreads();
  const int dp = dim / 8, items = nc * dp;      // item: (key head, piece)
  T* out = mixed + size_t(t) * p.Hq * p.Hkv * dim;
  for (int i = tid; i < (p.Hq + 3) / 4 * items; i += blockDim.x) {
    const int hb = i / items * 4, item = i % items, c = item / dp, d = (item - c * dp) * 8;
    float acc[4][8] = {};
    for (int g = 0; g < G; ++g) {
      float q[8];
      load8<float>(sq + (c * G + g) * dim + d, q);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float m = hb + j < p.Hq ? st[(hb + j) * nq + c * G + g] : 0.f;
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[j][e] = fmaf(m, q[e], acc[j][e]);
      }
    }
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (hb + j < p.Hq) store8(out + (size_t(hb + j) * p.Hkv + c0 + c) * dim + d, acc[j]);
  }
}

// ------------------------------------------------------------------------------------ experts' activations
// Rows of alternating (gate, up) columns.  kind 0: silu(g) * u; 1: min(g, limit) * sigmoid(alpha * min(g, limit)) * (clamp(u, +-limit) + 1).
// Rows without gates: kind 2: max(x, 0)^2.
template <typename T>
__global__ void expert_act_kernel(const T* __restrict__ gu, T* __restrict__ out, long n, int kind, float alpha, float limit) {
  pdl_launch_dependents();
  pdl_wait();
  for (long i = long(blockIdx.x) * blockDim.x + threadIdx.x; i < n; i += long(gridDim.x) * blockDim.x) {
    if (kind == 2) {
      const float x = fmaxf(to_f32(gu[i]), 0.f);
      out[i] = from_f32<T>(x * x);
      continue;
    }
    float g = to_f32(gu[2 * i]), u = to_f32(gu[2 * i + 1]), r;
    if (kind == 0) {
      r = g / (1.f + expf(-g)) * u;
    } else {
      if (limit > 0.f) { g = fminf(g, limit); u = fminf(fmaxf(u, -limit), limit); }
      r = g / (1.f + expf(-alpha * g)) * (u + 1.f);
    }
    out[i] = from_f32<T>(r);
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

OGB_API int ogb_embedding_stream(const int32_t* ids, const void* table, int table_fp32, float* out, void* copy, int T, int H, int vocab, float scale,
                                 void* stream) {
  if (T <= 0) return 0;
  auto s = static_cast<cudaStream_t>(stream);
  const dim3 block(H >= 256 ? 256 : 64);
  const bool ok = table_fp32 ? launch_pdl(embedding_stream_kernel<float>, dim3(T), block, 0, s, ids, static_cast<const float*>(table), out,
                                          static_cast<__nv_bfloat16*>(copy), H, vocab, scale)
                             : launch_pdl(embedding_stream_kernel<__nv_bfloat16>, dim3(T), block, 0, s, ids, static_cast<const __nv_bfloat16*>(table), out,
                                          static_cast<__nv_bfloat16*>(copy), H, vocab, scale);
  return ok ? 0 : -4;
}

OGB_API int ogb_embedding_bigram(const OgbBigram* p, const void* table, const void* bigram, float* out, void* stream) {
  if (p->T <= 0) return 0;
  if (p->B <= 0 || p->H <= 0 || p->vocab <= 0 || p->buckets <= 0 || p->block_size <= 0) return -1;
  auto s = static_cast<cudaStream_t>(stream);
  const bool vec = p->H % 8 == 0 && ((reinterpret_cast<uintptr_t>(table) | reinterpret_cast<uintptr_t>(bigram) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
  const int pieces = vec ? p->H / 8 : p->H;
  const dim3 block(pieces >= 256 ? 256 : (pieces + 31) / 32 * 32);
#define OGB_PAIRS(TY, V) launch_pdl(embedding_bigram_kernel<TY, V>, dim3(p->T), block, 0, s, *p, static_cast<const TY*>(table), static_cast<const TY*>(bigram), out)
  const bool ok = p->fp32 ? (vec ? OGB_PAIRS(float, 8) : OGB_PAIRS(float, 1)) : (vec ? OGB_PAIRS(__nv_bfloat16, 8) : OGB_PAIRS(__nv_bfloat16, 1));
#undef OGB_PAIRS
  return ok ? 0 : -4;
}

OGB_API int ogb_add_tanh_norm(const OgbTanhNorm* p, void* stream) {
  if (p->n_rows <= 0 || p->H <= 0) return 0;
  if (!p->h_in || !p->w || !p->b || !p->x || (p->inv_pos && (!p->y || !p->topk_w))) return -1;
  auto s = static_cast<cudaStream_t>(stream);
  auto addr = [](const void* a) { return reinterpret_cast<uintptr_t>(a); };
  const bool vec = p->H % 8 == 0 && (!p->y || p->ldy % 8 == 0) && (!p->y2 || p->ldy2 % 8 == 0) &&
                   ((addr(p->h_in) | addr(p->h_out) | addr(p->y) | addr(p->y2) | addr(p->first) | addr(p->step) | addr(p->w) | addr(p->b) | addr(p->x)) & 15) == 0;
  const int pieces = vec ? p->H / 8 : p->H;
  const dim3 block(pieces < 128 ? (pieces + 31) / 32 * 32 : 128), grid(p->n_rows, (pieces + block.x - 1) / block.x);
  if (grid.y > 65535) return -1;
  const bool ok = p->fp32 ? (vec ? launch_pdl(add_tanh_norm_kernel<float, 8>, grid, block, 0, s, *p) : launch_pdl(add_tanh_norm_kernel<float, 1>, grid, block, 0, s, *p))
                          : (vec ? launch_pdl(add_tanh_norm_kernel<__nv_bfloat16, 8>, grid, block, 0, s, *p)
                                 : launch_pdl(add_tanh_norm_kernel<__nv_bfloat16, 1>, grid, block, 0, s, *p));
  return ok ? 0 : -4;
}

OGB_API int ogb_norm_stream(const OgbNormStream* p, void* stream) {
  if (p->n_rows <= 0) return 0;
  if (p->H <= 0 || p->H > 48 * 1024 / 4 - 64 || (p->inv_pos && (!p->y || !p->topk_w)) || (p->w2 && !p->out2)) return -1;
  auto addr = [](const void* a) { return reinterpret_cast<uintptr_t>(a); };
  if (p->H % 4 == 0 && ((addr(p->x) | addr(p->w) | addr(p->b) | addr(p->w2) | addr(p->out) | addr(p->out2) | addr(p->y)) & (p->fp32 ? 15 : 7))) return -1;
  auto s = static_cast<cudaStream_t>(stream);
  const dim3 block(p->H >= 1024 ? 256 : 128), grid(p->n_rows);
  const size_t smem = size_t(p->H) * 4;
  using H = __nv_bfloat16;
  const bool ok = p->fp32 ? (p->y ? launch_pdl(norm_stream_kernel<float, true>, grid, block, smem, s, *p) : launch_pdl(norm_stream_kernel<float, false>, grid, block, smem, s, *p))
                          : (p->y ? launch_pdl(norm_stream_kernel<H, true>, grid, block, smem, s, *p) : launch_pdl(norm_stream_kernel<H, false>, grid, block, smem, s, *p));
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

OGB_API int ogb_add_normed(float* h, const void* y, int ldy, int y_fp32, const float* w, float eps, void* x, const int32_t* inv_pos, const float* topk_w,
                           int k, int T, int H, void* stream) {
  if (T <= 0 || H <= 0) return 0;
  auto s = static_cast<cudaStream_t>(stream);
  const AddNormed p{h, w, static_cast<__nv_bfloat16*>(x), inv_pos, topk_w, k, ldy, H, eps};
  const bool vec = H % ADN_VEC == 0 && ldy % ADN_VEC == 0 && H <= 256 * ADN_VEC * ADN_KEEP &&
                   ((reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(x)) & 15) == 0;
  // pieces of a row over the threads: every thread has one where the row has no more than 256
  const int pieces = vec ? (H / ADN_VEC + 31) / 32 * 32 : (H + 31) / 32 * 32;
  const dim3 block(pieces < 256 ? pieces : 256);
  bool ok;
  if (y_fp32) {
    const float* yf = static_cast<const float*>(y);
    ok = vec ? launch_pdl(add_normed_kernel<float, true>, dim3(T), block, 0, s, yf, p) : launch_pdl(add_normed_kernel<float, false>, dim3(T), block, 0, s, yf, p);
  } else {
    const __nv_bfloat16* yh = static_cast<const __nv_bfloat16*>(y);
    ok = vec ? launch_pdl(add_normed_kernel<__nv_bfloat16, true>, dim3(T), block, 0, s, yh, p)
             : launch_pdl(add_normed_kernel<__nv_bfloat16, false>, dim3(T), block, 0, s, yh, p);
  }
  return ok ? 0 : -4;
}

OGB_API int ogb_qkv_prep(void* proj, int ldp, int Hq, int Hkv, int Hv, int dim, int key_row, int value_row, const float* q_norm, const float* k_norm, float eps,
                         const int32_t* positions, const float* cos, const float* sin, int rot, int max_pos, const int32_t* slots, void* k_cache,
                         void* v_cache, int T, const float* talk, void* mixed, int fp32, void* stream) {
  if (T <= 0) return 0;
  if (Hq <= 0 || Hkv <= 0 || Hv <= 0 || dim <= 0 || dim > key_row || rot < 0 || rot > dim || (rot & 1) || (rot > 0 && (!cos || !sin || max_pos <= 0))) return -1;
  const QkvPrep p{ldp, Hq, Hkv, Hv, dim, key_row, value_row, rot, max_pos > 0 ? max_pos : 1, T, q_norm, k_norm, cos, sin, positions, slots, eps};
  const long items = long(T) * (Hq + Hkv + Hv);
  const dim3 grid(unsigned((items + 7) / 8));
  auto s = static_cast<cudaStream_t>(stream);
  const int elem = fp32 ? 4 : 2;
  if (talk) {
    const size_t smem = (size_t(Hq) * (Hq + key_row) + 1) * 4;
    if (!mixed || Hq % Hkv || key_row % 8 || smem > 200 * 1024 || (reinterpret_cast<uintptr_t>(mixed) & 15)) return -1;
    const dim3 block(256);
    const bool pieces = dim == key_row && dim % 8 == 0 && dim <= 256 && rot % 16 == 0 && value_row % 8 == 0 && ldp % 8 == 0 &&
                        ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(k_cache) | reinterpret_cast<uintptr_t>(v_cache) |
                          reinterpret_cast<uintptr_t>(cos) | reinterpret_cast<uintptr_t>(sin) | reinterpret_cast<uintptr_t>(q_norm) |
                          reinterpret_cast<uintptr_t>(k_norm)) & 15) == 0;
    if (pieces) {
      int lph = 1;
      while (lph * 8 < dim) lph *= 2;
      static bool p32[OGB_MAX_DEVICES] = {}, p16[OGB_MAX_DEVICES] = {};
      using B = __nv_bfloat16;
      if (fp32 ? !set_max_dyn_smem(qkv_prep_mixed_pieces_kernel<float>, 200 * 1024, p32) : !set_max_dyn_smem(qkv_prep_mixed_pieces_kernel<B>, 200 * 1024, p16)) return -3;
      const int parts = T >= 1200 ? 1 : (1200 / T < Hkv ? 1200 / T : Hkv), per = (Hkv + parts - 1) / parts;      // (256 tokens: 9.2 us; in one part 14)
      const dim3 g2(T, (Hkv + per - 1) / per);
      return (fp32 ? launch_pdl(qkv_prep_mixed_pieces_kernel<float>, g2, block, smem, s, static_cast<const float*>(proj), static_cast<float*>(k_cache),
                                static_cast<float*>(v_cache), p, talk, static_cast<float*>(mixed), lph, per)
                   : launch_pdl(qkv_prep_mixed_pieces_kernel<B>, g2, block, smem, s, static_cast<const B*>(proj), static_cast<B*>(k_cache),
                                static_cast<B*>(v_cache), p, talk, static_cast<B*>(mixed), lph, per)) ? 0 : -4;
    }
    static bool done32[OGB_MAX_DEVICES] = {}, done16[OGB_MAX_DEVICES] = {};
    if (fp32) {
      if (!set_max_dyn_smem(qkv_prep_mixed_kernel<float>, 200 * 1024, done32)) return -3;
      return launch_pdl(qkv_prep_mixed_kernel<float>, dim3(T), block, smem, s, static_cast<const float*>(proj), static_cast<float*>(k_cache), static_cast<float*>(v_cache),
                        p, talk, static_cast<float*>(mixed)) ? 0 : -4;
    }
    using B = __nv_bfloat16;
    if (!set_max_dyn_smem(qkv_prep_mixed_kernel<B>, 200 * 1024, done16)) return -3;
    return launch_pdl(qkv_prep_mixed_kernel<B>, dim3(T), block, smem, s, static_cast<const B*>(proj), static_cast<B*>(k_cache), static_cast<B*>(v_cache), p, talk,
                      static_cast<B*>(mixed)) ? 0 : -4;
  }
  if (!q_norm && !k_norm && dim == key_row && dim % 8 == 0 && rot % 16 == 0 && value_row % 8 == 0 && ldp % 8 == 0 &&
      ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(k_cache) | reinterpret_cast<uintptr_t>(v_cache) | reinterpret_cast<uintptr_t>(cos) |
        reinterpret_cast<uintptr_t>(sin)) & 15) == 0) {
    const int pieces = (Hq + Hkv) * (key_row / 8 - rot / 16) + Hv * (value_row / 8);
    const dim3 g2(T, T >= 1024 ? 1 : (pieces + 255) / 256), block(pieces < 256 ? (pieces + 31) / 32 * 32 : 256);
    const bool done = fp32 ? launch_pdl(qkv_prep_pieces_kernel<float>, g2, block, 0, s, static_cast<float*>(proj), static_cast<float*>(k_cache), static_cast<float*>(v_cache), p)
                           : launch_pdl(qkv_prep_pieces_kernel<__nv_bfloat16>, g2, block, 0, s, static_cast<__nv_bfloat16*>(proj),
                                        static_cast<__nv_bfloat16*>(k_cache), static_cast<__nv_bfloat16*>(v_cache), p);
    return done ? 0 : -4;
  }
  const bool two = dim % 2 == 0 && (rot / 2) % 2 == 0 && ldp % 2 == 0 && key_row % 2 == 0 && value_row % 2 == 0 &&
                   ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(k_cache) | reinterpret_cast<uintptr_t>(v_cache)) & (2 * elem - 1)) == 0;
#define OGB_PREP(TY, V) launch_pdl(qkv_prep_kernel<TY, V>, grid, dim3(256), 0, s, static_cast<TY*>(proj), static_cast<TY*>(k_cache), static_cast<TY*>(v_cache), p)
  const bool ok = fp32 ? (two ? OGB_PREP(float, 2) : OGB_PREP(float, 1)) : (two ? OGB_PREP(__nv_bfloat16, 2) : OGB_PREP(__nv_bfloat16, 1));
#undef OGB_PREP
  return ok ? 0 : -4;
}

OGB_API int ogb_expert_act(const void* gu, void* out, long long n, int I, int kind, float alpha, float limit, int fp32, void* stream) {
  const long total = long(n) * I;
  if (total <= 0) return 0;
  auto s = static_cast<cudaStream_t>(stream);
  const long nb = (total + 255) / 256;
  const dim3 grid(unsigned(nb < 148 * 16 ? nb : 148 * 16));
  const bool ok = fp32 ? launch_pdl(expert_act_kernel<float>, grid, dim3(256), 0, s, static_cast<const float*>(gu), static_cast<float*>(out), total, kind,
                                    alpha, limit)
                       : launch_pdl(expert_act_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, static_cast<const __nv_bfloat16*>(gu),
                                    static_cast<__nv_bfloat16*>(out), total, kind, alpha, limit);
  return ok ? 0 : -4;
}
