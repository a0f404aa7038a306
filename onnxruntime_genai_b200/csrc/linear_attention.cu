// Gated-delta-rule recurrence of a linear-attention (gated delta net) layer over packed sequences: the LinearAttention contrib op
// with update_rule "gated_delta" that the reference's builder emits for Qwen3-Next / Qwen3.5 style hybrids
// (src/python/py/models/builders/base.py:3419-3452, qwen.py:1842-1860; state handling src/models/recurrent_state.h:12-66).
//
// Two kernels over the same state pool (fp32, [slots][value heads][dk][dv] with a slot stride), for bf16 and fp32 activations and any
// dk / dv (rows and columns past the sizes are zeros):
//   gated_delta_kernel        decode-shaped steps.  One CTA = (request, value head, 32 columns of the head's state S [dk, dv]); a thread
//                             keeps 16 to 64 rows of one column, the lanes of a warp are neighbouring columns (the state streams in
//                             full lines), the row splits of a column meet in shared memory.
//   gated_delta_chunk_kernel  prompts.  The row splits of a column are lanes of one warp, so that the two dot products of a token are
//                             finished by shuffles and the token loop has no barrier; the keys and queries of a chunk of tokens
//                             are normalised into shared memory by all warps beforehand.
// Per token, with k_t, q_t of the head:
//     S[:, j] *= exp(g);   mem = sum_i S[i, j] k[i];   delta = (v[j] - mem) * beta;   S[i, j] += k[i] * delta;   o[j] = sum_i S[i, j] q[i]
// Tokens of a request are walked in order inside the kernel (a decode step is one token, a prompt chunk many); the state is read
// from / written to the request's slot once per launch.  A request whose past length is 0 starts from zero.
// This file is built without fast-math: the recurrence and all that feeds it is plain fp32.
#include "common.cuh"
#include "kernels.h"

namespace ogb {

template <typename T> __device__ __forceinline__ float act_f32(T v);
template <> __device__ __forceinline__ float act_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ float act_f32<__nv_bfloat16>(__nv_bfloat16 v) { return bf2f(v); }
template <typename T> __device__ __forceinline__ T act_from(float v);
template <> __device__ __forceinline__ float act_from<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 act_from<__nv_bfloat16>(float v) { return f2bf(v); }

template <typename T>
struct GdnParams {
  const T *q, *k, *v;                 // rows of token t at q + t * tok_stride (+ head offsets): separate tensors or slices of one projection
  long long tok_stride_qk, tok_stride_v;
  const float *g, *beta;              // [T, Hv] log-decay and write strength ...
  const T *b_raw, *a_raw;             // ... or (g == null) their raw projections [T, Hv] with a row stride: beta = sigmoid(b),
  long long ba_stride;                //     g = neg_exp_a[h] * softplus(a + dt_bias[h])
  const float *neg_exp_a, *dt_bias;
  int l2norm;                         // q and k are L2-normalised per head here (q then scaled by q_scale)
  float q_scale;
  float l2_eps;                       // > 0: unit vectors are x / sqrt(sum(x^2) + l2_eps); 0: x / max(sqrt(sum(x^2)), 1e-6)
  float* state;
  long long slot_stride;              // floats between the states of consecutive slots
  const int32_t *slots, *cu_seqlens, *past_lens;
  T* out;
  int Hk, Hv, dv, dk;
};

__device__ __forceinline__ float inv_length(float sumsq, float l2_eps) {
  return l2_eps > 0.f ? 1.f / sqrtf(sumsq + l2_eps) : 1.f / fmaxf(sqrtf(sumsq), 1e-6f);
}

// decay exp(g) and write strength beta of token t, value head h
template <typename T>
__device__ __forceinline__ void gdn_gates(const GdnParams<T>& p, int t, int h, float& decay, float& beta) {
  if (p.g) {
    decay = expf(p.g[size_t(t) * p.Hv + h]);
    beta = p.beta[size_t(t) * p.Hv + h];
  } else {
    const float ar = act_f32(p.a_raw[size_t(t) * p.ba_stride + h]) + p.dt_bias[h];
    const float soft = ar > 20.f ? ar : log1pf(expf(ar));
    decay = expf(p.neg_exp_a[h] * soft);
    beta = 1.f / (1.f + expf(-act_f32(p.b_raw[size_t(t) * p.ba_stride + h])));
  }
}

constexpr int GDN_MAX_DK = 1024, GDN_MAX_SPLITS = 16;

// FULL: dk is a multiple of NPT, no row is past the size.
template <typename T, int NPT, bool FULL>
__global__ void __launch_bounds__(512) gated_delta_kernel(GdnParams<T> p) {
  // thread (j, sp): column j of the state, rows [sp * NPT, (sp + 1) * NPT); the two dot products of a token (with k, then with q)
  // are summed over the splits through shared memory
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.x, h = blockIdx.y;
  const int Hk = p.Hk, Hv = p.Hv, dv = p.dv, dk = p.dk;
  const int splits = blockDim.x / 32;                         // 32 columns per CTA (blockIdx.z walks the column tiles)
  const int jj = threadIdx.x % 32, j = blockIdx.z * 32 + jj, sp = threadIdx.x / 32, n0 = sp * NPT;
  const int hk = h / (Hv / Hk);
  const int t0 = p.cu_seqlens[b], t1 = p.cu_seqlens[b + 1];
  if (t0 >= t1) return;
  __shared__ float sk[GDN_MAX_DK], sq[GDN_MAX_DK];
  __shared__ float sM[GDN_MAX_SPLITS][32], sO[GDN_MAX_SPLITS][32];
  __shared__ float sNorm[2][16];
  float* S = p.state + size_t(p.slots[b]) * p.slot_stride + (size_t(h) * dk + n0) * dv;
  float col[NPT];
  const bool live = j < dv;
  const bool fresh = p.past_lens[b] == 0;
#pragma unroll
  for (int i = 0; i < NPT; ++i) col[i] = (live && !fresh && (FULL || n0 + i < dk)) ? S[size_t(i) * dv + j] : 0.f;
  if (!FULL) for (int i = dk + threadIdx.x; i < splits * NPT; i += blockDim.x) { sk[i] = 0.f; sq[i] = 0.f; }
  for (int t = t0; t < t1; ++t) {
    __syncthreads();
    float ssk = 0.f, ssq = 0.f;
    for (int i = threadIdx.x; i < dk; i += blockDim.x) {
      const float kv_ = act_f32(p.k[size_t(t) * p.tok_stride_qk + size_t(hk) * dk + i]);
      const float qv_ = act_f32(p.q[size_t(t) * p.tok_stride_qk + size_t(hk) * dk + i]);
      sk[i] = kv_; sq[i] = qv_;
      ssk += kv_ * kv_; ssq += qv_ * qv_;
    }
    float rk = 1.f, rq = 1.f;
    if (p.l2norm) {
      ssk = warp_sum(ssk); ssq = warp_sum(ssq);
      if ((threadIdx.x & 31) == 0) { sNorm[0][threadIdx.x >> 5] = ssk; sNorm[1][threadIdx.x >> 5] = ssq; }
    }
    __syncthreads();
    if (p.l2norm) {
      float tk = 0.f, tq = 0.f;
      for (int w = 0; w < splits; ++w) { tk += sNorm[0][w]; tq += sNorm[1][w]; }
      rk = inv_length(tk, p.l2_eps);
      rq = p.q_scale * inv_length(tq, p.l2_eps);
    }
    float decay, bt;
    gdn_gates(p, t, h, decay, bt);
    float mem = 0.f;
#pragma unroll
    for (int i = 0; i < NPT; ++i) {
      col[i] *= decay;
      mem = fmaf(col[i], sk[n0 + i], mem);
    }
    if (splits > 1) {
      sM[sp][jj] = mem;
      __syncthreads();
      mem = 0.f;
      for (int s2 = 0; s2 < splits; ++s2) mem += sM[s2][jj];
    }
    const float vj = live ? act_f32(p.v[size_t(t) * p.tok_stride_v + size_t(h) * dv + j]) : 0.f;
    const float delta = (vj - mem * rk) * bt * rk;       // the normalised key is rk * sk: once in the read, once in the write
    float o = 0.f;
#pragma unroll
    for (int i = 0; i < NPT; ++i) {
      col[i] = fmaf(sk[n0 + i], delta, col[i]);
      o = fmaf(col[i], sq[n0 + i], o);
    }
    if (splits > 1) {
      sO[sp][jj] = o;
      __syncthreads();
      if (sp == 0)
        for (int s2 = 1; s2 < splits; ++s2) o += sO[s2][jj];
    }
    if (live && sp == 0) p.out[(size_t(t) * Hv + h) * dv + j] = act_from<T>(o * rq);
  }
  if (live) {
#pragma unroll
    for (int i = 0; i < NPT; ++i) if (FULL || n0 + i < dk) S[size_t(i) * dv + j] = col[i];
  }
}

// A thread owns two columns and NPT rows of each, 8 * NPT >= dk; the lanes of a warp are 4 column pairs x 8 row splits.  Row of split sp,
// register i: (i / 4) * 32 + sp * 4 + i % 4, so that a thread's rows come as groups of four and the splits of a warp read one
// 128-byte line of a key together.  CH tokens per chunk.
// Both dot products of a token are taken on the state before its update, which needs the two vectors once and one round of
// shuffles: with m = S^T k and r = S^T q (old state), delta = beta * (v - g m), S <- g S + k delta^T and S_new^T q = g r + (k . q) delta.
template <typename T, int NPT, int CH>
__global__ void __launch_bounds__(128) gated_delta_chunk_kernel(GdnParams<T> p) {
  constexpr int DKP = NPT * 8, G4 = NPT / 4;
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.x, h = blockIdx.y;
  const int Hv = p.Hv, dv = p.dv, dk = p.dk;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, sp = lane & 7;
  const int jj = warp * 8 + (lane >> 3) * 2, j = blockIdx.z * 32 + jj;      // columns j, j + 1
  const int hk = h / (Hv / p.Hk);
  const int t0 = p.cu_seqlens[b], t1 = p.cu_seqlens[b + 1];
  if (t0 >= t1) return;
  __shared__ __align__(16) float sk[CH][DKP];
  __shared__ __align__(16) float sq[CH][DKP];
  __shared__ __align__(8) float sv[CH][32];
  __shared__ float sdot[CH], sgate[2][CH];
  const bool live0 = j < dv, live1 = j + 1 < dv, fresh = p.past_lens[b] == 0;
  float* S = p.state + size_t(p.slots[b]) * p.slot_stride + size_t(h) * dk * dv;
  auto row_of = [&](int i) { return (i >> 2) * 32 + sp * 4 + (i & 3); };
  float c0[NPT], c1[NPT];
#pragma unroll
  for (int i = 0; i < NPT; ++i) {
    const bool ok = !fresh && row_of(i) < dk;
    c0[i] = ok && live0 ? S[size_t(row_of(i)) * dv + j] : 0.f;
    c1[i] = ok && live1 ? S[size_t(row_of(i)) * dv + j + 1] : 0.f;
  }

  // a chunk's raw keys / queries / values on their way from global memory: held in registers while the previous chunk is computed
  constexpr int PER = DKP / 32, TW = CH / 4;               // elements per lane of a row, rows per warp
  const T zero = act_from<T>(0.f);
  T rk[TW][PER], rq[TW][PER], rv[TW];
  float ga, gb;
  auto fetch = [&](int f0) {
#pragma unroll
    for (int w = 0; w < TW; ++w) {
      const int t = f0 + w * 4 + warp;
#pragma unroll
      for (int e = 0; e < PER; ++e) {
        const int i = e * 32 + lane;
        const bool ok = t < t1 && i < dk;
        rk[w][e] = ok ? p.k[size_t(t) * p.tok_stride_qk + size_t(hk) * dk + i] : zero;
        rq[w][e] = ok ? p.q[size_t(t) * p.tok_stride_qk + size_t(hk) * dk + i] : zero;
      }
      const int jc = blockIdx.z * 32 + lane;
      rv[w] = (t < t1 && jc < dv) ? p.v[size_t(t) * p.tok_stride_v + size_t(h) * dv + jc] : zero;
    }
    ga = gb = 0.f;
    if (threadIdx.x < CH && f0 + int(threadIdx.x) < t1) gdn_gates(p, f0 + threadIdx.x, h, ga, gb);
  };
  fetch(t0);
  for (int f0 = t0; f0 < t1; f0 += CH) {
    __syncthreads();                                       // the previous chunk is no longer read
#pragma unroll
    for (int w = 0; w < TW; ++w) {
      float ssk = 0.f, ssq = 0.f, skq = 0.f;
#pragma unroll
      for (int e = 0; e < PER; ++e) {
        const float kk = act_f32(rk[w][e]), qq = act_f32(rq[w][e]);
        ssk += kk * kk; ssq += qq * qq; skq += kk * qq;
      }
      float nk = 1.f, nq = 1.f;
      if (p.l2norm) {
        nk = inv_length(warp_sum(ssk), p.l2_eps);
        nq = p.q_scale * inv_length(warp_sum(ssq), p.l2_eps);
      }
      skq = warp_sum(skq) * nk * nq;
      const int tt = w * 4 + warp;
#pragma unroll
      for (int e = 0; e < PER; ++e) {
        sk[tt][e * 32 + lane] = act_f32(rk[w][e]) * nk;
        sq[tt][e * 32 + lane] = act_f32(rq[w][e]) * nq;
      }
      sv[tt][lane] = act_f32(rv[w]);
      if (lane == 0) sdot[tt] = skq;
    }
    if (threadIdx.x < CH) { sgate[0][threadIdx.x] = ga; sgate[1][threadIdx.x] = gb; }
    __syncthreads();
    if (f0 + CH < t1) fetch(f0 + CH);
    const int n = min(CH, t1 - f0);
    for (int tt = 0; tt < n; ++tt) {
      const float decay = sgate[0][tt], bt = sgate[1][tt], kq = sdot[tt];
      const float2 vj = *reinterpret_cast<const float2*>(&sv[tt][jj]);
      const float4* k4 = reinterpret_cast<const float4*>(sk[tt]) + sp;
      const float4* q4 = reinterpret_cast<const float4*>(sq[tt]) + sp;
      float4 kk[G4];
      float m0a = 0.f, m0b = 0.f, m1a = 0.f, m1b = 0.f, r0a = 0.f, r0b = 0.f, r1a = 0.f, r1b = 0.f;
#pragma unroll
      for (int i = 0; i < G4; ++i) {
        kk[i] = k4[i * 8];
        const float4 qq = q4[i * 8];
        m0a = fmaf(c0[4 * i], kk[i].x, m0a); m1a = fmaf(c1[4 * i], kk[i].x, m1a);
        m0b = fmaf(c0[4 * i + 1], kk[i].y, m0b); m1b = fmaf(c1[4 * i + 1], kk[i].y, m1b);
        m0a = fmaf(c0[4 * i + 2], kk[i].z, m0a); m1a = fmaf(c1[4 * i + 2], kk[i].z, m1a);
        m0b = fmaf(c0[4 * i + 3], kk[i].w, m0b); m1b = fmaf(c1[4 * i + 3], kk[i].w, m1b);
        r0a = fmaf(c0[4 * i], qq.x, r0a); r1a = fmaf(c1[4 * i], qq.x, r1a);
        r0b = fmaf(c0[4 * i + 1], qq.y, r0b); r1b = fmaf(c1[4 * i + 1], qq.y, r1b);
        r0a = fmaf(c0[4 * i + 2], qq.z, r0a); r1a = fmaf(c1[4 * i + 2], qq.z, r1a);
        r0b = fmaf(c0[4 * i + 3], qq.w, r0b); r1b = fmaf(c1[4 * i + 3], qq.w, r1b);
      }
      float m0 = m0a + m0b, m1 = m1a + m1b, r0 = r0a + r0b, r1 = r1a + r1b;
#pragma unroll
      for (int o = 1; o < 8; o <<= 1) {
        m0 += __shfl_xor_sync(0xffffffffu, m0, o);
        m1 += __shfl_xor_sync(0xffffffffu, m1, o);
        r0 += __shfl_xor_sync(0xffffffffu, r0, o);
        r1 += __shfl_xor_sync(0xffffffffu, r1, o);
      }
      const float d0 = (vj.x - decay * m0) * bt, d1 = (vj.y - decay * m1) * bt;
#pragma unroll
      for (int i = 0; i < G4; ++i) {
        c0[4 * i] = fmaf(kk[i].x, d0, decay * c0[4 * i]); c1[4 * i] = fmaf(kk[i].x, d1, decay * c1[4 * i]);
        c0[4 * i + 1] = fmaf(kk[i].y, d0, decay * c0[4 * i + 1]); c1[4 * i + 1] = fmaf(kk[i].y, d1, decay * c1[4 * i + 1]);
        c0[4 * i + 2] = fmaf(kk[i].z, d0, decay * c0[4 * i + 2]); c1[4 * i + 2] = fmaf(kk[i].z, d1, decay * c1[4 * i + 2]);
        c0[4 * i + 3] = fmaf(kk[i].w, d0, decay * c0[4 * i + 3]); c1[4 * i + 3] = fmaf(kk[i].w, d1, decay * c1[4 * i + 3]);
      }
      if (sp == 0) {
        T* dst = p.out + (size_t(f0 + tt) * Hv + h) * dv + j;
        if (live0) dst[0] = act_from<T>(fmaf(decay, r0, kq * d0));
        if (live1) dst[1] = act_from<T>(fmaf(decay, r1, kq * d1));
      }
    }
  }
#pragma unroll
  for (int i = 0; i < NPT; ++i) {
    if (row_of(i) >= dk) continue;
    if (live0) S[size_t(row_of(i)) * dv + j] = c0[i];
    if (live1) S[size_t(row_of(i)) * dv + j + 1] = c1[i];
  }
}

// Output gate of a gated-delta-net layer: per value head, RMS norm of the recurrence output times its weight, times silu of the gate
// projection z (a column slice of the layer's input projection).  One warp per (token, head); out rows have a stride of their own.
template <typename T>
__global__ void gdn_gate_norm_kernel(const T* __restrict__ o, const T* __restrict__ z, long long z_stride, const float* __restrict__ w, float eps,
                                     T* __restrict__ out, long long out_stride, int rows, int Hv, int dv) {
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (row >= rows) return;
  const int t = row / Hv, h = row % Hv;
  const T* src = o + size_t(row) * dv;
  float ss = 0.f;
  for (int e = lane; e < dv; e += 32) { const float x = act_f32(src[e]); ss += x * x; }
  ss = warp_sum(ss);
  const float inv = 1.f / sqrtf(ss / dv + eps);
  T* dst = out + size_t(t) * out_stride + size_t(h) * dv;
  for (int e = lane; e < dv; e += 32) {
    const float zz = act_f32(z[size_t(t) * z_stride + size_t(h) * dv + e]);
    dst[e] = act_from<T>(act_f32(src[e]) * inv * w[e] * (zz / (1.f + expf(-zz))));
  }
}

}  // namespace ogb

using namespace ogb;

template <typename T, int NPT>
static bool LaunchGdnDecode(const GdnParams<T>& p, int B, int splits, cudaStream_t s) {
  const dim3 grid(B, p.Hv, (p.dv + 31) / 32), block(32 * splits);
  return p.dk % NPT == 0 ? launch_pdl(gated_delta_kernel<T, NPT, true>, grid, block, 0, s, p)
                         : launch_pdl(gated_delta_kernel<T, NPT, false>, grid, block, 0, s, p);
}
template <typename T, int NPT, int CH>
static bool LaunchGdnChunk(const GdnParams<T>& p, int B, cudaStream_t s) {
  return launch_pdl(gated_delta_chunk_kernel<T, NPT, CH>, dim3(B, p.Hv, (p.dv + 31) / 32), dim3(128), 0, s, p);
}

// max_q_len: the most tokens a request of the launch feeds (1: the decode kernel; 0: unknown, treated as a prompt)
template <typename T>
static int LaunchGatedDelta(const GdnParams<T>& p, int B, int max_q_len, void* stream) {
  if (B <= 0) return 0;
  const int dk = p.dk, dv = p.dv;
  if (p.Hk <= 0 || p.Hv % p.Hk || dv <= 0 || dk <= 0) return -1;
  if (dk > GDN_MAX_DK) return -5;
  auto s = static_cast<cudaStream_t>(stream);
  bool ok;
  if (max_q_len != 1 && dk <= 256) {
    if (dk <= 32) ok = LaunchGdnChunk<T, 4, 32>(p, B, s);
    else if (dk <= 64) ok = LaunchGdnChunk<T, 8, 32>(p, B, s);
    else if (dk <= 128) ok = LaunchGdnChunk<T, 16, 32>(p, B, s);
    else ok = LaunchGdnChunk<T, 32, 16>(p, B, s);
    return ok ? 0 : -4;
  }
  // measured at Qwen3.5 shapes: 32 rows per thread 51 us, 16 rows 63 us, 64 rows 54 us (64 requests)
  if (dk <= 16) ok = LaunchGdnDecode<T, 16>(p, B, 1, s);
  else if (dk <= 32 * GDN_MAX_SPLITS) ok = LaunchGdnDecode<T, 32>(p, B, (dk + 31) / 32, s);
  else ok = LaunchGdnDecode<T, 64>(p, B, (dk + 63) / 64, s);
  return ok ? 0 : -4;
}

OGB_API int ogb_gated_delta(const void* q, const void* k, const void* v, const float* g, const float* beta, float* state, const int32_t* slots,
                            const int32_t* cu_seqlens, const int32_t* past_lens, void* out, int B, int Hk, int Hv, int dk, int dv, int max_q_len,
                            void* stream) {
  using T = __nv_bfloat16;
  GdnParams<T> p{};
  p.q = static_cast<const T*>(q); p.k = static_cast<const T*>(k); p.v = static_cast<const T*>(v);
  p.tok_stride_qk = static_cast<long long>(Hk) * dk; p.tok_stride_v = static_cast<long long>(Hv) * dv;
  p.g = g; p.beta = beta; p.l2norm = 0; p.q_scale = 1.f;
  p.state = state; p.slot_stride = static_cast<long long>(Hv) * dk * dv;
  p.slots = slots; p.cu_seqlens = cu_seqlens; p.past_lens = past_lens; p.out = static_cast<T*>(out);
  p.Hk = Hk; p.Hv = Hv; p.dv = dv; p.dk = dk;
  return LaunchGatedDelta(p, B, max_q_len, stream);
}

template <typename T>
static int GatedDeltaFused(const void* conv, long long conv_stride, long long q_off, long long k_off, long long v_off, const void* ba,
                           long long ba_stride, long long b_off, long long a_off, const float* neg_exp_a, const float* dt_bias, float q_scale,
                           float l2_eps, float* state, long long slot_stride, const int32_t* slots, const int32_t* cu_seqlens,
                           const int32_t* past_lens, void* out, int B, int Hk, int Hv, int dk, int dv, int max_q_len, void* stream) {
  GdnParams<T> p{};
  auto c = static_cast<const T*>(conv);
  auto r = static_cast<const T*>(ba);
  p.q = c + q_off; p.k = c + k_off; p.v = c + v_off; p.tok_stride_qk = conv_stride; p.tok_stride_v = conv_stride;
  p.g = nullptr; p.beta = nullptr; p.b_raw = r + b_off; p.a_raw = r + a_off; p.ba_stride = ba_stride;
  p.neg_exp_a = neg_exp_a; p.dt_bias = dt_bias; p.l2norm = 1; p.q_scale = q_scale; p.l2_eps = l2_eps;
  p.state = state; p.slot_stride = slot_stride > 0 ? slot_stride : static_cast<long long>(Hv) * dk * dv;
  p.slots = slots; p.cu_seqlens = cu_seqlens; p.past_lens = past_lens; p.out = static_cast<T*>(out);
  p.Hk = Hk; p.Hv = Hv; p.dv = dv; p.dk = dk;
  return LaunchGatedDelta(p, B, max_q_len, stream);
}

// The recurrence fed straight from the layer's tensors: q / k / v are column ranges of the convolved projection `conv` [T, row
// stride] (q at q_off, k at k_off, v at v_off), normalised here; the decay and the write strength come from the raw b / a
// projections (column ranges of `ba`, row stride ba_stride) with the layer's -exp(A_log) and dt_bias.  l2_eps, slot_stride and
// max_q_len as in GdnParams / LaunchGatedDelta (slot_stride 0: dense); fp32: element type of conv, ba and out (else bf16).
OGB_API int ogb_gated_delta_fused(const void* conv, long long conv_stride, long long q_off, long long k_off, long long v_off, const void* ba,
                                  long long ba_stride, long long b_off, long long a_off, const float* neg_exp_a, const float* dt_bias,
                                  float q_scale, float l2_eps, float* state, long long slot_stride, const int32_t* slots,
                                  const int32_t* cu_seqlens, const int32_t* past_lens, void* out, int B, int Hk, int Hv, int dk, int dv,
                                  int max_q_len, int fp32, void* stream) {
  return fp32 ? GatedDeltaFused<float>(conv, conv_stride, q_off, k_off, v_off, ba, ba_stride, b_off, a_off, neg_exp_a, dt_bias, q_scale, l2_eps,
                                       state, slot_stride, slots, cu_seqlens, past_lens, out, B, Hk, Hv, dk, dv, max_q_len, stream)
              : GatedDeltaFused<__nv_bfloat16>(conv, conv_stride, q_off, k_off, v_off, ba, ba_stride, b_off, a_off, neg_exp_a, dt_bias, q_scale,
                                               l2_eps, state, slot_stride, slots, cu_seqlens, past_lens, out, B, Hk, Hv, dk, dv, max_q_len, stream);
}

OGB_API int ogb_gdn_gate_norm(const void* o, const void* z, long long z_stride, const float* w, float eps, void* out, long long out_stride, int T,
                              int Hv, int dv, int fp32, void* stream) {
  if (T <= 0) return 0;
  if (dv <= 0) return -1;
  const int rows = T * Hv;
  const dim3 grid((rows + 7) / 8), block(256);
  auto s = static_cast<cudaStream_t>(stream);
  using H = __nv_bfloat16;
  return (fp32 ? launch_pdl(gdn_gate_norm_kernel<float>, grid, block, 0, s, static_cast<const float*>(o), static_cast<const float*>(z), z_stride, w, eps,
                            static_cast<float*>(out), out_stride, rows, Hv, dv)
               : launch_pdl(gdn_gate_norm_kernel<H>, grid, block, 0, s, static_cast<const H*>(o), static_cast<const H*>(z), z_stride, w, eps,
                            static_cast<H*>(out), out_stride, rows, Hv, dv)) ? 0 : -4;
}

// ---------------------------------------------------------------------------------------------- Mamba-2 selective scan
// The state-space recurrence of a Mamba-2 layer over packed sequences (GraniteMoeHybrid; reference: the Mamba2 branch of
// src/models/recurrent_state.cpp keeps its conv / ssm states, the layer itself is an opaque graph there).  Per head h with
// group gr = h / (heads / groups), per token t, with dt already softplus'ed:
//     S *= exp(dt[t, h] * A[h]);   S[n][p] += dt[t, h] * x[t, h, p] * B[t, gr, n];   y[t, h, p] = sum_n S[n][p] * C[t, gr, n] + D[h] * x[t, h, p]
// state [slots][heads][N][P] fp32, updated in place for the request slots (a request whose past length is 0 starts from a
// zero state).  One CTA per (request, head); a thread keeps 16 to 64 rows of one state column in registers (the rows of a column
// are split over up to 8 threads whose partial sums meet in shared memory), the token's B and C rows sit in
// shared memory; the tokens of a chunk are walked in order.
namespace ogb {
template <int NPT>
__global__ void __launch_bounds__(512) mamba2_scan_kernel(
    const __nv_bfloat16* __restrict__ x, const float* __restrict__ dt, const float* __restrict__ neg_a, const __nv_bfloat16* __restrict__ Bm,
    const __nv_bfloat16* __restrict__ Cm, const float* __restrict__ Dv, float* __restrict__ state, const int32_t* __restrict__ slots,
    const int32_t* __restrict__ cu_seqlens, const int32_t* __restrict__ past_lens, __nv_bfloat16* __restrict__ out, int heads, int groups, int P,
    int N, long long x_stride, long long bc_stride, const __nv_bfloat16* __restrict__ dt_raw, long long dt_stride,
    const float* __restrict__ dt_bias) {
  // x_stride / bc_stride: elements between the rows of consecutive tokens in x and in Bm / Cm (tensors of their own, or column
  // ranges of one convolved projection);
  // dt_raw (dt == null): the raw step projection [T, heads] with a row stride, step = softplus(dt_raw + dt_bias[h]) computed here
  // thread (j, sp): column j of the state, rows [sp * NPT, (sp + 1) * NPT); the partial dot products of the splits meet in shared memory
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.x, h = blockIdx.y;
  const int splits = N / NPT, Pp = blockDim.x / splits;
  const int j = threadIdx.x % Pp, sp = threadIdx.x / Pp, n0 = sp * NPT;
  const int gr = h / (heads / groups);
  const int t0 = cu_seqlens[b], t1 = cu_seqlens[b + 1];
  if (t0 >= t1) return;
  __shared__ float sB[256], sC[256];
  __shared__ float sY[8][128];
  float* S = state + ((size_t(slots[b]) * heads + h) * N + n0) * P;
  float col[NPT];
  const bool live = j < P;
  const bool fresh = past_lens[b] == 0;
#pragma unroll
  for (int i = 0; i < NPT; ++i) col[i] = (live && !fresh) ? S[size_t(i) * P + j] : 0.f;
  const float a = neg_a[h], d = Dv[h];
  for (int t = t0; t < t1; ++t) {
    __syncthreads();
    for (int i = threadIdx.x; i < N; i += blockDim.x) {
      sB[i] = bf2f(Bm[size_t(t) * bc_stride + size_t(gr) * N + i]);
      sC[i] = bf2f(Cm[size_t(t) * bc_stride + size_t(gr) * N + i]);
    }
    __syncthreads();
    float step;
    if (dt) step = dt[size_t(t) * heads + h];
    else {
      const float r = bf2f(dt_raw[size_t(t) * dt_stride + h]) + dt_bias[h];
      step = r > 20.f ? r : log1pf(__expf(r));
    }
    const float decay = __expf(step * a);
    const float xj = live ? bf2f(x[size_t(t) * x_stride + size_t(h) * P + j]) : 0.f;
    const float dx = step * xj;
    float y = 0.f;
#pragma unroll
    for (int i = 0; i < NPT; ++i) {
      col[i] = fmaf(col[i], decay, dx * sB[n0 + i]);
      y = fmaf(col[i], sC[n0 + i], y);
    }
    if (splits > 1) {
      sY[sp][j] = y;
      __syncthreads();
      if (sp == 0)
        for (int q = 1; q < splits; ++q) y += sY[q][j];
    }
    if (live && sp == 0) out[(size_t(t) * heads + h) * P + j] = f2bf(y + d * xj);
  }
  if (live) {
#pragma unroll
    for (int i = 0; i < NPT; ++i) S[size_t(i) * P + j] = col[i];
  }
}
}  // namespace ogb

static int LaunchMamba2(const void* x, const float* dt, const float* neg_a, const void* Bm, const void* Cm, const float* Dv, float* state,
                        const int32_t* slots, const int32_t* cu_seqlens, const int32_t* past_lens, void* out, int B, int heads, int groups, int P,
                        int N, long long x_stride, long long bc_stride, const void* dt_raw, long long dt_stride, const float* dt_bias, void* stream) {
  if (B <= 0) return 0;
  if (heads <= 0 || groups <= 0 || heads % groups || P <= 0 || P > 128) return -1;
  if (N < 16 || N > 256 || (N & (N - 1))) return -5;
  const int Pp = (P + 31) / 32 * 32;
  int npt = N < 32 ? N : 32;
  if (Pp * (N / npt) > 512) npt = 64;
  const int splits = N / npt;
  if (splits > 8 || Pp * splits > 512) return -5;
  dim3 grid(B, heads), block(Pp * splits);
  auto s = static_cast<cudaStream_t>(stream);
  auto X = static_cast<const __nv_bfloat16*>(x);
  auto Bp = static_cast<const __nv_bfloat16*>(Bm);
  auto Cp = static_cast<const __nv_bfloat16*>(Cm);
  auto O = static_cast<__nv_bfloat16*>(out);
  auto R = static_cast<const __nv_bfloat16*>(dt_raw);
  bool ok;
  switch (npt) {
    case 16: ok = ogb::launch_pdl(ogb::mamba2_scan_kernel<16>, grid, block, 0, s, X, dt, neg_a, Bp, Cp, Dv, state, slots, cu_seqlens, past_lens, O, heads, groups, P, N, x_stride, bc_stride, R, dt_stride, dt_bias); break;
    case 32: ok = ogb::launch_pdl(ogb::mamba2_scan_kernel<32>, grid, block, 0, s, X, dt, neg_a, Bp, Cp, Dv, state, slots, cu_seqlens, past_lens, O, heads, groups, P, N, x_stride, bc_stride, R, dt_stride, dt_bias); break;
    case 64: ok = ogb::launch_pdl(ogb::mamba2_scan_kernel<64>, grid, block, 0, s, X, dt, neg_a, Bp, Cp, Dv, state, slots, cu_seqlens, past_lens, O, heads, groups, P, N, x_stride, bc_stride, R, dt_stride, dt_bias); break;
    default: return -5;
  }
  return ok ? 0 : -4;
}

OGB_API int ogb_mamba2_scan(const void* x, const float* dt, const float* neg_a, const void* Bm, const void* Cm, const float* Dv, float* state,
                            const int32_t* slots, const int32_t* cu_seqlens, const int32_t* past_lens, void* out, int B, int heads, int groups,
                            int P, int N, void* stream) {
  return LaunchMamba2(x, dt, neg_a, Bm, Cm, Dv, state, slots, cu_seqlens, past_lens, out, B, heads, groups, P, N,
                      static_cast<long long>(heads) * P, static_cast<long long>(groups) * N, nullptr, 0, nullptr, stream);
}

// The scan fed straight from the layer's tensors: x / B / C are column ranges of the convolved projection `conv` (row stride
// conv_stride; x at 0, B at heads * P, C after B), the step comes from the raw dt projection (a column range of `proj`) with dt_bias.
OGB_API int ogb_mamba2_scan_fused(const void* conv, long long conv_stride, const void* dt_raw, long long dt_stride, const float* dt_bias,
                                  const float* neg_a, const float* Dv, float* state, const int32_t* slots, const int32_t* cu_seqlens,
                                  const int32_t* past_lens, void* out, int B, int heads, int groups, int P, int N, void* stream) {
  auto c = static_cast<const __nv_bfloat16*>(conv);
  const long long I = static_cast<long long>(heads) * P, GN = static_cast<long long>(groups) * N;
  return LaunchMamba2(c, nullptr, neg_a, c + I, c + I + GN, Dv, state, slots, cu_seqlens, past_lens, out, B, heads, groups, P, N, conv_stride,
                      conv_stride, dt_raw, dt_stride, dt_bias, stream);
}

// Output gate of a Mamba-2 layer: y * silu(z) (z a column range of the input projection), then an RMS norm over the whole width with
// the layer's weight.  One CTA per token.
namespace ogb {
__global__ void __launch_bounds__(256) mamba_gate_norm_kernel(const __nv_bfloat16* __restrict__ y, const __nv_bfloat16* __restrict__ z,
                                                             long long z_stride, const float* __restrict__ w, float eps,
                                                             __nv_bfloat16* __restrict__ out, int I) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  __shared__ float part[8];
  float v[16];
  float ss = 0.f;
  int n = 0;
  for (int e = threadIdx.x; e < I; e += blockDim.x, ++n) {
    const float zz = bf2f(z[size_t(t) * z_stride + e]);
    v[n] = bf2f(y[size_t(t) * I + e]) * (zz / (1.f + __expf(-zz)));
    ss += v[n] * v[n];
  }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
  for (int i = 0; i < int(blockDim.x >> 5); ++i) tot += part[i];
  const float inv = rsqrtf(tot / I + eps);
  n = 0;
  for (int e = threadIdx.x; e < I; e += blockDim.x, ++n) out[size_t(t) * I + e] = f2bf(v[n] * inv * w[e]);
}
}  // namespace ogb

OGB_API int ogb_mamba_gate_norm(const void* y, const void* z, long long z_stride, const float* w, float eps, void* out, int T, int I, void* stream) {
  if (T <= 0) return 0;
  if (I <= 0 || I > 16 * 256) return -1;
  return ogb::launch_pdl(ogb::mamba_gate_norm_kernel, dim3(T), dim3(256), 0, static_cast<cudaStream_t>(stream),
                         static_cast<const __nv_bfloat16*>(y), static_cast<const __nv_bfloat16*>(z), z_stride, w, eps,
                         static_cast<__nv_bfloat16*>(out), I) ? 0 : -4;
}

// ---------------------------------------------------------------------------------------------- state snapshots
// Copies the recurrent states of `count` slots between two pools of the same shape [layers][slots][slot_elems] (or inside
// one): dst[l][dst_slots[i]] = src[l][src_slots[i]].  Speculative decoding saves a request's state before the verification
// pass feeds draft tokens into it and puts it back when some of them are rejected (reference: CopyStateSlotsKernel,
// src/cuda/model_kernels.cu:488-520, used by src/models/recurrent_state.cpp for its snapshot slots).  16 bytes per thread.
namespace ogb {
__global__ void copy_state_slots_kernel(const float4* __restrict__ src, float4* __restrict__ dst, long long layer_vecs, long long slot_vecs,
                                        const int* __restrict__ src_slots, const int* __restrict__ dst_slots, int count) {
  const int pair = blockIdx.y % count, layer = blockIdx.y / count;
  const float4* s = src + size_t(layer) * layer_vecs + size_t(src_slots[pair]) * slot_vecs;
  float4* d = dst + size_t(layer) * layer_vecs + size_t(dst_slots[pair]) * slot_vecs;
  for (long long i = blockIdx.x * blockDim.x + threadIdx.x; i < slot_vecs; i += (long long)gridDim.x * blockDim.x) d[i] = s[i];
}
}  // namespace ogb

OGB_API int ogb_copy_state_slots(const float* src, float* dst, int layers, int slots, long long slot_elems, const int32_t* src_slots,
                                 const int32_t* dst_slots, int count, void* stream) {
  if (count <= 0 || layers <= 0) return 0;
  if (slot_elems <= 0 || (slot_elems % 4) || slots <= 0) return -1;
  if ((reinterpret_cast<uintptr_t>(src) | reinterpret_cast<uintptr_t>(dst)) & 15) return -1;
  if (static_cast<long long>(layers) * count > 65535) return -1;
  const long long slot_vecs = slot_elems / 4;
  const int threads = 256;
  int bx = int((slot_vecs + threads - 1) / threads);
  if (bx > 128) bx = 128;
  ogb::copy_state_slots_kernel<<<dim3(bx, layers * count), threads, 0, static_cast<cudaStream_t>(stream)>>>(
      reinterpret_cast<const float4*>(src), reinterpret_cast<float4*>(dst), static_cast<long long>(slots) * slot_vecs, slot_vecs, src_slots, dst_slots, count);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
