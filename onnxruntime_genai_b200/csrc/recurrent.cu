// Recurrent mixers of declared stacks over packed sequences, for bf16 and fp32 activations: the gated average (minGRU) and matrix memories (the mLSTM of
// xLSTM).  States are fp32 and live in the request's slot; a request whose past length is 0 starts from zero.  Built without fast-math: gates, decays and
// the recurrences are plain fp32.
//
// Gated average, every column on its own:   z = sigmoid(z'),  c = u + 1/2 (u >= 0) or sigmoid(u) (u < 0),  S <- (1 - z) S + z c,  out = S * silu(g) * scale.
//   min_gru_step_kernel   decode-shaped steps: a thread walks the tokens of one column, or of four.
//   min_gru_chunk_kernel  prompts, in two passes over chunks of tokens: what a chunk does to a state is an affine function per column; the second pass
//                         applies the functions of the chunks before its own to the first state and walks its tokens.
//
// Matrix memory, per head, with i and f the capped log gates and m the running maximum:
//   m' = max(f + m, i),  S <- exp(f + m - m') S + exp(i - m') k v^T,  n likewise with k alone,  o = S^T q / (max(|n . q|, exp(-m')) + 1e-6),
//   out = o / rms(o) * norm * sigmoid(g).
//   mlstm_step_kernel     any step.  A CTA, or a cluster that shares the columns, has a head of a request; the state passes through registers, where it
//                         stays over the tokens of a short portion.
//   chunk form (bf16)     requests with many tokens, 64 at a time.  With b_t the sum of the chunk's log forget gates up to t, c_t = i_t - b_t and
//                         M_t = max(m before the chunk, c_s for s <= t), the running maximum is b_t + M_t and the chunk's outputs and its end state are
//                         products:  num_t = e^(m - M_t) q_t S + sum_{s <= t} e^(c_s - M_t) (q_t . k_s) v_s,  S' = e^(m - M_L) S + sum_s e^(c_s - M_L) k_s v_s^T
//                         (every exponent is at most 0).  Four kernels: the gates of all tokens (prefix sums and maxima); every chunk's own sum of
//                         k v^T; the scan of these over a request's chunks, elementwise; every chunk's outputs.  Sums, decays and states are fp32; as operands of
//                         the tensor cores, weighted keys, states and weighted scores are split into two bf16 numbers (16 bits of mantissa), queries,
//                         keys and values are bf16 as the projection left them.
#include "common.cuh"
#include "kernels.h"

namespace ogb {

template <typename T> __device__ __forceinline__ float rec_f32(T v);
template <> __device__ __forceinline__ float rec_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ float rec_f32<__nv_bfloat16>(__nv_bfloat16 v) { return bf2f(v); }
template <typename T> __device__ __forceinline__ T rec_from(float v);
template <> __device__ __forceinline__ float rec_from<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 rec_from<__nv_bfloat16>(float v) { return f2bf(v); }

template <typename T> __device__ __forceinline__ float2 rec_ld2(const T* p);
template <> __device__ __forceinline__ float2 rec_ld2<float>(const float* p) { return *reinterpret_cast<const float2*>(p); }
template <> __device__ __forceinline__ float2 rec_ld2<__nv_bfloat16>(const __nv_bfloat16* p) { return unpack_bf16x2(*reinterpret_cast<const uint32_t*>(p)); }
__device__ __forceinline__ void rec_st2(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
__device__ __forceinline__ void rec_st2(__nv_bfloat16* p, float a, float b) { *reinterpret_cast<uint32_t*>(p) = pack_bf16x2(a, b); }

__device__ __forceinline__ float rec_sigmoid(float x) { return 1.f / (1.f + expf(-x)); }
// The same for models with 16-bit activations, with the hardware's exponential and reciprocal (relative error of a few 1e-7 where the argument is of the order of one).
template <typename T> __device__ __forceinline__ float rec_gate(float x) {
  if constexpr (sizeof(T) == 4) return rec_sigmoid(x);
  else return __fdividef(1.f, 1.f + __expf(-fmaxf(x, -80.f)));
}

// ------------------------------------------------------------------------------------ gated average
struct MinGruParams {
  const void *z, *x, *g;               // columns of the projection rows
  void* out;
  float* state;
  const int32_t *slots, *cu_seqlens, *past_lens;
  long long slot_stride;
  int ld, ldo, W;
  float scale;
};

template <typename T> __device__ __forceinline__ float mg_candidate(float u) { return u >= 0.f ? u + 0.5f : rec_gate<T>(u); }

template <int N> __device__ __forceinline__ void rec_load(const float* p, float (&v)[N]) {
  if constexpr (N == 4) { const float4 f = *reinterpret_cast<const float4*>(p); v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w; }
  else v[0] = *p;
}
template <int N> __device__ __forceinline__ void rec_load(const __nv_bfloat16* p, float (&v)[N]) {
  if constexpr (N == 4) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
  } else v[0] = bf2f(*p);
}
template <int N> __device__ __forceinline__ void rec_store(float* p, const float (&v)[N]) {
  if constexpr (N == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else *p = v[0];
}
template <int N> __device__ __forceinline__ void rec_store(__nv_bfloat16* p, const float (&v)[N]) {
  if constexpr (N == 4) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
  else *p = f2bf(v[0]);
}

// A thread has N neighbouring columns (N = 4: everything on boundaries of four).
template <typename T, int N>
__global__ void __launch_bounds__(128) min_gru_step_kernel(MinGruParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.y, c = (blockIdx.x * blockDim.x + threadIdx.x) * N;
  const int t0 = p.cu_seqlens[b], t1 = p.cu_seqlens[b + 1];
  if (c >= p.W || t0 >= t1) return;
  float* st = p.state + size_t(p.slots[b]) * p.slot_stride + c;
  const T *z = static_cast<const T*>(p.z) + c, *x = static_cast<const T*>(p.x) + c, *g = static_cast<const T*>(p.g) + c;
  float S[N] = {};
  if (p.past_lens[b] != 0) rec_load(st, S);
  for (int t = t0; t < t1; ++t) {
    float zz[N], u[N], gg[N], o[N];
    rec_load(z + size_t(t) * p.ld, zz);
    rec_load(x + size_t(t) * p.ld, u);
    rec_load(g + size_t(t) * p.ld, gg);
#pragma unroll
    for (int e = 0; e < N; ++e) {
      const float a = rec_gate<T>(zz[e]);
      S[e] = fmaf(a, mg_candidate<T>(u[e]), (1.f - a) * S[e]);
      o[e] = S[e] * gg[e] * rec_gate<T>(gg[e]) * p.scale;
    }
    rec_store(static_cast<T*>(p.out) + size_t(t) * p.ldo + c, o);
  }
  rec_store(st, S);
}

// Prompts, in chunks of MG_L tokens.  Pass 1: what a chunk does to a state, S -> A S + D, per column; the state before the request's first token is kept beside
// (the last chunk of pass 2 overwrites it).  Pass 2: the state before the chunk from the chunks before it, then the chunk's tokens.  A thread has two
// neighbouring columns.  Column count, strides and the columns' addresses are even.  Grid (.., chunks of the longest request, requests).
constexpr int MG_L = 64, MG_AHEAD = 8, MG_THREADS = 128;

__device__ __forceinline__ size_t mg_chunk(int t0, int b, int j) { return size_t(t0 / MG_L + b + j); }      // (unique: see mc_chunk)

template <typename T, bool OUT>
__global__ void __launch_bounds__(MG_THREADS) min_gru_chunk_kernel(MinGruParams p, float4* __restrict__ maps, float2* __restrict__ first) {
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.z, j = blockIdx.y, t0 = p.cu_seqlens[b], t1 = p.cu_seqlens[b + 1];
  const int pair = blockIdx.x * MG_THREADS + threadIdx.x, c = 2 * pair, begin = t0 + j * MG_L, end = min(t1, begin + MG_L);
  if (begin >= t1 || c >= p.W) return;
  const int pairs = p.W / 2;
  float* st = p.state + size_t(p.slots[b]) * p.slot_stride + c;
  const T *z = static_cast<const T*>(p.z) + c, *x = static_cast<const T*>(p.x) + c, *g = static_cast<const T*>(p.g) + c;
  T* out = static_cast<T*>(p.out) + c;
  float2 A = make_float2(1.f, 1.f), S = make_float2(0.f, 0.f);
  if constexpr (OUT) {
    S = first[size_t(b) * pairs + pair];
    const float4* m = maps + mg_chunk(t0, b, 0) * pairs + pair;
#pragma unroll 8
    for (int i = 0; i < j; ++i) {
      const float4 v = m[size_t(i) * pairs];
      S = make_float2(fmaf(v.x, S.x, v.z), fmaf(v.y, S.y, v.w));
    }
  } else if (j == 0) {
    first[size_t(b) * pairs + pair] = p.past_lens[b] == 0 ? S : make_float2(st[0], st[1]);
  }
  for (int t = begin; t < end; t += MG_AHEAD) {
    float2 zz[MG_AHEAD], u[MG_AHEAD], gg[MG_AHEAD];
#pragma unroll
    for (int i = 0; i < MG_AHEAD; ++i) {
      const int r = min(t + i, end - 1);
      zz[i] = rec_ld2(z + size_t(r) * p.ld);
      u[i] = rec_ld2(x + size_t(r) * p.ld);
      if constexpr (OUT) gg[i] = rec_ld2(g + size_t(r) * p.ld);
    }
#pragma unroll
    for (int i = 0; i < MG_AHEAD; ++i) {
      if (t + i >= end) break;
      const float s0 = rec_gate<T>(zz[i].x), s1 = rec_gate<T>(zz[i].y), a0 = 1.f - s0, a1 = 1.f - s1;
      S = make_float2(fmaf(a0, S.x, s0 * mg_candidate<T>(u[i].x)), fmaf(a1, S.y, s1 * mg_candidate<T>(u[i].y)));
      if constexpr (OUT) rec_st2(out + size_t(t + i) * p.ldo, S.x * gg[i].x * rec_gate<T>(gg[i].x) * p.scale, S.y * gg[i].y * rec_gate<T>(gg[i].y) * p.scale);
      else A = make_float2(A.x * a0, A.y * a1);
    }
  }
  if constexpr (OUT) {
    if (end == t1) { st[0] = S.x; st[1] = S.y; }
  } else {
    maps[mg_chunk(t0, b, j) * pairs + pair] = make_float4(A.x, A.y, S.x, S.y);
  }
}

// ------------------------------------------------------------------------------------ matrix memory
struct MlstmParams {
  const void *q, *k, *v, *g;           // columns of the projection rows: [H, d], [H, d], [H, dv], [H, dv]
  const float *gates, *gate_b;         // [T, 2 H] logits of the input and the forget gates (row stride ldg), their biases
  const float* norm_w;                 // [H, dv]
  void* out;
  float* state;                        // per slot [H, d, dv], [H, d], [H]
  const int32_t *slots, *cu_seqlens, *past_lens;
  long long slot_stride;
  int ld, ldg, ldo, H, d, dv;
  float cap, eps, q_scale;
  int long_tokens;                     // > 0: requests with at least that many tokens are left to the chunk kernels
};

struct MlstmGate { float keep, add, floor, m; };
// running maximum and factors of a token
__device__ __forceinline__ MlstmGate mlstm_gate(float zi, float zf, float cap, float m) {
  const float i = cap * tanhf(zi / cap), y = cap * tanhf(zf / cap);
  const float f = -(y < -20.f ? -y : log1pf(expf(-y)));
  const float fm = f + m, n = fmaxf(fm, i);
  return MlstmGate{expf(fm - n), expf(i - n), expf(-n), n};
}

constexpr int ML_THREADS = 256, ML_MAX_D = 1024, ML_MAX_CLUSTER = 8;

__device__ __forceinline__ void rec_cluster_arrive() { asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory"); }
__device__ __forceinline__ void rec_cluster_wait() { asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory"); }
__device__ __forceinline__ float rec_ld_peer(const float* local, uint32_t rank) {
  uint32_t a;
  float v;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(a) : "r"(smem_u32(local)), "r"(rank));
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(a) : "memory");
  return v;
}

// Grid (cluster, heads, requests).  The CTA owns columns [rank * cw, rank * cw + cw) of the head (cw a multiple of VEC, at most 256), a thread VEC columns of every
// groups-th row: NR rows in registers from the first token to the last, or (NR = 0) any number, read and written back at every token.
template <typename T, int VEC, int NR>
__global__ void __launch_bounds__(ML_THREADS) mlstm_step_kernel(MlstmParams p, int cw) {
  __shared__ float sk[ML_MAX_D], sq[ML_MAX_D], sn[ML_MAX_D];
  __shared__ float red[ML_THREADS * VEC];
  __shared__ float part[ML_THREADS / 32];
  __shared__ float sums[2];            // this CTA's sum of squares, by token parity
  pdl_launch_dependents();
  pdl_wait();
  const int rank = blockIdx.x, C = gridDim.x, h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int t0 = p.cu_seqlens[b], t1 = p.cu_seqlens[b + 1];
  const int d = p.d, dv = p.dv;
  if (t0 >= t1 || (p.long_tokens > 0 && t1 - t0 >= p.long_tokens)) return;      // (alike in all CTAs of a cluster)
  const bool fresh = p.past_lens[b] == 0;
  float* slot = p.state + size_t(p.slots[b]) * p.slot_stride;
  const int c0 = rank * cw, cols = min(cw, dv - c0);                // (may be <= 0)
  const int lanes = (cw + VEC - 1) / VEC;                           // column groups
  const int groups = ML_THREADS / lanes, cg = tid % lanes, rg = tid / lanes, col = cg * VEC;
  const bool mine = rg < groups && col < cols;
  float* S = slot + size_t(h) * d * dv + c0 + col;
  float* gn = slot + size_t(p.H) * d * dv + size_t(h) * d;
  float* gm = slot + size_t(p.H) * d * (dv + 1) + h;
  auto load = [&](int r, float (&s)[VEC]) {
    if constexpr (VEC == 4) {
      const float4 f = *reinterpret_cast<const float4*>(S + size_t(r) * dv);
      s[0] = f.x; s[1] = f.y; s[2] = f.z; s[3] = f.w;
    } else {
      s[0] = S[size_t(r) * dv];
    }
  };
  auto store = [&](int r, const float (&s)[VEC]) {
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(S + size_t(r) * dv) = make_float4(s[0], s[1], s[2], s[3]);
    else S[size_t(r) * dv] = s[0];
  };
  float st[NR > 0 ? NR : 1][VEC];
  if constexpr (NR > 0) {
#pragma unroll
    for (int i = 0; i < NR; ++i) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) st[i][e] = 0.f;
      if (mine && !fresh && rg + i * groups < d) load(rg + i * groups, st[i]);
    }
  }
  for (int i = tid; i < d; i += ML_THREADS) sn[i] = fresh ? 0.f : gn[i];
  float m = fresh ? 0.f : *gm;
  for (int t = t0; t < t1; ++t) {
    const T* qp = static_cast<const T*>(p.q) + size_t(t) * p.ld + size_t(h) * d;
    const T* kp = static_cast<const T*>(p.k) + size_t(t) * p.ld + size_t(h) * d;
    const float* gp = p.gates + size_t(t) * p.ldg;
    float v[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) v[e] = mine ? rec_f32(static_cast<const T*>(p.v)[size_t(t) * p.ld + size_t(h) * dv + c0 + col + e]) : 0.f;
    const MlstmGate gt = mlstm_gate(gp[h] + p.gate_b[h], gp[p.H + h] + p.gate_b[p.H + h], p.cap, m);
    m = gt.m;
    float nq = 0.f;
    for (int i = tid; i < d; i += ML_THREADS) {
      const float kk = gt.add * rec_f32(kp[i]), qq = rec_f32(qp[i]) * p.q_scale, n = fmaf(gt.keep, sn[i], kk);
      sk[i] = kk; sq[i] = qq; sn[i] = n;
      nq = fmaf(n, qq, nq);
    }
    nq = warp_sum(nq);
    if (lane == 0) part[warp] = nq;
    __syncthreads();
    nq = 0.f;
#pragma unroll
    for (int w = 0; w < ML_THREADS / 32; ++w) nq += part[w];
    float o[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) o[e] = 0.f;
    auto step = [&](int r, float (&s)[VEC]) {
      const float kk = sk[r], qq = sq[r];
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        s[e] = fmaf(gt.keep, s[e], kk * v[e]);
        o[e] = fmaf(qq, s[e], o[e]);
      }
    };
    if (mine) {
      if constexpr (NR > 0) {
#pragma unroll
        for (int i = 0; i < NR; ++i) if (rg + i * groups < d) step(rg + i * groups, st[i]);
      } else {
        for (int r = rg; r < d; r += groups) {
          float s[VEC];
#pragma unroll
          for (int e = 0; e < VEC; ++e) s[e] = 0.f;
          if (!(fresh && t == t0)) load(r, s);
          step(r, s);
          store(r, s);
        }
      }
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) red[tid * VEC + e] = o[e];
    __syncthreads();
    // column sums over the row groups: thread tid takes column tid
    float val = 0.f;
    if (tid < cols) {
#pragma unroll 8
      for (int r = 0; r < groups; ++r) val += red[r * lanes * VEC + tid];
      val /= fmaxf(fabsf(nq), gt.floor) + 1e-6f;
    }
    float ss = warp_sum(val * val);
    if (lane == 0) part[warp] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int w = 0; w < ML_THREADS / 32; ++w) ss += part[w];
    if (C > 1) {
      if (tid == 0) sums[t & 1] = ss;
      __syncthreads();
      rec_cluster_arrive();
      rec_cluster_wait();
      ss = 0.f;
      for (int r = 0; r < C; ++r) ss += rec_ld_peer(&sums[t & 1], r);
    }
    if (tid < cols) {
      const size_t at = size_t(h) * dv + c0 + tid;
      const float gate = rec_sigmoid(rec_f32(static_cast<const T*>(p.g)[size_t(t) * p.ld + at]));
      static_cast<T*>(p.out)[size_t(t) * p.ldo + at] = rec_from<T>(val / sqrtf(ss / dv + p.eps) * p.norm_w[at] * gate);
    }
    if (t + 1 < t1) __syncthreads();
  }
  if constexpr (NR > 0) {
    if (mine) {
#pragma unroll
      for (int i = 0; i < NR; ++i) if (rg + i * groups < d) store(rg + i * groups, st[i]);
    }
  }
  // (every CTA of the cluster has read the normaliser and the maximum: all have met at a token)
  if (rank == 0) {
    for (int i = tid; i < d; i += ML_THREADS) gn[i] = sn[i];
    if (tid == 0) *gm = m;
  }
  if (C > 1) { rec_cluster_arrive(); rec_cluster_wait(); }          // no CTA leaves while another may read its sums
}

// ------------------------------------------------------------------------------------ matrix memory, chunks of a prompt
constexpr int MC_L = 64;               // tokens of a chunk

struct MlstmChunk {
  float *c, *M, *floor;                // [H, T] per token: c_t, M_t, e^-(running maximum)
  float *m_in, *M_last;                // [chunks, H]: maximum before the chunk, M of its last token
  float* sums;                         // [chunks, H, KS, NT, 32 lanes, 4]: first a chunk's own sums (fp32), then the state before it (bf16 pairs)
  float* nsums;                        // [chunks, H, dp]: the same for the normalisers (fp32 throughout)
  int T, KS, NT;                       // 16-row groups of the keys' columns, 8-column groups of the values' (both padded to whole 16s)
  int min_tokens;                      // shorter requests are not served here
};
// chunk j of request b: ids are unique because a request starts at least as many ids after the one before it as that one has chunks
__device__ __forceinline__ int mc_chunk(int t0, int b, int j) { return t0 / MC_L + b + j; }

// One CTA per (head, request).  A warp takes chunks, a lane two of a chunk's tokens; then the maxima are chained over the chunks.
__global__ void __launch_bounds__(1024) mlstm_gates_kernel(MlstmParams p, MlstmChunk k) {
  extern __shared__ float sm[];        // per chunk: sum of log forget gates, largest c, maximum before the chunk
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, b = blockIdx.y, t0 = p.cu_seqlens[b], len = p.cu_seqlens[b + 1] - t0;
  if (len < k.min_tokens || len <= 0) return;
  const int n = (len + MC_L - 1) / MC_L, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  float *sb = sm, *sc = sm + n, *si = sm + 2 * n;
  const float bi = p.gate_b[h], bf = p.gate_b[p.H + h];
  float *gc = k.c + size_t(h) * k.T + t0, *gM = k.M + size_t(h) * k.T + t0, *gf = k.floor + size_t(h) * k.T + t0;
  for (int j = warp; j < n; j += blockDim.x >> 5) {
    float i[2], f[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = j * MC_L + 2 * lane + e;
      i[e] = -INFINITY;
      f[e] = 0.f;
      if (t < len) {
        const float* gp = p.gates + size_t(t0 + t) * p.ldg;
        i[e] = p.cap * tanhf((gp[h] + bi) / p.cap);
        const float y = p.cap * tanhf((gp[p.H + h] + bf) / p.cap);
        f[e] = -(y < -20.f ? -y : log1pf(expf(-y)));
      }
    }
    float s = f[0] + f[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) { const float v = __shfl_up_sync(0xffffffffu, s, o); if (lane >= o) s += v; }
    const float b1 = s, b0 = s - f[1], c0 = i[0] - b0, c1 = i[1] - b1;
    float x = fmaxf(c0, c1);
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) { const float v = __shfl_up_sync(0xffffffffu, x, o); if (lane >= o) x = fmaxf(x, v); }
    float before = __shfl_up_sync(0xffffffffu, x, 1);
    if (lane == 0) before = -INFINITY;
    const int t = j * MC_L + 2 * lane;
    if (t < len) { gc[t] = c0; gM[t] = fmaxf(before, c0); gf[t] = b0; }
    if (t + 1 < len) { gc[t + 1] = c1; gM[t + 1] = x; gf[t + 1] = b1; }
    if (lane == 31) { sb[j] = b1; sc[j] = x; }
  }
  __syncthreads();
  float* gm = p.state + size_t(p.slots[b]) * p.slot_stride + size_t(p.H) * p.d * (p.dv + 1) + h;
  if (threadIdx.x == 0) {
    float m = p.past_lens[b] == 0 ? 0.f : *gm;
    for (int j = 0; j < n; ++j) {
      const float M = fmaxf(m, sc[j]);
      const size_t at = size_t(mc_chunk(t0, b, j)) * p.H + h;
      k.m_in[at] = m;
      k.M_last[at] = M;
      si[j] = m;
      m = sb[j] + M;
    }
    *gm = m;
  }
  __syncthreads();
  for (int t = threadIdx.x; t < len; t += blockDim.x) {
    const float M = fmaxf(si[t / MC_L], gM[t]);
    gM[t] = M;
    gf[t] = expf(-(gf[t] + M));
  }
}

__device__ __forceinline__ void split_bf16(float v, __nv_bfloat16& hi, __nv_bfloat16& lo) {
  hi = f2bf(v);
  lo = f2bf(v - bf2f(hi));
}
__device__ __forceinline__ uint32_t pair_bits(__nv_bfloat16 a, __nv_bfloat16 b) {
  return uint32_t(__bfloat16_as_ushort(a)) | uint32_t(__bfloat16_as_ushort(b)) << 16;
}

// A chunk's own sums, transposed: rows are value columns, so that a thread's results are the two halves of its B operand in the output kernel.
// Grid (tiles of 64 key columns x 64 value columns, chunks of the longest request, requests x heads).
constexpr int MC_PITCH = 64 + 8;
__global__ void __launch_bounds__(128) mlstm_sums_kernel(MlstmParams p, MlstmChunk k) {
  __shared__ __align__(16) __nv_bfloat16 sv[MC_L * MC_PITCH], shi[MC_L * MC_PITCH], slo[MC_L * MC_PITCH];
  __shared__ float sw[MC_L];
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.z % p.H, b = blockIdx.z / p.H, j = blockIdx.y, t0 = p.cu_seqlens[b], len = p.cu_seqlens[b + 1] - t0;
  if (len < k.min_tokens || j * MC_L >= len) return;
  const int v_tiles = (k.NT + 7) / 8, v0 = blockIdx.x % v_tiles * 64, d0 = blockIdx.x / v_tiles * 64;
  const int n = min(MC_L, len - j * MC_L), first = t0 + j * MC_L, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int chunk = mc_chunk(t0, b, j);
  const float M = k.M_last[size_t(chunk) * p.H + h];
  if (tid < MC_L) sw[tid] = tid < n ? expf(k.c[size_t(h) * k.T + first + tid] - M) : 0.f;
  __syncthreads();
  for (int i = tid; i < MC_L * 8; i += 128) {
    const int t = i / 8, c = i % 8 * 8;
    const bool ok = t < n;
    const size_t row = size_t(first + t) * p.ld;
    uint4 v = make_uint4(0u, 0u, 0u, 0u), kk = v, hi, lo;
    if (ok && v0 + c < p.dv) v = *reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(p.v) + row + size_t(h) * p.dv + v0 + c);
    if (ok && d0 + c < p.d) kk = *reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(p.k) + row + size_t(h) * p.d + d0 + c);
    const uint32_t* in = &kk.x;
    uint32_t *ph = &hi.x, *pl = &lo.x;
    const float w = sw[t];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 f = unpack_bf16x2(in[e]);
      __nv_bfloat16 h0, l0, h1, l1;
      split_bf16(f.x * w, h0, l0);
      split_bf16(f.y * w, h1, l1);
      ph[e] = pair_bits(h0, h1);
      pl[e] = pair_bits(l0, l1);
    }
    *reinterpret_cast<uint4*>(sv + t * MC_PITCH + c) = v;
    *reinterpret_cast<uint4*>(shi + t * MC_PITCH + c) = hi;
    *reinterpret_cast<uint4*>(slo + t * MC_PITCH + c) = lo;
  }
  __syncthreads();
  if (v0 == 0 && tid < 64 && d0 + tid < k.KS * 16) {
    float s = 0.f;
    for (int t = 0; t < MC_L; ++t) s += bf2f(shi[t * MC_PITCH + tid]) + bf2f(slo[t * MC_PITCH + tid]);
    k.nsums[(size_t(chunk) * p.H + h) * k.KS * 16 + d0 + tid] = s;
  }
  if (v0 + warp * 16 >= k.NT * 8) return;
  float acc[8][4];
#pragma unroll
  for (int i = 0; i < 8; ++i) { acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f; }
#pragma unroll
  for (int ks = 0; ks < MC_L / 16; ++ks) {
    uint32_t a[4];
    ldmatrix_x4_trans(a, sv + (ks * 16 + (lane & 7) + (lane >> 4) * 8) * MC_PITCH + warp * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
    for (int g = 0; g < 4; ++g) {
      const int at = (ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * MC_PITCH + g * 16 + (lane >> 4) * 8;
      uint32_t w[4];
      ldmatrix_x4_trans(w, shi + at);
      mma_bf16_16816(acc[2 * g], a, w[0], w[1]);
      mma_bf16_16816(acc[2 * g + 1], a, w[2], w[3]);
      ldmatrix_x4_trans(w, slo + at);
      mma_bf16_16816(acc[2 * g], a, w[0], w[1]);
      mma_bf16_16816(acc[2 * g + 1], a, w[2], w[3]);
    }
  }
  float4* dst = reinterpret_cast<float4*>(k.sums) + (size_t(chunk) * p.H + h) * k.KS * k.NT * 32;
  const int nt = (v0 + warp * 16) / 8;
#pragma unroll
  for (int g = 0; g < 4; ++g) {
    const int ks = d0 / 16 + g;
    if (ks >= k.KS) break;
    dst[(size_t(ks) * k.NT + nt) * 32 + lane] = make_float4(acc[2 * g][0], acc[2 * g][1], acc[2 * g + 1][0], acc[2 * g + 1][1]);
    dst[(size_t(ks) * k.NT + nt + 1) * 32 + lane] = make_float4(acc[2 * g][2], acc[2 * g][3], acc[2 * g + 1][2], acc[2 * g + 1][3]);
  }
}

// The states before every chunk: S <- decay * S + sums, the four entries of a thread (rows 2 i, 2 i + 1, 2 i + 8, 2 i + 9 of a 16-row group, one column) kept
// over the chunks.  The last column of CTAs takes the normalisers.  Grid (.., heads, requests).
__global__ void __launch_bounds__(256) mlstm_scan_kernel(MlstmParams p, MlstmChunk k) {
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.y, b = blockIdx.z, t0 = p.cu_seqlens[b], len = p.cu_seqlens[b + 1] - t0;
  if (len < k.min_tokens || len <= 0) return;
  const int n = (len + MC_L - 1) / MC_L, chunk0 = mc_chunk(t0, b, 0);
  const bool fresh = p.past_lens[b] == 0;
  float* slot = p.state + size_t(p.slots[b]) * p.slot_stride;
  const float *m_in = k.m_in + size_t(chunk0) * p.H + h, *M_last = k.M_last + size_t(chunk0) * p.H + h;
  if (blockIdx.x == gridDim.x - 1) {
    const int dp = k.KS * 16;
    for (int i = threadIdx.x; i < dp; i += blockDim.x) {
      float* g = slot + size_t(p.H) * p.d * p.dv + size_t(h) * p.d + i;
      float S = fresh || i >= p.d ? 0.f : *g;
      for (int j = 0; j < n; ++j) {
        float* at = k.nsums + (size_t(chunk0 + j) * p.H + h) * dp + i;
        const float u = *at;
        *at = S;
        S = fmaf(expf(m_in[size_t(j) * p.H] - M_last[size_t(j) * p.H]), S, u);
      }
      if (i < p.d) *g = S;
    }
    return;
  }
  const int f = blockIdx.x * blockDim.x + threadIdx.x;
  if (f >= k.KS * k.NT * 32) return;
  const int lane = f & 31, nt = (f >> 5) % k.NT, ks = (f >> 5) / k.NT;
  const int v = nt * 8 + (lane >> 2), d = ks * 16 + (lane & 3) * 2;
  float* g = slot + size_t(h) * p.d * p.dv + v;
  float S[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const int r = d + (e >> 1) * 8 + (e & 1);
    S[e] = fresh || r >= p.d || v >= p.dv ? 0.f : g[size_t(r) * p.dv];
  }
  const size_t stride = size_t(p.H) * k.KS * k.NT * 32;
  float4* u = reinterpret_cast<float4*>(k.sums) + (size_t(chunk0) * p.H + h) * k.KS * k.NT * 32 + f;
  constexpr int AHEAD = 8;
  for (int j0 = 0; j0 < n; j0 += AHEAD) {
    float4 x[AHEAD];
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) if (j0 + i < n) x[i] = u[size_t(j0 + i) * stride];
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      if (j0 + i >= n) break;
      const float w = expf(m_in[size_t(j0 + i) * p.H] - M_last[size_t(j0 + i) * p.H]);
      __nv_bfloat16 hi[4], lo[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) split_bf16(S[e], hi[e], lo[e]);
      reinterpret_cast<uint4*>(u)[size_t(j0 + i) * stride] =
          make_uint4(pair_bits(hi[0], hi[1]), pair_bits(hi[2], hi[3]), pair_bits(lo[0], lo[1]), pair_bits(lo[2], lo[3]));
      S[0] = fmaf(w, S[0], x[i].x); S[1] = fmaf(w, S[1], x[i].y); S[2] = fmaf(w, S[2], x[i].z); S[3] = fmaf(w, S[3], x[i].w);
    }
  }
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const int r = d + (e >> 1) * 8 + (e & 1);
    if (r < p.d && v < p.dv) g[size_t(r) * p.dv] = S[e];
  }
}

// Outputs of a chunk.  Warp (rg, cg): rows rg * 32 .. + 31; scores of 16 keys each, then NTW 8-column groups of the values.  Grid (chunks, heads, requests).
template <int NTW>
__global__ void __launch_bounds__(256, NTW <= 8 ? 2 : 1) mlstm_out_kernel(MlstmParams p, MlstmChunk k) {
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ float sc[MC_L], sM[MC_L], sfl[MC_L], snq[MC_L], srow[4][MC_L];
  pdl_launch_dependents();
  pdl_wait();
  const int j = blockIdx.x, h = blockIdx.y, b = blockIdx.z, t0 = p.cu_seqlens[b], len = p.cu_seqlens[b + 1] - t0;
  if (len < k.min_tokens || j * MC_L >= len) return;
  const int dp = k.KS * 16, vp = k.NT * 8, qpitch = dp + 8, vpitch = vp + 8;
  __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(smem);
  __nv_bfloat16* sk = sq + MC_L * qpitch;
  __nv_bfloat16* sv = sk + MC_L * qpitch;
  __nv_bfloat16* phi = sv + MC_L * vpitch;
  __nv_bfloat16* plo = phi + MC_L * MC_PITCH;
  const int n = min(MC_L, len - j * MC_L), first = t0 + j * MC_L, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t4 = lane & 3;
  const int rg = warp >> 2, cg = warp & 3, chunk = mc_chunk(t0, b, j);
  const bool empty = j == 0 && p.past_lens[b] == 0;        // the state before the chunk is zero
  for (int i = tid; i < MC_L * (dp / 8); i += 256) {
    const int t = i / (dp / 8), c = i % (dp / 8) * 8;
    const bool ok = t < n && c < p.d;
    const size_t at = size_t(first + (ok ? t : 0)) * p.ld + size_t(h) * p.d + (ok ? c : 0);
    cp_async16(sq + t * qpitch + c, static_cast<const __nv_bfloat16*>(p.q) + at, ok);
    cp_async16(sk + t * qpitch + c, static_cast<const __nv_bfloat16*>(p.k) + at, ok);
  }
  cp_async_commit();
  for (int i = tid; i < MC_L * (vp / 8); i += 256) {
    const int t = i / (vp / 8), c = i % (vp / 8) * 8;
    const bool ok = t < n && c < p.dv;
    cp_async16(sv + t * vpitch + c, static_cast<const __nv_bfloat16*>(p.v) + size_t(first + (ok ? t : 0)) * p.ld + size_t(h) * p.dv + (ok ? c : 0), ok);
  }
  cp_async_commit();
  const float m = k.m_in[size_t(chunk) * p.H + h];
  if (tid < MC_L) {
    const size_t at = size_t(h) * k.T + first + tid;
    sc[tid] = tid < n ? k.c[at] : -INFINITY;
    sM[tid] = tid < n ? k.M[at] : 0.f;
    sfl[tid] = tid < n ? k.floor[at] : 1.f;
  }
  cp_async_wait<1>();
  __syncthreads();
  // ---- weighted scores
  {
    float acc[2][2][4] = {};
    if (cg * 16 <= rg * 32 + 31) {
      for (int ks = 0; ks < k.KS; ++ks) {
        uint32_t kb[4];
        ldmatrix_x4(kb, sk + (cg * 16 + (lane >> 4) * 8 + (lane & 7)) * qpitch + ks * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
        for (int mt = 0; mt < 2; ++mt) {
          uint32_t a[4];
          ldmatrix_x4(a, sq + (rg * 32 + mt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * qpitch + ks * 16 + (lane >> 4) * 8);
          mma_bf16_16816(acc[mt][0], a, kb[0], kb[1]);
          mma_bf16_16816(acc[mt][1], a, kb[2], kb[3]);
        }
      }
    }
#pragma unroll
    for (int mt = 0; mt < 2; ++mt)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int t = rg * 32 + mt * 16 + g + half * 8;
        const float M = sM[t];
        float sum = 0.f;
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          const int s = cg * 16 + nt * 8 + t4 * 2;
          __nv_bfloat16 hi[2], lo[2];
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const float w = s + e <= t ? acc[mt][nt][half * 2 + e] * p.q_scale * expf(sc[s + e] - M) : 0.f;
            sum += w;
            split_bf16(w, hi[e], lo[e]);
          }
          *reinterpret_cast<uint32_t*>(phi + t * MC_PITCH + s) = pair_bits(hi[0], hi[1]);
          *reinterpret_cast<uint32_t*>(plo + t * MC_PITCH + s) = pair_bits(lo[0], lo[1]);
        }
        sum += __shfl_xor_sync(0xffffffffu, sum, 1);
        sum += __shfl_xor_sync(0xffffffffu, sum, 2);
        if (t4 == 0) srow[cg][t] = sum;
      }
  }
  // ---- q . n of the state before the chunk: four threads per row
  {
    const int t = tid >> 2;
    float s = 0.f;
    if (!empty) {
      const float* nn = k.nsums + (size_t(chunk) * p.H + h) * dp;
      for (int i = tid & 3; i < dp; i += 4) s = fmaf(bf2f(sq[t * qpitch + i]), nn[i], s);
      s += __shfl_xor_sync(0xffffffffu, s, 1);
      s += __shfl_xor_sync(0xffffffffu, s, 2);
    }
    if ((tid & 3) == 0) snq[t] = s * p.q_scale * expf(m - sM[t]);
  }
  cp_async_wait<0>();
  __syncthreads();
  // ---- numerators
  float o[2][NTW][4];
#pragma unroll
  for (int mt = 0; mt < 2; ++mt)
#pragma unroll
    for (int i = 0; i < NTW; ++i) { o[mt][i][0] = o[mt][i][1] = o[mt][i][2] = o[mt][i][3] = 0.f; }
  const int nt0 = cg * NTW;
  if (!empty) {
    // (the next step's fragments are on their way while this one's are multiplied; groups past the last read it again)
    const uint4* S = reinterpret_cast<const uint4*>(k.sums) + (size_t(chunk) * p.H + h) * k.KS * k.NT * 32 + lane;
    constexpr int PF = NTW <= 8 ? NTW : 1;
    uint4 next[PF];
    auto fetch = [&](int ks, int i) { return S[(size_t(ks) * k.NT + min(nt0 + i, k.NT - 1)) * 32]; };
    if constexpr (PF == NTW) {
#pragma unroll
      for (int i = 0; i < PF; ++i) next[i] = fetch(0, i);
    }
    for (int ks = 0; ks < k.KS; ++ks) {
      uint32_t a[2][4];
      uint4 now[PF];
      if constexpr (PF == NTW) {
        const int after = min(ks + 1, k.KS - 1);
#pragma unroll
        for (int i = 0; i < PF; ++i) { now[i] = next[i]; next[i] = fetch(after, i); }
      }
#pragma unroll
      for (int mt = 0; mt < 2; ++mt) ldmatrix_x4(a[mt], sq + (rg * 32 + mt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * qpitch + ks * 16 + (lane >> 4) * 8);
#pragma unroll
      for (int i = 0; i < NTW; ++i) {
        if (nt0 + i >= k.NT) break;
        const uint4 f = PF == NTW ? now[i % PF] : fetch(ks, i);
#pragma unroll
        for (int mt = 0; mt < 2; ++mt) {
          mma_bf16_16816(o[mt][i], a[mt], f.x, f.y);
          mma_bf16_16816(o[mt][i], a[mt], f.z, f.w);
        }
      }
    }
#pragma unroll
    for (int mt = 0; mt < 2; ++mt) {
      const float w0 = p.q_scale * expf(m - sM[rg * 32 + mt * 16 + g]), w1 = p.q_scale * expf(m - sM[rg * 32 + mt * 16 + g + 8]);
#pragma unroll
      for (int i = 0; i < NTW; ++i) { o[mt][i][0] *= w0; o[mt][i][1] *= w0; o[mt][i][2] *= w1; o[mt][i][3] *= w1; }
    }
  }
#pragma unroll
  for (int ks = 0; ks < MC_L / 16; ++ks) {
    if (ks * 16 > rg * 32 + 31) break;
    uint32_t a[2][4], c[2][4];
#pragma unroll
    for (int mt = 0; mt < 2; ++mt) {
      const int at = (rg * 32 + mt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * MC_PITCH + ks * 16 + (lane >> 4) * 8;
      ldmatrix_x4(a[mt], phi + at);
      ldmatrix_x4(c[mt], plo + at);
    }
#pragma unroll
    for (int i = 0; i < NTW; i += 2) {
      if (nt0 + i >= k.NT) break;                          // (whole pairs of groups: NT is even)
      uint32_t vb[4];
      ldmatrix_x4_trans(vb, sv + (ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * vpitch + (nt0 + i + (lane >> 4)) * 8);
#pragma unroll
      for (int mt = 0; mt < 2; ++mt) {
        mma_bf16_16816(o[mt][i], a[mt], vb[0], vb[1]);
        mma_bf16_16816(o[mt][i], c[mt], vb[0], vb[1]);
        mma_bf16_16816(o[mt][i + 1], a[mt], vb[2], vb[3]);
        mma_bf16_16816(o[mt][i + 1], c[mt], vb[2], vb[3]);
      }
    }
  }
  // ---- denominators, norm over the head, gate
  float inv[2][2];
#pragma unroll
  for (int mt = 0; mt < 2; ++mt)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int t = rg * 32 + mt * 16 + g + half * 8;
      const float nq = snq[t] + ((srow[0][t] + srow[1][t]) + (srow[2][t] + srow[3][t]));
      inv[mt][half] = 1.f / (fmaxf(fabsf(nq), sfl[t]) + 1e-6f);
    }
  __syncthreads();                                          // (the row sums have been read)
#pragma unroll
  for (int mt = 0; mt < 2; ++mt)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < NTW; ++i)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const float x = o[mt][i][half * 2 + e] * inv[mt][half];
          o[mt][i][half * 2 + e] = x;
          ss = fmaf(x, x, ss);
        }
      ss += __shfl_xor_sync(0xffffffffu, ss, 1);
      ss += __shfl_xor_sync(0xffffffffu, ss, 2);
      if (t4 == 0) srow[cg][rg * 32 + mt * 16 + g + half * 8] = ss;
    }
  __syncthreads();
#pragma unroll
  for (int mt = 0; mt < 2; ++mt)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int t = rg * 32 + mt * 16 + g + half * 8;
      if (t >= n) continue;
      const float r = 1.f / sqrtf(((srow[0][t] + srow[1][t]) + (srow[2][t] + srow[3][t])) / p.dv + p.eps);
      const __nv_bfloat16* gp = static_cast<const __nv_bfloat16*>(p.g) + size_t(first + t) * p.ld + size_t(h) * p.dv;
      __nv_bfloat16* op = static_cast<__nv_bfloat16*>(p.out) + size_t(first + t) * p.ldo + size_t(h) * p.dv;
#pragma unroll
      for (int i = 0; i < NTW; ++i) {
        const int c = (nt0 + i) * 8 + t4 * 2;
        if (c >= p.dv) break;
        const float2 w = *reinterpret_cast<const float2*>(p.norm_w + size_t(h) * p.dv + c), gg = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(gp + c));
        *reinterpret_cast<uint32_t*>(op + c) =
            pack_bf16x2(o[mt][i][half * 2] * r * w.x * rec_sigmoid(gg.x), o[mt][i][half * 2 + 1] * r * w.y * rec_sigmoid(gg.y));
      }
    }
}

}  // namespace ogb

using namespace ogb;

OGB_API long long ogb_min_gru_scratch_bytes(int T, int B, int W) { return ((long long)(T / MG_L + B) * 16 + (long long)B * 8) * ((W + 1) / 2); }

// See kernels.h.
OGB_API int ogb_min_gru(const void* z, const void* x, const void* g, int ld, float* state, long long slot_stride, const int32_t* slots,
                        const int32_t* cu_seqlens, const int32_t* past_lens, void* out, int ldo, int T, int B, int W, float scale, int max_q_len,
                        void* scratch, long long scratch_bytes, int fp32, void* stream) {
  if (B <= 0 || W <= 0) return 0;
  if (B > 65535 || slot_stride < W) return -1;
  const MinGruParams p{z, x, g, out, state, slots, cu_seqlens, past_lens, slot_stride, ld, ldo, W, scale};
  auto s = static_cast<cudaStream_t>(stream);
  auto addr = [](const void* a) { return reinterpret_cast<uintptr_t>(a); };
  const bool even = W % 2 == 0 && ld % 2 == 0 && ldo % 2 == 0 && ((addr(z) | addr(x) | addr(g) | addr(out)) & (fp32 ? 7 : 3)) == 0;
  using H = __nv_bfloat16;
  if (!scratch || !even) {
    const bool four = W % 4 == 0 && ld % 4 == 0 && ldo % 4 == 0 && slot_stride % 4 == 0 && (addr(state) & 15) == 0 &&
                      ((addr(z) | addr(x) | addr(g) | addr(out)) & (fp32 ? 15 : 7)) == 0;
    const dim3 grid(four ? (W / 4 + 127) / 128 : (W + 127) / 128, B), block(128);
    if (four) return (fp32 ? launch_pdl(min_gru_step_kernel<float, 4>, grid, block, 0, s, p) : launch_pdl(min_gru_step_kernel<H, 4>, grid, block, 0, s, p)) ? 0 : -4;
    return (fp32 ? launch_pdl(min_gru_step_kernel<float, 1>, grid, block, 0, s, p) : launch_pdl(min_gru_step_kernel<H, 1>, grid, block, 0, s, p)) ? 0 : -4;
  }
  if (scratch_bytes < ogb_min_gru_scratch_bytes(T, B, W) || (addr(scratch) & 15)) return -2;
  auto* maps = static_cast<float4*>(scratch);
  auto* first = reinterpret_cast<float2*>(maps + size_t(T / MG_L + B) * (W / 2));
  const dim3 grid((W / 2 + MG_THREADS - 1) / MG_THREADS, (max_q_len + MG_L - 1) / MG_L, B), block(MG_THREADS);
  if (grid.y > 65535) return -1;
  const bool ok = fp32 ? launch_pdl(min_gru_chunk_kernel<float, false>, grid, block, 0, s, p, maps, first) && launch_pdl(min_gru_chunk_kernel<float, true>, grid, block, 0, s, p, maps, first)
                       : launch_pdl(min_gru_chunk_kernel<H, false>, grid, block, 0, s, p, maps, first) && launch_pdl(min_gru_chunk_kernel<H, true>, grid, block, 0, s, p, maps, first);
  return ok ? 0 : -4;
}

template <typename T, int VEC, int NR>
static bool LaunchMlstmStepRows(const MlstmParams& p, int B, int cw, int C, cudaStream_t s) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(C, p.H, B);
  cfg.blockDim = dim3(ML_THREADS);
  cfg.stream = s;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  attr[1].id = cudaLaunchAttributeClusterDimension;
  attr[1].val.clusterDim.x = C; attr[1].val.clusterDim.y = 1; attr[1].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = C > 1 ? 2 : 1;
  return cudaLaunchKernelEx(&cfg, mlstm_step_kernel<T, VEC, NR>, p, cw) == cudaSuccess;
}
template <typename T, int VEC>
static bool LaunchMlstmStep(const MlstmParams& p, int B, int cw, int C, int rows, cudaStream_t s) {
  if (rows <= 4) return LaunchMlstmStepRows<T, VEC, 4>(p, B, cw, C, s);
  if (rows <= 8) return LaunchMlstmStepRows<T, VEC, 8>(p, B, cw, C, s);
  if (rows <= 16) return LaunchMlstmStepRows<T, VEC, 16>(p, B, cw, C, s);
  return LaunchMlstmStepRows<T, VEC, 0>(p, B, cw, C, s);
}

// Sizes of the chunk form's scratch, or false where its kernels cannot run.
static bool MlstmChunkSizes(int T, int B, int H, int d, int dv, MlstmChunk* k, long long* floats) {
  if (d % 8 || dv % 8 || d > 256 || dv > 512) return false;
  k->T = T; k->KS = (d + 15) / 16; k->NT = (dv + 15) / 16 * 2;
  const long long chunks = T / MC_L + B, per = (long long)H * k->KS * k->NT * 128;
  *floats = 3LL * H * T + 2 * chunks * H + chunks * per + chunks * H * k->KS * 16 + 64;
  return true;
}

OGB_API long long ogb_mlstm_scratch_bytes(int T, int B, int H, int d, int dv) {
  MlstmChunk k;
  long long n = 0;
  return MlstmChunkSizes(T, B, H, d, dv, &k, &n) ? n * 4 : 0;
}

template <int NTW>
static bool LaunchMlstmOut(const MlstmParams& p, const MlstmChunk& k, dim3 grid, cudaStream_t s) {
  const int smem = (MC_L * (2 * (k.KS * 16 + 8) + k.NT * 8 + 8) + 2 * MC_L * MC_PITCH) * 2;
  static bool done[OGB_MAX_DEVICES] = {};
  return set_max_dyn_smem(mlstm_out_kernel<NTW>, 200 * 1024, done) && launch_pdl(mlstm_out_kernel<NTW>, grid, dim3(256), smem, s, p, k);
}

static int LaunchMlstmChunks(const MlstmParams& p, const OgbMlstm* a, cudaStream_t s) {
  MlstmChunk k;
  long long floats = 0;
  if (!MlstmChunkSizes(a->T, a->B, a->H, a->d, a->dv, &k, &floats)) return -5;
  if (floats * 4 > a->scratch_bytes) return -2;
  auto addr = [](const void* x) { return reinterpret_cast<uintptr_t>(x); };
  if (((addr(a->q) | addr(a->k) | addr(a->v) | addr(a->scratch)) & 15) || a->ld % 8 || a->ldo % 2 || ((addr(a->g) | addr(a->out)) & 3) || (addr(a->norm_w) & 7)) return -1;
  k.min_tokens = a->long_tokens;
  const long long chunks = a->T / MC_L + a->B, HT = (long long)a->H * a->T;
  k.sums = static_cast<float*>(a->scratch);                 // (16-byte pieces: first)
  k.nsums = k.sums + chunks * a->H * k.KS * k.NT * 128;
  k.c = k.nsums + chunks * a->H * k.KS * 16;
  k.M = k.c + HT; k.floor = k.M + HT;
  k.m_in = k.floor + HT; k.M_last = k.m_in + chunks * a->H;
  const int n = (a->max_q_len + MC_L - 1) / MC_L;
  if (n > 65535 || (long long)a->B * a->H > 65535) return -1;
  const size_t gsmem = size_t(3) * n * 4;
  if (gsmem > 48 * 1024) return -5;
  if (!launch_pdl(mlstm_gates_kernel, dim3(a->H, a->B), dim3(n >= 16 ? 1024 : (n >= 8 ? 512 : 256)), gsmem, s, p, k)) return -4;
  if (!launch_pdl(mlstm_sums_kernel, dim3(((k.NT + 7) / 8) * ((k.KS + 3) / 4), n, a->B * a->H), dim3(128), 0, s, p, k)) return -4;
  if (!launch_pdl(mlstm_scan_kernel, dim3((k.KS * k.NT * 32 + 255) / 256 + 1, a->H, a->B), dim3(256), 0, s, p, k)) return -4;
  const dim3 grid(n, a->H, a->B);
  const bool ok = k.NT <= 16 ? LaunchMlstmOut<4>(p, k, grid, s) : (k.NT <= 32 ? LaunchMlstmOut<8>(p, k, grid, s) : LaunchMlstmOut<16>(p, k, grid, s));
  return ok ? 0 : -4;
}

OGB_API int ogb_mlstm(const OgbMlstm* a, void* stream) {
  if (a->B <= 0 || a->H <= 0) return 0;
  if (a->d <= 0 || a->d > ML_MAX_D || a->dv <= 0 || a->B > 65535 || a->H > 65535 || a->cap <= 0.f) return -5;
  MlstmParams p{};
  p.q = a->q; p.k = a->k; p.v = a->v; p.g = a->g; p.gates = a->gates; p.gate_b = a->gate_b; p.norm_w = a->norm_w; p.out = a->out; p.state = a->state;
  p.slots = a->slots; p.cu_seqlens = a->cu_seqlens; p.past_lens = a->past_lens; p.slot_stride = a->slot_stride;
  p.ld = a->ld; p.ldg = a->ldg; p.ldo = a->ldo; p.H = a->H; p.d = a->d; p.dv = a->dv; p.cap = a->cap; p.eps = a->eps;
  p.q_scale = 1.f / sqrtf(float(a->d));
  auto s = static_cast<cudaStream_t>(stream);
  if (a->long_tokens > 0) {
    if (a->fp32) return -5;
    const int rc = LaunchMlstmChunks(p, a, s);
    if (rc != 0 || a->all_long) return rc;
    p.long_tokens = a->long_tokens;
  }
  // states in whole 16-byte pieces (a slot's first float is on a 16-byte boundary, heads and rows are multiples of four)
  const bool vec = a->dv % 4 == 0 && a->slot_stride % 4 == 0 && (reinterpret_cast<uintptr_t>(a->state) & 15) == 0;
  const int unit = vec ? 4 : 1;
  // CTAs that share a head: no more than it takes for two CTAs per SM, and for 16 rows of a thread to hold the state; no fewer than 32 columns each
  int C = 1, cw = 0, rows = 0;
  for (;; C *= 2) {
    cw = ((a->dv + C - 1) / C + unit - 1) / unit * unit;
    rows = cw <= 256 ? (a->d + ML_THREADS / ((cw + unit - 1) / unit) - 1) / (ML_THREADS / ((cw + unit - 1) / unit)) : 1 << 20;
    if (C == ML_MAX_CLUSTER || (cw <= 256 && (cw < 64 || (rows <= 16 && (long long)a->B * a->H * C >= 296)))) break;
  }
  if (cw > 256) return -5;
  const bool ok = a->fp32 ? (vec ? LaunchMlstmStep<float, 4>(p, a->B, cw, C, rows, s) : LaunchMlstmStep<float, 1>(p, a->B, cw, C, rows, s))
                          : (vec ? LaunchMlstmStep<__nv_bfloat16, 4>(p, a->B, cw, C, rows, s) : LaunchMlstmStep<__nv_bfloat16, 1>(p, a->B, cw, C, rows, s));
  return ok ? 0 : -4;
}
