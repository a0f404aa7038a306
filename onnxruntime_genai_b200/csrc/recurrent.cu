// Recurrent mixers of declared stacks over packed sequences, for bf16 and fp32 activations: the gated average (minGRU) and matrix memories (the mLSTM of
// xLSTM).  States are fp32 and live in the request's slot; a request whose past length is 0 starts from zero.  Built without fast-math: gates, decays and
// the recurrences are plain fp32.
//
// Gated average, every column on its own:   z = sigmoid(z'),  c = u + 1/2 (u >= 0) or sigmoid(u) (u < 0),  S <- (1 - z) S + z c,  out = S * silu(g) * scale.
//   min_gru_step_kernel   decode-shaped steps: a thread walks the tokens of its columns.
//   min_gru_scan_kernel   prompts: a CTA takes 16 columns and 512 tokens at a time, a thread 8 tokens of two columns.  S_t is an affine function of the
//                         state before the thread's tokens, these functions are composed by a scan over the threads of a column, and the thread's
//                         tokens are replayed from the state found.
//
// Matrix memory, per head, with i and f the capped log gates and m the running maximum:
//   m' = max(f + m, i),  S <- exp(f + m - m') S + exp(i - m') k v^T,  n likewise with k alone,  o = S^T q / (max(|n . q|, exp(-m')) + 1e-6),
//   out = o / rms(o) * norm * sigmoid(g).
//   mlstm_step_kernel     any step.  A cluster of CTAs shares the columns of a head; the state streams through registers once per token.
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

__device__ __forceinline__ float mg_candidate(float u) { return u >= 0.f ? u + 0.5f : rec_sigmoid(u); }

template <typename T>
__global__ void __launch_bounds__(128) min_gru_step_kernel(MinGruParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
  const int t0 = p.cu_seqlens[b], t1 = p.cu_seqlens[b + 1];
  if (c >= p.W || t0 >= t1) return;
  float* st = p.state + size_t(p.slots[b]) * p.slot_stride + c;
  const T *z = static_cast<const T*>(p.z) + c, *x = static_cast<const T*>(p.x) + c, *g = static_cast<const T*>(p.g) + c;
  float S = p.past_lens[b] == 0 ? 0.f : *st;
  for (int t = t0; t < t1; ++t) {
    const float zz = rec_sigmoid(rec_f32(z[size_t(t) * p.ld])), gg = rec_f32(g[size_t(t) * p.ld]);
    S = fmaf(zz, mg_candidate(rec_f32(x[size_t(t) * p.ld])), (1.f - zz) * S);
    static_cast<T*>(p.out)[size_t(t) * p.ldo + c] = rec_from<T>(S * gg * rec_sigmoid(gg) * p.scale);
  }
  *st = S;
}

constexpr int MG_COLS = 16, MG_L = 8, MG_SEGS = 64, MG_THREADS = MG_SEGS * MG_COLS / 2;

// Column count, strides and the columns' addresses are even.
template <typename T>
__global__ void __launch_bounds__(MG_THREADS) min_gru_scan_kernel(MinGruParams p) {
  __shared__ float sa[MG_COLS][MG_SEGS + 1], sb[MG_COLS][MG_SEGS + 1];
  __shared__ float carry[MG_COLS];
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.y, t0 = p.cu_seqlens[b], t1 = p.cu_seqlens[b + 1];
  if (t0 >= t1) return;
  const int tid = threadIdx.x, seg = tid / (MG_COLS / 2), cc = tid % (MG_COLS / 2) * 2, c = blockIdx.x * MG_COLS + cc;
  const bool live = c < p.W;
  float* st = p.state + size_t(p.slots[b]) * p.slot_stride;
  const T *z = static_cast<const T*>(p.z) + c, *x = static_cast<const T*>(p.x) + c, *g = static_cast<const T*>(p.g) + c;
  T* out = static_cast<T*>(p.out) + c;
  if (tid < MG_COLS) carry[tid] = p.past_lens[b] == 0 || blockIdx.x * MG_COLS + tid >= p.W ? 0.f : st[blockIdx.x * MG_COLS + tid];
  for (int base = t0; base < t1; base += MG_SEGS * MG_L) {
    // S after a token: a * S + d
    float2 a[MG_L], d[MG_L], gate[MG_L];
    const int ts = base + seg * MG_L;
    float2 A = make_float2(1.f, 1.f), D = make_float2(0.f, 0.f);
#pragma unroll
    for (int i = 0; i < MG_L; ++i) {
      const bool ok = live && ts + i < t1;
      float2 zz = make_float2(0.f, 0.f), u = zz;
      gate[i] = zz;
      if (ok) {
        zz = rec_ld2(z + size_t(ts + i) * p.ld);
        u = rec_ld2(x + size_t(ts + i) * p.ld);
        gate[i] = rec_ld2(g + size_t(ts + i) * p.ld);
      }
      const float s0 = ok ? rec_sigmoid(zz.x) : 0.f, s1 = ok ? rec_sigmoid(zz.y) : 0.f;
      a[i] = make_float2(1.f - s0, 1.f - s1);
      d[i] = make_float2(s0 * mg_candidate(u.x), s1 * mg_candidate(u.y));
      D = make_float2(fmaf(a[i].x, D.x, d[i].x), fmaf(a[i].y, D.y, d[i].y));
      A = make_float2(A.x * a[i].x, A.y * a[i].y);
    }
    sa[cc][seg] = A.x; sa[cc + 1][seg] = A.y;
    sb[cc][seg] = D.x; sb[cc + 1][seg] = D.y;
    __syncthreads();
    // one warp per column: the state before every segment
    {
      const int w = tid >> 5, lane = tid & 31;
      float a0 = sa[w][2 * lane], a1 = sa[w][2 * lane + 1], b0 = sb[w][2 * lane], b1 = sb[w][2 * lane + 1];
      float pa = a0 * a1, pb = fmaf(a1, b0, b1);
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float qa = __shfl_up_sync(0xffffffffu, pa, o), qb = __shfl_up_sync(0xffffffffu, pb, o);
        if (lane >= o) { pb = fmaf(pa, qb, pb); pa *= qa; }
      }
      const float ea = __shfl_up_sync(0xffffffffu, pa, 1), eb = __shfl_up_sync(0xffffffffu, pb, 1), s0 = carry[w];
      const float before = lane ? fmaf(ea, s0, eb) : s0;
      sb[w][2 * lane] = before;
      sb[w][2 * lane + 1] = fmaf(a0, before, b0);
      const float end = __shfl_sync(0xffffffffu, fmaf(pa, s0, pb), 31);
      __syncwarp();
      if (lane == 0) carry[w] = end;
    }
    __syncthreads();
    float2 S = make_float2(sb[cc][seg], sb[cc + 1][seg]);
#pragma unroll
    for (int i = 0; i < MG_L; ++i) {
      S = make_float2(fmaf(a[i].x, S.x, d[i].x), fmaf(a[i].y, S.y, d[i].y));
      if (live && ts + i < t1)
        rec_st2(out + size_t(ts + i) * p.ldo, S.x * gate[i].x * rec_sigmoid(gate[i].x) * p.scale, S.y * gate[i].y * rec_sigmoid(gate[i].y) * p.scale);
    }
    __syncthreads();
  }
  if (tid < MG_COLS && blockIdx.x * MG_COLS + tid < p.W) st[blockIdx.x * MG_COLS + tid] = carry[tid];
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

// Grid (cluster, heads, requests).  The CTA owns columns [rank * cw, rank * cw + cw) of the head, cw = a multiple of VEC of at most 256; thread
// (row group, column group of VEC).  Every token: the factors, n . q (by all CTAs alike), then the state's rows through registers.  The state of a step
// of several tokens is read back by the thread that wrote it.
template <typename T, int VEC>
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
  float* S = slot + size_t(h) * d * dv;
  float* gn = slot + size_t(p.H) * d * dv + size_t(h) * d;
  float* gm = slot + size_t(p.H) * d * (dv + 1) + h;
  const int c0 = rank * cw, cols = min(cw, dv - c0);                // (may be <= 0)
  const int lanes = (cw + VEC - 1) / VEC;                           // column groups
  const int groups = ML_THREADS / lanes, cg = tid % lanes, rg = tid / lanes, col = cg * VEC;
  const bool mine = rg < groups && col < cols;
  for (int i = tid; i < d; i += ML_THREADS) sn[i] = fresh ? 0.f : gn[i];
  float m = fresh ? 0.f : *gm;
  if (C > 1) { __syncthreads(); rec_cluster_arrive(); rec_cluster_wait(); }      // n and m have been read by every CTA
  for (int t = t0; t < t1; ++t) {
    const T* qp = static_cast<const T*>(p.q) + size_t(t) * p.ld + size_t(h) * d;
    const T* kp = static_cast<const T*>(p.k) + size_t(t) * p.ld + size_t(h) * d;
    const float* gp = p.gates + size_t(t) * p.ldg;
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
    float o[VEC], v[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) o[e] = 0.f;
    if (mine) {
      const T* vp = static_cast<const T*>(p.v) + size_t(t) * p.ld + size_t(h) * dv + c0 + col;
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[e] = rec_f32(vp[e]);
      const bool zero = fresh && t == t0;
#pragma unroll 4
      for (int r = rg; r < d; r += groups) {
        float* sp = S + size_t(r) * dv + c0 + col;
        float s[VEC];
        if (zero) {
#pragma unroll
          for (int e = 0; e < VEC; ++e) s[e] = 0.f;
        } else if constexpr (VEC == 4) {
          const float4 f = *reinterpret_cast<const float4*>(sp);
          s[0] = f.x; s[1] = f.y; s[2] = f.z; s[3] = f.w;
        } else {
          s[0] = *sp;
        }
        const float kk = sk[r], qq = sq[r];
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          s[e] = fmaf(gt.keep, s[e], kk * v[e]);
          o[e] = fmaf(qq, s[e], o[e]);
        }
        if constexpr (VEC == 4) *reinterpret_cast<float4*>(sp) = make_float4(s[0], s[1], s[2], s[3]);
        else *sp = s[0];
      }
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) red[tid * VEC + e] = o[e];
    __syncthreads();
    // column sums over the row groups: thread tid takes column tid
    float val = 0.f;
    if (tid < cols) {
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
    __syncthreads();
  }
  if (rank == 0) {
    for (int i = tid; i < d; i += ML_THREADS) gn[i] = sn[i];
    if (tid == 0) *gm = m;
  }
  if (C > 1) { rec_cluster_arrive(); rec_cluster_wait(); }          // no CTA leaves while another may read its sums
}

}  // namespace ogb

using namespace ogb;

// See kernels.h.
OGB_API int ogb_min_gru(const void* z, const void* x, const void* g, int ld, float* state, long long slot_stride, const int32_t* slots,
                        const int32_t* cu_seqlens, const int32_t* past_lens, void* out, int ldo, int B, int W, float scale, int max_q_len, int fp32,
                        void* stream) {
  if (B <= 0 || W <= 0) return 0;
  if (B > 65535 || slot_stride < W) return -1;
  const MinGruParams p{z, x, g, out, state, slots, cu_seqlens, past_lens, slot_stride, ld, ldo, W, scale};
  auto s = static_cast<cudaStream_t>(stream);
  auto addr = [](const void* a) { return reinterpret_cast<uintptr_t>(a); };
  const bool even = W % 2 == 0 && ld % 2 == 0 && ldo % 2 == 0 && ((addr(z) | addr(x) | addr(g) | addr(out)) & (fp32 ? 7 : 3)) == 0;
  using H = __nv_bfloat16;
  if (max_q_len <= 16 || !even) {
    const dim3 grid((W + 127) / 128, B), block(128);
    return (fp32 ? launch_pdl(min_gru_step_kernel<float>, grid, block, 0, s, p) : launch_pdl(min_gru_step_kernel<H>, grid, block, 0, s, p)) ? 0 : -4;
  }
  const dim3 grid((W + MG_COLS - 1) / MG_COLS, B), block(MG_THREADS);
  return (fp32 ? launch_pdl(min_gru_scan_kernel<float>, grid, block, 0, s, p) : launch_pdl(min_gru_scan_kernel<H>, grid, block, 0, s, p)) ? 0 : -4;
}

template <typename T, int VEC>
static bool LaunchMlstmStep(const MlstmParams& p, int B, int cw, int C, cudaStream_t s) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(C, p.H, B);
  cfg.blockDim = dim3(ML_THREADS);
  cfg.stream = s;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = C; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = 2;
  return cudaLaunchKernelEx(&cfg, mlstm_step_kernel<T, VEC>, p, cw) == cudaSuccess;
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
  // states in whole 16-byte pieces (a slot's first float is on a 16-byte boundary, heads and rows are multiples of four)
  const bool vec = a->dv % 4 == 0 && a->slot_stride % 4 == 0 && (reinterpret_cast<uintptr_t>(a->state) & 15) == 0;
  const int unit = vec ? 4 : 1;
  // columns of a CTA: 32 where that needs no more than a cluster of eight (so that few requests still use many SMs), at most 256
  int cw = 32;
  while ((a->dv + cw - 1) / cw > ML_MAX_CLUSTER) cw *= 2;
  if (cw > 256) return -5;
  int C = (a->dv + cw - 1) / cw;
  while (C & (C - 1)) ++C;              // (a CTA without columns only meets the others)
  if (C == 1) cw = (a->dv + unit - 1) / unit * unit;
  const bool ok = a->fp32 ? (vec ? LaunchMlstmStep<float, 4>(p, a->B, cw, C, s) : LaunchMlstmStep<float, 1>(p, a->B, cw, C, s))
                          : (vec ? LaunchMlstmStep<__nv_bfloat16, 4>(p, a->B, cw, C, s) : LaunchMlstmStep<__nv_bfloat16, 1>(p, a->B, cw, C, s));
  return ok ? 0 : -4;
}
