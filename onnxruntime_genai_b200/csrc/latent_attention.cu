// Latent attention over a paged cache.  A token's cache row is its normalised latent c (R values) followed by one rotated key part
// (rot values) that all heads share; per-head keys and values are linear maps of c.  With the key map folded into the query
// (qlat[t, h] = W_uk[h]^T q[t, h], made by a per-head product beforehand) a head's score against cached position j is
//     (qlat[t, h] . c_j + q_rot[t, h] . k_rot_j) * scale
// and its result before the value map is sum_j p_j c_j: every head of a token reads the same rows, once, for scores and values.
// Kernels:
//   latent_prep_kernel   RMS norm of the latent and rotation of the key part into the cache; rotation of the queries' rotary parts.
//   latent_mma_kernel    decode steps and short portions: one CTA = (request, up to 64 (token, head) rows, key split); tiles of 32
//                        cache rows, one bulk copy per row into a double buffer, serve as K (all columns) and as V (the first R columns) of
//                        warp-level MMAs; two CTAs share an SM (up to 16 rows of 576 columns), so that one's copies and softmax run
//                        under the other's MMAs.  Like paged_attention_kernel (attention.cu) it is bound by the cache stream and its rows are
//                        few; long prompts take the tensor-memory kernel (attention_tc.cu) on expanded keys and values instead.
//   latent_simt_kernel   the same op in plain fp32 arithmetic for fp32 models and for sizes the other kernels cannot address.
//   latent_gather_kernel cached rows of some requests into a dense matrix (input of the key / value expansion of long prompts).
//   gate_rows_kernel     an output gate: rows times the sigmoid of other rows, in place.
// A query at position p sees keys (p - window, p] (window > 0) or [0, p]; a head may have a sink, a logit in its denominator.  Built without fast-math.
#include <cstdlib>
#include "common.cuh"
#include "kernels.h"

namespace ogb {

constexpr float LAT_LOG2E = 1.4426950408889634f;

template <typename T> __device__ __forceinline__ float lat_f32(T v);
template <> __device__ __forceinline__ float lat_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ float lat_f32<__nv_bfloat16>(__nv_bfloat16 v) { return bf2f(v); }
template <typename T> __device__ __forceinline__ T lat_from(float v);
template <> __device__ __forceinline__ float lat_from<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 lat_from<__nv_bfloat16>(float v) { return f2bf(v); }

// ------------------------------------------------------------------------------------ norm + rotation + append
// Row t of q (null: not here): H heads of (dim | rot); of down (null: not here): R latent values, rot shared key values; of cq (null: none):
// the queries' own latent.  q and cq may be column ranges of down's matrix that do not overlap it.  One CTA per token.
template <typename T>
__global__ void __launch_bounds__(128) latent_prep_kernel(T* q_, int ldq, const T* down_, int ldd, T* cq_, int ldcq, int q_rank,
                                                          const float* __restrict__ cq_w, OgbLatentShape sh, const float* __restrict__ norm_w, float eps,
                                                          const int32_t* __restrict__ positions, const float* __restrict__ cosc,
                                                          const float* __restrict__ sinc, int max_pos, const int32_t* __restrict__ slots,
                                                          T* __restrict__ cache, int ldcache) {
  __shared__ float part[8];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const T* down = down_ ? down_ + size_t(t) * ldd : nullptr;
  T* cq = cq_ ? cq_ + size_t(t) * ldcq : nullptr;
  const int pos = min(max(positions[t], 0), max_pos - 1), slot = down ? slots[t] : -1;
  const int half = sh.rot_dims / 2;
  const float *cs = cosc + size_t(pos) * half, *sn = sinc + size_t(pos) * half;
  float ss = 0.f, sq = 0.f;
  if (down)
    for (int i = threadIdx.x; i < sh.R; i += 128) { const float v = lat_f32(down[i]); ss += v * v; }
  if (cq)
    for (int i = threadIdx.x; i < q_rank; i += 128) { const float v = lat_f32(cq[i]); sq += v * v; }
  ss = warp_sum(ss);
  sq = warp_sum(sq);
  if (lane == 0) { part[warp] = ss; part[4 + warp] = sq; }
  __syncthreads();
  if (cq) {
    const float inv = 1.f / sqrtf((part[4] + part[5] + part[6] + part[7]) / q_rank + eps);
    for (int i = threadIdx.x; i < q_rank; i += 128) cq[i] = lat_from<T>(lat_f32(cq[i]) * inv * cq_w[i]);
  }
  if (slot >= 0) {
    const float inv = 1.f / sqrtf((part[0] + part[1] + part[2] + part[3]) / sh.R + eps);
    T* dst = cache + size_t(slot) * ldcache;
    for (int i = threadIdx.x; i < sh.R; i += 128) dst[i] = lat_from<T>(lat_f32(down[i]) * inv * norm_w[i]);
    for (int i = threadIdx.x; i < sh.rot; i += 128) {
      float v = lat_f32(down[sh.R + i]);
      if (i < half) v = v * cs[i] - lat_f32(down[sh.R + i + half]) * sn[i];
      else if (i < 2 * half) v = v * cs[i - half] + lat_f32(down[sh.R + i - half]) * sn[i - half];
      dst[sh.R + i] = lat_from<T>(v);
    }
  }
  if (!q_) return;
  for (int idx = threadIdx.x; idx < sh.H * half; idx += 128) {
    const int h = idx / half, i = idx - h * half;
    T* q = q_ + size_t(t) * ldq + h * (sh.dim + sh.rot) + sh.dim;
    const float u = lat_f32(q[i]), v = lat_f32(q[i + half]);
    q[i] = lat_from<T>(u * cs[i] - v * sn[i]);
    q[i + half] = lat_from<T>(v * cs[i] + u * sn[i]);
  }
}

// ------------------------------------------------------------------------------------ warp-MMA kernel
// Contiguous copy global -> shared (16-byte aligned addresses, a multiple of 16 bytes), completion on an mbarrier.
__device__ __forceinline__ void bulk_load(void* smem_dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
               ::"r"(smem_u32(smem_dst)), "l"(src), "r"(bytes), "r"(smem_u32(bar)) : "memory");
}

struct LatentParams {
  const __nv_bfloat16* qlat;      // [T, H, R]
  const __nv_bfloat16* proj;      // rotary query parts at row t, column h * (dim + rot) + dim
  int ldp, dim;
  const __nv_bfloat16* cache; int ldcache;
  const int32_t *cu, *past, *table; int table_cols, block_size, block_shift;      // log2(block_size) or -1
  __nv_bfloat16* out;             // [T, H, R]
  float* part_o; float* part_ml;
  const float* sinks;             // [H] a logit in each head's denominator, or null
  float scale;
  int window, B, H, R, rot, kp, pitch, splits, total_rows, skip_q_len;
  const int32_t* order;           // [B] requests in issue order (longest first), or null
  int* status;                    // device status word (bounded waits)
};

constexpr int LAT_MAX_SPLITS = 32, LAT_MAX_SMEM = 226 * 1024;          // (some static shared memory beside the dynamic part)
constexpr int LAT_BN = 32, LAT_THREADS = 256, LAT_PP = LAT_BN + 8, LAT_SP = LAT_BN + 4;   // keys per tile; pitches of P and score rows

template <int MT>
struct LatCfg {
  static constexpr int BM = MT * 16;
  // The score sums are divided over KH warps by columns of the rows.  16 rows: every warp takes all keys and an eighth of the columns,
  // its part of the queries stays in registers (the staged queries make room for the partial scores), a cache row is read once.
  static constexpr int KH = MT == 4 ? 1 : (MT == 2 ? 2 : 8);
  static constexpr int TPR = LAT_THREADS / BM;         // threads of one row in the softmax
  static constexpr int KPT = LAT_BN / TPR;             // keys of each of them
  static constexpr int S_BYTES = KH * BM * LAT_SP * 4;
  static constexpr int q_bytes(int pitch) { return MT == 1 && S_BYTES > BM * pitch * 2 ? S_BYTES : BM * pitch * 2; }
  static constexpr int smem(int pitch) { return q_bytes(pitch) + 2 * LAT_BN * pitch * 2 + BM * LAT_PP * 2 + (MT == 1 ? 0 : S_BYTES) + BM * 8 + 64; }
};

template <int MT, int NTW>
__global__ void __launch_bounds__(LAT_THREADS, MT == 4 ? 1 : 2) latent_mma_kernel(LatentParams p) {
  using Cfg = LatCfg<MT>;
  constexpr int BM = Cfg::BM, KH = Cfg::KH, TPR = Cfg::TPR, KPT = Cfg::KPT;
  extern __shared__ __align__(128) uint8_t smem[];
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(smem);
  __nv_bfloat16* sK = sQ + Cfg::q_bytes(p.pitch) / 2;  // [2][LAT_BN][pitch]
  __nv_bfloat16* sP = sK + 2 * LAT_BN * p.pitch;       // [BM][LAT_PP]
  float* sS = MT == 1 ? reinterpret_cast<float*>(sQ) : reinterpret_cast<float*>(sP + BM * LAT_PP);     // [KH][BM][LAT_SP] partial scores
  float* sA = MT == 1 ? reinterpret_cast<float*>(sP + BM * LAT_PP) : sS + KH * BM * LAT_SP;             // [BM] factor of the old output; at the end the row sums
  float* sM = sA + BM;                                 // [BM] at the end the row maxima
  __shared__ uint64_t full[2];                         // a tile's rows (tile 0: and the queries) have landed
  __shared__ int abort_flag;
  volatile int* abort_p = &abort_flag;
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int bz = blockIdx.z / p.splits, split = blockIdx.z % p.splits;
  const int b = p.order ? p.order[bz] : bz;
  const int H = p.H, tok0 = p.cu[b], q_len = p.cu[b + 1] - tok0, rows = q_len * H;
  const int row0 = blockIdx.x * BM;
  if (row0 >= rows || (p.skip_q_len > 0 && q_len >= p.skip_q_len)) return;
  const int past = p.past[b];
  const int32_t* table = p.table + size_t(b) * p.table_cols;
  // this tile's keys, then the part of them this split owns
  const int kv_hi = past + min(q_len - 1, (row0 + BM - 1) / H) + 1;
  const int kv_lo = p.window > 0 ? max(0, past + row0 / H - p.window + 1) : 0;
  const int per = ((kv_hi - kv_lo + LAT_BN - 1) / LAT_BN + p.splits - 1) / p.splits * LAT_BN;
  const int lo = kv_lo + split * per, hi = min(kv_hi, lo + per);
  if (p.splits > 1 && lo >= hi) {
    for (int r = tid; r < BM; r += LAT_THREADS)
      if (row0 + r < rows) {
        float* pm = p.part_ml + (size_t(split) * p.total_rows + size_t(tok0) * H + row0 + r) * 2;
        pm[0] = -INFINITY; pm[1] = 0.f;
      }
    return;
  }
  const int n_tiles = (hi - lo + LAT_BN - 1) / LAT_BN;
  const int kc = (p.R + p.rot) / 8;                    // 16-byte chunks of a cache row
  const uint32_t row_bytes = (p.R + p.rot) * 2;
  if (tid == 0) {
    mbar_init(&full[0], 1);
    mbar_init(&full[1], 1);
    abort_flag = 0;
    mbar_fence_init();
  }
  if (kc * 8 < p.kp) {                                 // columns between the row's end and the next multiple of 16 are zeros
    for (int r = tid; r < BM; r += LAT_THREADS) *reinterpret_cast<uint4*>(sQ + r * p.pitch + kc * 8) = make_uint4(0, 0, 0, 0);
    for (int r = tid; r < 2 * LAT_BN; r += LAT_THREADS) *reinterpret_cast<uint4*>(sK + r * p.pitch + kc * 8) = make_uint4(0, 0, 0, 0);
  }
  __syncthreads();
  // Warp 0 copies a tile, one row per lane; the rows' blocks are looked up one tile ahead of the copy and not touched before it, so that
  // it does not wait for the table.  Rows past the range repeat its last row (their weights are zero).
  auto key_of = [&](int it) { return min(lo + it * LAT_BN + lane, hi - 1); };
  auto lookup = [&](int it) {
    const int j = key_of(it);
    return table[p.block_shift >= 0 ? j >> p.block_shift : j / p.block_size];
  };
  auto load = [&](int it, int block) {
    const int j = key_of(it);
    const int slot = p.block_shift >= 0 ? (block << p.block_shift) + (j & (p.block_size - 1)) : block * p.block_size + j % p.block_size;
    bulk_load(sK + ((it & 1) * LAT_BN + lane) * p.pitch, p.cache + size_t(slot) * p.ldcache, row_bytes, &full[it & 1]);
  };
  int block_next = 0;
  if (warp == 0) {
    if (lane == 0) mbar_expect_tx(&full[0], (BM + LAT_BN) * row_bytes);
    __syncwarp();
    // queries: latent part from qlat, rotary part from the projection; rows past the request's repeat its last one
    for (int r = lane; r < BM; r += 32) {
      const int gr = min(row0 + r, rows - 1);
      const size_t tr = size_t(tok0) * H + gr;
      bulk_load(sQ + r * p.pitch, p.qlat + tr * p.R, p.R * 2, &full[0]);
      if (p.rot > 0)
        bulk_load(sQ + r * p.pitch + p.R, p.proj + size_t(tok0 + gr / H) * p.ldp + size_t(gr % H) * (p.dim + p.rot) + p.dim, p.rot * 2, &full[0]);
    }
    load(0, lookup(0));
    block_next = lookup(1);
  }

  // softmax: TPR neighbouring threads share row sr, KPT keys each
  const int sr = tid / TPR, sk0 = (tid % TPR) * KPT;
  const bool s_valid = row0 + sr < rows;
  const int s_pos = past + (row0 + sr) / H;
  const float sc2 = p.scale * LAT_LOG2E;
  float mx = -INFINITY, l = 0.f;                       // the row's running maximum; the sum over this thread's keys
  // scores: warp -> 16 rows (mt), a group of keys (kg), a share of the columns (kh)
  const int ksteps = p.kp / 16;
  constexpr int KS = NTW == 8 ? 5 : (NTW == 4 ? 3 : 2);                        // column steps of a warp (16 rows), at most
  const int mt = warp % MT, kg = (warp / MT) & 1, kh = KH == 8 ? warp : (KH == 2 ? warp >> 2 : 0);
  const int ks0 = kh * ksteps / KH, ks1 = (kh + 1) * ksteps / KH;
  uint32_t qreg[KS][4];
  const int c0 = warp * NTW * 8;                       // output columns [c0, c0 + 8 * NTW) of every row
  float o[MT][NTW][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < NTW; ++n) o[m][n][0] = o[m][n][1] = o[m][n][2] = o[m][n][3] = 0.f;

  for (int it = 0; it < n_tiles; ++it) {
    if (!mbar_wait_bounded(&full[it & 1], (it >> 1) & 1, abort_p)) {
      *abort_p = 1;
      if (p.status) atomicMax(p.status, int(OGB_ERR_WAIT_TMA));
    }
    __syncthreads();                                   // tile it has landed; every warp is done with tile it - 1
    if (*abort_p) break;                               // (set before the barrier or not at all: all threads leave together)
    if (warp == 0 && it + 1 < n_tiles) {
      if (lane == 0) mbar_expect_tx(&full[(it + 1) & 1], LAT_BN * row_bytes);
      __syncwarp();
      load(it + 1, block_next);
      block_next = lookup(it + 2);
    }
    const __nv_bfloat16* tk = sK + (it & 1) * LAT_BN * p.pitch;
    const __nv_bfloat16* qa = sQ + (mt * 16 + (lane & 15)) * p.pitch + (lane >> 4) * 8;
    float* ps = sS + (kh * BM + mt * 16 + g) * LAT_SP + t4 * 2;
    if constexpr (MT == 1) {
      // 16 rows x 32 keys over this warp's columns
      if (it == 0) {
#pragma unroll
        for (int i = 0; i < KS; ++i) if (ks0 + i < ks1) ldmatrix_x4(qreg[i], qa + (ks0 + i) * 16);
        __syncthreads();                               // the staged queries are no longer needed: the scores take their place
      }
      float s[4][4] = {};
      const __nv_bfloat16* ka = tk + ((lane >> 4) * 8 + (lane & 7)) * p.pitch + ((lane >> 3) & 1) * 8 + ks0 * 16;
      // the next step's fragments are read ahead of this step's MMAs
      uint32_t k0[2][4], k1[2][4];
      if (ks0 < ks1) {
        ldmatrix_x4(k0[0], ka);
        ldmatrix_x4(k1[0], ka + 16 * p.pitch);
      }
#pragma unroll
      for (int i = 0; i < KS; ++i) {
        if (i + 1 < KS && ks0 + i + 1 < ks1) {
          ldmatrix_x4(k0[(i + 1) & 1], ka + (i + 1) * 16);
          ldmatrix_x4(k1[(i + 1) & 1], ka + 16 * p.pitch + (i + 1) * 16);
        }
        if (ks0 + i < ks1) {
          mma_bf16_16816(s[0], qreg[i], k0[i & 1][0], k0[i & 1][1]);
          mma_bf16_16816(s[1], qreg[i], k0[i & 1][2], k0[i & 1][3]);
          mma_bf16_16816(s[2], qreg[i], k1[i & 1][0], k1[i & 1][1]);
          mma_bf16_16816(s[3], qreg[i], k1[i & 1][2], k1[i & 1][3]);
        }
      }
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        *reinterpret_cast<float2*>(ps + n * 8) = make_float2(s[n][0], s[n][1]);
        *reinterpret_cast<float2*>(ps + 8 * LAT_SP + n * 8) = make_float2(s[n][2], s[n][3]);
      }
    } else {
      // 16 rows x 16 keys
      float s[2][2][4] = {};
      const __nv_bfloat16* ka = tk + (kg * 16 + (lane >> 4) * 8 + (lane & 7)) * p.pitch + ((lane >> 3) & 1) * 8;
#pragma unroll 2
      for (int ks = ks0; ks < ks1; ks += 2) {
        uint32_t qf[4], kb[4], qf2[4], kb2[4];
        const int k2 = min(ks + 1, ks1 - 1);
        ldmatrix_x4(qf, qa + ks * 16);
        ldmatrix_x4(kb, ka + ks * 16);
        ldmatrix_x4(qf2, qa + k2 * 16);
        ldmatrix_x4(kb2, ka + k2 * 16);
        mma_bf16_16816(s[0][0], qf, kb[0], kb[1]);
        mma_bf16_16816(s[0][1], qf, kb[2], kb[3]);
        if (ks + 1 < ks1) {
          mma_bf16_16816(s[1][0], qf2, kb2[0], kb2[1]);
          mma_bf16_16816(s[1][1], qf2, kb2[2], kb2[3]);
        }
      }
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        *reinterpret_cast<float2*>(ps + kg * 16 + n * 8) = make_float2(s[0][n][0] + s[1][n][0], s[0][n][1] + s[1][n][1]);
        *reinterpret_cast<float2*>(ps + 8 * LAT_SP + kg * 16 + n * 8) = make_float2(s[0][n][2] + s[1][n][2], s[0][n][3] + s[1][n][3]);
      }
    }
    __syncthreads();
    // ---- softmax of the tile's scores
    float x[KPT], tmax = -INFINITY;
#pragma unroll
    for (int e = 0; e < KPT; ++e) {
      float v = sS[sr * LAT_SP + sk0 + e];
#pragma unroll
      for (int k = 1; k < KH; ++k) v += sS[(k * BM + sr) * LAT_SP + sk0 + e];
      const int j = lo + it * LAT_BN + sk0 + e;
      x[e] = s_valid && j < hi && j <= s_pos && (p.window <= 0 || j > s_pos - p.window) ? v * sc2 : -INFINITY;
      tmax = fmaxf(tmax, x[e]);
    }
#pragma unroll
    for (int w = TPR / 2; w > 0; w >>= 1) tmax = fmaxf(tmax, __shfl_xor_sync(0xffffffffu, tmax, w));
    const float mn = fmaxf(mx, tmax), ms = mn == -INFINITY ? 0.f : mn;
    const float al = mn == -INFINITY ? 1.f : exp2f(mx - mn);
    mx = mn;
    l *= al;
#pragma unroll
    for (int e = 0; e < KPT; e += 2) {
      const float p0 = exp2f(x[e] - ms), p1 = exp2f(x[e + 1] - ms);
      l += p0 + p1;
      *reinterpret_cast<uint32_t*>(sP + sr * LAT_PP + sk0 + e) = pack_bf16x2(p0, p1);
    }
    if (sk0 == 0) sA[sr] = al;
    __syncthreads();
    // ---- O = O * alpha + P C
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const float al0 = sA[m * 16 + g], al1 = sA[m * 16 + g + 8];
      if (!__any_sync(0xffffffffu, al0 != 1.f || al1 != 1.f)) continue;        // no maximum moved
#pragma unroll
      for (int n = 0; n < NTW; ++n) { o[m][n][0] *= al0; o[m][n][1] *= al0; o[m][n][2] *= al1; o[m][n][3] *= al1; }
    }
#pragma unroll
    for (int kk = 0; kk < LAT_BN / 16; ++kk) {
      uint32_t pa[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m) ldmatrix_x4(pa[m], sP + (m * 16 + (lane & 15)) * LAT_PP + kk * 16 + (lane >> 4) * 8);
      uint32_t vb[NTW / 2][4];                         // (all fragments first: an MMA would hold back the reads behind it)
#pragma unroll
      for (int np = 0; np < NTW / 2; ++np)
        if (c0 + np * 16 < p.R) ldmatrix_x4_trans(vb[np], tk + (kk * 16 + (lane & 15)) * p.pitch + c0 + np * 16 + (lane >> 4) * 8);
#pragma unroll
      for (int np = 0; np < NTW / 2; ++np) {
        if (c0 + np * 16 >= p.R) break;
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          mma_bf16_16816(o[m][np * 2], pa[m], vb[np][0], vb[np][1]);
          mma_bf16_16816(o[m][np * 2 + 1], pa[m], vb[np][2], vb[np][3]);
        }
      }
    }
  }
  if (*abort_p) {                                      // a wait ran out: let copies in flight land before the shared memory goes away
    int never = 0;
    mbar_wait_bounded(&full[0], 0, &never, 20000000ull);
    mbar_wait_bounded(&full[1], 0, &never, 20000000ull);
    return;
  }
#pragma unroll
  for (int w = TPR / 2; w > 0; w >>= 1) l += __shfl_xor_sync(0xffffffffu, l, w);
  __syncthreads();
  if (sk0 == 0) { sA[sr] = l; sM[sr] = mx; }
  __syncthreads();
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = m * 16 + g + e * 8;
      if (row0 + r >= rows) continue;
      const float lr = sA[r];
      const size_t orow = size_t(tok0) * H + row0 + r;
      if (p.splits > 1) {
        float* po = p.part_o + (size_t(split) * p.total_rows + orow) * p.R;
#pragma unroll
        for (int n = 0; n < NTW; ++n)
          if (c0 + n * 8 < p.R) *reinterpret_cast<float2*>(po + c0 + n * 8 + t4 * 2) = make_float2(o[m][n][e * 2], o[m][n][e * 2 + 1]);
        if (warp == 0 && t4 == 0) {
          float* pm = p.part_ml + (size_t(split) * p.total_rows + orow) * 2;
          pm[0] = sM[r]; pm[1] = lr;
        }
      } else {
        float inv = lr > 0.f ? 1.f / lr : 0.f;
        if (p.sinks) {
          const float sk = p.sinks[(row0 + r) % H] * LAT_LOG2E, top = fmaxf(sM[r], sk), old = exp2f(sM[r] - top);
          inv = old / (lr * old + exp2f(sk - top));
        }
        __nv_bfloat16* po = p.out + orow * p.R;
#pragma unroll
        for (int n = 0; n < NTW; ++n)
          if (c0 + n * 8 < p.R) *reinterpret_cast<uint32_t*>(po + c0 + n * 8 + t4 * 2) = pack_bf16x2(o[m][n][e * 2] * inv, o[m][n][e * 2 + 1] * inv);
      }
    }
}

// One CTA per (token, head) row: merges the split partials.
__global__ void __launch_bounds__(128) latent_combine_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml,
                                                             __nv_bfloat16* __restrict__ out, int total_rows, int R, int splits,
                                                             const float* __restrict__ sinks, int H) {
  __shared__ float w[LAT_MAX_SPLITS];
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x, lane = threadIdx.x & 31;
  if (threadIdx.x < 32) {
    float2 ml = make_float2(-INFINITY, 0.f);
    if (lane < splits) ml = *reinterpret_cast<const float2*>(part_ml + (size_t(lane) * total_rows + row) * 2);
    const float sk = sinks ? sinks[row % H] * LAT_LOG2E : -INFINITY;
    const float M = fmaxf(warp_max(ml.x), sk);
    const float e = ml.x == -INFINITY ? 0.f : exp2f(ml.x - M);
    const float L = warp_sum(e * ml.y) + (sinks ? exp2f(sk - M) : 0.f);
    w[lane] = L > 0.f ? e / L : 0.f;
  }
  __syncthreads();
  for (int c = threadIdx.x * 4; c < R; c += 512) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
    for (int s = 0; s < splits; ++s) {
      const float f = w[s];
      const float4 v = *reinterpret_cast<const float4*>(part_o + (size_t(s) * total_rows + row) * R + c);
      if (f != 0.f) { a.x += f * v.x; a.y += f * v.y; a.z += f * v.z; a.w += f * v.w; }      // (an empty split's values are not defined)
    }
    *reinterpret_cast<uint2*>(out + size_t(row) * R + c) = make_uint2(pack_bf16x2(a.x, a.y), pack_bf16x2(a.z, a.w));
  }
}

// ------------------------------------------------------------------------------------ plain kernel
constexpr int LAT_SIMT_COLS = 16;                      // latent columns per thread (R <= 2048)
template <typename T>
__global__ void __launch_bounds__(128) latent_simt_kernel(const T* __restrict__ qlat, const T* __restrict__ proj, int ldp, OgbLatentShape sh,
                                                          const T* __restrict__ cache, int ldcache, const int32_t* __restrict__ cu,
                                                          const int32_t* __restrict__ past_lens, const int32_t* __restrict__ tables, int table_cols,
                                                          int block_size, T* __restrict__ out, float scale, int window, const float* __restrict__ sinks, int B,
                                                          int skip_q_len) {
  extern __shared__ float sq[];                        // [R + rot] query, then 32 scores
  float* ssc = sq + sh.R + sh.rot;
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, h = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  int rlo = 0, rhi = B - 1;
  while (rlo < rhi) {
    const int mid = (rlo + rhi + 1) >> 1;
    if (cu[mid] <= t) rlo = mid; else rhi = mid - 1;
  }
  const int b = rlo, q_len = cu[b + 1] - cu[b];
  if (t >= cu[b + 1] || (skip_q_len > 0 && q_len >= skip_q_len)) return;
  const int pos = past_lens[b] + t - cu[b], n = sh.R + sh.rot;
  const int lo = window > 0 ? max(0, pos - window + 1) : 0;
  const int32_t* table = tables + size_t(b) * table_cols;
  for (int i = threadIdx.x; i < n; i += 128)
    sq[i] = lat_f32(i < sh.R ? qlat[(size_t(t) * sh.H + h) * sh.R + i] : proj[size_t(t) * ldp + size_t(h) * (sh.dim + sh.rot) + sh.dim + i - sh.R]);
  float acc[LAT_SIMT_COLS];
#pragma unroll
  for (int c = 0; c < LAT_SIMT_COLS; ++c) acc[c] = 0.f;
  // the sink takes part in the maximum and the sum from the start
  float m = sinks ? sinks[h] : -INFINITY, l = sinks ? 1.f : 0.f;
  auto row_of = [&](int j) { return cache + (size_t(table[j / block_size]) * block_size + j % block_size) * ldcache; };
  for (int j0 = lo; j0 <= pos; j0 += 32) {
    __syncthreads();
    for (int k = warp; k < 32; k += 4) {
      const int j = j0 + k;
      float d = 0.f;
      if (j <= pos) {
        const T* row = row_of(j);
        for (int i = lane; i < n; i += 32) d = fmaf(sq[i], lat_f32(row[i]), d);
      }
      d = warp_sum(d);
      if (lane == 0) ssc[k] = j <= pos ? d * scale : -INFINITY;
    }
    __syncthreads();
    float mn = m;
    for (int k = 0; k < 32; ++k) mn = fmaxf(mn, ssc[k]);
    const float al = expf(m - mn);                     // m = -inf at first: 0
    l *= al;
#pragma unroll
    for (int c = 0; c < LAT_SIMT_COLS; ++c) acc[c] *= al;
    for (int k = 0; k < 32 && j0 + k <= pos; ++k) {
      const float pr = expf(ssc[k] - mn);
      l += pr;
      const T* row = row_of(j0 + k);
#pragma unroll
      for (int c = 0; c < LAT_SIMT_COLS; ++c) {
        const int i = c * 128 + threadIdx.x;
        if (i < sh.R) acc[c] = fmaf(pr, lat_f32(row[i]), acc[c]);
      }
    }
    m = mn;
  }
  const float inv = 1.f / l;
#pragma unroll
  for (int c = 0; c < LAT_SIMT_COLS; ++c) {
    const int i = c * 128 + threadIdx.x;
    if (i < sh.R) out[(size_t(t) * sh.H + h) * sh.R + i] = lat_from<T>(acc[c] * inv);
  }
}

// ------------------------------------------------------------------------------------ gate
template <typename T>
__global__ void gate_rows_kernel(T* __restrict__ out, int ldo, const T* __restrict__ gate, int ldg, int T_, int n) {
  pdl_launch_dependents();
  pdl_wait();
  const long all = long(T_) * n;
  for (long i = long(blockIdx.x) * blockDim.x + threadIdx.x; i < all; i += long(gridDim.x) * blockDim.x) {
    const long t = i / n, c = i % n;
    out[t * ldo + c] = lat_from<T>(lat_f32(out[t * ldo + c]) / (1.f + expf(-lat_f32(gate[t * ldg + c]))));
  }
}

// ------------------------------------------------------------------------------------ gather
// Dense row i holds cached position first_kv[k] + i - row_base[k] of request req[k], k the last with row_base[k] <= i; rows past
// kv_len[k] are zeros (a request's rows are padded to a multiple of 16).
__global__ void latent_gather_kernel(const uint4* __restrict__ cache, int ldvec, const int32_t* __restrict__ tables, int table_cols, int block_size,
                                     const int32_t* __restrict__ row_base, const int32_t* __restrict__ first_kv, const int32_t* __restrict__ kv_len,
                                     const int32_t* __restrict__ req, int n_req, int rows, int nvec, uint4* __restrict__ out, int ldo) {
  pdl_launch_dependents();
  pdl_wait();
  const int i = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (i >= rows) return;
  int lo = 0, hi = n_req - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (row_base[mid] <= i) lo = mid; else hi = mid - 1;
  }
  const int j = first_kv[lo] + i - row_base[lo];
  const bool ok = j < kv_len[lo];
  const uint4* src = cache;
  if (ok) src += (size_t(tables[size_t(req[lo]) * table_cols + j / block_size]) * block_size + j % block_size) * ldvec;
  for (int c = lane; c < nvec; c += 32) out[size_t(i) * ldo + c] = ok ? src[c] : make_uint4(0, 0, 0, 0);
}

template <int MT, int NTW>
static int LaunchLatentMma(const LatentParams& p, int max_q_len, cudaStream_t s) {
  auto kern = latent_mma_kernel<MT, NTW>;
  static bool configured[OGB_MAX_DEVICES] = {};
  if (!set_max_dyn_smem(kern, LAT_MAX_SMEM, configured)) return -3;
  const dim3 grid((max_q_len * p.H + MT * 16 - 1) / (MT * 16), 1, p.B * p.splits);
  if (!launch_pdl(kern, grid, dim3(LAT_THREADS), LatCfg<MT>::smem(p.pitch), s, p)) return -4;
  if (p.splits > 1 && !launch_pdl(latent_combine_kernel, dim3(p.total_rows), dim3(128), 0, s, static_cast<const float*>(p.part_o),
                                  static_cast<const float*>(p.part_ml), p.out, p.total_rows, p.R, p.splits, p.sinks, p.H))
    return -4;
  return 0;
}
template <int MT>
static int LaunchLatentMt(const LatentParams& p, int max_q_len, cudaStream_t s) {
  if (p.R <= 128) return LaunchLatentMma<MT, 2>(p, max_q_len, s);
  if (p.R <= 256) return LaunchLatentMma<MT, 4>(p, max_q_len, s);
  return LaunchLatentMma<MT, 8>(p, max_q_len, s);
}

static int lat_pitch(const OgbLatentShape* sh) { return (sh->R + sh->rot + 15) / 16 * 16 + 8; }     // an odd number of 16-byte chunks

}  // namespace ogb

using namespace ogb;

OGB_API int ogb_latent_prep(void* q, int ldq, const void* down, int ldd, void* cq, int ldcq, int q_rank, const float* cq_w, const OgbLatentShape* sh,
                            const float* norm_w, float eps, const int32_t* positions, const float* cos, const float* sin, int max_pos,
                            const int32_t* slots, void* cache, int ldcache, int T, int fp32, void* stream) {
  if (T <= 0) return 0;
  if (sh->rot_dims < 0 || sh->rot_dims > sh->rot || (sh->rot_dims & 1) || (sh->rot_dims > 0 && (!cos || !sin || max_pos <= 0))) return -1;
  if ((down && sh->R + sh->rot > ldcache) || (cq && (q_rank <= 0 || !cq_w))) return -1;
  auto s = static_cast<cudaStream_t>(stream);
#define OGB_LAT_PREP(TY) launch_pdl(latent_prep_kernel<TY>, dim3(T), dim3(128), 0, s, static_cast<TY*>(q), ldq, static_cast<const TY*>(down), ldd, \
                                    static_cast<TY*>(cq), ldcq, q_rank, cq_w, *sh, norm_w, eps, positions, cos, sin, max_pos, slots, \
                                    static_cast<TY*>(cache), ldcache)
  const bool ok = fp32 ? OGB_LAT_PREP(float) : OGB_LAT_PREP(__nv_bfloat16);
#undef OGB_LAT_PREP
  return ok ? 0 : -4;
}

OGB_API int ogb_gate_rows(void* out, int ldo, const void* gate, int ldg, int T, int n, int fp32, void* stream) {
  if (T <= 0 || n <= 0) return 0;
  auto s = static_cast<cudaStream_t>(stream);
  const long nb = (long(T) * n + 255) / 256;
  const dim3 grid(unsigned(nb < 148 * 16 ? nb : 148 * 16));
  using Hf = __nv_bfloat16;
  return (fp32 ? launch_pdl(gate_rows_kernel<float>, grid, dim3(256), 0, s, static_cast<float*>(out), ldo, static_cast<const float*>(gate), ldg, T, n)
               : launch_pdl(gate_rows_kernel<Hf>, grid, dim3(256), 0, s, static_cast<Hf*>(out), ldo, static_cast<const Hf*>(gate), ldg, T, n)) ? 0 : -4;
}

// 1 when the warp-MMA kernel can address these sizes (16-byte pieces everywhere, the tile fits in shared memory).
OGB_API int ogb_latent_mma_supported(const OgbLatentShape* sh) {
  return sh->R % 8 == 0 && sh->rot % 8 == 0 && sh->dim % 8 == 0 && sh->R >= 8 && sh->R <= 512 && sh->rot <= 128 && LatCfg<1>::smem(lat_pitch(sh)) <= LAT_MAX_SMEM;
}

// Rows of (token, head) a CTA takes for requests of at most max_q_len tokens.  17 .. 32 rows go as two tiles of 16: two of these CTAs share an SM
// and one's copies run under the other's MMAs, while the 32-row form is alone on it (measured with 32 heads of 576 columns, 64 requests of 2049
// keys in two parts: 87 against 108 us; 256 of 1025: 165 against 208).
OGB_API int ogb_latent_rows_per_tile(int H, int max_q_len) {
  const int rows = H * max_q_len;
  return rows <= 32 ? 16 : 64;
}

OGB_API long long ogb_latent_scratch_bytes(int total_rows, int R, int splits) {
  return splits <= 1 ? 0 : (long long)splits * total_rows * (R + 2) * 4;
}

// bf16.  skip_q_len > 0: requests with at least that many tokens are left to another kernel (their rows of `out` are unspecified).
OGB_API int ogb_latent_attention(const void* qlat, const void* proj, int ldp, const OgbLatentShape* sh, const void* cache, int ldcache,
                                 const int32_t* cu_seqlens, const int32_t* past_lens, const int32_t* block_table, int table_cols, int block_size,
                                 void* out, float scale, int window, const float* sinks, int B, int T, int max_q_len, int skip_q_len, int splits,
                                 void* scratch, long long scratch_bytes, const int32_t* order, int* status, void* stream) {
  if (B <= 0 || T <= 0 || max_q_len <= 0) return 0;
  if (!ogb_latent_mma_supported(sh)) return -5;
  if ((ldp % 8) || (ldcache % 8) || block_size <= 0) return -1;
  if ((reinterpret_cast<uintptr_t>(qlat) | reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(cache) | reinterpret_cast<uintptr_t>(out)) & 15) return -1;
  splits = splits < 1 ? 1 : (splits > LAT_MAX_SPLITS ? LAT_MAX_SPLITS : splits);
  const int rows = T * sh->H;
  if (ogb_latent_scratch_bytes(rows, sh->R, splits) > scratch_bytes || (long long)B * splits > 65535) return -2;
  LatentParams p;
  p.qlat = static_cast<const __nv_bfloat16*>(qlat); p.proj = static_cast<const __nv_bfloat16*>(proj); p.ldp = ldp; p.dim = sh->dim;
  p.cache = static_cast<const __nv_bfloat16*>(cache); p.ldcache = ldcache;
  p.cu = cu_seqlens; p.past = past_lens; p.table = block_table; p.table_cols = table_cols; p.block_size = block_size;
  p.block_shift = -1;
  for (int k = 0; k < 16; ++k) if (block_size == 1 << k) p.block_shift = k;
  p.out = static_cast<__nv_bfloat16*>(out);
  p.part_o = static_cast<float*>(scratch);
  p.part_ml = p.part_o ? p.part_o + size_t(splits) * rows * sh->R : nullptr;
  p.sinks = sinks; p.scale = scale; p.window = window; p.B = B; p.H = sh->H; p.R = sh->R; p.rot = sh->rot;
  p.kp = (sh->R + sh->rot + 15) / 16 * 16; p.pitch = lat_pitch(sh);
  p.splits = splits; p.total_rows = rows; p.skip_q_len = skip_q_len; p.order = order; p.status = status;
  auto s = static_cast<cudaStream_t>(stream);
  int bm = ogb_latent_rows_per_tile(sh->H, skip_q_len > 0 && skip_q_len - 1 < max_q_len ? skip_q_len - 1 : max_q_len);
  if (bm == 64 && LatCfg<4>::smem(p.pitch) > LAT_MAX_SMEM) bm = 32;
  if (bm == 32 && LatCfg<2>::smem(p.pitch) > LAT_MAX_SMEM) bm = 16;
  if (skip_q_len > 0 && max_q_len > skip_q_len - 1) max_q_len = skip_q_len - 1;
  if (max_q_len <= 0) return 0;
  if (bm == 16) return LaunchLatentMt<1>(p, max_q_len, s);
  if (bm == 32) return LaunchLatentMt<2>(p, max_q_len, s);
  return LaunchLatentMt<4>(p, max_q_len, s);
}

OGB_API int ogb_latent_attention_simt(const void* qlat, const void* proj, int ldp, const OgbLatentShape* sh, const void* cache, int ldcache,
                                      const int32_t* cu_seqlens, const int32_t* past_lens, const int32_t* block_table, int table_cols, int block_size,
                                      void* out, float scale, int window, const float* sinks, int B, int T, int skip_q_len, int fp32, void* stream) {
  if (B <= 0 || T <= 0) return 0;
  if (sh->R > 128 * LAT_SIMT_COLS || sh->H > 65535 || block_size <= 0) return -5;
  const int smem = (sh->R + sh->rot + 32) * 4;
  if (smem > 48 * 1024) return -5;
  auto s = static_cast<cudaStream_t>(stream);
  using Hf = __nv_bfloat16;
  return (fp32 ? launch_pdl(latent_simt_kernel<float>, dim3(T, sh->H), dim3(128), smem, s, static_cast<const float*>(qlat), static_cast<const float*>(proj),
                            ldp, *sh, static_cast<const float*>(cache), ldcache, cu_seqlens, past_lens, block_table, table_cols, block_size,
                            static_cast<float*>(out), scale, window, sinks, B, skip_q_len)
               : launch_pdl(latent_simt_kernel<Hf>, dim3(T, sh->H), dim3(128), smem, s, static_cast<const Hf*>(qlat), static_cast<const Hf*>(proj), ldp, *sh,
                            static_cast<const Hf*>(cache), ldcache, cu_seqlens, past_lens, block_table, table_cols, block_size, static_cast<Hf*>(out), scale,
                            window, sinks, B, skip_q_len)) ? 0 : -4;
}

// width, ldcache, ldo in bf16 elements, multiples of 8
OGB_API int ogb_latent_gather(const void* cache, int ldcache, const int32_t* block_table, int table_cols, int block_size, const int32_t* row_base,
                              const int32_t* first_kv, const int32_t* kv_len, const int32_t* req, int n_req, int rows, int width, void* out, int ldo,
                              void* stream) {
  if (rows <= 0 || n_req <= 0) return 0;
  if ((width % 8) || (ldcache % 8) || (ldo % 8) || block_size <= 0) return -1;
  return launch_pdl(latent_gather_kernel, dim3((rows + 7) / 8), dim3(256), 0, static_cast<cudaStream_t>(stream), static_cast<const uint4*>(cache),
                    ldcache / 8, block_table, table_cols, block_size, row_base, first_kv, kv_len, req, n_req, rows, width / 8, static_cast<uint4*>(out),
                    ldo / 8) ? 0 : -4;
}
