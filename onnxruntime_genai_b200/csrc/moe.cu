// Mixture-of-experts routing around the grouped tcgen05 expert GEMM (ogb_moe_gemm in gemm_tcgen05.cu).
//
//   router logits [T, E] (fp32, from the GEMM)  -- moe_topk -->  expert ids + routing weights [T, k]
//   -- moe_sort -->  token rows grouped by expert: per-expert row ranges, source token of every sorted row,
//                    sorted row of every (token, j) assignment, and the list of token tiles for the GEMM grid
//   -- gather rows, grouped gate/up GEMM (+ clamped SwiGLU), grouped down GEMM --
//   -- moe_combine -->  out[t] = sum_j w[t, j] * y[row(t, j)]  (j order, fp32: deterministic)
//
// Everything stays on the device (no counts are read back), so a decode step with experts replays inside
// a CUDA graph.  With expert parallelism a rank passes its expert range to moe_sort: assignments to other
// ranks' experts get row -1 and are skipped by the combine, whose partial result is then all-reduced.
//
// Reference semantics: the MoE / QMoE contrib op emitted by src/python/py/models/builders/base.py:4176-4408
// (k, normalize_routing_weights, swiglu_fusion) and the router of builders/gptoss.py:653-847.
#include "common.cuh"
#include "kernels.h"

namespace ogb {

// One warp per token.  mode 0: softmax over the k selected logits; mode 1: softmax over all experts, the
// selected probabilities unchanged; mode 2: softmax over all experts, renormalised over the selected.  shared: every token also gets expert E
// with weight 1 (rows of k + 1 entries).
__global__ void moe_topk_kernel(const float* __restrict__ logits, int ld, int T, int E, int k, int mode, int shared, int* __restrict__ topk_idx,
                                float* __restrict__ topk_w) {
  const int warp = (blockIdx.x * blockDim.x + threadIdx.x) >> 5, lane = threadIdx.x & 31;
  if (warp >= T) return;
  const float* row = logits + size_t(warp) * ld;
  uint32_t taken = 0;  // bit i: this lane's element lane + 32*i is already selected (E <= 1024)
  float all_max = -INFINITY, all_sum = 0.f;
  if (mode != 0) {
    for (int e = lane; e < E; e += 32) all_max = fmaxf(all_max, row[e]);
    all_max = warp_max(all_max);
    for (int e = lane; e < E; e += 32) all_sum += expf(row[e] - all_max);
    all_sum = warp_sum(all_sum);
  }
  float my_val = 0.f;   // lane j keeps the j-th selected logit
  int my_idx = 0;
  float first = 0.f;
  for (int j = 0; j < k; ++j) {
    float best = -INFINITY;
    int best_e = 0x7fffffff;
    for (int i = 0, e = lane; e < E; ++i, e += 32) {
      if (taken >> i & 1) continue;
      const float v = row[e];
      if (v > best || (v == best && e < best_e)) { best = v; best_e = e; }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, o);
      const int oe = __shfl_xor_sync(0xffffffffu, best_e, o);
      if (ov > best || (ov == best && oe < best_e)) { best = ov; best_e = oe; }
    }
    if (best_e != 0x7fffffff && (best_e & 31) == lane) taken |= 1u << (best_e >> 5);
    if (j == 0) first = best;
    if (lane == j) { my_val = best; my_idx = best_e == 0x7fffffff ? 0 : best_e; }
  }
  float w;
  if (mode == 0) {
    const float ex = lane < k ? expf(my_val - first) : 0.f;
    w = ex / warp_sum(ex);
  } else {
    const float pr = lane < k ? expf(my_val - all_max) / all_sum : 0.f;
    w = mode == 2 ? pr / warp_sum(pr) : pr;
  }
  const int per = k + shared;
  if (lane < per) {
    topk_idx[size_t(warp) * per + lane] = lane < k ? my_idx : E;
    topk_w[size_t(warp) * per + lane] = lane < k ? w : 1.f;
  }
}

// A float as an unsigned number of the same order.
__device__ __forceinline__ uint32_t order_bits(float v) {
  const uint32_t u = __float_as_uint(v);
  return u & 0x80000000u ? ~u : u | 0x80000000u;
}
// Entry with the largest key of the warp's lanes (each brings its best and where that is; 0: nothing), the smallest place among equal ones.
__device__ __forceinline__ int warp_argmax(uint32_t key, int at) {
  const uint32_t top = __reduce_max_sync(0xffffffffu, key);
  return int(__reduce_min_sync(0xffffffffu, key == top ? uint32_t(at) : 0x7fffffffu));
}

// One warp per token: experts chosen by sigmoid(logit) + correction among the `keep` of `groups` groups of neighbours whose two largest choice
// scores have the largest sums; weights: the chosen sigmoids divided by their sum (+ 1e-20), times scale.  A lane holds every 32nd expert, PER of them; the
// scores also sit in shared memory for the groups' sums.
template <int PER>
__global__ void __launch_bounds__(128) moe_topk_grouped_kernel(const float* __restrict__ logits, int ld, int T, int E, int k, const float* __restrict__ correction,
                                                               int groups, int keep, float scale, int* __restrict__ topk_idx, float* __restrict__ topk_w) {
  extern __shared__ float choice_all[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x * (blockDim.x >> 5) + warp;
  if (t >= T) return;
  float* c = choice_all + size_t(warp) * E;
  const float* row = logits + size_t(t) * ld;
  float s[PER];
  uint32_t key[PER];                       // 0: not to be chosen
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int e = i * 32 + lane;
    s[i] = 0.f;
    key[i] = 0;
    if (e >= E) continue;
    s[i] = 1.f / (1.f + expf(-row[e]));
    const float v = s[i] + correction[e];
    key[i] = order_bits(v);
    if (groups > 1) c[e] = v;
  }
  if (groups > 1) {
    __syncwarp();
    const int per = E / groups;
    // groups in rounds of 32, one per lane; a round's kept groups compete with those kept so far
    uint32_t kept[32];                     // bit g % 32 of word g / 32
    const int words = (groups + 31) / 32;
#pragma unroll 1
    for (int w = 0; w < words; ++w) {
      const int g = w * 32 + lane;
      uint32_t mine = 0;
      if (g < groups) {
        float a = -INFINITY, b = -INFINITY;
        for (int e = g * per; e < (g + 1) * per; ++e) {
          const float v = c[e];
          b = fmaxf(b, fminf(a, v));
          a = fmaxf(a, v);
        }
        mine = order_bits(per > 1 ? a + b : a);
      }
      kept[w] = mine;
    }
    // `keep` times the best group that is left
    uint32_t open_[32];
    for (int w = 0; w < words; ++w) open_[w] = 0;
    for (int j = 0; j < keep; ++j) {
      uint32_t best = 0;
      int at = 0x7fffffff;
      for (int w = 0; w < words; ++w) if (kept[w] > best) { best = kept[w]; at = w * 32 + lane; }
      const int g = warp_argmax(best, at);
      if (g >= groups) break;
      if ((g & 31) == lane) kept[g >> 5] = 0;
      open_[g >> 5] |= 1u << (g & 31);
    }
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      const int g = min(i * 32 + lane, E - 1) / per;
      if (!(open_[g >> 5] >> (g & 31) & 1)) key[i] = 0;
    }
  }
  float w = 0.f;
  int mine = 0;
  for (int j = 0; j < k; ++j) {
    uint32_t best = 0;
    int at = 0x7fffffff;
    float sv = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i) if (key[i] > best) { best = key[i]; at = i * 32 + lane; sv = s[i]; }
    const int e = min(warp_argmax(best, at), E - 1);       // (there are always enough experts to choose from)
    sv = __shfl_sync(0xffffffffu, sv, e & 31);
#pragma unroll
    for (int i = 0; i < PER; ++i) if (i * 32 + lane == e) key[i] = 0;
    if (lane == j) { mine = e; w = sv; }
  }
  const float sum = warp_sum(w) + 1e-20f;
  if (lane < k) {
    topk_idx[size_t(t) * k + lane] = mine;
    topk_w[size_t(t) * k + lane] = w / sum * scale;
  }
}

// Single CTA: counting sort of the n = T*k assignments by expert (local experts [e_lo, e_hi) only).
__global__ void __launch_bounds__(1024)
moe_sort_kernel(const int* __restrict__ topk_idx, int n, int k, int E, int e_lo, int e_hi, int bt, int* __restrict__ expert_offsets,
                int* __restrict__ sorted_token, int* __restrict__ inv_pos, int* __restrict__ tile_expert, int* __restrict__ tile_row0,
                int* __restrict__ tile_rows, int* __restrict__ num_tiles, int max_tiles) {
  extern __shared__ int sm[];
  int* cnt = sm;               // [E]
  int* off = sm + E;           // [E + 1] rows
  int* tbase = off + E + 1;    // [E + 1] tiles
  for (int e = threadIdx.x; e < E; e += blockDim.x) cnt[e] = 0;
  __syncthreads();
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    const int e = topk_idx[i];
    if (e >= e_lo && e < e_hi) atomicAdd(&cnt[e], 1);
  }
  __syncthreads();
  if (threadIdx.x == 0) {  // E is small (<= 1024): a serial scan costs less than a microsecond
    int r = 0, t = 0;
    for (int e = 0; e < E; ++e) {
      off[e] = r; tbase[e] = t;
      r += cnt[e];
      t += (cnt[e] + bt - 1) / bt;
    }
    off[E] = r; tbase[E] = t;
    *num_tiles = t < max_tiles ? t : max_tiles;
  }
  __syncthreads();
  for (int e = threadIdx.x; e <= E; e += blockDim.x) expert_offsets[e] = off[e];
  for (int e = threadIdx.x; e < E; e += blockDim.x) {
    const int c = cnt[e];
    for (int j = 0, t = tbase[e]; j * bt < c && t < max_tiles; ++j, ++t) {
      tile_expert[t] = e - e_lo;   // index into this rank's slice of the expert weights
      tile_row0[t] = off[e] + j * bt;
      tile_rows[t] = min(bt, c - j * bt);
    }
  }
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += blockDim.x) cnt[e] = 0;   // reuse as cursors
  __syncthreads();
  // Rows of one expert keep assignment order only up to the atomics' order; every sorted row is computed
  // independently of its neighbours, so the result does not depend on that order.
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    const int e = topk_idx[i];
    if (e >= e_lo && e < e_hi) {
      const int pos = off[e] + atomicAdd(&cnt[e], 1);
      sorted_token[pos] = i / k;
      inv_pos[i] = pos;
    } else {
      inv_pos[i] = -1;
    }
  }
  // Rows past the last assignment feed tail tiles of the grouped GEMM: give them a valid source.
  for (int i = off[E] + threadIdx.x; i < n; i += blockDim.x) sorted_token[i] = 0;
}

// out[t, :] = (residual[t, :]) + sum_j w[t, j] * y[inv_pos[t, j], :]   (8 features per thread)
__global__ void moe_combine_kernel(const __nv_bfloat16* __restrict__ y, int ldy, const int* __restrict__ inv_pos,
                                   const float* __restrict__ topk_w, int T, int k, int H, const __nv_bfloat16* __restrict__ residual,
                                   int ldr, __nv_bfloat16* __restrict__ out, int ldo) {
  const int t = blockIdx.x;
  for (int c = threadIdx.x * 8; c < H; c += blockDim.x * 8) {
    float acc[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (residual) {
      const uint4 q = *reinterpret_cast<const uint4*>(residual + size_t(t) * ldr + c);
      const float2 a = unpack_bf16x2(q.x), b = unpack_bf16x2(q.y), cc = unpack_bf16x2(q.z), d = unpack_bf16x2(q.w);
      acc[0] = a.x; acc[1] = a.y; acc[2] = b.x; acc[3] = b.y; acc[4] = cc.x; acc[5] = cc.y; acc[6] = d.x; acc[7] = d.y;
    }
    for (int j = 0; j < k; ++j) {
      const int pos = inv_pos[size_t(t) * k + j];
      if (pos < 0) continue;
      const float w = topk_w[size_t(t) * k + j];
      const uint4 q = *reinterpret_cast<const uint4*>(y + size_t(pos) * ldy + c);
      const float2 a = unpack_bf16x2(q.x), b = unpack_bf16x2(q.y), cc = unpack_bf16x2(q.z), d = unpack_bf16x2(q.w);
      acc[0] += w * a.x; acc[1] += w * a.y; acc[2] += w * b.x; acc[3] += w * b.y;
      acc[4] += w * cc.x; acc[5] += w * cc.y; acc[6] += w * d.x; acc[7] += w * d.y;
    }
    *reinterpret_cast<uint4*>(out + size_t(t) * ldo + c) =
        make_uint4(pack_bf16x2(acc[0], acc[1]), pack_bf16x2(acc[2], acc[3]), pack_bf16x2(acc[4], acc[5]), pack_bf16x2(acc[6], acc[7]));
  }
}

}  // namespace ogb

using namespace ogb;

OGB_API int ogb_moe_topk(const float* logits, int ld, int T, int E, int k, int mode, int shared, int32_t* topk_idx, float* topk_w, void* stream) {
  if (T <= 0) return 0;
  shared = shared ? 1 : 0;
  if (E <= 0 || E > 1024 || k <= 0 || k + shared > 32 || k > E || mode < 0 || mode > 2) return -1;
  const int threads = 128, warps_per_block = threads / 32;
  moe_topk_kernel<<<(T + warps_per_block - 1) / warps_per_block, threads, 0, static_cast<cudaStream_t>(stream)>>>(
      logits, ld, T, E, k, mode, shared, topk_idx, topk_w);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

OGB_API int ogb_moe_topk_grouped(const float* logits, int ld, int T, int E, int k, const float* correction, int groups, int keep, float scale,
                                 int32_t* topk_idx, float* topk_w, void* stream) {
  if (T <= 0) return 0;
  if (E <= 0 || E > 1024 || k <= 0 || k > 32 || k > E || groups < 1 || E % groups || keep < 1 || keep > groups || k > E / groups * keep || !correction) return -1;
  const int warps = 4;
  const dim3 grid((T + warps - 1) / warps), block(warps * 32);
  const size_t smem = groups > 1 ? size_t(warps) * E * sizeof(float) : 0;
  auto st = static_cast<cudaStream_t>(stream);
#define OGB_GROUPED(PER) moe_topk_grouped_kernel<PER><<<grid, block, smem, st>>>(logits, ld, T, E, k, correction, groups, keep, scale, topk_idx, topk_w)
  if (E <= 32) OGB_GROUPED(1);
  else if (E <= 64) OGB_GROUPED(2);
  else if (E <= 128) OGB_GROUPED(4);
  else if (E <= 256) OGB_GROUPED(8);
  else OGB_GROUPED(32);
#undef OGB_GROUPED
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// Upper bound of the tile-list length for n assignments over `experts` experts at token tile `bt`.
OGB_API int ogb_moe_max_tiles(int n, int experts, int bt) {
  const int by_rows = n / bt + experts;   // sum of ceil(c_e / bt) <= n / bt + (experts with a remainder)
  return by_rows < n ? by_rows : n;
}

OGB_API int ogb_moe_sort(const int32_t* topk_idx, int T, int k, int E, int e_lo, int e_hi, int bt, int32_t* expert_offsets,
                         int32_t* sorted_token, int32_t* inv_pos, int32_t* tile_expert, int32_t* tile_row0, int32_t* tile_rows,
                         int32_t* num_tiles, int max_tiles, void* stream) {
  if (T <= 0) return 0;
  if (E <= 0 || E > 1024 || k <= 0 || bt <= 0 || max_tiles <= 0) return -1;
  const size_t smem = size_t(3 * E + 2) * sizeof(int);
  moe_sort_kernel<<<1, 1024, smem, static_cast<cudaStream_t>(stream)>>>(topk_idx, T * k, k, E, e_lo, e_hi, bt, expert_offsets,
                                                                         sorted_token, inv_pos, tile_expert, tile_row0, tile_rows,
                                                                         num_tiles, max_tiles);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

OGB_API int ogb_moe_combine(const void* y, int ldy, const int32_t* inv_pos, const float* topk_w, int T, int k, int H,
                            const void* residual, int ldr, void* out, int ldo, void* stream) {
  if (T <= 0) return 0;
  if ((H % 8) || (ldy % 8) || (ldo % 8) || (residual && (ldr % 8))) return -1;
  if ((reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(residual)) & 15) return -1;
  int threads = (H / 8 + 31) / 32 * 32;
  if (threads > 512) threads = 512;
  moe_combine_kernel<<<T, threads, 0, static_cast<cudaStream_t>(stream)>>>(
      static_cast<const __nv_bfloat16*>(y), ldy, inv_pos, topk_w, T, k, H, static_cast<const __nv_bfloat16*>(residual), ldr,
      static_cast<__nv_bfloat16*>(out), ldo);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
