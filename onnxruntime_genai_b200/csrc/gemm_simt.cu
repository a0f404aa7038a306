// Linear layers outside the tensor cores: true fp32 products of the 32-bit models (fp32 operands, fp32 multiply-adds, no reduced
// precision mode), and bf16 products whose sizes or addresses TMA cannot take (strides that are not multiples of 16 bytes).
//   C[m, z * c_cols + n] = sum_k A[m, z * a_cols + k] * W[z * N + n, k]   (+ bias[n], + residual[m, n], fp32)
// and the grouped form over token rows sorted by expert (tile list of moe.cu): C[r, n] = sum_k A[map(r), k] * W[expert(r) * N + n, k].
// One CTA = a 64 x 64 output tile, 16 columns of K at a time through shared memory, 4 x 4 outputs per thread.
#include "common.cuh"
#include "gemm_common.cuh"
#include "kernels.h"

namespace ogb {

struct SimtGemmParams {
  const void* A; const void* W; void* C; const float* residual; const void* bias;
  int lda, a_cols, ldw, ldc, c_cols, ldr;
  int M, N, K;
  int act;      // 0 none, else 1 + activation (see act_one)
  // grouped form: per token tile (blockIdx.y) its expert, first row and rows; row_map (may be null): row of A for every sorted row
  const int32_t *tile_expert, *tile_row0, *tile_rows, *num_tiles, *row_map;
};

template <typename T> __device__ __forceinline__ float ld_f32(const T* p);
template <> __device__ __forceinline__ float ld_f32<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float ld_f32<__nv_bfloat16>(const __nv_bfloat16* p) { return bf2f(*p); }

template <typename T, typename TO>
__global__ void __launch_bounds__(256) gemm_simt_kernel(SimtGemmParams p) {
  constexpr int BM = 64, BN = 64, BK = 16;
  __shared__ float sA[BK][BM + 4], sW[BK][BN + 4];
  pdl_launch_dependents();
  pdl_wait();
  const bool grouped = p.tile_expert != nullptr;
  if (grouped && int(blockIdx.y) >= *p.num_tiles) return;
  const int z = blockIdx.z, m0 = grouped ? p.tile_row0[blockIdx.y] : blockIdx.y * BM, n0 = blockIdx.x * BN;
  const int m_end = grouped ? m0 + min(BM, p.tile_rows[blockIdx.y]) : p.M;
  const T* A = static_cast<const T*>(p.A) + size_t(z) * p.a_cols;
  const T* W = static_cast<const T*>(p.W) + size_t(grouped ? p.tile_expert[blockIdx.y] : z) * p.N * p.ldw;
  const int tid = threadIdx.x, tx = tid % 16, ty = tid / 16;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < p.K; k0 += BK) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int idx = tid + i * 256, r = idx / BK, k = idx % BK;
      const int m = m0 + r;
      sA[k][r] = (m < m_end && k0 + k < p.K) ? ld_f32(A + size_t(grouped && p.row_map ? p.row_map[m] : m) * p.lda + k0 + k) : 0.f;
      sW[k][r] = (n0 + r < p.N && k0 + k < p.K) ? ld_f32(W + size_t(n0 + r) * p.ldw + k0 + k) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < BK; ++k) {
      float a[4], w[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { a[i] = sA[k][ty * 4 + i]; w[i] = sW[k][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], w[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= m_end) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= p.N) continue;
      float v = acc[i][j];
      if (p.bias) v += ld_f32(static_cast<const T*>(p.bias) + n);
      if (p.act) v = act_one(p.act, v);
      if (p.residual) v += p.residual[size_t(m) * p.ldr + n];
      TO* dst = static_cast<TO*>(p.C) + size_t(m) * p.ldc + size_t(z) * p.c_cols + n;
      if constexpr (sizeof(TO) == 4) *dst = v; else *dst = f2bf(v);
    }
  }
}

}  // namespace ogb

using namespace ogb;

// in_fp32 / out_fp32: element types of A and W / of C (else bf16).  residual (fp32, may be C itself) and bias [N] (in A's type)
// only with batch == 1.  act: 0, or 1 + the activation of the result (numbers as in ogb_gemm_bf16), before the residual.
OGB_API int ogb_gemm_simt(const void* A, int lda, int a_cols, const void* W, int ldw, void* C, int ldc, int c_cols, int M, int N, int K,
                          int batch, const float* residual, int ldr, const void* bias, int act, int in_fp32, int out_fp32, void* stream_) {
  if (M <= 0 || N <= 0 || K <= 0 || batch <= 0) return 0;
  if ((residual || bias) && batch != 1) return -1;
  if (M > 64 * 65535 || batch > 65535) return -1;
  SimtGemmParams p{A, W, C, residual, bias, lda, a_cols, ldw, ldc, c_cols, ldr, M, N, K, act, nullptr, nullptr, nullptr, nullptr, nullptr};
  const dim3 grid((N + 63) / 64, (M + 63) / 64, batch);
  auto s = static_cast<cudaStream_t>(stream_);
  bool ok;
  if (in_fp32) ok = out_fp32 ? launch_pdl(gemm_simt_kernel<float, float>, grid, dim3(256), 0, s, p)
                             : launch_pdl(gemm_simt_kernel<float, __nv_bfloat16>, grid, dim3(256), 0, s, p);
  else ok = out_fp32 ? launch_pdl(gemm_simt_kernel<__nv_bfloat16, float>, grid, dim3(256), 0, s, p)
                     : launch_pdl(gemm_simt_kernel<__nv_bfloat16, __nv_bfloat16>, grid, dim3(256), 0, s, p);
  return ok ? 0 : -4;
}

// Grouped expert product: W [experts, N, K] dense, token tiles of at most 64 rows.  row_map (may be null): sorted row r reads row
// row_map[r] of A.  C has the element type of A and W.
OGB_API int ogb_moe_gemm_simt(const void* A, int lda, const void* W, void* C, int ldc, int N, int K, const int32_t* tile_expert, const int32_t* tile_row0,
                              const int32_t* tile_rows, const int32_t* num_tiles, int max_tiles, int token_tile, const int32_t* row_map, int fp32,
                              void* stream_) {
  if (N <= 0 || K <= 0 || max_tiles <= 0) return 0;
  if (token_tile > 64 || max_tiles > 65535 || !tile_expert || !tile_row0 || !tile_rows || !num_tiles) return -1;
  SimtGemmParams p{A, W, C, nullptr, nullptr, lda, 0, K, ldc, 0, 0, 0, N, K, 0, tile_expert, tile_row0, tile_rows, num_tiles, row_map};
  const dim3 grid((N + 63) / 64, max_tiles, 1);
  auto s = static_cast<cudaStream_t>(stream_);
  const bool ok = fp32 ? launch_pdl(gemm_simt_kernel<float, float>, grid, dim3(256), 0, s, p)
                       : launch_pdl(gemm_simt_kernel<__nv_bfloat16, __nv_bfloat16>, grid, dim3(256), 0, s, p);
  return ok ? 0 : -4;
}
