// Prefill attention on the tensor cores: the launches for heads of 64 and 128 columns and of the latent form (the kernel is in
// attention_tc.cuh; heads of other widths are in attention_tc_mixed.cu), and the entry points.
#include "attention_tc.cuh"

namespace ogb {

template <int NOPE, int ROT, int DV, int BN>
static int LaunchTcLatent(const TcAttnParams& p, const CUtensorMap& mk, const CUtensorMap& mv, const CUtensorMap& mr, int max_q_len, cudaStream_t stream) {
  using Cfg = TcaCfg<NOPE + ROT, DV, BN>;
  auto kern = attention_tc_kernel<NOPE + ROT, DV, BN, true, NOPE>;
  static bool configured[OGB_MAX_DEVICES] = {};
  if (!set_max_dyn_smem(kern, Cfg::SMEM, configured)) return -3;
  dim3 grid((max_q_len + TCA_BM - 1) / TCA_BM, p.Hkv, p.B);
  launch_pdl(kern, grid, dim3(TCA_THREADS), Cfg::SMEM, stream, mk, mv, mr, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

int LaunchTcUniform(const TcAttnParams& p, int D, const void* k_cache, const void* v_cache, int max_q_len, int cache_slots, cudaStream_t stream) {
  // 128 keys per tile (measured on B200 against 64: 457 vs 429 TFLOP/s at 4096 tokens, head_dim 128)
  if (D == 128) return LaunchTc<128, 128, 128>(p, k_cache, v_cache, max_q_len, cache_slots, stream);
  if (D == 64) return LaunchTc<64, 64, 128>(p, k_cache, v_cache, max_q_len, cache_slots, stream);
  return -5;
}

}  // namespace ogb

using namespace ogb;

// 1 when the tensor-core prefill kernel can serve this configuration (the caller then launches both kernels: this one takes the
// requests with at least `min_rows` query rows, ogb_paged_attention with skip_rows = min_rows the others).
OGB_API int ogb_attention_tc_supported(int D, int block_size, int kv_bits, int cache_slots) {
  return (D == 64 || D == 128) && block_size % 16 == 0 && kv_bits == 16 && cache_slots >= 16;
}

OGB_API int ogb_attention_tc(const void* q, int q_stride, const void* k_cache, const void* v_cache, const int32_t* cu_seqlens,
                             const int32_t* past_lens, const int32_t* block_table, int table_cols, int block_size, void* out, int out_stride,
                             const float* sinks, float scale, float softcap, int window, int B, int max_q_len, int Hq, int Hkv, int D,
                             int min_rows, int cache_slots, int* status, void* stream_) {
  if (B <= 0 || max_q_len <= 0) return 0;
  if (!ogb_attention_tc_supported(D, block_size, 16, cache_slots)) return -5;
  if (Hkv <= 0 || Hq % Hkv || (q_stride % 8) || (out_stride % 8)) return -1;
  if (((reinterpret_cast<uintptr_t>(k_cache) | reinterpret_cast<uintptr_t>(v_cache) | reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(out)) & 15) != 0) return -1;
  TcAttnParams p{};
  p.out_scale = 1.f;
  p.q = static_cast<const __nv_bfloat16*>(q); p.q_stride = q_stride;
  p.cu_seqlens = cu_seqlens; p.past_lens = past_lens; p.block_table = block_table; p.table_cols = table_cols; p.block_size = block_size;
  p.out = static_cast<__nv_bfloat16*>(out); p.out_stride = out_stride;
  p.sinks = sinks; p.scale = scale; p.softcap = softcap; p.window = window;
  p.B = B; p.Hq = Hq; p.Hkv = Hkv; p.min_rows = min_rows; p.status = status;
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  return LaunchTcUniform(p, D, k_cache, v_cache, max_q_len, cache_slots, stream);
}

// 1 when the latent form can serve these sizes: 16-byte pieces everywhere, unrotated part up to 192 columns, rotated part up to 64,
// values up to 128.
OGB_API int ogb_attention_tc_latent_supported(int dim, int rot, int vdim) {
  return dim % 8 == 0 && rot % 8 == 0 && vdim % 8 == 0 && dim > 0 && dim <= 192 && rot > 0 && rot <= 64 && vdim > 0 && vdim <= 128;
}

// Long prompts of a latent-attention layer.  q: row t holds H heads of (dim | rot) rotated queries; kv [rows, >= H * (dim + vdim)]: the
// expanded keys (head-major columns) then values; kr [rows, >= kr_col + rot]: the shared rotated key part from column kr_col on.
// row_base / first_kv [B]: dense row of each request's first expanded position (a multiple of 16) and that position; row_base < 0
// leaves the request out.  Output row t: H heads of vdim columns, times the sigmoid of gate [T, H * vdim] (may be null).  sinks (may be null) [H].
OGB_API int ogb_attention_tc_latent(const void* q, int q_stride, const void* kv, int ldkv, const void* kr, int ldkr, int kr_col, int rows,
                                    const int32_t* cu_seqlens, const int32_t* past_lens, const int32_t* row_base, const int32_t* first_kv, void* out,
                                    int out_stride, float scale, int window, const float* sinks, const void* gate, int gate_stride, int B, int max_q_len,
                                    int H, int dim, int rot, int vdim, int* status, void* stream_) {
  if (B <= 0 || max_q_len <= 0 || rows <= 0) return 0;
  if (!ogb_attention_tc_latent_supported(dim, rot, vdim)) return -5;
  if ((q_stride % 8) || (out_stride % 8) || (ldkv % 8) || (ldkr % 8) || (kr_col % 8)) return -1;
  if (gate && ((gate_stride % 8) || (reinterpret_cast<uintptr_t>(gate) & 15))) return -1;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(kv) | reinterpret_cast<uintptr_t>(kr) | reinterpret_cast<uintptr_t>(out)) & 15) return -1;
  TcAttnParams p{};
  p.out_scale = 1.f;
  p.q = static_cast<const __nv_bfloat16*>(q); p.q_stride = q_stride;
  p.cu_seqlens = cu_seqlens; p.past_lens = past_lens; p.block_size = 16;
  p.out = static_cast<__nv_bfloat16*>(out); p.out_stride = out_stride;
  p.scale = scale; p.window = window; p.B = B; p.Hq = H; p.Hkv = H; p.min_rows = 1; p.status = status;
  p.sinks = sinks; p.gate = static_cast<const __nv_bfloat16*>(gate); p.gate_stride = gate_stride; p.gate_wide = gate != nullptr;
  p.lat.row_base = row_base; p.lat.first_kv = first_kv; p.lat.dim = dim; p.lat.rot = rot; p.lat.vdim = vdim; p.lat.kr_col = kr_col;
  CUtensorMap mk, mv, mr;
  const __nv_bfloat16* base = static_cast<const __nv_bfloat16*>(kv);
  if ((H * dim) % 8) return -1;
  if (!MakeMapBf16(&mk, base, rows, H * dim, ldkv, 16) || !MakeMapBf16(&mv, base + size_t(H) * dim, rows, H * vdim, ldkv, 16) ||
      !MakeMapBf16(&mr, kr, rows, kr_col + rot, ldkr, 16))
    return -2;
  cudaStream_t s = static_cast<cudaStream_t>(stream_);
  // tiles of 128 keys where two stages of both rings fit beside the query tile, else 64
  const int nope = (dim + 63) / 64;
  if (vdim <= 64) {
    if (nope == 1) return LaunchTcLatent<64, 64, 64, 128>(p, mk, mv, mr, max_q_len, s);
    if (nope == 2) return LaunchTcLatent<128, 64, 64, 128>(p, mk, mv, mr, max_q_len, s);
    return LaunchTcLatent<192, 64, 64, 64>(p, mk, mv, mr, max_q_len, s);
  }
  if (nope == 1) return LaunchTcLatent<64, 64, 128, 128>(p, mk, mv, mr, max_q_len, s);
  if (nope == 2) return LaunchTcLatent<128, 64, 128, 128>(p, mk, mv, mr, max_q_len, s);
  return LaunchTcLatent<192, 64, 128, 64>(p, mk, mv, mr, max_q_len, s);
}
