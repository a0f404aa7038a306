// Prefill attention on the tensor cores (attention_tc.cuh) for layers whose heads have sizes of their own: queries and keys of dk columns
// staged as 64, 128, 192 or 256, values of dv columns staged as 64, 128 or 256.  Joint layers (a query meets the keys of all key heads) also with keys of up to 1024
// columns, which arrive in parts of 128 (beyond 512 columns to tiles of 64 query rows).
#include "attention_tc.cuh"

namespace ogb {

int LaunchTcUniform(const TcAttnParams& p, int D, const void* k_cache, const void* v_cache, int max_q_len, int cache_slots, cudaStream_t stream);

// tiles of 128 keys where three score buffers and the output fit in tensor memory and two stages of both rings beside the query tile
template <int DK, int DV>
static int LaunchTcMixed(const TcAttnParams& p, const void* k, const void* v, int max_q_len, int cache_slots, cudaStream_t s) {
  constexpr int BN = DV <= 128 && DK <= 128 ? 128 : 64;
  return LaunchTc<DK, DV, BN, true>(p, k, v, max_q_len, cache_slots, s);
}
template <int DK>
static int LaunchTcMixedKeys(const TcAttnParams& p, const void* k, const void* v, int max_q_len, int cache_slots, cudaStream_t s) {
  if (p.dv <= 64) return LaunchTcMixed<DK, 64>(p, k, v, max_q_len, cache_slots, s);
  if (p.dv <= 128) return LaunchTcMixed<DK, 128>(p, k, v, max_q_len, cache_slots, s);
  return LaunchTcMixed<DK, 256>(p, k, v, max_q_len, cache_slots, s);
}

template <int DK, int DV>
static int LaunchTcWide(const TcAttnParams& p, const void* k, const void* v, int max_q_len, int cache_slots, cudaStream_t s) {
  constexpr int QR = DK <= 512 ? TCA_BM : 64;
  return p.softcap > 0.f ? LaunchTcForm<DK, DV, 64, true, true, 128, QR>(p, k, v, max_q_len, cache_slots, s)
                         : LaunchTcForm<DK, DV, 64, true, false, 128, QR>(p, k, v, max_q_len, cache_slots, s);
}
template <int DK>
static int LaunchTcWideKeys(const TcAttnParams& p, const void* k, const void* v, int max_q_len, int cache_slots, cudaStream_t s) {
  if (p.dv <= 64) return LaunchTcWide<DK, 64>(p, k, v, max_q_len, cache_slots, s);
  if (p.dv <= 128) return LaunchTcWide<DK, 128>(p, k, v, max_q_len, cache_slots, s);
  return LaunchTcWide<DK, 256>(p, k, v, max_q_len, cache_slots, s);
}

}  // namespace ogb

using namespace ogb;

OGB_API int ogb_attention_tc_joint_supported(int dk, int dv, int block_size, int cache_slots) {
  return dk > 0 && dv > 0 && dk % 8 == 0 && dv % 8 == 0 && dk <= 1024 && dv <= 256 && block_size % 16 == 0 && cache_slots >= 16;
}

OGB_API int ogb_attention_tc_mixed_supported(int dk, int dv, int block_size, int cache_slots) {
  return dk > 0 && dv > 0 && dk % 8 == 0 && dv % 8 == 0 && dk <= 256 && dv <= 256 && block_size % 16 == 0 && cache_slots >= 16;
}

// Serves the requests with at least min_rows (token, head of a group) rows; their rows of `out` are written, no others.
OGB_API int ogb_attention_tc_mixed(const OgbAttnLayer* a, const void* q, int q_stride, const void* k_cache, const void* v_cache, const int32_t* cu_seqlens,
                                   const int32_t* past_lens, const int32_t* block_table, int table_cols, int block_size, void* out, int out_stride, int B,
                                   int max_q_len, int min_rows, int cache_slots, int splits, int total_tokens, void* scratch,
                                   long long scratch_bytes, int* status, void* stream_) {
  if (B <= 0 || max_q_len <= 0) return 0;
  if (!(a->joint ? ogb_attention_tc_joint_supported(a->dk, a->dv, block_size, cache_slots) : ogb_attention_tc_mixed_supported(a->dk, a->dv, block_size, cache_slots))) return -5;
  const int maps = a->maps > 1 ? a->maps : 1;
  if (splits < 1) splits = 1;
  if (a->dk % (8 * maps) || a->Hkv * maps > 65535 || (a->Hq / a->Hkv) % maps || (a->raw && (a->sinks || !scratch))) return -1;
  if (a->raw && (long long)splits * total_tokens * a->Hq * (a->dv + 2) * 4 > scratch_bytes) return -2;
  if (a->gate && a->gate_wide && ((a->gate_stride % 8) || (reinterpret_cast<uintptr_t>(a->gate) & 15))) return -1;
  if (a->Hkv <= 0 || a->Hq % a->Hkv || (q_stride % 8) || (out_stride % 8) || a->Hkv > 65535 || B > 65535) return -1;
  if ((reinterpret_cast<uintptr_t>(k_cache) | reinterpret_cast<uintptr_t>(v_cache) | reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(out)) & 15) return -1;
  TcAttnParams p{};
  p.q = static_cast<const __nv_bfloat16*>(q); p.q_stride = q_stride;
  p.cu_seqlens = cu_seqlens; p.past_lens = past_lens; p.block_table = block_table; p.table_cols = table_cols; p.block_size = block_size;
  p.out = static_cast<__nv_bfloat16*>(out); p.out_stride = out_stride;
  p.sinks = a->sinks; p.scale = a->scale; p.softcap = a->softcap; p.window = a->window; p.local = a->chunk;
  p.B = B; p.Hq = a->Hq; p.Hkv = a->Hkv * maps; p.min_rows = min_rows; p.status = status;
  p.joint = a->joint; p.out_scale = a->out_scale;
  if (a->joint && maps > 1) return -1;
  p.dk = a->dk / maps; p.dv = a->dv; p.maps = maps;
  p.gate_wide = a->gate && a->gate_wide;
  if (a->raw) {
    p.splits = splits; p.total_rows = total_tokens * a->Hq;
    p.part_o = static_cast<float*>(scratch);
    p.part_ml = p.part_o + size_t(splits) * p.total_rows * a->dv;
  }
  p.gate = static_cast<const __nv_bfloat16*>(a->gate); p.gate_stride = a->gate_stride;
  cudaStream_t s = static_cast<cudaStream_t>(stream_);
  if (maps == 1 && !a->raw && !a->joint && a->dk == a->dv && (a->dk == 64 || a->dk == 128)) return LaunchTcUniform(p, a->dk, k_cache, v_cache, max_q_len, cache_slots, s);
  if (p.dk <= 64) return LaunchTcMixedKeys<64>(p, k_cache, v_cache, max_q_len, cache_slots, s);
  if (p.dk <= 128) return LaunchTcMixedKeys<128>(p, k_cache, v_cache, max_q_len, cache_slots, s);
  if (p.dk <= 192) return LaunchTcMixedKeys<192>(p, k_cache, v_cache, max_q_len, cache_slots, s);
  if (p.dk <= 256) return LaunchTcMixedKeys<256>(p, k_cache, v_cache, max_q_len, cache_slots, s);
  if (p.dk <= 384) return LaunchTcWideKeys<384>(p, k_cache, v_cache, max_q_len, cache_slots, s);
  if (p.dk <= 512) return LaunchTcWideKeys<512>(p, k_cache, v_cache, max_q_len, cache_slots, s);
  if (p.dk <= 768) return LaunchTcWideKeys<768>(p, k_cache, v_cache, max_q_len, cache_slots, s);
  return LaunchTcWideKeys<1024>(p, k_cache, v_cache, max_q_len, cache_slots, s);
}
