// Attention over a paged cache for layers whose heads have sizes of their own (declared stacks): queries and keys of dk columns, values of
// dv columns, an optional gate per head, keys limited to a window or to the query's own run of positions.  Decode rows and short portions:
// the warp-MMA kernel of attention_paged.cuh with rows filled up with zeros to 64, 128, 192 (keys) or 256 columns (heads that are 64, 96 or 128 wide
// throughout take its exact forms).  Long portions are served by attention_tc_mixed.cu, fp32 models and other sizes by attention_simt.cu.
#include "attention_paged.cuh"

namespace ogb {

int LaunchAttentionUniform(const AttnParams& p, int D, int max_q_len, cudaStream_t stream);      // attention.cu

template <int DK, int DV>
static int LaunchMixed(const AttnParams& p, int max_q_len, cudaStream_t stream) {
  if (max_q_len * (p.Hq / p.Hkv) <= 16) return LaunchAttentionMode<DK, DV, true, false, false>(p, max_q_len, stream);
  return LaunchAttentionMode<DK, DV, false, false, false>(p, max_q_len, stream);
}
template <int DK>
static int LaunchMixedKeys(const AttnParams& p, int max_q_len, cudaStream_t stream) {
  if (p.dv <= 64) return LaunchMixed<DK, 64>(p, max_q_len, stream);
  if (p.dv <= 128) return LaunchMixed<DK, 128>(p, max_q_len, stream);
  return LaunchMixed<DK, 256>(p, max_q_len, stream);
}

}  // namespace ogb

using namespace ogb;

OGB_API int ogb_attention_mixed_supported(int dk, int dv) { return dk > 0 && dv > 0 && dk % 8 == 0 && dv % 8 == 0 && dk <= 256 && dv <= 256; }

// skip_rows > 0: requests with at least that many (token, head of a group) rows are left to ogb_attention_tc_mixed.
OGB_API int ogb_attention_mixed(const OgbAttnLayer* a, const void* q, int q_stride, const void* k_cache, const void* v_cache, const int32_t* cu_seqlens,
                                const int32_t* past_lens, const int32_t* block_table, int table_cols, int block_size, void* out, int out_stride, int B,
                                int total_tokens, int max_q_len, int splits, int kv_chunk, void* scratch, long long scratch_bytes, const int32_t* order,
                                int* status, void* stream_, int skip_rows) {
  if (B <= 0 || total_tokens <= 0 || max_q_len <= 0) return 0;
  if (a->joint || !ogb_attention_mixed_supported(a->dk, a->dv)) return -5;
  if (a->Hkv <= 0 || a->Hq % a->Hkv || (q_stride % 8) || (out_stride % 2) || block_size <= 0 || a->Hkv > 65535) return -1;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k_cache) | reinterpret_cast<uintptr_t>(v_cache)) & 15) return -1;
  if (reinterpret_cast<uintptr_t>(out) & 3) return -1;
  if (splits < 1) splits = 1;
  if (kv_chunk < 0 || (kv_chunk % ATT_BN) || (long long)B * splits > 65535) return -1;
  if ((splits > 1 || a->raw) && (long long)splits * total_tokens * a->Hq * (a->dv + 2) * 4 > scratch_bytes) return -2;
  const int maps = a->maps > 1 ? a->maps : 1;
  if (a->dk % (8 * maps) || (a->raw && (a->sinks || !scratch))) return -1;
  AttnParams p{};
  p.q = static_cast<const __nv_bfloat16*>(q); p.q_stride = q_stride;
  p.k_cache = static_cast<const __nv_bfloat16*>(k_cache); p.v_cache = static_cast<const __nv_bfloat16*>(v_cache);
  p.cu_seqlens = cu_seqlens; p.past_lens = past_lens; p.block_table = block_table; p.table_cols = table_cols; p.block_size = block_size;
  p.out = static_cast<__nv_bfloat16*>(out); p.out_stride = out_stride;
  p.total_rows = total_tokens * a->Hq;
  p.part_o = static_cast<float*>(scratch);
  p.part_ml = p.part_o ? p.part_o + size_t(splits) * p.total_rows * a->dv : nullptr;
  p.sinks = a->sinks; p.scale = a->scale; p.softcap = a->softcap; p.window = a->window; p.local = a->chunk;
  p.B = B; p.Hq = a->Hq; p.Hkv = a->Hkv; p.splits = splits; p.chunk = splits > 1 ? kv_chunk : 0;
  p.status = status; p.order = order; p.skip_rows = skip_rows;
  p.dk = a->dk; p.dv = a->dv;
  p.gate = static_cast<const __nv_bfloat16*>(a->gate); p.gate_stride = a->gate_stride; p.gate_wide = a->gate && a->gate_wide;
  p.maps = maps; p.raw = a->raw; p.out_scale = a->out_scale;
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (a->dk == a->dv && (a->dk == 64 || a->dk == 96 || a->dk == 128)) return LaunchAttentionUniform(p, a->dk, max_q_len, stream);
  if (a->dk <= 64) return LaunchMixedKeys<64>(p, max_q_len, stream);
  if (a->dk <= 128) return LaunchMixedKeys<128>(p, max_q_len, stream);
  if (a->dk <= 192) return LaunchMixedKeys<192>(p, max_q_len, stream);
  return LaunchMixedKeys<256>(p, max_q_len, stream);
}
