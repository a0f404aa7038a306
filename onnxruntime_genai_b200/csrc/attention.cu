// Paged attention: the launches for heads of 64, 96 and 128 columns, keys and values alike (the kernel is in attention_paged.cuh; heads of
// other widths are in attention_mixed.cu), and the entry points.
#include "attention_paged.cuh"

namespace ogb {

template <int D>
static int LaunchAttention(const AttnParams& p, int max_q_len, cudaStream_t stream) {
  const int G = p.Hq / p.Hkv;
  if (p.kv8) {
    if (max_q_len * G <= 16) return LaunchAttentionMode<D, D, true, true>(p, max_q_len, stream);
    return LaunchAttentionMode<D, D, false, true>(p, max_q_len, stream);
  }
  if (max_q_len * G <= 16) return LaunchAttentionMode<D, D, true>(p, max_q_len, stream);
  return LaunchAttentionMode<D, D, false>(p, max_q_len, stream);
}

int LaunchAttentionUniform(const AttnParams& p, int D, int max_q_len, cudaStream_t stream) {
  switch (D) {
    case 64: return LaunchAttention<64>(p, max_q_len, stream);
    case 96: return LaunchAttention<96>(p, max_q_len, stream);
    case 128: return LaunchAttention<128>(p, max_q_len, stream);
  }
  return -5;
}

}  // namespace ogb

using namespace ogb;

// Bytes of fp32 scratch needed for `splits` > 1.
OGB_API long long ogb_attention_scratch_bytes(int total_tokens, int Hq, int D, int splits) {
  if (splits <= 1) return 0;
  return (long long)splits * total_tokens * Hq * (D + 2) * 4;
}

static int PagedAttention(const void* q, int q_stride, const void* k_cache, const void* v_cache, const int32_t* cu_seqlens,
                          const int32_t* past_lens, const int32_t* block_table, int table_cols, int block_size, void* out,
                          int out_stride, const float* sinks, float scale, float softcap, int window, int B, int total_tokens,
                          int max_q_len, int Hq, int Hkv, int D, int splits, int kv_chunk, void* scratch,
                          long long scratch_bytes, int cache_slots, const int32_t* order, int* status, void* stream_, int kv_bits,
                          int skip_rows = 0) {
  if (B <= 0 || total_tokens <= 0) return 0;
  if (kv_bits != 16 && kv_bits != 8) return -1;
  if (Hkv <= 0 || Hq % Hkv || (q_stride % 8) || (out_stride % 2)) return -1;
  if (splits < 1) splits = 1;
  if (kv_chunk < 0 || (kv_chunk % ATT_BN)) return -1;
  if (splits > 1 && ogb_attention_scratch_bytes(total_tokens, Hq, D, splits) > scratch_bytes) return -2;
  AttnParams p{};
  p.out_scale = 1.f;
  p.chunk = splits > 1 ? kv_chunk : 0;
  p.status = status;
  p.order = order;
  p.kv8 = kv_bits == 8;
  p.skip_rows = skip_rows;
  p.q = static_cast<const __nv_bfloat16*>(q); p.q_stride = q_stride;
  p.k_cache = static_cast<const __nv_bfloat16*>(k_cache); p.v_cache = static_cast<const __nv_bfloat16*>(v_cache);
  p.cu_seqlens = cu_seqlens; p.past_lens = past_lens; p.block_table = block_table; p.table_cols = table_cols;
  p.block_size = block_size; p.out = static_cast<__nv_bfloat16*>(out); p.out_stride = out_stride;
  p.total_rows = total_tokens * Hq;
  p.part_o = static_cast<float*>(scratch);
  p.part_ml = p.part_o ? p.part_o + size_t(splits) * p.total_rows * D : nullptr;
  p.sinks = sinks; p.scale = scale; p.softcap = softcap; p.window = window;
  p.B = B; p.Hq = Hq; p.Hkv = Hkv; p.splits = splits; p.dk = p.dv = D;
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  return LaunchAttentionUniform(p, D, max_q_len, stream);
}

OGB_API int ogb_paged_attention(const void* q, int q_stride, const void* k_cache, const void* v_cache, const int32_t* cu_seqlens,
                                const int32_t* past_lens, const int32_t* block_table, int table_cols, int block_size, void* out,
                                int out_stride, const float* sinks, float scale, float softcap, int window, int B, int total_tokens,
                                int max_q_len, int Hq, int Hkv, int D, int splits, int kv_chunk, void* scratch,
                                long long scratch_bytes, int cache_slots, const int32_t* order, int* status, void* stream_) {
  return PagedAttention(q, q_stride, k_cache, v_cache, cu_seqlens, past_lens, block_table, table_cols, block_size, out, out_stride, sinks,
                        scale, softcap, window, B, total_tokens, max_q_len, Hq, Hkv, D, splits, kv_chunk, scratch, scratch_bytes,
                        cache_slots, order, status, stream_, 16);
}

// Same, leaving the requests with at least `skip_rows` query rows to ogb_attention_tc (their output rows are not written here;
// with splits > 1 the combine pass writes unspecified values there, so the tensor-core launch must come afterwards).
OGB_API int ogb_paged_attention_skip(const void* q, int q_stride, const void* k_cache, const void* v_cache, const int32_t* cu_seqlens,
                                     const int32_t* past_lens, const int32_t* block_table, int table_cols, int block_size, void* out,
                                     int out_stride, const float* sinks, float scale, float softcap, int window, int B, int total_tokens,
                                     int max_q_len, int Hq, int Hkv, int D, int splits, int kv_chunk, void* scratch,
                                     long long scratch_bytes, int cache_slots, const int32_t* order, int* status, void* stream_, int skip_rows) {
  return PagedAttention(q, q_stride, k_cache, v_cache, cu_seqlens, past_lens, block_table, table_cols, block_size, out, out_stride, sinks,
                        scale, softcap, window, B, total_tokens, max_q_len, Hq, Hkv, D, splits, kv_chunk, scratch, scratch_bytes,
                        cache_slots, order, status, stream_, 16, skip_rows);
}

// Same over an 8-bit cache: rows of head_dim int8 values + fp32 scale + 12 bytes of padding (see AttnParams::kv8).
OGB_API int ogb_paged_attention_kv8(const void* q, int q_stride, const void* k_cache, const void* v_cache, const int32_t* cu_seqlens,
                                    const int32_t* past_lens, const int32_t* block_table, int table_cols, int block_size, void* out,
                                    int out_stride, const float* sinks, float scale, float softcap, int window, int B, int total_tokens,
                                    int max_q_len, int Hq, int Hkv, int D, int splits, int kv_chunk, void* scratch,
                                    long long scratch_bytes, int cache_slots, const int32_t* order, int* status, void* stream_) {
  return PagedAttention(q, q_stride, k_cache, v_cache, cu_seqlens, past_lens, block_table, table_cols, block_size, out, out_stride, sinks,
                        scale, softcap, window, B, total_tokens, max_q_len, Hq, Hkv, D, splits, kv_chunk, scratch, scratch_bytes,
                        cache_slots, order, status, stream_, 8);
}

// ------------------------------------------------------------------------------------------------
// Entry point that allocates nothing (see noalloc.h): the split-KV partials live in a fixed array of
// the library's device image instead of caller-provided scratch.
#include "noalloc.h"

static __device__ __align__(256) unsigned char g_noalloc_scratch[OGB_NOALLOC_SCRATCH_BYTES];
// Device address of g_noalloc_scratch per device, resolved on the first call with that device current.
static void* g_noalloc_scratch_addr[16] = {};

OGB_API long long ogb_paged_attention_noalloc_required_bytes(int total_tokens, int Hq, int D, int splits) {
  return ogb_attention_scratch_bytes(total_tokens, Hq, D, splits);
}

OGB_API int ogb_paged_attention_noalloc(const void* q, int q_stride, const void* k_cache, const void* v_cache,
                                        const int32_t* cu_seqlens, const int32_t* past_lens, const int32_t* block_table,
                                        int table_cols, int block_size, void* out, int out_stride, const float* sinks, float scale,
                                        float softcap, int window, int B, int total_tokens, int max_q_len, int Hq, int Hkv, int D,
                                        int splits, void* stream) {
  if (splits < 1) splits = 1;
  const long long need = ogb_attention_scratch_bytes(total_tokens, Hq, D, splits);
  if (need > OGB_NOALLOC_SCRATCH_BYTES) return OGB_ERR_NOALLOC_TOO_LARGE;
  int dev = -1;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 16) return OGB_ERR_NOALLOC_SETUP;
  if (!g_noalloc_scratch_addr[dev]) {
    // In host code `g_noalloc_scratch` names a host-side shadow of the symbol; the kernel needs the
    // address the array has on the current device.
    void* p = nullptr;
    if (cudaGetSymbolAddress(&p, g_noalloc_scratch) != cudaSuccess || !p) return OGB_ERR_NOALLOC_SETUP;
    g_noalloc_scratch_addr[dev] = p;
  }
  return ogb_paged_attention(q, q_stride, k_cache, v_cache, cu_seqlens, past_lens, block_table, table_cols, block_size, out,
                             out_stride, sinks, scale, softcap, window, B, total_tokens, max_q_len, Hq, Hkv, D, splits, 0,
                             g_noalloc_scratch_addr[dev], OGB_NOALLOC_SCRATCH_BYTES, 0, nullptr, nullptr, stream);
}
