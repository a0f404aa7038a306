// C entry points of libogb200_kernels.so (sm_100a).  Every launcher takes raw device pointers and
// a CUDA stream (void* = cudaStream_t), launches asynchronously and returns 0 on success or a
// negative code: -1 bad argument / alignment, -2 scratch or tensor-map failure, -3 attribute
// failure, -4 launch failure, -5 unsupported shape.  None of them allocates device memory.
#pragma once
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

// ---- runtime.cu
int ogb_runtime_init(int device);                 // allocates the per-device status word (call outside graph capture)
int* ogb_status_device_ptr(int device);           // device address of the status word
int ogb_status_read_and_clear(int device);        // synchronises the device; returns the OgbStatus code seen since last call
int ogb_sm_count(int device);
const char* ogb_last_cuda_error();

// ---- gemm_tcgen05.cu
int ogb_gemm_token_tile(int M, int dual);
int ogb_gemm_max_active_clusters(int bt, int splits);
int ogb_gemm_auto_splits(int M, int N, int K, int dual, int sm_count);
int ogb_comm_register(int device, int world, int rank, void** buf, void* epoch, long long plane_elems);
int ogb_comm_register_nvls(int device, void* data, void* data_mc, void* out, void* out_mc, void* ctr, void* ctr_mc, void* expected,
                           long long plane_elems);
int ogb_comm_has_nvls(int device);
int ogb_comm_set_options(int use_nvls, long long two_shot_bytes, int p2p_two_hop);   // negative (-2 for the last): leave unchanged
long long ogb_comm_capacity(int device);
// flags: bit 0 fp32 output, bit 1 paired silu(gate)*up epilogue, bit 2 fused tensor-parallel all-reduce,
// bit 3 fused reduce-scatter by token rows (sequence-parallel form), bit 5 the residual is fp32, bit 6 the paired activation is
// max(gate, 0) * up, bits 8 .. 10: 1 + the activation of every output column (0: none; 0 SiLU, 1 GELU(tanh), 2 ReLU, 3 GELU(erf), 4 ReLU^2)
int ogb_gemm_bf16(const void* A, int lda, const void* W, int ldw, void* C, int ldc, int M, int N, int K, const void* bias,
                  const void* residual, int ldr, int flags, int splits, int device, int* status, int sm_count, void* stream);

// Decode-step fusions of ogb_gemm_bf16_fused (all pointers are device pointers).
typedef struct OgbGemmFused {
  float norm_eps;            // > 0: RMS norm folded into the GEMM (row scale rsqrt(mean(x^2) + eps); the weight carries the norm's weight)
  const int32_t* positions;  // != NULL: QKV projection with rotary embedding + KV-cache append in the epilogue
  const int32_t* slots;      // cache row of each token (< 0: not stored)
  const float* cos;          // [max_pos, rot / 2]
  const float* sin;
  void* k_cache;             // bf16 [slots, Hkv, D]
  void* v_cache;
  int Hq, Hkv, D, rot, max_pos;
} OgbGemmFused;
int ogb_gemm_bf16_fused(const void* A, int lda, const void* W, int ldw, void* C, int ldc, int M, int N, int K, const void* bias,
                        const void* residual, int ldr, int flags, int splits, int device, int* status, int sm_count, void* stream,
                        const OgbGemmFused* fused);

// Per-head products over the same rows of A: C[:, z * c_cols + n] = sum_k A[:, z * a_cols + k] * W[z * N + n, k]
int ogb_gemm_bf16_batched(const void* A, int lda, int a_width, int a_cols, const void* W, int ldw, void* C, int ldc, int c_cols, int M, int N,
                          int K, int batch, const void* gate, int ldg, int* status, void* stream);

// ---- gemm_simt.cu: fp32 products and bf16 products TMA cannot address
int ogb_gemm_simt(const void* A, int lda, int a_cols, const void* W, int ldw, void* C, int ldc, int c_cols, int M, int N, int K, int batch,
                  const float* residual, int ldr, const void* bias, int act, int in_fp32, int out_fp32, void* stream);

// Grouped expert product over token rows sorted by expert in plain arithmetic (tile list of ogb_moe_sort, tiles of at most 64 rows).
int ogb_moe_gemm_simt(const void* A, int lda, const void* W, void* C, int ldc, int N, int K, const int32_t* tile_expert, const int32_t* tile_row0,
                      const int32_t* tile_rows, const int32_t* num_tiles, int max_tiles, int token_tile, const int32_t* row_map, int fp32, void* stream);

// ---- layer_ops.cu: fp32 residual stream
// (copy, may be null: the rows as bf16 beside the stream)
int ogb_embedding_stream(const int32_t* ids, const void* table, int table_fp32, float* out, void* copy, int T, int H, int vocab, float scale, void* stream);
// Norm of rows of the fp32 stream x [.., H]: out[i] = norm(x[r]) * w + b, r = rows ? rows[i] : i; w2 (may be null): out2[i] = norm(x[r]) * w2.  RMS norm, or
// layer norm.  y (may be null): y[r] (in the compute type, like out), or (inv_pos not null) the weighted sum of experts' rows sum_j topk_w[r, j] *
// y[inv_pos[r, j]], j < k, is added to the row first, in place where rows is null.
typedef struct OgbNormStream {
  float* x;
  const int32_t* rows;
  const float *w, *b, *w2;
  void *out, *out2;
  const void* y;
  const int32_t* inv_pos; const float* topk_w;
  int ldy, k, n_rows, H, layernorm, fp32;
  float eps;
} OgbNormStream;
int ogb_norm_stream(const OgbNormStream* p, void* stream);
// Head norms, rotation and cache append of an attention layer: proj row t holds Hq query heads and Hkv key heads of key_row columns (the
// first `dim` are the head, the rest zeros) and Hkv value heads of value_row columns.  Queries are replaced in place, keys and values go to
// row slots[t] of the caches (slot < 0: nowhere).  Norm weights fp32 [dim] (null: no norm), cos / sin fp32 [max_pos, rot / 2] (rot 0: none).
// talk (may be null) fp32 [Hq, Hq]: the queries are not replaced; mixed row t [Hq][Hkv][key_row] gets sum over the heads g of key head c's group
// of talk[h, g] * q_g as part c of head h.
int ogb_qkv_prep(void* proj, int ldp, int Hq, int Hkv, int Hv, int dim, int key_row, int value_row, const float* q_norm, const float* k_norm, float eps,
                 const int32_t* positions, const float* cos, const float* sin, int rot, int max_pos, const int32_t* slots, void* k_cache,
                 void* v_cache, int T, const float* talk, void* mixed, int fp32, void* stream);
// h[t] += w * v / sqrt(mean(v^2) + eps), x[t] = h[t] as bf16 (x may be null).  v = y[t], or (inv_pos not null) the weighted sum of the
// experts' rows sum_j topk_w[t, j] * y[inv_pos[t, j]], j < k.
int ogb_add_normed(float* h, const void* y, int ldy, int y_fp32, const float* w, float eps, void* x, const int32_t* inv_pos, const float* topk_w, int k,
                   int T, int H, void* stream);
// Sum into the fp32 stream and tanh norm of the result: n = h_in[r] + v + y2[r] + first[r] + step, h_out[r] = n (h_out may be null, or h_in),
// x[i] = tanh(alpha * n) * w + b, r = rows ? rows[i] : i.  v = y[r] (y may be null), or the weighted sum of experts' rows as above; y, y2 and x
// in the compute type; first (fp32 rows) and step (one fp32 row) may be null.
typedef struct OgbTanhNorm {
  const float* h_in; float* h_out;
  const void* y; const void* y2;
  const int32_t* inv_pos; const float* topk_w;
  const float* first; const float* step;
  const float* w; const float* b;
  void* x; const int32_t* rows;
  int ldy, ldy2, k, n_rows, H, fp32;
  float alpha;
} OgbTanhNorm;
int ogb_add_tanh_norm(const OgbTanhNorm* p, void* stream);
// Token embedding plus a row hashed from (previous token, token): out[t] = table[id] * scale + bigram[(prev * mul_prev + id * mul_cur) mod buckets],
// row `buckets` for a sequence's first token (position 0).  The previous token of a step's first token comes from the paged pool `tokens` [slots]; every
// token of the step is stored there.
typedef struct OgbBigram {
  const int32_t *ids, *slots, *positions, *cu_seqlens, *block_table;
  int32_t* tokens;
  int table_cols, block_size, B, T, H, vocab, buckets, fp32;
  long long mul_prev, mul_cur;
  float scale;
} OgbBigram;
int ogb_embedding_bigram(const OgbBigram* p, const void* table, const void* bigram, float* out, void* stream);
// Expert activations on rows of alternating (gate, up) columns [n, 2 I]: kind 0 silu(g) * u, 1 clamped g * sigmoid(alpha g) * (u + 1);
// on rows [n, I]: kind 2 max(x, 0)^2.
int ogb_expert_act(const void* gu, void* out, long long n, int I, int kind, float alpha, float limit, int fp32, void* stream);
int ogb_act_mul_rows(const void* x, int ldx, void* out, int ldo, int T, int I, int act, int fp32, void* stream);
int ogb_causal_conv_rows(const void* x, int ldx, const void* w, const void* bias, void* cache, int ldcache, const int32_t* slots,
                         const int32_t* positions, const int32_t* cu_seqlens, const int32_t* past_lens, const int32_t* block_table, int table_cols,
                         int block_size, void* out, int T, int B, int C, int L, int silu, int fp32, void* stream);

// ---- recurrent.cu: recurrent mixers over packed sequences (states fp32, at state + slot * slot_stride; a request without a past starts from zero)
// Gated average per column: S <- (1 - sigmoid(z)) S + sigmoid(z) * c(x), c(x) = x + 1/2 for x >= 0, sigmoid(x) below; out = S * silu(g) * scale.
// z, x, g: columns of rows of ld elements, W each.  scratch (may be null) of ogb_min_gru_scratch_bytes: requests of many tokens, T in the step.
int ogb_min_gru(const void* z, const void* x, const void* g, int ld, float* state, long long slot_stride, const int32_t* slots, const int32_t* cu_seqlens,
                const int32_t* past_lens, void* out, int ldo, int T, int B, int W, float scale, int max_q_len, void* scratch, long long scratch_bytes, int fp32,
                void* stream);
long long ogb_min_gru_scratch_bytes(int T, int B, int W);
// Matrix memories of H heads with keys of d and values of dv columns.  q, k, v, g: columns of rows of ld elements ([H, d], [H, d], [H, dv], [H, dv]); gates:
// fp32 rows of ldg, H logits of the input gates and H of the forget gates, to which gate_b [2 H] is added; out rows of ldo.  State of a slot: memories
// [H, d, dv], normalisers [H, d], maxima [H].  max_q_len: the most tokens a request of the step feeds, T the step's tokens.  long_tokens > 0 (bf16):
// requests with at least that many tokens run in the chunk form, in ogb_mlstm_scratch_bytes of scratch (0: these sizes have none); all_long: no request of the
// step has fewer.
typedef struct OgbMlstm {
  const void *q, *k, *v, *g;
  const float *gates, *gate_b, *norm_w;
  void* out;
  float* state;
  const int32_t *slots, *cu_seqlens, *past_lens;
  long long slot_stride;
  int ld, ldg, ldo, B, H, d, dv, T, max_q_len, fp32, long_tokens, all_long;
  float cap, eps;
  void* scratch;
  long long scratch_bytes;
} OgbMlstm;
long long ogb_mlstm_scratch_bytes(int T, int B, int H, int d, int dv);
int ogb_mlstm(const OgbMlstm* a, void* stream);

// ---- attention_tc.cu, latent form (long prompts over expanded keys and values)
int ogb_attention_tc_latent_supported(int dim, int rot, int vdim);
int ogb_attention_tc_latent(const void* q, int q_stride, const void* kv, int ldkv, const void* kr, int ldkr, int kr_col, int rows,
                            const int32_t* cu_seqlens, const int32_t* past_lens, const int32_t* row_base, const int32_t* first_kv, void* out,
                            int out_stride, float scale, int window, const float* sinks, const void* gate, int gate_stride, int B, int max_q_len,
                            int H, int dim, int rot, int vdim, int* status, void* stream);

// ---- attention_mixed.cu, attention_tc_mixed.cu, attention_simt.cu: attention layers with sizes of their own.  Hq query heads over Hkv key /
// value heads (q rows: Hq heads of dk columns first; caches [slots, Hkv, dk] and [slots, Hkv, dv]; out rows: Hq heads of dv columns).
// window > 0: position p sees (p - window, p]; chunk > 0: the keys of p's own run of `chunk` positions; 0: every earlier key.
// sinks (may be null) [Hq]: a logit in each head's denominator.  gate (may be null) [tokens, gate_stride], in the model's element type: a
// head's output is multiplied by the sigmoid of its entry (gate_wide: a row holds Hq * dv entries, one for every output column).
// joint: dk counts the columns of all key heads of a position (caches [slots, dk] and [slots, Hkv, dv]); every query is that wide and meets all of
// them.  The result is multiplied by out_scale (not in raw calls).
// softcap > 0: a scaled score s becomes softcap * tanh(s / softcap).  maps > 1: query vector h belongs to map h % maps, is dk / maps columns
// wide and meets only that map's columns of its key head (Hq counts query vectors, a key head holds the vectors of all maps side by side).
// raw: instead of `out`, fp32 partial results go to scratch: [splits, tokens * Hq, dv] sums and, behind them, [splits, tokens * Hq, 2] (maximum
// in log2 units, sum of the weights); ogb_attention_diff_merge reads them.
typedef struct OgbAttnLayer {
  int Hq, Hkv, dk, dv, window, chunk, gate_stride;
  float scale;
  const float* sinks;
  const void* gate;
  int gate_wide, maps, raw;
  float softcap;
  int joint;
  float out_scale;
} OgbAttnLayer;
// Differential attention on raw partial results of H heads with two maps each (query vectors 2 h and 2 h + 1): with a1 and a2 the maps'
// results, o = a1 - lambda * a2, out = o / sqrt(mean(o^2) + eps) * post over the head's first vdim columns (columns vdim .. dv - 1 are zeros),
// times the sigmoid of gate [T, H * dv] (may be null).
int ogb_attention_diff_merge(const float* part, int splits, int T, int part_tokens, int H, int dv, int vdim, float lambda, float post, float eps,
                             const void* gate, int gate_stride, void* out, int out_stride, int fp32, void* stream);
int ogb_attention_mixed_supported(int dk, int dv);
int ogb_attention_mixed(const OgbAttnLayer* a, const void* q, int q_stride, const void* k_cache, const void* v_cache, const int32_t* cu_seqlens,
                        const int32_t* past_lens, const int32_t* block_table, int table_cols, int block_size, void* out, int out_stride, int B,
                        int total_tokens, int max_q_len, int splits, int kv_chunk, void* scratch, long long scratch_bytes, const int32_t* order,
                        int* status, void* stream, int skip_rows);
// attention_joint.cu: joint layers, decode steps and short portions
int ogb_attention_joint_supported(int dk, int v_cols);
int ogb_attention_joint(const OgbAttnLayer* l, const void* q, int q_stride, const void* k_cache, const void* v_cache, const int32_t* cu_seqlens,
                        const int32_t* past_lens, const int32_t* block_table, int table_cols, int block_size, void* out, int out_stride, int B,
                        int total_tokens, int max_q_len, int splits, void* scratch, long long scratch_bytes, const int32_t* order, int* status,
                        void* stream, int skip_rows);
int ogb_attention_tc_mixed_supported(int dk, int dv, int block_size, int cache_slots);
int ogb_attention_tc_joint_supported(int dk, int dv, int block_size, int cache_slots);
int ogb_attention_tc_mixed(const OgbAttnLayer* a, const void* q, int q_stride, const void* k_cache, const void* v_cache, const int32_t* cu_seqlens,
                           const int32_t* past_lens, const int32_t* block_table, int table_cols, int block_size, void* out, int out_stride, int B,
                           int max_q_len, int min_rows, int cache_slots, int splits, int total_tokens, void* scratch, long long scratch_bytes,
                           int* status, void* stream);
int ogb_attention_simt(const OgbAttnLayer* a, const void* q, int q_stride, const void* k_cache, const void* v_cache, const int32_t* cu_seqlens,
                       const int32_t* past_lens, const int32_t* block_table, int table_cols, int block_size, void* out, int out_stride, int B, int T,
                       void* scratch, long long scratch_bytes, int fp32, void* stream);

// ---- latent_attention.cu: attention over a paged cache of latent rows [c (R) | rotated key (rot)]
typedef struct OgbLatentShape { int H, dim, rot, vdim, R, rot_dims; } OgbLatentShape;
// q (may be null) [T, H * (dim | rot)]: the rotary parts are rotated in place; down (may be null) [T, R | rot]: normed and rotated into the cache;
// cq (may be null) [T, q_rank]: RMS-normed in place with weight cq_w.
int ogb_latent_prep(void* q, int ldq, const void* down, int ldd, void* cq, int ldcq, int q_rank, const float* cq_w, const OgbLatentShape* sh,
                    const float* norm_w, float eps, const int32_t* positions, const float* cos, const float* sin, int max_pos, const int32_t* slots,
                    void* cache, int ldcache, int T, int fp32, void* stream);
// out[t, i] *= sigmoid(gate[t, i]), i < n
int ogb_gate_rows(void* out, int ldo, const void* gate, int ldg, int T, int n, int fp32, void* stream);
int ogb_latent_mma_supported(const OgbLatentShape* sh);
int ogb_latent_rows_per_tile(int H, int max_q_len);
long long ogb_latent_scratch_bytes(int total_rows, int R, int splits);
int ogb_latent_attention(const void* qlat, const void* proj, int ldp, const OgbLatentShape* sh, const void* cache, int ldcache,
                         const int32_t* cu_seqlens, const int32_t* past_lens, const int32_t* block_table, int table_cols, int block_size,
                         void* out, float scale, int window, const float* sinks, int B, int T, int max_q_len, int skip_q_len, int splits,
                         void* scratch, long long scratch_bytes, const int32_t* order, int* status, void* stream);
int ogb_latent_attention_simt(const void* qlat, const void* proj, int ldp, const OgbLatentShape* sh, const void* cache, int ldcache,
                              const int32_t* cu_seqlens, const int32_t* past_lens, const int32_t* block_table, int table_cols, int block_size,
                              void* out, float scale, int window, const float* sinks, int B, int T, int skip_q_len, int fp32, void* stream);
int ogb_latent_gather(const void* cache, int ldcache, const int32_t* block_table, int table_cols, int block_size, const int32_t* row_base,
                      const int32_t* first_kv, const int32_t* kv_len, const int32_t* req, int n_req, int rows, int width, void* out, int ldo,
                      void* stream);

// Grouped expert GEMM over token rows sorted by expert (tile list from ogb_moe_sort); act_kind 1 = silu(gate)*up,
// 2 = clamped SwiGLU(alpha, limit); flags as above (bit 2 unused).
int ogb_moe_gemm(const void* A, int lda, const void* W, int ldw, void* C, int ldc, int rows_total, int N, int K, int experts,
                 const void* bias, int flags, int act_kind, float act_alpha, float act_limit, const int* tile_expert,
                 const int* tile_row0, const int* tile_rows, const int* num_tiles, int max_tiles, int token_tile, int* status,
                 void* stream);

// ---- collectives.cu: mode 0 all-reduce, 1 all-gather, 2 reduce-scatter over the registered symmetric buffers (bf16)
int ogb_collective(int mode, const void* in, void* out, const void* residual, long long n, int device, int* status, int sm_count,
                   void* stream);

// ---- moe.cu
// shared: row t gets one more entry, expert E with weight 1 (rows of k + 1).
int ogb_moe_topk(const float* logits, int ld, int T, int E, int k, int mode, int shared, int32_t* topk_idx, float* topk_w, void* stream);
int ogb_moe_max_tiles(int n, int experts, int bt);
int ogb_moe_fp4_reads_row_map(int token_tile, int K, int half);
int ogb_moe_sort(const int32_t* topk_idx, int T, int k, int E, int e_lo, int e_hi, int bt, int32_t* expert_offsets,
                 int32_t* sorted_token, int32_t* inv_pos, int32_t* tile_expert, int32_t* tile_row0, int32_t* tile_rows,
                 int32_t* num_tiles, int max_tiles, void* stream);
int ogb_moe_combine(const void* y, int ldy, const int32_t* inv_pos, const float* topk_w, int T, int k, int H, const void* residual,
                    int ldr, void* out, int ldo, void* stream);

// ---- gemm_w4.cu (int4 block-32 weights, repacked by ops.pack_w4)
long long ogb_w4_packed_bytes(int N, int K);
int ogb_gemm_w4(const void* A, int lda, const void* Wpacked, void* C, int ldc, int M, int N, int K, const void* bias,
                const void* residual, int ldr, int flags, int splits, int* status, int sm_count, void* stream);

// ---- gemm_fp4.cu (MXFP4 experts kept packed: e2m1 codes + e8m0 block scales, repacked by ops/fp4.py)
long long ogb_fp4_packed_bytes(int experts, int N, int K);
int ogb_moe_gemm_fp4(const void* A, int lda, const void* Wpacked, void* C, int ldc, int rows_total, int N, int K, int experts,
                     const void* bias, int flags, int act_kind, float act_alpha, float act_limit, const int* tile_expert,
                     const int* tile_row0, const int* tile_rows, const int* num_tiles, int max_tiles, int token_tile,
                     int max_rows_per_tile, const int32_t* row_map, int* status, void* stream);

// ---- elementwise.cu
int ogb_embedding(const int32_t* ids, const void* table, void* out, int T, int H, int vocab, float scale, void* stream);
int ogb_norm(const void* x, const void* residual_in, void* residual_out, const void* weight, const void* bias, void* out,
             int rows, int H, float eps, int layernorm, void* stream);
int ogb_norm_moe_combine(const void* y, int ldy, const int32_t* inv_pos, const float* topk_w, int k, const void* residual_in, void* residual_out,
                         const void* weight, const void* bias, void* out, int rows, int H, float eps, int layernorm, void* stream);
int ogb_rope_kv_append(void* qkv, int qkv_stride, const int32_t* positions, const int32_t* slots, const float* cos_cache,
                       const float* sin_cache, void* k_cache, void* v_cache, const void* q_norm_w, const void* k_norm_w,
                       float norm_eps, int T, int Hq, int Hkv, int D, int rot, int interleaved, int max_pos, void* stream);
int ogb_rope_kv_append_bits(void* qkv, int qkv_stride, const int32_t* positions, const int32_t* slots, const float* cos_cache,
                       const float* sin_cache, void* k_cache, void* v_cache, const void* q_norm_w, const void* k_norm_w,
                       float norm_eps, int T, int Hq, int Hkv, int D, int rot, int interleaved, int max_pos, int kv_bits, const int32_t* positions3, int sec0, int sec1, void* stream);
int ogb_embedding_q4(const int32_t* ids, const void* q, const void* scales, const void* zps, void* out, int T, int K, int vocab,
                     float mult, void* stream);
int ogb_act_mul(const void* x, void* out, int T, int I, int act, void* stream);
int ogb_act(const void* x, void* out, long long n, int act, void* stream);
int ogb_causal_conv(const void* x, int x_stride, const void* weight, const void* bias, void* cache, const int32_t* slots,
                    const int32_t* positions, const int32_t* cu_seqlens, const int32_t* past_lens, const int32_t* block_table,
                    int table_cols, int block_size, void* out, int T, int B, int C, int L, int cache_stride, int silu, void* stream);
int ogb_short_conv(const void* bcx, int bcx_stride, const void* weight, const void* bias, void* cache, const int32_t* slots,
                   const int32_t* positions, const int32_t* cu_seqlens, const int32_t* past_lens, const int32_t* block_table,
                   int table_cols, int block_size, void* out, int T, int B, int C, int L, void* stream);
int ogb_decode_advance(const int32_t* sampled, int32_t* input_ids, int32_t* positions, int32_t* past_lens, int32_t* slot_mapping,
                       int32_t* sample_pos, const int32_t* block_table, int table_cols, int block_size, int B, void* stream);
int ogb_logits_edit(float* logits, int vocab, const int32_t* rows, const int32_t* tokens, const int32_t* ops,
                    const float* values, int n, void* stream);
int ogb_logits_bitmask(float* logits, int rows, int vocab, const uint32_t* mask, const int32_t* mask_rows, void* stream);
int ogb_bf16_to_f32(const void* in, float* out, long long n, void* stream);
int ogb_gather_rows(const void* in, const int32_t* rows, void* out, int n_rows, int row_bytes, void* stream);
int ogb_gather_rows_f16(const void* in, const int32_t* rows, void* out, int n_rows, int row_bytes, void* stream);  // bf16 -> fp16

// ---- linear_attention.cu: gated delta rule over packed sequences; state [slots, Hv, dk, dv] fp32 updated in place
int ogb_gated_delta_fused(const void* conv, long long conv_stride, long long q_off, long long k_off, long long v_off, const void* ba,
                          long long ba_stride, long long b_off, long long a_off, const float* neg_exp_a, const float* dt_bias,
                          float q_scale, float l2_eps, float* state, long long slot_stride, const int32_t* slots, const int32_t* cu_seqlens,
                          const int32_t* past_lens, void* out, int B, int Hk, int Hv, int dk, int dv, int max_q_len, int fp32, void* stream);
int ogb_gdn_gate_norm(const void* o, const void* z, long long z_stride, const float* w, float eps, void* out, long long out_stride, int T, int Hv,
                      int dv, int fp32, void* stream);
int ogb_gated_delta(const void* q, const void* k, const void* v, const float* g, const float* beta, float* state, const int32_t* slots,
                    const int32_t* cu_seqlens, const int32_t* past_lens, void* out, int B, int Hk, int Hv, int dk, int dv, int max_q_len, void* stream);
int ogb_mamba2_scan_fused(const void* conv, long long conv_stride, const void* dt_raw, long long dt_stride, const float* dt_bias, const float* neg_a,
                          const float* Dv, float* state, const int32_t* slots, const int32_t* cu_seqlens, const int32_t* past_lens, void* out, int B,
                          int heads, int groups, int P, int N, void* stream);
int ogb_mamba_gate_norm(const void* y, const void* z, long long z_stride, const float* w, float eps, void* out, int T, int I, void* stream);
int ogb_mamba2_scan(const void* x, const float* dt, const float* neg_a, const void* Bm, const void* Cm, const float* Dv, float* state,
                    const int32_t* slots, const int32_t* cu_seqlens, const int32_t* past_lens, void* out, int B, int heads, int groups, int P, int N,
                    void* stream);
int ogb_copy_state_slots(const float* src, float* dst, int layers, int slots, long long slot_elems, const int32_t* src_slots,
                         const int32_t* dst_slots, int count, void* stream);

// ---- attention.cu
long long ogb_attention_scratch_bytes(int total_tokens, int Hq, int D, int splits);
// cache_slots (rows of the key / value cache) and status (device status word) enable the TMA-fed K/V path; 0 / null keep
// the cp.async path.  order: optional [B] permutation of the requests in which the CTAs are issued (longest first balances
// a batch of mixed lengths).  splits > 1 divides a request's keys between CTAs: evenly (kv_chunk 0) or in fixed ranges of kv_chunk keys (multiple of 64).
int ogb_paged_attention(const void* q, int q_stride, const void* k_cache, const void* v_cache, const int32_t* cu_seqlens,
                        const int32_t* past_lens, const int32_t* block_table, int table_cols, int block_size, void* out,
                        int out_stride, const float* sinks, float scale, float softcap, int window, int B, int total_tokens,
                        int max_q_len, int Hq, int Hkv, int D, int splits, int kv_chunk, void* scratch, long long scratch_bytes,
                        int cache_slots, const int32_t* order, int* status, void* stream);
// attention_tc.cu: tcgen05 prefill attention for the requests of a launch with at least `min_rows` query rows (bf16 cache,
// head_dim 64 / 128, cache blocks of a multiple of 16 tokens); ogb_paged_attention_skip serves the others.
int ogb_attention_tc_supported(int D, int block_size, int kv_bits, int cache_slots);
int ogb_attention_tc(const void* q, int q_stride, const void* k_cache, const void* v_cache, const int32_t* cu_seqlens,
                     const int32_t* past_lens, const int32_t* block_table, int table_cols, int block_size, void* out, int out_stride,
                     const float* sinks, float scale, float softcap, int window, int B, int max_q_len, int Hq, int Hkv, int D,
                     int min_rows, int cache_slots, int* status, void* stream);
int ogb_paged_attention_skip(const void* q, int q_stride, const void* k_cache, const void* v_cache, const int32_t* cu_seqlens,
                             const int32_t* past_lens, const int32_t* block_table, int table_cols, int block_size, void* out,
                             int out_stride, const float* sinks, float scale, float softcap, int window, int B, int total_tokens,
                             int max_q_len, int Hq, int Hkv, int D, int splits, int kv_chunk, void* scratch,
                             long long scratch_bytes, int cache_slots, const int32_t* order, int* status, void* stream, int skip_rows);
int ogb_paged_attention_kv8(const void* q, int q_stride, const void* k_cache, const void* v_cache, const int32_t* cu_seqlens,
                        const int32_t* past_lens, const int32_t* block_table, int table_cols, int block_size, void* out,
                        int out_stride, const float* sinks, float scale, float softcap, int window, int B, int total_tokens,
                        int max_q_len, int Hq, int Hkv, int D, int splits, int kv_chunk, void* scratch, long long scratch_bytes,
                        int cache_slots, const int32_t* order, int* status, void* stream);

// ---- sampling.cu
int ogb_sample(const float* logits, long long row_stride, int rows, int vocab, const int32_t* top_k, const float* top_p,
               const float* temperature, const unsigned long long* seeds, const int32_t* positions, int32_t* out, void* stream);
int ogb_argmax(const float* logits, long long row_stride, int rows, int vocab, int32_t* out, void* stream);
int ogb_topk(const float* x, long long row_stride, int rows, int n, int k, int mode, const float* add, float* out_vals,
             int32_t* out_idx, void* stream);
int ogb_beam_merge(const float* in_vals, const int32_t* in_idx, int batch, int beams, int cand, float* out_scores,
                   int32_t* out_tokens, int32_t* out_beams, void* stream);
// Beam scorer + sequence append on the device (beam_scorer.cu)
int ogb_beam_scorer_step(const float* cand_scores, const int32_t* cand_tokens, const int32_t* cand_beams, void* seq0, void* seq1, int cur, int len,
                         void* scores, void* hyp_tokens, void* hyp_len, void* hyp_score, void* hyp_order, void* hyp_count, void* done, void* out,
                         int batch, int num_beams, int max_length, int pad_token, int early_stopping, float length_penalty, const int32_t* eos,
                         int n_eos, void* stream);
int ogb_beam_scorer_finalize(void* seq0, void* seq1, int cur, int len, void* scores, void* hyp_tokens, void* hyp_len, void* hyp_score,
                             void* hyp_order, void* hyp_count, void* done, void* out, int batch, int num_beams, int max_length, int pad_token,
                             int early_stopping, float length_penalty, const int32_t* eos, int n_eos, void* stream);
int ogb_verify_sampled(const float* logits, long long row_stride, int vocab, int K, const int32_t* top_k, const float* top_p,
                       const float* temperature, const unsigned long long* seeds, const int32_t* positions, const int32_t* draft,
                       const int32_t* q_idx, const float* q_prob, const int32_t* q_n, int q_stride, int32_t* scratch,
                       float* accept_prob, int32_t* accepted, int32_t* commit, int32_t* status, void* stream);
int ogb_verify_greedy(const int32_t* draft, const int32_t* target_argmax, int k, int32_t* accepted, int32_t* commit, void* stream);

#ifdef __cplusplus
}
#endif
