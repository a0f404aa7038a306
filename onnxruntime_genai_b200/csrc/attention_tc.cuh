// Prefill attention on the 5th-generation tensor cores: Q K^T and P V are tcgen05.mma instructions with the score tile S and
// the output tile O in tensor memory, K/V tiles arrive through the block table as TMA boxes, and four warps run the online
// softmax with one thread per query row (a TMEM lane), so row maxima and sums need no shuffles.
//
// Same semantics as paged_attention_kernel (attention.cu: packed variable-length queries over a block-table cache, GQA rows
// (token, head of the group) sharing one K/V stream, causal / sliding-window / bidirectional masks, sinks, soft-capping;
// reference ops: GroupQueryAttention / PagedAttention, src/python/py/models/builders/base.py:3315-3386, 3484-3536).  It serves
// the requests of a launch that have at least TCA_MIN_ROWS query rows; the other requests (decode rows, short verify rows) are
// left to the bandwidth-bound kernel, which skips the ones taken here.
//
// One CTA = (request, kv head, 128 query rows).  Roles:
//   warps 0-7  softmax: a row (TMEM lane) is shared by two threads, one per half of the tile's key columns (warp w serves the
//              lane quarter w % 4, which is the only one it may address, and column half w / 4).  Per K/V tile: read S from TMEM,
//              scale / soft-cap / mask, row maximum (the two halves meet through shared memory), exponentials, bf16 P written
//              over S in TMEM (the A operand of P V is read from tensor memory), rescale O in TMEM when the maximum moved.
//   warps 8,9  TMA producers of the K ring and of the V ring: per 16 keys and 64 dims one box (the cache as a 2-D tensor
//              [slots, kv_heads * head_dim], 128-byte swizzle); the lanes look their blocks up in parallel.
//   warp 10    MMA issuer (one lane): S[b] = Q K_j^T into one of three S buffers, two tiles ahead of the softmax warps;
//              O += P_j V_j with V as the MN-major B operand (keys are its K dimension) as soon as P_j is there.
// The softmax loop is plain (read S, mask, maximum, exchange, exponentials, P back into TMEM): a software-pipelined form
// (exponentials of tile j interleaved with the load and maximum of tile j + 1) measured slower, 457 against 591 TFLOP/s at 4096
// tokens, because its loop body outgrew the instruction cache and its extra waits cost more than the overlap gave.  The scale is
// folded into the exponent's multiply-add.  Registers move from the producer / issuer warps to the softmax warps (setmaxnreg).
// Row tiles are dispatched from the end of the prompt (most keys) to its start, so the grid's tail is short CTAs (591 -> 658).
//
// Every wait on an mbarrier is bounded (mbar_wait_bounded); a wait that runs out sets the CTA's abort flag and the device status
// word; the producers and the issuer leave their loops, the softmax warps keep walking theirs without waiting (they share a
// named barrier per warp pair, which has no time limit, so none of them may leave early), the producer waits (bounded) for
// copies in flight, TMEM is freed and the kernel returns.
// The latent form (LAT) serves long prompts of latent-attention layers: keys and values of the request's visible positions were
// expanded into dense matrices beforehand ([rows, H * dim] and [rows, H * vdim] column ranges of one product, and the rotated key
// part that all heads share as columns of the gathered latents), so a row of K is put together from two tensor maps (the head's
// unrotated part, then the shared rotated part, each padded to 64 columns that meet zeros in Q), and key position j of request b
// is dense row row_base[b] + j - first_kv[b] instead of a block-table lookup.  Every head has keys of its own: one CTA = (request,
// head, 128 tokens).
// The cache must hold finite values in every slot of a block that is in use (PagedKVCache allocates zeros): keys past the end
// of a request inside its last 16-key group are masked (P = 0) but still multiplied.
#pragma once
#include <cstdlib>
#include <cstring>

#include "common.cuh"
#include "kernels.h"

namespace ogb {

bool MakeMapBf16(CUtensorMap* out, const void* ptr, int rows, int cols, int ld, int box_rows);  // gemm_tcgen05.cu

constexpr int TCA_BM = 128;
constexpr int TCA_SOFTMAX_THREADS = 256;
constexpr int TCA_THREADS = TCA_SOFTMAX_THREADS + 128;      // warps 8..11: K producer, V producer, MMA issuer, one spare
constexpr int TCA_K_WARP = 8, TCA_V_WARP = 9, TCA_MMA_WARP = 10;
constexpr int TCA_REGS_SOFTMAX = 224, TCA_REGS_OTHER = 40;   // after setmaxnreg: 256 x 224 + 128 x 40 registers
constexpr float TCA_LOG2E = 1.4426950408889634f;
constexpr float TCA_RESCALE_GAP = 8.f;   // log2 units

// Latent form: where a request's expanded rows start, and how a head's columns are laid out (see LAT above).
struct TcLatent {
  const int32_t *row_base, *first_kv;      // per request of the batch; row_base < 0: the request is not served here
  int dim, rot, vdim;                      // a query head is (dim | rot) columns of q
  int kr_col;                              // column of the shared rotated part in its matrix
};

struct TcAttnParams {
  const __nv_bfloat16* q; int q_stride;
  const int32_t* cu_seqlens; const int32_t* past_lens;
  const int32_t* block_table; int table_cols; int block_size;
  __nv_bfloat16* out; int out_stride;
  const float* sinks;
  float scale, softcap;
  int window, B, Hq, Hkv, min_rows;
  int* status;
  TcLatent lat;
  int dk, dv;        // columns of a key (query) head and of a value head (MIX)
  int local;         // > 0: a query sees the keys of its own run of `local` positions only (runs are counted from position 0)
  const __nv_bfloat16* gate; int gate_stride;      // (may be null) [tokens, Hq]: a head's output is multiplied by the sigmoid of its entry
  int gate_wide;     // gate [tokens, Hq * dv]: one entry per output column
  // maps > 1 (MIX): Hkv counts the key vectors of all maps; key vector v meets the query vectors h of its group with h % maps == v % maps and
  // the value head v / maps.
  int maps;
  // part_o (may be null; MIX): instead of `out`, sums [total_rows, dv], and (maximum, sum of weights) in part_ml [splits, total_rows, 2], whose
  // entries of the other splits are marked empty.
  float *part_o, *part_ml;
  int splits, total_rows;
  int joint;         // (MIX) one key of dk columns per cache row, which every query head meets; values by key head
  float out_scale;   // multiplies the result
};
// entry of a query row in a grid of key vectors
__device__ __forceinline__ int tca_query(int kvh, int i, int G, int maps) { return maps > 1 ? ((kvh / maps) * G + i) * maps + kvh % maps : kvh * G + i; }

// KC: key columns of a ring slot (DK, or a part of it where whole tiles of wide keys would not fit twice beside the queries).  QR: query rows of a tile, 128, or
// 64 where 128 rows of queries would not leave room for the rings: the lower half of the accumulators then belongs to no row (as operand rows 64 .. 127
// the MMA reads whatever follows 64 rows in shared memory; rows do not mix).
template <int DK, int DV, int BN, int KC = DK, int QR = TCA_BM>
struct TcaCfg {
  static constexpr int K_PARTS = DK / KC, K_HALVES = KC / 64, V_HALVES = DV / 64;
  static_assert(DK % KC == 0 && (QR == 64 || QR == TCA_BM), "a key row is whole parts");
  static constexpr int Q_BYTES = QR * DK * 2, Q_HALF = QR * 128;      // 64 columns of the rows
  static constexpr int K_TILE = BN * KC * 2, V_TILE = BN * DV * 2;
  // K and V tiles have rings of their own: a K tile is free as soon as its Q K^T is done (one tile period earlier than the
  // V tile of the same keys), and the loads must run two to three tile periods ahead of their use to hide their latency.
  static constexpr int BUDGET = 227 * 1024 - 1024 - 1536 - Q_BYTES;      // 1 KiB of alignment slack, static shared memory
  static constexpr int PAIRS = K_PARTS > 1 ? 2 : (BUDGET / (K_TILE + V_TILE) >= 4 ? 4 : BUDGET / (K_TILE + V_TILE));
  static constexpr int V_STAGES = PAIRS;
  static constexpr int K_STAGES = K_PARTS > 1 ? (BUDGET - 2 * V_TILE) / K_TILE
                                              : (PAIRS < 4 && BUDGET - PAIRS * (K_TILE + V_TILE) >= K_TILE ? PAIRS + 1 : PAIRS);
  static_assert(PAIRS >= 2 && K_STAGES >= 2, "the rings need two stages each");
  static constexpr int SMEM = 1024 + Q_BYTES + K_STAGES * K_TILE + V_STAGES * V_TILE;
  static constexpr int S_BUFS = 3;
  static constexpr int S_COLS = BN, O_COL = S_BUFS * BN;
  static constexpr int COLS_USED = S_BUFS * BN + DV;
  static_assert(COLS_USED <= 512, "scores and output must fit in tensor memory");
  static constexpr int TMEM_COLS = COLS_USED <= 128 ? 128 : (COLS_USED <= 256 ? 256 : 512);
  static constexpr int CTAS_PER_SM = 1;
};

// MN-major operand with the 128-byte swizzle: 64 contiguous elements per 128-byte row, rows are K indices; 8-row groups along
// K are `sbo` bytes apart, 64-element groups along MN are `lbo` bytes apart.
__device__ __forceinline__ uint64_t umma_desc_sw128_mn(uint32_t smem_addr, uint32_t lbo, uint32_t sbo) {
  uint64_t d = 0;
  d |= uint64_t((smem_addr & 0x3FFFF) >> 4);
  d |= uint64_t((lbo >> 4) & 0x3FFF) << 16;
  d |= uint64_t((sbo >> 4) & 0x3FFF) << 32;
  d |= uint64_t(1) << 46;
  d |= uint64_t(2) << 61;
  return d;
}

__device__ __forceinline__ void tmem_st16(uint32_t taddr, const uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};"
      ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]),
        "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
      : "memory");
}
// D[tmem] (+)= A[tmem] * B[smem desc]: A is 128 lanes x K values, two 16-bit values per 32-bit column.
__device__ __forceinline__ void umma_f16_ta(uint32_t tmem_d, uint32_t tmem_a, uint64_t desc_b, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}"
      ::"r"(tmem_d), "r"(tmem_a), "l"(desc_b), "r"(idesc), "r"(accumulate)
      : "memory");
}
__device__ __forceinline__ void tmem_st_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ void fence_proxy_async_smem() { asm volatile("fence.proxy.async.shared::cta;" ::: "memory"); }

// DK: width of the staged query and key rows; DV: width of the value rows; LAT: the latent form, whose first NOPE of the DK columns
// are the unrotated part; MIX: heads of p.dk and p.dv columns (multiples of 8).  The boxes of a head narrower than the staged rows reach
// into the next head's columns, which meet zeros in Q (keys) or give output columns that are not stored (values).  CAP: scores are soft-capped
// (a kernel of its own: the loop body of the others has to stay within the instruction cache).
template <int DK, int DV, int BN, bool LAT = false, int NOPE = DK, bool MIX = false, bool CAP = false, int KC = DK, int QR = TCA_BM>
__global__ void __launch_bounds__(TCA_THREADS, TcaCfg<DK, DV, BN, KC, QR>::CTAS_PER_SM)
attention_tc_kernel(const __grid_constant__ CUtensorMap tmap_k, const __grid_constant__ CUtensorMap tmap_v, const __grid_constant__ CUtensorMap tmap_r,
                    TcAttnParams p) {
  using Cfg = TcaCfg<DK, DV, BN, KC, QR>;
  static_assert(KC == DK || (MIX && !LAT), "keys in parts: only layers with sizes of their own");
  constexpr int KS = Cfg::K_STAGES, VS = Cfg::V_STAGES;
  extern __shared__ __align__(128) uint8_t smem_dyn[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_dyn) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = smem;                                  // [HALVES][QR rows][128 B]
  uint8_t* sK = sQ + Cfg::Q_BYTES;                     // [KS][HALVES][BN keys][128 B]
  uint8_t* sV = sK + KS * Cfg::K_TILE;                 // [VS][HALVES][BN keys][128 B]
  __shared__ uint64_t k_full[KS], k_empty[KS], v_full[VS], v_empty[VS], s_full[Cfg::S_BUFS], p_full[Cfg::S_BUFS], o_done[Cfg::S_BUFS], q_full;
  __shared__ uint32_t tmem_slot;
  __shared__ int abort_flag;
  // Row maxima of the two column halves, [tile parity][half][row] as bf16 (rounded up: a reference maximum only has to be
  // the same on both sides and not below the true one); at the end the same bytes carry the halves' sums as [half][row] fp32.
  __shared__ __align__(16) __nv_bfloat16 xchg[2][2][TCA_BM];

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  pdl_wait();
  const int kvh = blockIdx.y, b = blockIdx.z;
  const int G = p.Hq / p.Hkv;
  const int tok0 = p.cu_seqlens[b];
  const int q_len = p.cu_seqlens[b + 1] - tok0;
  const int rows = q_len * G;
  // CTAs are dispatched in block-index order: the last row tiles of a causal prompt see the most keys, so they go first and
  // the tail of the grid is made of short CTAs
  const int row0 = int(gridDim.x - 1 - blockIdx.x) * QR;
  if (rows * (MIX ? p.maps : 1) < p.min_rows || row0 >= rows) return;      // before anything is allocated
  if (LAT && p.lat.row_base[b] < 0) return;
  const int past = p.past_lens[b];
  const bool full = p.window < 0;
  const int32_t* table = p.block_table + size_t(b) * p.table_cols;
  const int last_tq = min(q_len - 1, (row0 + QR - 1) / G);
  const int kv_hi = full ? past : past + last_tq + 1;
  int kv_lo = 0;
  if (p.window > 0) kv_lo = max(0, past + row0 / G - p.window + 1);
  if (p.local > 0) kv_lo = (past + row0 / G) / p.local * p.local;
  const int tile_begin = kv_lo / BN;
  const int lat_row0 = LAT ? p.lat.row_base[b] - p.lat.first_kv[b] : 0;      // dense row of key position 0 (may be negative)
  const int lat_first = LAT ? p.lat.first_kv[b] : 0;                          // positions before it were not expanded (never visible)
  const int n_tiles = kv_hi > kv_lo ? (kv_hi + BN - 1) / BN - tile_begin : 0;

  if (tid == 0) {
    for (int i = 0; i < KS; ++i) { mbar_init(&k_full[i], 1); mbar_init(&k_empty[i], 1); }
    for (int i = 0; i < VS; ++i) { mbar_init(&v_full[i], 1); mbar_init(&v_empty[i], 1); }
    for (int i = 0; i < Cfg::S_BUFS; ++i) mbar_init(&s_full[i], 1);
    for (int i = 0; i < Cfg::S_BUFS; ++i) { mbar_init(&p_full[i], TCA_SOFTMAX_THREADS); mbar_init(&o_done[i], 1); }
    mbar_init(&q_full, TCA_SOFTMAX_THREADS);
    abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == TCA_K_WARP) {
    tmem_alloc(&tmem_slot, Cfg::TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  pdl_launch_dependents();        // only now: a dependent grid that also wants tensor memory starts after this CTA owns its share
  const uint32_t tmem_base = tmem_slot;
  volatile int* abort_p = &abort_flag;
  auto fail = [&](int code) {
    *abort_p = 1;
    if (p.status) atomicMax(p.status, code);
  };

  if (warp >= TCA_K_WARP) {
  asm volatile("setmaxnreg.dec.sync.aligned.u32 %0;" ::"n"(TCA_REGS_OTHER));
  if (warp == TCA_K_WARP || warp == TCA_V_WARP) {
    // ------------------------------------------------------------------------------ TMA producers (K ring, V ring)
    const bool is_k = warp == TCA_K_WARP;
    const CUtensorMap* tmap = is_k ? &tmap_k : &tmap_v;
    uint64_t* full = is_k ? k_full : v_full;
    uint64_t* empty = is_k ? k_empty : v_empty;
    uint8_t* ring = is_k ? sK : sV;
    const int NS = is_k ? KS : VS;
    const int tile_bytes = is_k ? Cfg::K_TILE : Cfg::V_TILE;
    if (lane == 0) tma_prefetch_desc(tmap);
    const int last_group = max(0, (kv_hi - 1) / 16 * 16);
    int issued = 0;
    const int parts = is_k ? Cfg::K_PARTS : 1;             // slots per tile
    for (int n = 0; n < n_tiles * parts; ++n) {
      const int st = n % NS, it = Cfg::K_PARTS > 1 ? n / parts : n, part = Cfg::K_PARTS > 1 ? n - it * parts : 0;
      if (n >= NS && !mbar_wait_bounded(&empty[st], ((n / NS) - 1) & 1, abort_p)) { if (lane == 0) fail(OGB_ERR_WAIT_TMA); break; }
      if (lane == 0) mbar_expect_tx(&full[st], tile_bytes);
      __syncwarp();
      // Key groups past the end of the range re-read the last valid group (their scores are masked), so every stage
      // receives the same byte count.
      if (lane < BN / 16) {
        int j0 = min((tile_begin + it) * BN + lane * 16, last_group);
        uint8_t* dst = ring + st * tile_bytes + lane * 16 * 128;
        if constexpr (LAT) {
          j0 = max(j0, lat_first);                     // (key groups ahead of the first expanded row are masked as well)
          if (is_k) {
#pragma unroll
            for (int h = 0; h < Cfg::K_HALVES; ++h) {
              if (h < NOPE / 64) tma_load_2d(dst + h * (BN * 128), &tmap_k, &full[st], kvh * p.lat.dim + h * 64, lat_row0 + j0);
              else tma_load_2d(dst + h * (BN * 128), &tmap_r, &full[st], p.lat.kr_col + (h - NOPE / 64) * 64, lat_row0 + j0);
            }
          } else {
#pragma unroll
            for (int h = 0; h < Cfg::V_HALVES; ++h) tma_load_2d(dst + h * (BN * 128), &tmap_v, &full[st], kvh * p.lat.vdim + h * 64, lat_row0 + j0);
          }
        } else {
          const int slot0 = table[j0 / p.block_size] * p.block_size + j0 % p.block_size;
          if constexpr (MIX) {
            if (is_k) {
#pragma unroll
              for (int h = 0; h < Cfg::K_HALVES; ++h) tma_load_2d(dst + h * (BN * 128), tmap, &full[st], (p.joint ? 0 : kvh * p.dk) + part * KC + h * 64, slot0);
            } else {
#pragma unroll
              for (int h = 0; h < Cfg::V_HALVES; ++h) tma_load_2d(dst + h * (BN * 128), tmap, &full[st], kvh / p.maps * p.dv + h * 64, slot0);
            }
          } else {
#pragma unroll
            for (int h = 0; h < Cfg::K_HALVES; ++h) tma_load_2d(dst + h * (BN * 128), tmap, &full[st], kvh * DK + h * 64, slot0);
          }
        }
      }
      issued = n + 1;
    }
    if (*abort_p) {
      // copies in flight must land before the shared memory goes away
      for (int it = max(0, issued - NS); it < issued; ++it) {
        int dummy = 0;
        mbar_wait_bounded(&full[it % NS], (it / NS) & 1, &dummy, 20000000ull);
      }
    }
  } else if (warp == TCA_MMA_WARP) {
    // ------------------------------------------------------------------------------ MMA issuer
    constexpr uint32_t idesc_qk = umma_idesc_f16(TCA_BM, BN, 1);
    constexpr uint32_t idesc_pv = umma_idesc_f16(TCA_BM, DV, 1) | (1u << 16);    // B operand MN-major
    const uint32_t q_addr = smem_u32(sQ), k_ring = smem_u32(sK), v_ring = smem_u32(sV);
    constexpr uint32_t lbo = BN * 128, sbo = 1024;       // between the 64-dim halves of V; between 8-key groups
    bool ok = mbar_wait_bounded(&q_full, 0, abort_p);
    if (!ok && lane == 0) fail(OGB_ERR_WAIT_MMA);
    auto issue_qk = [&](int it) -> bool {
#pragma unroll 1
      for (int part = 0; part < Cfg::K_PARTS; ++part) {
        const int n = it * Cfg::K_PARTS + part, st = n % KS;
        if (!mbar_wait_bounded(&k_full[st], (n / KS) & 1, abort_p)) return false;
        tc_fence_after();
        if (lane == 0) {
          const uint32_t k_addr = k_ring + st * Cfg::K_TILE, q_part = q_addr + part * (KC / 64) * Cfg::Q_HALF;
#pragma unroll
          for (int ks = 0; ks < KC / 16; ++ks) {
            const uint64_t da = umma_desc_sw128(q_part + (ks >> 2) * Cfg::Q_HALF + (ks & 3) * 32);
            const uint64_t db = umma_desc_sw128(k_addr + (ks >> 2) * (BN * 128) + (ks & 3) * 32);
            umma_f16(tmem_base + (it % Cfg::S_BUFS) * Cfg::S_COLS, da, db, idesc_qk, part > 0 || ks > 0);
          }
          if (part == Cfg::K_PARTS - 1) umma_commit(&s_full[it % Cfg::S_BUFS]);
          umma_commit(&k_empty[st]);
        }
        __syncwarp();
      }
      return true;
    };
    // Q K^T runs three tiles ahead (three S buffers; P_j replaces S_j in place and the buffer is free again after P_j V_j,
    // which the in-order tensor pipe finishes before the Q K^T issued behind it starts)
    for (int it = 0; ok && it < min(Cfg::S_BUFS, n_tiles); ++it) ok = issue_qk(it);
    if (!ok && lane == 0) fail(OGB_ERR_WAIT_TMA);
    for (int it = 0; ok && it < n_tiles; ++it) {
      // (barriers per S buffer: a waiter can then never be two phases behind, whichever side runs ahead)
      if (!mbar_wait_bounded(&p_full[it % Cfg::S_BUFS], (it / Cfg::S_BUFS) & 1, abort_p)) { if (lane == 0) fail(OGB_ERR_WAIT_MMA); ok = false; break; }
      const int st = it % VS;
      if (!mbar_wait_bounded(&v_full[st], (it / VS) & 1, abort_p)) { if (lane == 0) fail(OGB_ERR_WAIT_TMA); ok = false; break; }
      tc_fence_after();
      if (lane == 0) {
        const uint32_t v_addr = v_ring + st * Cfg::V_TILE;
#pragma unroll
        for (int ks = 0; ks < BN / 16; ++ks) {
          const uint64_t db = umma_desc_sw128_mn(v_addr + ks * 16 * 128, lbo, sbo);
          umma_f16_ta(tmem_base + Cfg::O_COL, tmem_base + (it % Cfg::S_BUFS) * Cfg::S_COLS + ks * 8, db, idesc_pv, (it > 0 || ks > 0) ? 1u : 0u);
        }
        umma_commit(&v_empty[st]);
        umma_commit(&o_done[it % Cfg::S_BUFS]);
      }
      __syncwarp();
      if (it + Cfg::S_BUFS < n_tiles && !issue_qk(it + Cfg::S_BUFS)) { if (lane == 0) fail(OGB_ERR_WAIT_TMA); ok = false; break; }
    }
  }
  // (warp 11 is the spare of the fourth warpgroup: register reallocation works on whole warpgroups)
  } else {
    // ------------------------------------------------------------------------------ softmax warps
    asm volatile("setmaxnreg.inc.sync.aligned.u32 %0;" ::"n"(TCA_REGS_SOFTMAX));
    constexpr int HC = BN / 2;                 // key columns per thread and tile
    constexpr int OC = DV / 2;                 // output columns per thread
    const int quarter = warp & 3, half = warp >> 2;
    const int r = quarter * 32 + lane;
    const int gr = row0 + r;
    const bool valid = gr < rows && (QR == TCA_BM || r < QR);
    const int tq = valid ? gr / G : q_len - 1;
    const int hq = MIX ? tca_query(kvh, valid ? gr % G : 0, G, p.maps) : kvh * G + (valid ? gr % G : 0);
    const int qpos = past + tq;
    const int first_local = p.local > 0 ? qpos / p.local * p.local : 0;
    // The two warps of a lane quarter meet on a named barrier.  It has no time limit, so no softmax warp ever leaves the tile loop
    // early: after a bounded wait gave up (abort flag set) a warp keeps walking the loop - its waits then return at once - and
    // still arrives at every barrier its partner arrives at.
    auto pair_sync = [&]() { asm volatile("bar.sync %0, 64;" ::"r"(quarter + 1) : "memory"); };
    {
      const __nv_bfloat16* src = p.q + size_t(tok0 + tq) * p.q_stride + size_t(hq) * (LAT ? p.lat.dim + p.lat.rot : (MIX ? p.dk : DK));
#pragma unroll
      for (int cc = 0; cc < DK / 16; ++cc) {
        const int c = half * (DK / 16) + cc;
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if constexpr (LAT) {
          // columns past a part's own width are zeros: what K holds there (other heads' columns) does not count
          const int col = c * 8 < NOPE ? c * 8 : c * 8 - NOPE, width = c * 8 < NOPE ? p.lat.dim : p.lat.rot;
          if (valid && col < width) v = *reinterpret_cast<const uint4*>(src + (c * 8 < NOPE ? col : p.lat.dim + col));
        } else if (valid && (!MIX || c * 8 < p.dk)) v = *reinterpret_cast<const uint4*>(src + c * 8);
        if (QR == TCA_BM || r < QR) *reinterpret_cast<uint4*>(sQ + (c >> 3) * Cfg::Q_HALF + r * 128 + (((c & 7) ^ (r & 7)) << 4)) = v;
      }
      fence_proxy_async_smem();
      mbar_arrive(&q_full);
    }
    const uint32_t lane_base = tmem_base + (uint32_t(quarter * 32) << 16);
    const float kmul = CAP ? 1.f : p.scale * TCA_LOG2E;        // exponent = s * kmul - reference maximum
    const float inv_cap = CAP ? p.scale / p.softcap : 0.f, capl = p.softcap * TCA_LOG2E;
    // a tile every key of which every row of this lane quarter sees needs no masks
    const int wq_lo = past + min(q_len - 1, (row0 + quarter * 32) / G), wq_hi = past + min(q_len - 1, (row0 + quarter * 32 + 31) / G);
    const bool rows_full = row0 + quarter * 32 + 31 < rows && quarter * 32 < QR;
    auto tile_interior = [&](int it) {
      const int j0 = (tile_begin + it) * BN;
      return j0 >= kv_lo && j0 + BN <= kv_hi && (full || j0 + BN - 1 <= wq_lo) && (p.window <= 0 || j0 > wq_hi - p.window) &&
             (p.local <= 0 || j0 >= wq_hi / p.local * p.local) && rows_full;
    };
    auto issue_loads = [&](int it, float (&dst)[HC]) {
#pragma unroll
      for (int c = 0; c < HC / 16; ++c) {
        uint32_t v[16];
        tmem_ld16(lane_base + (it % Cfg::S_BUFS) * Cfg::S_COLS + half * HC + c * 16, v);
#pragma unroll
        for (int e = 0; e < 16; ++e) dst[c * 16 + e] = __uint_as_float(v[e]);
      }
    };
    // soft-cap / mask 16 scores of tile `it` in place and return their maximum (raw units: times kmul gives the exponent)
    auto prep16 = [&](int it, float (&x)[HC], int c, bool interior) -> float {
      if constexpr (CAP) {
        // (most scores lie where the polynomial holds: one vote spares the others the exponential and the division)
        float far = 0.f;
#pragma unroll
        for (int e = 0; e < 16; ++e) { x[c * 16 + e] *= inv_cap; far = fmaxf(far, fabsf(x[c * 16 + e])); }
        if (__any_sync(0xffffffffu, far > SOFT_CAP_NEAR)) {
#pragma unroll
          for (int e = 0; e < 16; ++e) x[c * 16 + e] = capl * tanh_capped(x[c * 16 + e]);
        } else {
#pragma unroll
          for (int e = 0; e < 16; ++e) x[c * 16 + e] = capl * tanh_near(x[c * 16 + e]);
        }
      }
      if (!interior) {
        const int jb = (tile_begin + it) * BN + half * HC + c * 16;
#pragma unroll
        for (int e = 0; e < 16; ++e) {
          const int j = jb + e;
          bool vis = valid && j >= kv_lo && j < kv_hi && (full || j <= qpos);
          if (p.window > 0) vis = vis && j > qpos - p.window;
          if (p.local > 0) vis = vis && j >= first_local;
          x[c * 16 + e] = vis ? x[c * 16 + e] : -INFINITY;
        }
      }
      float m4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int e = 0; e < 16; e += 4) {
        m4[0] = fmaxf(m4[0], x[c * 16 + e]); m4[1] = fmaxf(m4[1], x[c * 16 + e + 1]);
        m4[2] = fmaxf(m4[2], x[c * 16 + e + 2]); m4[3] = fmaxf(m4[3], x[c * 16 + e + 3]);
      }
      return fmaxf(fmaxf(m4[0], m4[1]), fmaxf(m4[2], m4[3]));
    };
    // row maximum of a tile from this half's maximum: meet the partner half through shared memory
    auto exchange_max = [&](int it, float mx_raw) -> float {
      const __nv_bfloat16 mxb = __float2bfloat16_ru(mx_raw * kmul);
      xchg[it & 1][half][r] = mxb;
      pair_sync();
      return fmaxf(__bfloat162float(mxb), __bfloat162float(xchg[it & 1][half ^ 1][r]));
    };
    float m_ref = -INFINITY, l = 0.f;
    bool ok = true;
    for (int it = 0; it < n_tiles; ++it) {
      if (ok && !mbar_wait_bounded(&s_full[it % Cfg::S_BUFS], (it / Cfg::S_BUFS) & 1, abort_p)) { fail(OGB_ERR_WAIT_MMA); ok = false; }
      tc_fence_after();
      float sc[HC];
      issue_loads(it, sc);
      tmem_ld_wait();
      const bool interior = tile_interior(it);
      float mx_raw = -INFINITY;
#pragma unroll
      for (int c = 0; c < HC / 16; ++c) mx_raw = fmaxf(mx_raw, prep16(it, sc, c, interior));
      const float mx_cur = exchange_max(it, mx_raw);
      // lazy maximum: move the reference only when the row maximum outgrew it by more than the gap (both halves decide alike)
      float alpha = 1.f;
      bool moved = false;
      if (mx_cur > m_ref + TCA_RESCALE_GAP || (m_ref == -INFINITY && mx_cur > -INFINITY)) {
        alpha = m_ref == -INFINITY ? 0.f : exp2f(m_ref - mx_cur);
        m_ref = mx_cur;
        moved = true;
      }
      const float nms = m_ref == -INFINITY ? 0.f : -m_ref;
      float sum4[4] = {0.f, 0.f, 0.f, 0.f};
      uint32_t pk[HC / 2];
#pragma unroll
      for (int e = 0; e < HC; e += 4) {
        const float p0 = exp2f(fmaf(sc[e], kmul, nms)), p1 = exp2f(fmaf(sc[e + 1], kmul, nms));
        const float p2 = exp2f(fmaf(sc[e + 2], kmul, nms)), p3 = exp2f(fmaf(sc[e + 3], kmul, nms));
        sum4[0] += p0; sum4[1] += p1; sum4[2] += p2; sum4[3] += p3;
        pk[e / 2] = pack_bf16x2(p0, p1);
        pk[e / 2 + 1] = pack_bf16x2(p2, p3);
      }
      l = l * alpha + ((sum4[0] + sum4[1]) + (sum4[2] + sum4[3]));
      if (it > 0 && __any_sync(0xffffffffu, moved)) {
        if (ok && !mbar_wait_bounded(&o_done[(it - 1) % Cfg::S_BUFS], ((it - 1) / Cfg::S_BUFS) & 1, abort_p)) { fail(OGB_ERR_WAIT_MMA); ok = false; }
        tc_fence_after();
#pragma unroll
        for (int c = 0; c < OC / 16; ++c) {
          uint32_t v[16];
          tmem_ld16(lane_base + Cfg::O_COL + half * OC + c * 16, v);
          tmem_ld_wait();
#pragma unroll
          for (int e = 0; e < 16; ++e) v[e] = __float_as_uint(__uint_as_float(v[e]) * alpha);
          tmem_st16(lane_base + Cfg::O_COL + half * OC + c * 16, v);
        }
      }
      // P replaces S in place: two bf16 values per 32-bit column, this half's keys in columns [half * HC / 2, +HC / 2)
#pragma unroll
      for (int c = 0; c < HC / 32; ++c) {
        uint32_t v[16];
#pragma unroll
        for (int e = 0; e < 16; ++e) v[e] = pk[c * 16 + e];
        tmem_st16(lane_base + (it % Cfg::S_BUFS) * Cfg::S_COLS + half * (HC / 2) + c * 16, v);
      }
      tmem_st_wait();
      tc_fence_before();
      mbar_arrive(&p_full[it % Cfg::S_BUFS]);
    }
    // the gate's columns of this row are fetched while the last P V runs (ranges start on 16-byte boundaries)
    const bool wide = p.gate_wide;
    const int v_cols = LAT ? p.lat.vdim : (MIX ? p.dv : DV);
    uint4 gq[OC / 8];
#pragma unroll
    for (int c = 0; c < OC / 8; ++c) {
      gq[c] = make_uint4(0u, 0u, 0u, 0u);
      if (wide && valid && half * OC + c * 8 < v_cols)
        gq[c] = *reinterpret_cast<const uint4*>(p.gate + size_t(tok0 + tq) * p.gate_stride + size_t(hq) * v_cols + half * OC + c * 8);
    }
    ok = ok && !*abort_p;
    if (ok && n_tiles > 0 && !mbar_wait_bounded(&o_done[(n_tiles - 1) % Cfg::S_BUFS], ((n_tiles - 1) / Cfg::S_BUFS) & 1, abort_p)) { fail(OGB_ERR_WAIT_MMA); ok = false; }
    tc_fence_after();
    // the row's sum is the two halves' sums (same reference maximum on both sides)
    pair_sync();                                                // the partner is done reading the last tile's maxima
    float* lsum = reinterpret_cast<float*>(&xchg[0][0][0]);     // [half][row]
    lsum[half * TCA_BM + r] = l;
    pair_sync();
    l += lsum[(half ^ 1) * TCA_BM + r];
    if (ok && !*abort_p) {
      float scale_o = 1.f;
      if (p.sinks) {
        const float sk = p.sinks[hq] * TCA_LOG2E;
        const float mm = fmaxf(m_ref, sk);
        scale_o = m_ref == -INFINITY ? 0.f : exp2f(m_ref - mm);
        l = l * scale_o + exp2f(sk - mm);
      }
      float inv = l > 0.f ? scale_o / l * p.out_scale : 0.f;
      if (p.gate && !wide) inv /= 1.f + __expf(-bf2f(p.gate[size_t(tok0 + tq) * p.gate_stride + hq]));
      __nv_bfloat16* po = p.out + size_t(tok0 + tq) * p.out_stride + size_t(hq) * v_cols + half * OC;
      const bool raw = MIX && p.part_o;
      const size_t part_row = size_t(tok0 + tq) * p.Hq + hq;
      if (raw && valid && half == 0) {
        p.part_ml[part_row * 2] = m_ref;
        p.part_ml[part_row * 2 + 1] = l;
        for (int s = 1; s < p.splits; ++s) p.part_ml[(size_t(s) * p.total_rows + part_row) * 2] = -INFINITY;
      }
#pragma unroll
      for (int c = 0; c < OC / 16; ++c) {
        uint32_t v[16];
        if (n_tiles > 0) {
          tmem_ld16(lane_base + Cfg::O_COL + half * OC + c * 16, v);
          tmem_ld_wait();
        } else {
#pragma unroll
          for (int e = 0; e < 16; ++e) v[e] = 0u;
        }
        if (wide) {
#pragma unroll
          for (int h8 = 0; h8 < 2; ++h8) {
            const uint4 q = gq[c * 2 + h8];
            const uint32_t qw[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const float2 g = unpack_bf16x2(qw[e]);
              const int i = h8 * 8 + 2 * e;
              v[i] = __float_as_uint(__fdividef(__uint_as_float(v[i]), 1.f + __expf(-g.x)));
              v[i + 1] = __float_as_uint(__fdividef(__uint_as_float(v[i + 1]), 1.f + __expf(-g.y)));
            }
          }
        }
        if (raw) {
          float* pr = p.part_o + part_row * p.dv + half * OC + c * 16;
#pragma unroll
          for (int e = 0; e < 16; e += 4)
            if (valid && half * OC + c * 16 + e < v_cols)
              *reinterpret_cast<float4*>(pr + e) = make_float4(__uint_as_float(v[e]), __uint_as_float(v[e + 1]), __uint_as_float(v[e + 2]), __uint_as_float(v[e + 3]));
        } else if (valid) {
          uint4 lo, hi;
          lo.x = pack_bf16x2(__uint_as_float(v[0]) * inv, __uint_as_float(v[1]) * inv);
          lo.y = pack_bf16x2(__uint_as_float(v[2]) * inv, __uint_as_float(v[3]) * inv);
          lo.z = pack_bf16x2(__uint_as_float(v[4]) * inv, __uint_as_float(v[5]) * inv);
          lo.w = pack_bf16x2(__uint_as_float(v[6]) * inv, __uint_as_float(v[7]) * inv);
          hi.x = pack_bf16x2(__uint_as_float(v[8]) * inv, __uint_as_float(v[9]) * inv);
          hi.y = pack_bf16x2(__uint_as_float(v[10]) * inv, __uint_as_float(v[11]) * inv);
          hi.z = pack_bf16x2(__uint_as_float(v[12]) * inv, __uint_as_float(v[13]) * inv);
          hi.w = pack_bf16x2(__uint_as_float(v[14]) * inv, __uint_as_float(v[15]) * inv);
          if (!(LAT || MIX) || half * OC + c * 16 < v_cols) *reinterpret_cast<uint4*>(po + c * 16) = lo;
          if (!(LAT || MIX) || half * OC + c * 16 + 8 < v_cols) *reinterpret_cast<uint4*>(po + c * 16 + 8) = hi;
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == TCA_K_WARP) tmem_dealloc(tmem_base, Cfg::TMEM_COLS);
}

template <int DK, int DV, int BN, bool MIX, bool CAP, int KC = DK, int QR = TCA_BM>
static int LaunchTcForm(const TcAttnParams& p, const void* k_cache, const void* v_cache, int max_q_len, int cache_slots, cudaStream_t stream) {
  using Cfg = TcaCfg<DK, DV, BN, KC, QR>;
  auto kern = attention_tc_kernel<DK, DV, BN, false, DK, MIX, CAP, KC, QR>;
  const int kw = MIX && p.joint ? p.dk : p.Hkv * (MIX ? p.dk : DK), vw = MIX ? p.Hkv / p.maps * p.dv : p.Hkv * DV;      // row widths of the caches
  static bool configured[OGB_MAX_DEVICES] = {};
  if (!set_max_dyn_smem(kern, Cfg::SMEM, configured)) return -3;
  CUtensorMap mk, mv;
  memset(&mk, 0, sizeof(mk));
  memset(&mv, 0, sizeof(mv));
  if (!MakeMapBf16(&mk, k_cache, cache_slots, kw, kw, 16)) return -2;
  if (!MakeMapBf16(&mv, v_cache, cache_slots, vw, vw, 16)) return -2;
  const int G = p.Hq / p.Hkv;
  dim3 grid((max_q_len * G + QR - 1) / QR, p.Hkv, p.B);
  launch_pdl(kern, grid, dim3(TCA_THREADS), Cfg::SMEM, stream, mk, mv, mv, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

template <int DK, int DV, int BN, bool MIX = false>
static int LaunchTc(const TcAttnParams& p, const void* k_cache, const void* v_cache, int max_q_len, int cache_slots, cudaStream_t stream) {
  return p.softcap > 0.f ? LaunchTcForm<DK, DV, BN, MIX, true>(p, k_cache, v_cache, max_q_len, cache_slots, stream)
                         : LaunchTcForm<DK, DV, BN, MIX, false>(p, k_cache, v_cache, max_q_len, cache_slots, stream);
}

}  // namespace ogb
