// Attention of heads whose scores are mixed (every query head meets the keys of all key heads of a position as one key of dk columns, values by key head), for
// decode steps and short portions over a paged cache: windows, sinks, soft-capped scores, gates and key splits as in attention_paged.cuh.  One CTA = (query
// token, up to 32 heads, key split): a cache row, keys and values of all key heads, is read once for all heads.  Rows arrive by one bulk copy each for the key and
// the value, several tiles ahead.  Per tile of BN keys: every warp multiplies its share of the key columns (warp-level MMAs, query fragments in registers), the
// partial scores meet in shared memory, the softmax runs in fp32, then every warp multiplies the weights with its share of the value columns.  The kernel is
// bound by the cache stream; its rows are the heads of one token, far fewer than tcgen05 wants.  Long prompts take attention_tc_mixed.cu.
// Every wait on an mbarrier is bounded: after one that ran out the CTA sets the status word, waits (bounded) for the copies in flight and leaves.
#include "attention_paged.cuh"

namespace ogb {

constexpr int AJ_MAX_STAGES = 4, AJ_FEW = 32;

__device__ __forceinline__ void aj_bulk_load(void* smem_dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
               ::"r"(smem_u32(smem_dst)), "l"(src), "r"(bytes), "r"(smem_u32(bar)) : "memory");
}

struct JointParams {
  AttnParams a;          // (Hkv: value heads; dk: columns of a key row, dv: of a value head)
  int stages, head_tiles;
  int block_shift;       // log2 of the block size, or -1
};

// MT: 16-head tiles; KSW: 16-column steps of the keys per warp; NP: pairs of 8-column groups of the values per warp; BN: keys per tile; CTAS: per SM.
// ONE: the heads of a key head's group are all in one head tile (16 is a multiple of the group), so that a group of value columns needs one accumulator.
template <int AJ_WARPS, int MT, int KSW, int NP, int BN, int CTAS, bool ONE>
__global__ void __launch_bounds__(AJ_WARPS * 32, CTAS) attention_joint_kernel(JointParams jp) {
  constexpr int AJ_THREADS = AJ_WARPS * 32, ROWS = 16 * MT, TPR = AJ_THREADS / ROWS, MO = ONE ? 1 : MT, KPT = BN / TPR, SP = BN + 2, PP = BN + 8;
  // elements between the rows of a tile: an odd number of 16-byte pieces, as wide as the form's widest rows (fixed, so that addresses are offsets)
  constexpr int KPITCH = AJ_WARPS * KSW * 16 + 8, VPITCH = AJ_WARPS * NP * 16 + 8;
  static_assert(KPT >= 1 && BN % TPR == 0, "a row's keys are divided over its threads");
  const AttnParams& p = jp.a;
  extern __shared__ __align__(128) uint8_t smem_dyn[];
  __nv_bfloat16* sK = reinterpret_cast<__nv_bfloat16*>(smem_dyn);                   // [stages][BN][kpitch]
  __nv_bfloat16* sV = sK + size_t(jp.stages) * BN * KPITCH;                       // [stages][BN][vpitch]
  float* sS = reinterpret_cast<float*>(sV + size_t(jp.stages) * BN * VPITCH);     // [8 warps][ROWS][SP]
  __nv_bfloat16* sP = reinterpret_cast<__nv_bfloat16*>(sS + AJ_WARPS * ROWS * SP);   // [ROWS][PP]
  float* sA = reinterpret_cast<float*>(sP + ROWS * PP);                              // [ROWS] factor of the old output; at the end the factor of the result
  volatile int* moved = reinterpret_cast<int*>(sA + ROWS);                           // the last tile that changed a factor
  __shared__ uint64_t full[AJ_MAX_STAGES];
  __shared__ int abort_flag;
  volatile int* abort_p = &abort_flag;
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int bz = blockIdx.z / p.splits, split = blockIdx.z % p.splits;
  const int b = p.order ? p.order[bz] : bz;
  const int tq = blockIdx.x / jp.head_tiles, h0 = blockIdx.x % jp.head_tiles * ROWS;
  const int tok0 = p.cu_seqlens[b], q_len = p.cu_seqlens[b + 1] - tok0, G = p.Hq / p.Hkv;
  if (tq >= q_len || (p.skip_rows > 0 && q_len * G >= p.skip_rows)) return;
  const int tok = tok0 + tq, pos = p.past_lens[b] + tq;
  const int32_t* table = p.block_table + size_t(b) * p.table_cols;
  // keys of the token, then the part of them this split owns
  const int kv_lo = p.window > 0 ? max(0, pos - p.window + 1) : 0, kv_hi = pos + 1;
  const int per = ((kv_hi - kv_lo + BN - 1) / BN + p.splits - 1) / p.splits * BN;
  const int lo = kv_lo + split * per, hi = min(kv_hi, lo + per);
  const bool partial = p.splits > 1;
  if (lo >= hi) {                                     // (only with splits: a token sees itself)
    for (int r = tid; r < ROWS; r += AJ_THREADS)
      if (h0 + r < p.Hq) {
        float* pm = p.part_ml + (size_t(split) * p.total_rows + size_t(tok) * p.Hq + h0 + r) * 2;
        pm[0] = -INFINITY; pm[1] = 0.f;
      }
    return;
  }
  const int n_tiles = (hi - lo + BN - 1) / BN, stages = jp.stages;
  const int v_cols = p.Hkv * p.dv, k_steps = (p.dk + 15) / 16, v_groups = v_cols / 8;
  const uint32_t k_bytes = p.dk * 2, v_bytes = v_cols * 2;
  if (tid == 0) {
    *moved = 0;
    for (int i = 0; i < stages; ++i) mbar_init(&full[i], 1);
    abort_flag = 0;
    mbar_fence_init();
  }
  // columns past the rows' ends that a step or a pair of groups reaches are zeros
  for (int r = tid; r < stages * BN; r += AJ_THREADS) {
    if (p.dk < k_steps * 16) *reinterpret_cast<uint4*>(sK + size_t(r) * KPITCH + p.dk) = make_uint4(0, 0, 0, 0);
    if (v_groups & 1) *reinterpret_cast<uint4*>(sV + size_t(r) * VPITCH + v_cols) = make_uint4(0, 0, 0, 0);
  }
  __syncthreads();

  // A tile's rows are divided over the warps, one copy per lane: KW keys, then their values (rows past the range repeat its last one).  A copy takes the issuing
  // warp's time, so that one warp alone would hold up the others.  Blocks are looked up a tile ahead.
  constexpr int KW = BN / AJ_WARPS;
  const int my_row = warp * KW + lane % KW;
  const bool copies = lane < 2 * KW, is_key = lane < KW;
  const uint32_t my_bytes = is_key ? k_bytes : v_bytes;
  const __nv_bfloat16* my_cache = is_key ? p.k_cache : p.v_cache;
  const int my_cols = is_key ? p.dk : v_cols, my_pitch = is_key ? KPITCH : VPITCH;
  __nv_bfloat16* my_ring = is_key ? sK : sV;
  auto key_of = [&](int it) { return min(lo + it * BN + my_row, hi - 1); };
  auto lookup = [&](int it) { const int j = key_of(it); return table[jp.block_shift >= 0 ? j >> jp.block_shift : j / p.block_size]; };
  auto load = [&](int it, int st, int block) {
    const int j = key_of(it);
    if (tid == 0) mbar_expect_tx(&full[st], BN * (k_bytes + v_bytes));
    if (copies) {
      const size_t slot = jp.block_shift >= 0 ? (size_t(block) << jp.block_shift) + (j & (p.block_size - 1)) : size_t(block) * p.block_size + j % p.block_size;
      aj_bulk_load(my_ring + (size_t(st) * BN + my_row) * my_pitch, my_cache + slot * my_cols, my_bytes, &full[st]);
    }
  };
  int block_next = lookup(0), issued = 0, issue_st = 0;      // tiles issued, stage of the next one
  auto issue = [&]() {
    const int block = block_next;
    block_next = lookup(issued + 1);
    load(issued, issue_st, block);
    ++issued;
    issue_st = issue_st + 1 == stages ? 0 : issue_st + 1;
  };
  while (issued < min(stages - 1, n_tiles)) issue();

  // query fragments: rows are heads, this warp's steps of the columns are warp, warp + 8, ..
  uint32_t qf[KSW][MT][4];
#pragma unroll
  for (int i = 0; i < KSW; ++i)
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int h = h0 + mt * 16 + g + (e & 1) * 8, c = (warp + i * AJ_WARPS) * 16 + t4 * 2 + (e >> 1) * 8;
        qf[i][mt][e] = h < p.Hq && c < p.dk ? *reinterpret_cast<const uint32_t*>(p.q + size_t(tok) * p.q_stride + size_t(h) * p.dk + c) : 0u;
      }
  // which head tiles this warp's groups of value columns belong to
  uint32_t hit = 0;
#pragma unroll
  for (int i = 0; i < NP; ++i)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int group = (warp + i * AJ_WARPS) * 2 + e, c = group * 8 / p.dv;
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
        if (group < v_groups && c * G < h0 + mt * 16 + 16 && (c + 1) * G > h0 + mt * 16) hit |= 1u << ((i * 2 + e) * MT + mt);
    }
  const int sr = tid / TPR, sk0 = (tid % TPR) * KPT;      // softmax: row and first key of this thread
  const float sc2 = p.scale * LOG2E;
  float mx = -INFINITY, l = 0.f;
  float o[NP][2][MO][4];
#pragma unroll
  for (int i = 0; i < NP; ++i)
#pragma unroll
    for (int e = 0; e < 2; ++e)
#pragma unroll
      for (int mt = 0; mt < MO; ++mt) { o[i][e][mt][0] = o[i][e][mt][1] = o[i][e][mt][2] = o[i][e][mt][3] = 0.f; }

  bool ok = true;
  uint32_t phase = 0;
  for (int it = 0, st = 0; it < n_tiles; ++it) {
    bool there = false;
    for (int i = 0; i < 32 && !there; ++i) there = mbar_try_wait(&full[st], phase);      // (the clock of the bounded wait is slow to read)
    if (!there && !mbar_wait_bounded(&full[st], phase, abort_p)) {
      *abort_p = 1;
      if (p.status) atomicMax(p.status, OGB_ERR_WAIT_TMA);
    }
    const __nv_bfloat16* tk = sK + size_t(st) * BN * KPITCH;
    const __nv_bfloat16* tv = sV + size_t(st) * BN * VPITCH;
    {
      float s[MT][BN / 8][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int i = 0; i < BN / 8; ++i) { s[mt][i][0] = s[mt][i][1] = s[mt][i][2] = s[mt][i][3] = 0.f; }
#pragma unroll
      for (int i = 0; i < KSW; ++i) {
        const int ks = warp + i * AJ_WARPS;
        if (ks >= k_steps) break;
#pragma unroll
        for (int np = 0; np < BN / 16; ++np) {
          uint32_t kb[4];
          ldmatrix_x4(kb, tk + ((np * 2 + (lane >> 4)) * 8 + (lane & 7)) * KPITCH + ks * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
          for (int mt = 0; mt < MT; ++mt) {
            mma_bf16_16816(s[mt][np * 2], qf[i][mt], kb[0], kb[1]);
            mma_bf16_16816(s[mt][np * 2 + 1], qf[i][mt], kb[2], kb[3]);
          }
        }
      }
      float* ps = sS + warp * ROWS * SP;
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int i = 0; i < BN / 8; ++i) {
          *reinterpret_cast<float2*>(ps + (mt * 16 + g) * SP + i * 8 + t4 * 2) = make_float2(s[mt][i][0], s[mt][i][1]);
          *reinterpret_cast<float2*>(ps + (mt * 16 + g + 8) * SP + i * 8 + t4 * 2) = make_float2(s[mt][i][2], s[mt][i][3]);
        }
    }
    __syncthreads();                                      // partial scores are there; the tile before is no longer read
    if (*abort_p) { ok = false; break; }                  // (set before the barrier, so all leave alike)
    if (issued < n_tiles) issue();
    {
      float x[KPT], top = -INFINITY;
#pragma unroll
      for (int e = 0; e < KPT; ++e) {
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < AJ_WARPS; ++w) v += sS[(w * ROWS + sr) * SP + sk0 + e];
        if (p.softcap > 0.f) v = p.softcap * tanh_capped(v * p.scale / p.softcap) * LOG2E;
        else v *= sc2;
        x[e] = lo + it * BN + sk0 + e < hi ? v : -INFINITY;
        top = fmaxf(top, x[e]);
      }
#pragma unroll
      for (int q = 1; q < TPR; q <<= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, q));
      // the reference moves only where a row's maximum outgrew it by more than 2^8 (a tile has at least one key)
      float al = 1.f;
      if (top > mx + 8.f || it == 0) {
        al = exp2f(mx - top);
        mx = top;
        l *= al;
        *moved = it;
      }
#pragma unroll
      for (int e = 0; e < KPT; ++e) {
        x[e] = exp2f(x[e] - mx);
        l += x[e];
      }
      if constexpr (KPT == 1) sP[sr * PP + sk0] = f2bf(x[0]);
      else {
#pragma unroll
        for (int e = 0; e < KPT; e += 2) *reinterpret_cast<uint32_t*>(sP + sr * PP + sk0 + e) = pack_bf16x2(x[e], x[e + 1]);
      }
      if (tid % TPR == 0) sA[sr] = al;
    }
    __syncthreads();
    {
      if (it > 0 && *moved == it) {
        float a[MT][2];
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) { a[mt][0] = sA[mt * 16 + g]; a[mt][1] = sA[mt * 16 + g + 8]; }
#pragma unroll
        for (int i = 0; i < NP; ++i)
#pragma unroll
          for (int e = 0; e < 2; ++e)
#pragma unroll
            for (int mo = 0; mo < MO; ++mo) {
              const bool second = MT > 1 && (ONE ? hit >> ((i * 2 + e) * MT + 1) & 1 : mo > 0);
              const float a0 = second ? a[MT - 1][0] : a[0][0], a1 = second ? a[MT - 1][1] : a[0][1];
              o[i][e][mo][0] *= a0; o[i][e][mo][1] *= a0; o[i][e][mo][2] *= a1; o[i][e][mo][3] *= a1;
            }
      }
#pragma unroll
      for (int kk = 0; kk < BN / 16; ++kk) {
        uint32_t pa[MT][4];
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) ldmatrix_x4(pa[mt], sP + (mt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * PP + kk * 16 + (lane >> 4) * 8);
#pragma unroll
        for (int i = 0; i < NP; ++i) {
          const int pair = warp + i * AJ_WARPS;
          if (pair * 2 >= v_groups) break;
          uint32_t vb[4];
          ldmatrix_x4_trans(vb, tv + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * VPITCH + (pair * 2 + (lane >> 4)) * 8);
#pragma unroll
          for (int mt = 0; mt < MT; ++mt) {
            if (MT == 1 || (hit >> (i * 2 * MT + mt) & 1)) mma_bf16_16816(o[i][0][mt % MO], pa[mt], vb[0], vb[1]);
            if (MT == 1 || (hit >> ((i * 2 + 1) * MT + mt) & 1)) mma_bf16_16816(o[i][1][mt % MO], pa[mt], vb[2], vb[3]);
          }
        }
      }
    }
    if (++st == stages) { st = 0; phase ^= 1; }
  }
  if (!ok) {
    // copies in flight must land before the shared memory goes away
    for (int i = max(0, issued - stages); i < issued; ++i) {
      int dummy = 0;
      mbar_wait_bounded(&full[i % stages], (i / stages) & 1, &dummy, 20000000ull);
    }
    return;
  }
#pragma unroll
  for (int q = 1; q < TPR; q <<= 1) l += __shfl_xor_sync(0xffffffffu, l, q);
  __syncthreads();                                        // the last tile's factors have been read
  if (tid % TPR == 0 && h0 + sr < p.Hq) {
    if (partial) {
      float* pm = p.part_ml + (size_t(split) * p.total_rows + size_t(tok) * p.Hq + h0 + sr) * 2;
      pm[0] = mx; pm[1] = l;
    } else {
      float f = 1.f;
      if (p.sinks) {
        const float sk = p.sinks[h0 + sr] * LOG2E, mm = fmaxf(mx, sk);
        f = exp2f(mx - mm);
        l = l * f + exp2f(sk - mm);
      }
      sA[sr] = f / l * p.out_scale * (p.gate_wide ? 1.f : attn_gate(p.gate, p.gate_stride, tok, h0 + sr));
    }
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < NP; ++i)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int group = (warp + i * AJ_WARPS) * 2 + e;
      if (group >= v_groups) continue;
      const int c = group * 8 / p.dv, col = group * 8 - c * p.dv + t4 * 2;
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int r = mt * 16 + g + half * 8, h = h0 + r;
          if (h >= p.Hq || h / G != c) continue;
          const float x = o[i][e][mt % MO][half * 2], y = o[i][e][mt % MO][half * 2 + 1];
          if (partial) {
            *reinterpret_cast<float2*>(p.part_o + (size_t(split) * p.total_rows + size_t(tok) * p.Hq + h) * p.dv + col) = make_float2(x, y);
          } else {
            const float f = sA[r];
            const float2 gt = p.gate_wide ? attn_gate2(p.gate + size_t(tok) * p.gate_stride + size_t(h) * p.dv + col) : make_float2(1.f, 1.f);
            *reinterpret_cast<uint32_t*>(p.out + size_t(tok) * p.out_stride + size_t(h) * p.dv + col) = pack_bf16x2(x * f * gt.x, y * f * gt.y);
          }
        }
    }
}

template <int AJ_WARPS, int MT, int KSW, int NP, int BN, int CTAS, bool ONE = false>
static int LaunchJoint(const AttnParams& a, int max_q_len, cudaStream_t stream) {
  JointParams jp{};
  jp.a = a;
  jp.block_shift = (a.block_size & (a.block_size - 1)) == 0 ? __builtin_ctz(a.block_size) : -1;
  constexpr int KPITCH = AJ_WARPS * KSW * 16 + 8, VPITCH = AJ_WARPS * NP * 16 + 8;
  const int rows = 16 * MT, stage = BN * (KPITCH + VPITCH) * 2, rest = AJ_WARPS * rows * (BN + 2) * 4 + rows * (BN + 8) * 2 + rows * 4 + 16;
  const int room = (CTAS > 1 ? 226 * 1024 / CTAS - 1024 : 224 * 1024) - rest;
  jp.stages = room / stage < AJ_MAX_STAGES ? room / stage : AJ_MAX_STAGES;
  if (jp.stages < 2) return -5;
  jp.head_tiles = (a.Hq + rows - 1) / rows;
  const long long gx = (long long)max_q_len * jp.head_tiles;
  if (gx > 0x7fffffff) return -1;
  auto kern = attention_joint_kernel<AJ_WARPS, MT, KSW, NP, BN, CTAS, ONE>;
  static bool configured[OGB_MAX_DEVICES] = {};
  if (!set_max_dyn_smem(kern, 224 * 1024, configured)) return -3;
  if (!launch_pdl(kern, dim3(unsigned(gx), 1, a.B * a.splits), dim3(AJ_WARPS * 32), size_t(jp.stages) * stage + rest, stream, jp)) return -4;
  if (a.splits > 1) {
    const int warps = 4;
    const dim3 grid((a.total_rows + warps - 1) / warps), block(warps * 32);
    const float *po = a.part_o, *ml = a.part_ml;
    const bool ok = a.dv <= 128 ? launch_pdl(attention_combine_kernel<128, false>, grid, block, 0, stream, po, ml, a.sinks, a.out, a.out_stride, a.total_rows, a.Hq, a.splits,
                                             a.dv, a.gate, a.gate_stride, a.gate_wide, a.out_scale)
                                : launch_pdl(attention_combine_kernel<1024, false>, grid, block, 0, stream, po, ml, a.sinks, a.out, a.out_stride, a.total_rows, a.Hq,
                                             a.splits, a.dv, a.gate, a.gate_stride, a.gate_wide, a.out_scale);
    if (!ok) return -4;
  }
  return 0;
}

}  // namespace ogb

using namespace ogb;

OGB_API int ogb_attention_joint_supported(int dk, int v_cols) { return dk > 0 && v_cols > 0 && dk % 8 == 0 && v_cols % 8 == 0 && dk <= 1024 && v_cols <= 1024; }

// Serves the requests with fewer than skip_rows (token, head of a group) rows (0: all); splits > 1: partial results and their merge in scratch.
OGB_API int ogb_attention_joint(const OgbAttnLayer* l, const void* q, int q_stride, const void* k_cache, const void* v_cache, const int32_t* cu_seqlens,
                                const int32_t* past_lens, const int32_t* block_table, int table_cols, int block_size, void* out, int out_stride, int B,
                                int total_tokens, int max_q_len, int splits, void* scratch, long long scratch_bytes, const int32_t* order, int* status,
                                void* stream_, int skip_rows) {
  if (B <= 0 || total_tokens <= 0 || max_q_len <= 0) return 0;
  if (!l->joint || !ogb_attention_joint_supported(l->dk, l->Hkv * l->dv) || l->dv % 8) return -5;
  if (l->Hkv <= 0 || l->Hq % l->Hkv || q_stride % 2 || out_stride % 2 || block_size <= 0 || l->chunk > 0 || l->maps > 1 || l->raw) return -1;
  if ((reinterpret_cast<uintptr_t>(k_cache) | reinterpret_cast<uintptr_t>(v_cache)) & 15) return -1;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(out)) & 3) return -1;
  if (l->gate && l->gate_wide && (l->gate_stride % 2 || (reinterpret_cast<uintptr_t>(l->gate) & 3))) return -1;
  if (splits < 1) splits = 1;
  if ((long long)B * splits > 65535) return -1;
  if (splits > 1 && (!scratch || (long long)splits * total_tokens * l->Hq * (l->dv + 2) * 4 > scratch_bytes)) return -2;
  AttnParams p{};
  p.q = static_cast<const __nv_bfloat16*>(q); p.q_stride = q_stride;
  p.k_cache = static_cast<const __nv_bfloat16*>(k_cache); p.v_cache = static_cast<const __nv_bfloat16*>(v_cache);
  p.cu_seqlens = cu_seqlens; p.past_lens = past_lens; p.block_table = block_table; p.table_cols = table_cols; p.block_size = block_size;
  p.out = static_cast<__nv_bfloat16*>(out); p.out_stride = out_stride;
  p.total_rows = total_tokens * l->Hq;
  p.part_o = static_cast<float*>(scratch);
  p.part_ml = p.part_o ? p.part_o + size_t(splits) * p.total_rows * l->dv : nullptr;
  p.sinks = l->sinks; p.scale = l->scale; p.softcap = l->softcap; p.window = l->window;
  p.B = B; p.Hq = l->Hq; p.Hkv = l->Hkv; p.splits = splits; p.status = status; p.order = order; p.skip_rows = skip_rows;
  p.dk = l->dk; p.dv = l->dv;
  p.gate = static_cast<const __nv_bfloat16*>(l->gate); p.gate_stride = l->gate_stride; p.gate_wide = l->gate && l->gate_wide;
  p.out_scale = l->out_scale;
  auto s = static_cast<cudaStream_t>(stream_);
  const int cols = max(p.dk, p.Hkv * p.dv);
  const bool one = p.Hq <= 16;
  if (cols > 512 && !one && 16 % (p.Hq / p.Hkv) == 0) return LaunchJoint<16, 2, 4, 4, 16, 1, true>(p, max_q_len, s);
  if (cols > 512) return one ? LaunchJoint<8, 1, 8, 8, 16, 1>(p, max_q_len, s) : LaunchJoint<16, 2, 4, 4, 16, 1>(p, max_q_len, s);
  if (cols <= 256) return one ? LaunchJoint<4, 1, 4, 4, 32, 2>(p, max_q_len, s) : LaunchJoint<4, 2, 4, 4, 32, 2>(p, max_q_len, s);
  // few CTAs: taller tiles, one CTA per SM; else two, whose phases overlap (64 requests: 46.5 us against 50.1, 16 requests: 27.7 against 26.1)
  if ((long long)B * max_q_len <= AJ_FEW) return one ? LaunchJoint<8, 1, 4, 4, 32, 1>(p, max_q_len, s) : LaunchJoint<8, 2, 4, 4, 32, 1>(p, max_q_len, s);
  return one ? LaunchJoint<8, 1, 4, 4, 16, 2>(p, max_q_len, s) : LaunchJoint<8, 2, 4, 4, 16, 2>(p, max_q_len, s);
}
