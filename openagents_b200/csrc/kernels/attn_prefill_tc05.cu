// Causal grouped-query flash attention for prefill on the 5th-generation tensor cores.
//
// Head sizes are template parameters (queries / keys DK = 64..256, values DV = 64 or 128, multiples of 64; other sizes are padded
// in the cache); the figures below are those of DK = DV = 128.  An optional gate per head (or per output element) multiplies the output
// by a sigmoid.  Differential attention gives a key/value head two key rows side by side: the query heads of either map load theirs.
// Latent attention (LATENT): keys and values are plain rows of a workspace that holds the expanded context, and the last columns
// of every key, the rotated part all heads share, come from the paged latent cache.
//
// One CTA = 128 query rows of one head.  Roles: warps 0 and 10 are the TMA producers (a ring of K / V
// blocks of 64 keys gathered page by page from the paged fp16 cache), warps 1 and 11 issue the two
// kinds of tcgen05.mma, warps 2..9 do the online softmax: two warps per 32 query rows (the two share a tensor-memory lane
// quarter), one taking keys 0..63 of a block and output columns 0..63, the other the rest; they swap
// their partial row maxima through shared memory once per block.  Two warps per scheduler is what
// hides the latencies of tensor-memory loads, exponentials and barriers.  Per key block j:
//   S_j = Q K_j^T        tcgen05.mma 128 x 128 x 128 into one of two S accumulators in tensor memory
//   softmax              S_j -> registers (tcgen05.ld), mask, running max / sum, P_j (fp16 pairs) -> tensor
//                        memory over the S columns it came from, where the next MMA reads it as its A operand
//   O += P_j V_j         tcgen05.mma 128 x 128 x 128 accumulating in ONE O tile that stays in tensor memory
//                        for the whole row block, V taken as it lies in the cache ([key][dim], i.e. the
//                        MN-major form of the B operand)
// The exponent offset of a row (its running maximum) is only moved when the maximum has grown by more
// than 8 (a factor 256, well inside fp16 for P and fp32 for O and the row sum); then the row's owner
// thread rescales the O row in tensor memory (tcgen05.ld / st) between two PV products.  After the
// first key blocks of a causal row that is rare, so the steady state has no O traffic at all.
// Sliding windows, chunks, learned sink logits and a context that is longer than the chunk (chunked prefill,
// prefix reuse) are handled by the mask and the block range.  Math as in the reference's attention
// (apps/openagents.com/workers/api/src/cs336-a1-real-gradient-workload.ts:478-518: max-subtract,
// exp, normalise).  Every wait is bounded; a wait that runs out sets the status word and the CTA
// leaves through the common exit, which frees its tensor memory.
#include "tc05.cuh"

using namespace b200;
using namespace b200::tc;

namespace {

constexpr int QB = 128, KB = 128;
constexpr int BOX_BYTES = KB * 128;             // one 64-dim column block of a K or V tile: [128 keys][128 bytes]
constexpr uint32_t TMEM_COLS = 512;             // S: 2 x 128 (P is written over the S columns it came from), O: DV, Q: DK / 2
constexpr float kRescaleStep = 8.f;             // log2 units
constexpr float kLog2e = 1.4426950408889634f;

struct PrefillArgs {
  const int* page_table;   // [n_seqs][max_pages]
  const int* q_start;      // [n_seqs]
  const int* q_len;        // [n_seqs]
  const int* ctx_len;      // [n_seqs]
  const float* sinks;      // [Hq] or null
  __nv_bfloat16* out;      // [T_total][Hq * DV]
  int* status;
  const __half* q;         // [T_total][Hq * DK], rotated and scaled
  const float* gate;       // [T_total][ldg] or null: head h's output is multiplied by sigmoid(gate[t][h])
  int ldg;
  int max_pages, Hq, Hkv, window, T_total;
  int chunk;               // > 0: a query sees its own chunk of that many positions only
  int maps;                // 2: key/value heads have two key rows of DK columns (query heads in the order (kv head, map, head of the group))
  int gate_elem;           // the gate has a column per output column instead of one per head
  float* out_f32;          // written instead of out where given
  // LATENT
  const int* base;         // [n_seqs] first workspace row of each sequence
  int k_boxes, v_col, r_col;   // 64-column boxes of a key's own part; first value column of the workspace; first rotated column of the cache
};

template <int DK, int DV>
constexpr int kv_stages() { return 196608 / (KB * (DK + DV) * 2) < 4 ? 196608 / (KB * (DK + DV) * 2) : 4; }

template <int DK, int DV, bool LATENT>
__global__ void __launch_bounds__(384, 1) attn_prefill_tc05_kernel(const __grid_constant__ CUtensorMap tmK,
                                                                   const __grid_constant__ CUtensorMap tmV,
                                                                   const __grid_constant__ CUtensorMap tmR,
                                                                   const PrefillArgs a) {
  constexpr int K_BYTES = KB * DK * 2, V_BYTES = KB * DV * 2, STAGE_BYTES = K_BYTES + V_BYTES, KV_STAGES = kv_stages<DK, DV>();
  static_assert(256 + DV + DK / 2 <= (int)TMEM_COLS && KV_STAGES >= 2, "head sizes");
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  uint8_t* sKV = smem;                                    // KV_STAGES x (K, V)
  uint64_t* bars = (uint64_t*)(sKV + KV_STAGES * STAGE_BYTES);
  uint64_t* q_full = bars;                                // [1]
  uint64_t* kv_full = bars + 1;                           // [KV_STAGES]
  uint64_t* kv_empty = kv_full + KV_STAGES;               // [KV_STAGES]
  uint64_t* s_full = kv_empty + KV_STAGES;                // [2]
  uint64_t* s_empty = s_full + 2;                         // [2]
  uint64_t* p_full = s_empty + 2;                         // [2]
  uint64_t* pv_done = p_full + 2;                         // [2]: PV product of the blocks that used P buffer b
  uint64_t* x_full = pv_done + 2;                          // [4 quarters][2]: both warps of a pair have posted their half
  uint32_t* tmem_holder = (uint32_t*)(x_full + 8);
  volatile int* abort_flag = (volatile int*)(tmem_holder + 1);
  float* xch = (float*)(bars + 32);                       // [2 (block parity)][2 (half)][128 rows] partial row maxima / sums

  const int seq = blockIdx.z, h = blockIdx.y, qb = gridDim.x - 1 - blockIdx.x;   // longest (latest) query blocks first
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  if (threadIdx.x == 0) {
    mbar_init(smem_u32(q_full), 4);
    for (int s = 0; s < KV_STAGES; s++) {
      mbar_init(smem_u32(kv_full + s), 1);
      mbar_init(smem_u32(kv_empty + s), 1);
    }
    for (int s = 0; s < 2; s++) {
      mbar_init(smem_u32(s_full + s), 1);
      mbar_init(smem_u32(s_empty + s), 8);
      mbar_init(smem_u32(p_full + s), 8);
    }
    mbar_init(smem_u32(pv_done), 1);
    mbar_init(smem_u32(pv_done + 1), 1);
    for (int s = 0; s < 8; s++) mbar_init(smem_u32(x_full + s), 2);
    *abort_flag = 0;
    fence_barrier_init();
    tma_prefetch_desc(&tmK);
    tma_prefetch_desc(&tmV);
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(tmem_holder), TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_holder;
  pdl_trigger();
  pdl_wait();

  const int qlen = a.q_len[seq];
  const int q0 = qb * QB;
  const bool live = q0 < qlen;            // a dead CTA still goes through the common exit (it holds tensor memory)
  const int ctx = a.ctx_len[seq], qs = a.q_start[seq];
  const int row_k = h / (a.Hq / (a.Hkv * a.maps)), kh = row_k / a.maps, k_col = row_k % a.maps * DK;
  const int pos0 = ctx - qlen + q0;       // absolute position of this CTA's first query row
  const int k_hi = min(ctx, pos0 + QB);   // keys [k_lo, k_hi) can matter to some row
  const int k_lo = a.chunk > 0 ? pos0 / a.chunk * a.chunk : a.window > 0 ? max(0, pos0 - a.window + 1) : 0;
  const int jb0 = k_lo / KB, jb1 = live ? (k_hi + KB - 1) / KB : jb0;   // key blocks [jb0, jb1)
  const int nb = jb1 - jb0;
  const uint32_t S_T = tmem_base, O_T = tmem_base + 256;   // S buffers at +0, +128; O at +256
  const uint32_t Q_T = O_T + DV;                           // Q (fp16 pairs, DK / 2 columns)
  // P_j (fp16 pairs) overwrites S_j: the warp that owns keys [64 h, 64 h + 64) of a block writes columns [64 h, 64 h + 32)

  // Four single-thread roles, each in a warp of its own, because what a thread can issue is the bound here:
  // about 55 cycles per tcgen05.mma and 100-200 per TMA load, barrier wait, fence or commit.
  //   warp 0: K loads (and the byte count of the whole stage)      warp 10: V loads
  //   warp 1: S_j = Q K_j^T                                         warp 11: O += P_j V_j, releases the stage
  if (warp == 0 || warp == 10) {
    if (lane == 0 && nb > 0) {
      const bool is_k = warp == 0;
      const int* pt = a.page_table + (size_t)seq * a.max_pages;
      for (int j = 0; j < nb; j++) {
        const int s = j % KV_STAGES;
        const uint32_t ph = (j / KV_STAGES) & 1;
        if (!mbar_wait(smem_u32(kv_empty + s), ph ^ 1, abort_flag)) break;
        const uint32_t bar = smem_u32(kv_full + s);
        // the barrier holds one pending arrival until this arrive.expect_tx, so V bytes that land first cannot
        // complete the phase early
        if (is_k) mbar_expect_tx(bar, STAGE_BYTES);
        uint8_t* dst = sKV + (size_t)s * STAGE_BYTES + (is_k ? 0 : K_BYTES);
        const int boxes = (is_k ? DK : DV) / 64;
        const CUtensorMap* tm = is_k ? &tmK : &tmV;
        if constexpr (LATENT) {
          const int row = a.base[seq] + (jb0 + j) * KB;             // 128 workspace rows at a time; rows past the context are masked
          if (!is_k) {
            for (int c = 0; c < DV / 64; c++) tma_load_2d(smem_u32(dst + c * BOX_BYTES), tm, bar, a.v_col + h * DV + c * 64, row);
          } else {
            for (int c = 0; c < a.k_boxes; c++) tma_load_2d(smem_u32(dst + c * BOX_BYTES), tm, bar, (h * a.k_boxes + c) * 64, row);
#pragma unroll
            for (int p = 0; p < KB / 16; p++) {
              const int pi = (jb0 + j) * (KB / 16) + p;
              const int page = (pi * 16 < ctx) ? pt[pi] : 0;
              for (int c = a.k_boxes; c < DK / 64; c++)
                tma_load_2d(smem_u32(dst + c * BOX_BYTES + p * 2048), &tmR, bar, a.r_col + (c - a.k_boxes) * 64, page * 16);
            }
          }
          continue;
        }
#pragma unroll
        for (int p = 0; p < KB / 16; p++) {
          const int pi = (jb0 + j) * (KB / 16) + p;
          const int page = (pi * 16 < ctx) ? pt[pi] : 0;          // pages past the context are masked anyway
          const int row = (page * a.Hkv + kh) * 16;
          for (int hf = 0; hf < boxes; hf++)
            tma_load_2d(smem_u32(dst + hf * BOX_BYTES + p * 2048), tm, bar, (is_k ? k_col : 0) + hf * 64, row);
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0 && nb > 0) {
      constexpr uint32_t idesc_s = idesc_f16(QB, KB, false);
      bool ok = mbar_wait(smem_u32(q_full), 0, abort_flag);
      for (int j = 0; j < nb && ok; j++) {
        const int s = j % KV_STAGES, b = j & 1;
        if (!mbar_wait(smem_u32(kv_full + s), (j / KV_STAGES) & 1, abort_flag)) break;
        if (!mbar_wait(smem_u32(s_empty + b), ((j >> 1) & 1) ^ 1, abort_flag)) break;
        if (j >= 2 && !mbar_wait(smem_u32(pv_done + b), ((j - 2) >> 1) & 1, abort_flag)) break;   // P_{j-2} sits in S buffer b
        tc_fence_after();
        const uint32_t ka = smem_u32(sKV + (size_t)s * STAGE_BYTES);
#pragma unroll
        for (int kk = 0; kk < DK / 16; kk++)
          umma_ts(S_T + b * KB, Q_T + 8 * kk, smem_desc_sw128(ka + (kk >> 2) * BOX_BYTES) + 2 * (kk & 3), idesc_s,
                  kk != 0 ? 1u : 0u);
        umma_commit(smem_u32(s_full + b));
      }
    }
  } else if (warp == 11) {
    if (lane == 0 && nb > 0) {
      constexpr uint32_t idesc_o = idesc_f16(QB, DV, true);
      for (int j = 0; j < nb; j++) {
        const int s = j % KV_STAGES, b = j & 1;
        if (!mbar_wait(smem_u32(kv_full + s), (j / KV_STAGES) & 1, abort_flag)) break;       // V_j has landed
        if (!mbar_wait(smem_u32(p_full + b), (j >> 1) & 1, abort_flag)) break;                // P_j written, O rows rescaled if needed
        tc_fence_after();
        const uint32_t va = smem_u32(sKV + (size_t)s * STAGE_BYTES + K_BYTES);
#pragma unroll
        for (int kk = 0; kk < KB / 16; kk++)
          umma_ts(O_T, S_T + b * KB + (kk >> 2) * 64 + 8 * (kk & 3), smem_desc_sw128_mn(va + kk * 2048, BOX_BYTES), idesc_o,
                  (j != 0 || kk != 0) ? 1u : 0u);
        // a commit covers this thread's MMAs only; S_j is known to be done because the softmax of block j needed it
        umma_commit(smem_u32(pv_done + b));
        umma_commit(smem_u32(kv_empty + s));
      }
    }
  } else if (warp < 10 && nb > 0) {
    const int q = warp & 3;                      // tensor-memory lane quarter this warp may read
    const int hsel = (warp - 2) >> 2;            // 0: keys 0..31 of a block, output columns 0..63; 1: the other half
    const int row = q * 32 + lane;               // query row of this thread (shared with the partner warp's same lane)
    const int qpos = pos0 + row;
    const int row_lo = a.chunk > 0 ? qpos / a.chunk * a.chunk : a.window > 0 ? qpos - a.window + 1 : 0;     // first key this row sees
    const int lo_max = a.chunk > 0 ? (pos0 + QB - 1) / a.chunk * a.chunk : a.window > 0 ? pos0 + QB - a.window : 0;   // of the CTA's last row
    const uint32_t lane_addr = (uint32_t)(q * 32) << 16;
    constexpr int HK = KB / 2, HO = DV / 2;
    float m_used = -INFINITY, l = 0.f;     // exponent offset of this row (log2 units) and this warp's part of the row sum
    bool ok = true;
    // post this warp's half and wait (bounded, like every wait here) for the partner's; use number `u` of buffer `bb`
    if (hsel == 0) {
      // This row of Q (fp16, already rotated and scaled) goes to tensor memory once: column j = dims 2j, 2j + 1.
      const bool in = qs + q0 + row < a.T_total;
      const uint4* qrow = (const uint4*)(a.q + ((size_t)(qs + q0 + (in ? row : 0)) * a.Hq + h) * DK);
#pragma unroll
      for (int c = 0; c < DK / 64; c++) {
        uint32_t r[32];
#pragma unroll
        for (int i = 0; i < 8; i++) {
          const uint4 v = in ? qrow[c * 8 + i] : make_uint4(0u, 0u, 0u, 0u);
          r[4 * i] = v.x; r[4 * i + 1] = v.y; r[4 * i + 2] = v.z; r[4 * i + 3] = v.w;
        }
        tmem_st32(Q_T + lane_addr + c * 32, r);
      }
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(q_full));
    }
    auto pair_sync = [&](int bb, int u) -> bool {
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(x_full + q * 2 + bb));
      bool k = mbar_wait(smem_u32(x_full + q * 2 + bb), (uint32_t)u & 1, abort_flag);
      return __all_sync(0xffffffffu, k && !*abort_flag);
    };

    for (int j = 0; j < nb; j++) {
      const int b = j & 1;
      ok = mbar_wait(smem_u32(s_full + b), (j >> 1) & 1, abort_flag);
      ok = __all_sync(0xffffffffu, ok && !*abort_flag);
      if (!ok) break;
      tc_fence_after();
      float sv[HK];
      {
        uint32_t r[32];
#pragma unroll
        for (int c = 0; c < HK / 32; c++) {
          tmem_ld32(S_T + b * KB + lane_addr + hsel * HK + c * 32, r);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; i++) sv[c * 32 + i] = __uint_as_float(r[i]);
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(s_empty + b));
      // mask, maximum of this half, swap with the partner warp
      const int kb0 = (jb0 + j) * KB;
      const bool edge = kb0 + KB - 1 > pos0 || kb0 + KB > ctx || kb0 < lo_max;
      if (edge) {
#pragma unroll
        for (int i = 0; i < HK; i++) {
          const int kp = kb0 + hsel * HK + i;
          if (kp > qpos || kp >= ctx || kp < row_lo) sv[i] = -INFINITY;
        }
      }
      float mx0 = fmaxf(sv[0], sv[1]), mx1 = fmaxf(sv[2], sv[3]);
#pragma unroll
      for (int i = 4; i < HK; i += 4) {
        mx0 = max3(mx0, sv[i], sv[i + 1]);
        mx1 = max3(mx1, sv[i + 2], sv[i + 3]);
      }
      float* xb = xch + b * 256;
      xb[hsel * 128 + row] = fmaxf(mx0, mx1);
      ok = pair_sync(b, j >> 1);
      if (!ok) break;
      const float bmax = fmaxf(fmaxf(mx0, mx1), xb[(hsel ^ 1) * 128 + row]) * kLog2e;
      // move the exponent offset only when it is far behind (or not set yet); both warps of a pair decide alike
      const bool unset = m_used == -INFINITY;
      const bool behind = bmax > m_used + kRescaleStep;          // false while bmax is -inf
      if (j > 0 && __any_sync(0xffffffffu, behind && !unset)) {
        const float m_new = fmaxf(m_used, bmax);
        const float scale = (m_new == -INFINITY) ? 1.f : ex2_approx(m_used - m_new);
        ok = mbar_wait(smem_u32(pv_done + ((j - 1) & 1)), ((j - 1) >> 1) & 1, abort_flag);       // PV_{j-1} has finished
        ok = __all_sync(0xffffffffu, ok && !*abort_flag);
        if (!ok) break;
        tc_fence_after();
#pragma unroll
        for (int c = 0; c < HO / 32; c++) {
          uint32_t r[32];
          tmem_ld32(O_T + lane_addr + hsel * HO + c * 32, r);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; i++) r[i] = __float_as_uint(__uint_as_float(r[i]) * scale);
          tmem_st32(O_T + lane_addr + hsel * HO + c * 32, r);
        }
        tmem_st_wait();
        tc_fence_before();
        l *= scale;
        m_used = m_new;
      } else if (unset) {
        m_used = bmax;                             // nothing accumulated yet under the old offset (O row and l are zero)
      }
      const float off = (m_used == -INFINITY) ? 0.f : m_used;
      float sum0 = 0.f, sum1 = 0.f, sum2 = 0.f, sum3 = 0.f;
      // P row (fp16 pairs) straight into tensor memory, where the PV product reads it as its A operand:
      // this warp's 64 keys become 32 columns at the start of its own half of S buffer b
      uint32_t pw[HK / 2];
#pragma unroll
      for (int i = 0; i < HK / 2; i++) {
        const float p0 = ex2_approx(fmaf(sv[2 * i], kLog2e, -off)), p1 = ex2_approx(fmaf(sv[2 * i + 1], kLog2e, -off));
        if (i & 1) { sum2 += p0; sum3 += p1; } else { sum0 += p0; sum1 += p1; }
        const __half2 hh = __floats2half2_rn(p0, p1);
        pw[i] = *(const uint32_t*)&hh;
      }
      // (S buffer b is free for P_j: S_j was only issued once PV_{j-2}, the last reader of these columns, had finished)
      tmem_st32(S_T + b * KB + lane_addr + hsel * HK, pw);
      tmem_st_wait();
      l += (sum0 + sum1) + (sum2 + sum3);
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(p_full + b));
    }
    if (ok) {
      ok = mbar_wait(smem_u32(pv_done + ((nb - 1) & 1)), ((nb - 1) >> 1) & 1, abort_flag);          // last PV product
      ok = __all_sync(0xffffffffu, ok && !*abort_flag);
    }
    // row sum = both halves (the partner is at the same point: every exit above is taken by whole CTAs' worth of
    // warps only through the abort flag, in which case nothing is written)
    if (__all_sync(0xffffffffu, ok)) {
      float* xl = xch + (nb & 1) * 256;            // the buffer the last block did not use
      xl[hsel * 128 + row] = l;
      ok = pair_sync(nb & 1, nb >> 1);
      l += xl[(hsel ^ 1) * 128 + row];
      tc_fence_after();
      if (a.sinks) l += (m_used == -INFINITY) ? 1.f : ex2_approx(a.sinks[h] * kLog2e - m_used);
      float inv = l > 0.f ? 1.f / l : 0.f;
      const bool wr = ok && row < qlen - q0;
      if (a.gate && !a.gate_elem && wr) inv *= 1.f / (1.f + __expf(-a.gate[(size_t)(qs + q0 + row) * a.ldg + h]));
      const size_t at = (size_t)(qs + q0 + row) * a.Hq * DV + (size_t)h * DV + hsel * HO;
      __nv_bfloat16* dst = a.out + at;
      const float* gp = a.gate && a.gate_elem ? a.gate + (size_t)(qs + q0 + row) * a.ldg + (size_t)h * DV + hsel * HO : nullptr;
#pragma unroll
      for (int c = 0; c < HO / 32; c++) {
        uint32_t r[32];
        tmem_ld32(O_T + lane_addr + hsel * HO + c * 32, r);
        tmem_ld_wait();
        if (wr && gp) {
#pragma unroll
          for (int i = 0; i < 32; i += 4) {
            const float4 g = *(const float4*)(gp + c * 32 + i);
            r[i] = __float_as_uint(__uint_as_float(r[i]) / (1.f + __expf(-g.x)));
            r[i + 1] = __float_as_uint(__uint_as_float(r[i + 1]) / (1.f + __expf(-g.y)));
            r[i + 2] = __float_as_uint(__uint_as_float(r[i + 2]) / (1.f + __expf(-g.z)));
            r[i + 3] = __float_as_uint(__uint_as_float(r[i + 3]) / (1.f + __expf(-g.w)));
          }
        }
        if (wr && a.out_f32) {
#pragma unroll
          for (int i = 0; i < 32; i += 4)
            *(float4*)(a.out_f32 + at + c * 32 + i) = make_float4(__uint_as_float(r[i]) * inv, __uint_as_float(r[i + 1]) * inv,
                                                                  __uint_as_float(r[i + 2]) * inv, __uint_as_float(r[i + 3]) * inv);
        } else if (wr) {
#pragma unroll
          for (int i = 0; i < 32; i += 8) {
            uint4 v;
            __nv_bfloat162* p = (__nv_bfloat162*)&v;
#pragma unroll
            for (int k = 0; k < 4; k++)
              p[k] = __floats2bfloat162_rn(__uint_as_float(r[i + 2 * k]) * inv, __uint_as_float(r[i + 2 * k + 1]) * inv);
            *(uint4*)(dst + c * 32 + i) = v;
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem_base, TMEM_COLS);
  if (threadIdx.x == 0 && *abort_flag && a.status) atomicExch(a.status, (int)B200_ERR_TIMEOUT_MMA);
}

template <int DK, int DV, bool LATENT>
int run_prefill(const CUtensorMap& tk, const CUtensorMap& tv, const CUtensorMap& tr, const PrefillArgs& a, int n_seqs, int max_q, cudaStream_t st) {
  constexpr size_t smem = 1024 + (size_t)kv_stages<DK, DV>() * KB * (DK + DV) * 2 + 32 * 8 + 2 * 2 * 128 * 4;
  static_assert(smem <= 232448, "shared memory per CTA");
  auto kern = attn_prefill_tc05_kernel<DK, DV, LATENT>;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  dim3 grid((max_q + QB - 1) / QB, a.Hq, n_seqs);
  return launch_pdl(kern, grid, dim3(384), smem, st, tk, tv, tr, a);
}

template <int DK, int DV>
int launch_prefill(const void* kc, const void* vc, int n_pages, const PrefillArgs& a, int n_seqs, int max_q, cudaStream_t st) {
  CUtensorMap tk, tv;
  const uint64_t rows = (uint64_t)n_pages * a.Hkv * 16;
  int rc = make_tmap_2d(&tk, kc, 2, rows, (uint64_t)a.maps * DK, (uint64_t)a.maps * DK * 2, 16, 64, true);
  if (rc) return rc;
  rc = make_tmap_2d(&tv, vc, 2, rows, DV, (uint64_t)DV * 2, 16, 64, true);
  if (rc) return rc;
  return run_prefill<DK, DV, false>(tk, tv, tk, a, n_seqs, max_q, st);
}

}  // namespace

// q fp16 [T_total][Hq * dk] (rotated, pre-scaled); kc fp16 [n_pages][Hkv][16][maps * dk], vc [n_pages][Hkv][16][dv];
// out bf16 [T_total][Hq * dv], or the same in fp32 to out_f32.  Sequences as in b200_attn_prefill; max_q = longest chunk.
B200_API int b200_attn_prefill_tc05(const void* q, const void* kc, const void* vc, const int* page_table, int max_pages,
                                    int n_pages, const int* q_start, const int* q_len, const int* ctx_len, int n_seqs,
                                    int max_q, int T_total, int Hq, int Hkv, int dk, int dv, int window, const float* sinks,
                                    const float* gate, int ldg, void* out, int chunk, int maps, float* out_f32, int* status, cudaStream_t st) {
  if (Hkv < 1 || maps < 1 || Hq % (Hkv * maps) || n_seqs < 1 || max_q < 1 || !page_table || chunk < 0 || (chunk && window) || (!out && !out_f32))
    return B200_ERR_BAD_ARG;
  PrefillArgs a = {};
  a.chunk = chunk; a.maps = maps; a.out_f32 = out_f32;
  a.q = (const __half*)q; a.T_total = T_total; a.gate = gate; a.ldg = ldg;
  a.page_table = page_table; a.q_start = q_start; a.q_len = q_len; a.ctx_len = ctx_len; a.sinks = sinks;
  a.out = (__nv_bfloat16*)out; a.status = status; a.max_pages = max_pages; a.Hq = Hq; a.Hkv = Hkv; a.window = window;
  switch (dk * 1000 + dv) {
    case 64064: return launch_prefill<64, 64>(kc, vc, n_pages, a, n_seqs, max_q, st);
    case 64128: return launch_prefill<64, 128>(kc, vc, n_pages, a, n_seqs, max_q, st);
    case 128064: return launch_prefill<128, 64>(kc, vc, n_pages, a, n_seqs, max_q, st);
    case 128128: return launch_prefill<128, 128>(kc, vc, n_pages, a, n_seqs, max_q, st);
    case 192064: return launch_prefill<192, 64>(kc, vc, n_pages, a, n_seqs, max_q, st);
    case 192128: return launch_prefill<192, 128>(kc, vc, n_pages, a, n_seqs, max_q, st);
    case 256064: return launch_prefill<256, 64>(kc, vc, n_pages, a, n_seqs, max_q, st);
    case 256128: return launch_prefill<256, 128>(kc, vc, n_pages, a, n_seqs, max_q, st);
  }
  return B200_ERR_BAD_ARG;
}

// The same over an expanded context (latent attention): ws fp16 [ws_rows][ldw] holds, at row base[seq] + key, the keys' own parts (head h at
// column h * kn) and from v_col on the values (head h at h * dv); the last rr columns of every key lie in the paged cache [n_pages][16][ks] from
// column r_col on.  q fp16 [T_total][H * (kn + rr)]; gate fp32 [T_total][ldg] (or null) has a column per output column; kn, rr, dv multiples of 64.
// ws must hold no infinities or NaNs anywhere (rows past a context meet zero weights).
B200_API int b200_attn_prefill_latent(const void* q, const void* ws, long ws_rows, int ldw, int v_col, const int* base, const void* cache, int n_pages,
                                      int ks, int r_col, const int* page_table, int max_pages, const int* q_start, const int* q_len, const int* ctx_len,
                                      int n_seqs, int max_q, int T_total, int H, int kn, int rr, int dv, const float* sinks, const float* gate, int ldg,
                                      void* out, int* status, cudaStream_t st) {
  if (H < 1 || n_seqs < 1 || max_q < 1 || kn < 64 || kn % 64 || rr < 64 || rr % 64 || v_col % 8 || r_col % 8 || ldw % 8 || ks % 8 || v_col < H * kn ||
      ldw < v_col + H * dv || ks < r_col + rr || (gate && (ldg % 4 || ldg < H * dv || ((uintptr_t)gate & 15))))
    return B200_ERR_BAD_ARG;
  PrefillArgs a = {};
  a.q = (const __half*)q; a.T_total = T_total; a.gate = gate; a.ldg = ldg; a.gate_elem = 1; a.maps = 1;
  a.page_table = page_table; a.q_start = q_start; a.q_len = q_len; a.ctx_len = ctx_len; a.sinks = sinks;
  a.out = (__nv_bfloat16*)out; a.status = status; a.max_pages = max_pages; a.Hq = H; a.Hkv = H;
  a.base = base; a.k_boxes = kn / 64; a.v_col = v_col; a.r_col = r_col;
  CUtensorMap tw, tr;
  int rc = make_tmap_2d(&tw, ws, 2, (uint64_t)ws_rows, (uint64_t)ldw, (uint64_t)ldw * 2, KB, 64, true);
  if (rc) return rc;
  rc = make_tmap_2d(&tr, cache, 2, (uint64_t)n_pages * 16, (uint64_t)ks, (uint64_t)ks * 2, 16, 64, true);
  if (rc) return rc;
  switch ((kn + rr) * 1000 + dv) {
    case 128064: return run_prefill<128, 64, true>(tw, tw, tr, a, n_seqs, max_q, st);
    case 128128: return run_prefill<128, 128, true>(tw, tw, tr, a, n_seqs, max_q, st);
    case 192064: return run_prefill<192, 64, true>(tw, tw, tr, a, n_seqs, max_q, st);
    case 192128: return run_prefill<192, 128, true>(tw, tw, tr, a, n_seqs, max_q, st);
    case 256064: return run_prefill<256, 64, true>(tw, tw, tr, a, n_seqs, max_q, st);
    case 256128: return run_prefill<256, 128, true>(tw, tw, tr, a, n_seqs, max_q, st);
  }
  return B200_ERR_BAD_ARG;
}
