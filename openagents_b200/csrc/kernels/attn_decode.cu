// Paged-KV grouped-query attention for decode: one query token per sequence against a paged
// fp16 K/V cache with 16-token pages, optional sliding window, chunks and learned sink logits.
//
// Work split: grid = (splits, kv_heads, sequences).  A CTA streams its share of one sequence's
// pages for one KV head exactly once and serves all G query heads that share that KV head, so the
// cache is read once per KV head, not once per query head.  Pages arrive through swizzled 2-D TMA
// loads into a ring of shared-memory slots; each warp consumes whole pages on mma.sync tiles with
// the query heads of the group as the (padded) M dimension.  Splits are merged by whichever CTA
// finishes last (a counter, no waiting).
//
// Query / key heads and value heads have sizes of their own (DK, DV: multiples of 64; other sizes are padded in the cache), and
// an optional gate per head multiplies the output by a sigmoid.
//
// The softmax follows the reference formulation (max-subtract, exp, normalise:
// apps/openagents.com/workers/api/src/cs336-a1-real-gradient-workload.ts:478-518).
#include "tc05.cuh"
#include "warp_mma.cuh"

using namespace b200;

struct AttnDecArgs {
  const float* q;          // [B][Hq*DK], rotated and pre-scaled
  const __half* kc;        // [pages][Hkv][16][DK]
  const __half* vc;        // [pages][Hkv][16][DV]
  const int* page_table;   // [B][max_pages]
  const int* seq_lens;     // [B] keys to attend (includes the current token)
  const float* sinks;      // [Hq] or null
  int max_pages, Hq, Hkv, window, chunk, S;   // chunk > 0: keys of the token's own chunk of that many positions only
  int kv_rep, Hkv_cache;   // virtual KV heads per cache head (splits wide groups), heads in the cache
  int G;                   // query heads per (virtual) KV head
  const float* gate;       // [B][ldg] or null: head h's output is multiplied by sigmoid(gate[b][h])
  int ldg;
  float* out_f32;          // [B][Hq*DV] or null
  __nv_bfloat16* out_bf16; // [B][Hq*DV] or null
  int8_t* oq;              // quantized output for a following mat-vec, or null
  float* od;
  float* os16;
  float* part_acc;         // [B*Hkv*S*G][DV]
  float* part_ml;          // [B*Hkv*S*G][2]
  int* counters;           // [B*Hkv], zero before first use; left zero on exit
  int* status;             // set non-zero if a copy never arrived (may be null)
};

__device__ __forceinline__ float exp_scale(float m, float M) {
  return m == -INFINITY ? 0.f : __expf(m - M);
}

template <int DV>
__device__ __forceinline__ void write_out(const AttnDecArgs& a, int b, int h, int e, float o) {
  const int col = h * DV + e;
  const size_t row = (size_t)b * a.Hq * DV;
  if (a.out_f32) a.out_f32[row + col] = o;
  if (a.out_bf16) a.out_bf16[row + col] = __float2bfloat16(o);
  if (a.oq) {
    const int lane = threadIdx.x & 31;
    const int blk = col >> 5;
    const size_t nblk = (size_t)a.Hq * DV / 32;
    quantize_block32(o, lane, a.oq + row + (size_t)blk * 32, a.od + (size_t)b * nblk + blk,
                     a.os16 + ((size_t)b * nblk + blk) * 2);
  }
}

constexpr int kStages = 8;   // pages in flight per CTA (two per warp)

// One CTA = (split, kv head, sequence).  Warp w owns pages w, w+4, w+8, ... of the CTA's range and
// the ring slots w and w+4: it waits for its own page, runs QK^T and PV on tensor-core tiles with
// the G query heads padded to a 16-row tile, and re-issues the TMA load for its next page itself,
// so no CTA-wide synchronisation happens inside the loop.  K/V tiles land in shared memory with the
// 128-byte swizzle, which makes every ldmatrix conflict-free.
// GT = rows reserved for query heads; EXACT: the group has exactly GT of them, else a.G <= GT.
template <int DK, int DV, int GT, bool EXACT>
__global__ void __launch_bounds__(128) attn_decode_kernel(const __grid_constant__ CUtensorMap tmK,
                                                           const __grid_constant__ CUtensorMap tmV,
                                                           const AttnDecArgs a) {
  constexpr int KBOX = DK / 64, VBOX = DV / 64;   // 64-column (128-byte) boxes per tile
  constexpr int BOX = 16 * 128;                   // bytes of one box: 16 tokens x 128 bytes
  constexpr int KTILE = KBOX * BOX, SLOT = (KBOX + VBOX) * BOX;     // bytes of a (page, head) K tile, of K and V together
  const int G = EXACT ? GT : a.G;
  extern __shared__ uint8_t dyn_raw[];
  uint8_t* ring = (uint8_t*)(((uintptr_t)dyn_raw + 1023) & ~(uintptr_t)1023);   // kStages x (K, V)
  uint64_t* bars = (uint64_t*)(ring + kStages * SLOT);
  int* s_pid = (int*)(bars + kStages);
  __shared__ float s_acc[4][GT][DV];
  __shared__ float s_ml[4][GT][2];
  __shared__ int s_last;
  __shared__ int s_abort;

  const int split = blockIdx.x, kh = blockIdx.y, b = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g4 = lane >> 2, t4 = lane & 3;
  if (tid == 0) {
    for (int s = 0; s < kStages; s++) tc::mbar_init(tc::smem_u32(bars + s), 1);
    s_abort = 0;
    tc::fence_barrier_init();
    tc::tma_prefetch_desc(&tmK);
    tc::tma_prefetch_desc(&tmV);
  }
  // Everything above touches only this CTA's shared memory; lengths, page table, queries and the
  // cache come from earlier kernels.
  pdl_trigger();
  pdl_wait();
  const int len = a.seq_lens[b];
  const int first = a.chunk > 0 ? (len - 1) / a.chunk * a.chunk : (a.window > 0 && len > a.window) ? len - a.window : 0;
  const int p_first = first >> 4, p_last = (len + 15) >> 4;
  const int per = (p_last - p_first + a.S - 1) / a.S;
  const int pa = p_first + split * per;
  const int pb = min(p_last, pa + per);
  const int np = max(0, pb - pa);
  const int kh_cache = kh / a.kv_rep;

  const int* pt = a.page_table + (size_t)b * a.max_pages;
  for (int i = tid; i < np; i += 128) s_pid[i] = pt[pa + i];
  __syncthreads();

  auto issue = [&](int i) {   // one lane: fetch page i of the range into ring slot i % kStages
    const int s = i % kStages;
    const uint32_t bar = tc::smem_u32(bars + s);
    const int row = (s_pid[i] * a.Hkv_cache + kh_cache) * 16;
    tc::mbar_expect_tx(bar, SLOT);
#pragma unroll
    for (int c = 0; c < KBOX; c++) tc::tma_load_2d(tc::smem_u32(ring + (size_t)s * SLOT + c * BOX), &tmK, bar, c * 64, row);
#pragma unroll
    for (int c = 0; c < VBOX; c++) tc::tma_load_2d(tc::smem_u32(ring + (size_t)s * SLOT + KTILE + c * BOX), &tmV, bar, c * 64, row);
  };
  if (lane == 0) {
    if (warp < np) issue(warp);
    if (warp + 4 < np) issue(warp + 4);
  }

  // Q as the A operand: rows = query heads (zero beyond G), fp16, DK/16 k-steps.
  uint32_t qf[DK / 16][4];
  {
    const float* q0 = a.q + (size_t)b * a.Hq * DK + (size_t)(kh * G) * DK;
#pragma unroll
    for (int kk = 0; kk < DK / 16; kk++) {
      const int c0 = kk * 16 + t4 * 2;
      float2 v00 = make_float2(0.f, 0.f), v01 = v00, v10 = v00, v11 = v00;
      if (g4 < G) {
        v00 = *(const float2*)(q0 + g4 * DK + c0);
        v01 = *(const float2*)(q0 + g4 * DK + c0 + 8);
      }
      if (g4 + 8 < G) {
        v10 = *(const float2*)(q0 + (g4 + 8) * DK + c0);
        v11 = *(const float2*)(q0 + (g4 + 8) * DK + c0 + 8);
      }
      qf[kk][0] = pack_h2(v00.x, v00.y);
      qf[kk][1] = pack_h2(v10.x, v10.y);
      qf[kk][2] = pack_h2(v01.x, v01.y);
      qf[kk][3] = pack_h2(v11.x, v11.y);
    }
  }
  float o[DV / 8][4];
#pragma unroll
  for (int j = 0; j < DV / 8; j++) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;   // rows g4 and g4 + 8

  for (int i = warp; i < np; i += 4) {
    const int s = i % kStages;
    bool ok = tc::mbar_wait(tc::smem_u32(bars + s), (uint32_t)((i / kStages) & 1), &s_abort);
    ok = __all_sync(0xffffffffu, ok);
    if (!ok) break;
    const uint8_t* kt = ring + (size_t)s * SLOT;
    const uint8_t* vt = kt + KTILE;
    // ---- S = Q K^T : 16 heads x 16 tokens
    float sc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
    for (int kk = 0; kk < DK / 16; kk++) {
      const int r = (lane >> 4) * 8 + (lane & 7);            // token row
      const int c = 2 * kk + ((lane >> 3) & 1);              // 16-byte chunk of the full row
      const uint8_t* p = kt + (c >> 3) * BOX + r * 128 + (((c & 7) ^ (r & 7)) << 4);
      uint32_t b0, b1, b2, b3;
      ldsm_x4(tc::smem_u32(p), b0, b1, b2, b3);
      mma16816(sc[0], qf[kk], b0, b1);
      mma16816(sc[1], qf[kk], b2, b3);
    }
    // ---- mask, online softmax (rows g4, g4+8; this thread holds tokens 2*t4, 2*t4+1 of each 8)
    const int tbase = (pa + i) * 16;
    float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
    for (int j = 0; j < 2; j++)
#pragma unroll
      for (int e = 0; e < 4; e++) {
        const int t = tbase + j * 8 + t4 * 2 + (e & 1);
        if (!(t >= first && t < len)) sc[j][e] = -INFINITY;
        if (e < 2) mx0 = fmaxf(mx0, sc[j][e]); else mx1 = fmaxf(mx1, sc[j][e]);
      }
    mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
    mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
    mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
    mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
    const float mn0 = fmaxf(m0, mx0), mn1 = fmaxf(m1, mx1);
    const float c0 = exp_scale(m0, mn0), c1 = exp_scale(m1, mn1);
    const float sub0 = mn0 == -INFINITY ? 0.f : mn0, sub1 = mn1 == -INFINITY ? 0.f : mn1;
    uint32_t pf[4];
    float rs0 = 0.f, rs1 = 0.f;
#pragma unroll
    for (int j = 0; j < 2; j++) {
      const float p0 = __expf(sc[j][0] - sub0), p1 = __expf(sc[j][1] - sub0);
      const float p2 = __expf(sc[j][2] - sub1), p3 = __expf(sc[j][3] - sub1);
      rs0 += p0 + p1;
      rs1 += p2 + p3;
      pf[j * 2] = pack_h2(p0, p1);
      pf[j * 2 + 1] = pack_h2(p2, p3);
    }
    l0 = l0 * c0 + rs0;
    l1 = l1 * c1 + rs1;
    m0 = mn0;
    m1 = mn1;
#pragma unroll
    for (int j = 0; j < DV / 8; j++) {
      o[j][0] *= c0; o[j][1] *= c0; o[j][2] *= c1; o[j][3] *= c1;
    }
    // ---- O += P V
#pragma unroll
    for (int jd = 0; jd < DV / 8; jd += 2) {
      const int r = (lane & 7) + ((lane >> 3) & 1) * 8;      // token row
      const int c = jd + (lane >> 4);
      const uint8_t* p = vt + (c >> 3) * BOX + r * 128 + (((c & 7) ^ (r & 7)) << 4);
      uint32_t b0, b1, b2, b3;
      ldsm_x4_t(tc::smem_u32(p), b0, b1, b2, b3);
      mma16816(o[jd], pf, b0, b1);
      mma16816(o[jd + 1], pf, b2, b3);
    }
    __syncwarp();
    if (lane == 0 && i + kStages < np) issue(i + kStages);
  }
  if (tid == 0 && s_abort && a.status) atomicExch(a.status, (int)B200_ERR_TIMEOUT_TMA);

  // row sums live in the four lanes of a quad
  l0 += __shfl_xor_sync(0xffffffffu, l0, 1);
  l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
  l1 += __shfl_xor_sync(0xffffffffu, l1, 1);
  l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
  // this warp's partial (m, l, O) for each real head -> shared
  if (g4 < GT && g4 < G) {
#pragma unroll
    for (int j = 0; j < DV / 8; j++) {
      s_acc[warp][g4][j * 8 + t4 * 2] = o[j][0];
      s_acc[warp][g4][j * 8 + t4 * 2 + 1] = o[j][1];
    }
    if (t4 == 0) {
      s_ml[warp][g4][0] = m0;
      s_ml[warp][g4][1] = l0;
    }
  }
  if (g4 + 8 < GT && g4 + 8 < G) {
#pragma unroll
    for (int j = 0; j < DV / 8; j++) {
      s_acc[warp][g4 + 8][j * 8 + t4 * 2] = o[j][2];
      s_acc[warp][g4 + 8][j * 8 + t4 * 2 + 1] = o[j][3];
    }
    if (t4 == 0) {
      s_ml[warp][g4 + 8][0] = m1;
      s_ml[warp][g4 + 8][1] = l1;
    }
  }
  __syncthreads();

  // merge the four warps: thread e owns output dim e
  const int e = tid;
  const size_t pbase = (((size_t)b * a.Hkv + kh) * a.S + split) * G;
  float fm[GT], fl[GT], fa[GT];
#pragma unroll
  for (int g = 0; g < GT; g++) {
    if (g >= G) continue;
    float M = -INFINITY;
#pragma unroll
    for (int w = 0; w < 4; w++) M = fmaxf(M, s_ml[w][g][0]);
    float L = 0.f, A = 0.f;
#pragma unroll
    for (int w = 0; w < 4; w++) {
      const float c = exp_scale(s_ml[w][g][0], M);
      L += s_ml[w][g][1] * c;
      if (e < DV) A += s_acc[w][g][e] * c;
    }
    fm[g] = M; fl[g] = L; fa[g] = A;
  }

  if (a.S > 1) {
#pragma unroll
    for (int g = 0; g < GT; g++) {
      if (g >= G) continue;
      if (e < DV) a.part_acc[(pbase + g) * DV + e] = fa[g];
      if (e == 0) {
        a.part_ml[(pbase + g) * 2] = fm[g];
        a.part_ml[(pbase + g) * 2 + 1] = fl[g];
      }
    }
    __threadfence();
    __syncthreads();
    if (tid == 0) {
      const int done = atomicAdd(a.counters + b * a.Hkv + kh, 1);
      s_last = (done == a.S - 1);
      if (s_last) a.counters[b * a.Hkv + kh] = 0;
    }
    __syncthreads();
    if (!s_last) return;
    __threadfence();
    const size_t p0 = ((size_t)b * a.Hkv + kh) * a.S * G;
#pragma unroll
    for (int g = 0; g < GT; g++) {
      if (g >= G) continue;
      float M = -INFINITY;
      for (int s = 0; s < a.S; s++) M = fmaxf(M, __ldcg(a.part_ml + (p0 + (size_t)s * G + g) * 2));
      float L = 0.f, A = 0.f;
      for (int s = 0; s < a.S; s++) {
        const size_t idx = p0 + (size_t)s * G + g;
        const float c = exp_scale(__ldcg(a.part_ml + idx * 2), M);
        L += __ldcg(a.part_ml + idx * 2 + 1) * c;
        if (e < DV) A += __ldcg(a.part_acc + idx * DV + e) * c;
      }
      fm[g] = M; fl[g] = L; fa[g] = A;
    }
  }

  if (warp * 32 < DV) {  // warps that own real output dims (all four when DV = 128)
#pragma unroll
    for (int g = 0; g < GT; g++) {
      if (g >= G) continue;
      float M = fm[g], L = fl[g], A = fa[g];
      if (a.sinks) {
        const float sk = a.sinks[kh * G + g];
        const float M2 = fmaxf(M, sk);
        const float c = exp_scale(M, M2);
        L = L * c + __expf(sk - M2);
        A *= c;
      }
      float o = L > 0.f ? A / L : 0.f;
      if (a.gate) o *= 1.f / (1.f + __expf(-a.gate[(size_t)b * a.ldg + kh * G + g]));
      write_out<DV>(a, b, kh * G + g, e, o);
    }
  }
}

template <int DK, int DV, int GT, bool EXACT>
static int launch(const AttnDecArgs& a, int B, int n_pages, cudaStream_t st) {
  dim3 grid(a.S, a.Hkv, B);
  const int pages_per_cta = (a.max_pages + a.S - 1) / a.S + 1;
  const size_t smem = 1024 + (size_t)kStages * 16 * (DK + DV) * 2 + kStages * 8 + (size_t)pages_per_cta * 4;
  if (smem > 180 * 1024) return B200_ERR_BAD_ARG;
  auto kern = attn_decode_kernel<DK, DV, GT, EXACT>;
  static size_t configured = 0;
  if (smem > configured) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = smem;
  }
  // The caches as 2-D tensors: one row per (page, head, token).
  CUtensorMap tk, tv;
  const uint64_t rows = (uint64_t)n_pages * a.Hkv_cache * 16;
  int rc = make_tmap_2d(&tk, a.kc, 2, rows, DK, (uint64_t)DK * 2, 16, 64, true);
  if (rc) return rc;
  rc = make_tmap_2d(&tv, a.vc, 2, rows, DV, (uint64_t)DV * 2, 16, 64, true);
  if (rc) return rc;
  return launch_pdl(kern, grid, dim3(128), smem, st, tk, tv, a);
}

template <int HD>
static int launch_exact(const AttnDecArgs& a, int B, int n_pages, cudaStream_t st) {
  switch (a.G) {
    case 1: return launch<HD, HD, 1, true>(a, B, n_pages, st);
    case 2: return launch<HD, HD, 2, true>(a, B, n_pages, st);
    case 4: return launch<HD, HD, 4, true>(a, B, n_pages, st);
    case 8: return launch<HD, HD, 8, true>(a, B, n_pages, st);
    case 16: return launch<HD, HD, 16, true>(a, B, n_pages, st);
  }
  return a.G < 8 ? launch<HD, HD, 8, false>(a, B, n_pages, st) : launch<HD, HD, 16, false>(a, B, n_pages, st);
}
template <int DK, int DV>
static int launch_any(const AttnDecArgs& a, int B, int n_pages, cudaStream_t st) {
  if (a.G == 1) return launch<DK, DV, 1, true>(a, B, n_pages, st);
  return a.G <= 4 ? launch<DK, DV, 4, false>(a, B, n_pages, st) : launch<DK, DV, 16, false>(a, B, n_pages, st);
}

// Floats of scratch the split-merge needs: part_acc then part_ml (hd = value head size), plus one int of counters per
// sequence and query head at most.
B200_API size_t b200_attn_decode_scratch_floats(int B, int Hq, int Hkv, int hd, int S) {
  return (size_t)B * Hq * S * (hd + 2);
}

// hd: query / key head size, dv: value head size (64..256 and 64..128, multiples of 64).  counters: B * Hq ints, zero before first use.
B200_API int b200_attn_decode(const float* q, const void* kc, const void* vc, const int* page_table,
                              int max_pages, int n_pages, const int* seq_lens, const float* sinks, int B,
                              int Hq, int Hkv, int hd, int dv, int window, int chunk, int S, const float* gate, int ldg, float* out_f32,
                              void* out_bf16, void* oq, float* od, float* os16, float* scratch, int* counters, int* status,
                              cudaStream_t st) {
  if (Hkv < 1 || Hq % Hkv || S < 1 || chunk < 0 || (chunk && window)) return B200_ERR_BAD_ARG;
  int G = Hq / Hkv, rep = 1;
  while (G % rep || G / rep > 16) rep++;            // a group wider than the 16-row tile is served as several
  AttnDecArgs a;
  a.q = q; a.kc = (const __half*)kc; a.vc = (const __half*)vc; a.page_table = page_table;
  a.seq_lens = seq_lens; a.sinks = sinks; a.max_pages = max_pages; a.Hq = Hq; a.Hkv = Hkv * rep;
  a.window = window; a.chunk = chunk; a.S = S; a.kv_rep = rep; a.Hkv_cache = Hkv; a.G = G / rep; a.gate = gate; a.ldg = ldg;
  a.out_f32 = out_f32; a.out_bf16 = (__nv_bfloat16*)out_bf16;
  a.oq = (int8_t*)oq; a.od = od; a.os16 = os16;
  a.part_acc = scratch;
  a.part_ml = scratch ? scratch + (size_t)B * Hq * S * dv : nullptr;
  a.counters = counters;
  a.status = status;
  if (S > 1 && (!scratch || !counters)) return B200_ERR_BAD_ARG;
  if (hd == dv && hd == 128) return launch_exact<128>(a, B, n_pages, st);
  if (hd == dv && hd == 64) return launch_exact<64>(a, B, n_pages, st);
  switch (hd * 1000 + dv) {
    case 64128: return launch_any<64, 128>(a, B, n_pages, st);
    case 128064: return launch_any<128, 64>(a, B, n_pages, st);
    case 192064: return launch_any<192, 64>(a, B, n_pages, st);
    case 192128: return launch_any<192, 128>(a, B, n_pages, st);
    case 256064: return launch_any<256, 64>(a, B, n_pages, st);
    case 256128: return launch_any<256, 128>(a, B, n_pages, st);
  }
  return B200_ERR_BAD_ARG;
}
