// Attention whose heads' scores are mixed ahead of the softmax: score_h <- sum_g T[h][g] score_g, with keys that are the values too, a bias
// that grows with the distance, a sliding window and a term of one in the softmax's denominator.
//
// The mixture is linear in the queries, so it can be taken either on them or on the scores:
//   sum_g T[h][g] (q_g . k_c(g)) = Q'_h . K,   K = [k_0 | k_1 | ...] (all key heads of a token side by side),
//                                              Q'_h = [sum over g of group 0 of T[h][g] q_g | the same of group 1 | ...]
// Prompts take the first form: every head then attends on its own, with wide queries on a key row that all heads share, whose slice of the
// head's group is the value; the tensor cores have the room for the longer products.  Decoding takes the second: a token's raw scores fit one warp's
// registers, so that the mixture is one more small product there.  Distances: the biases of the mixture add up to one slope per head.
// A cache row is K: [page][16][G * DK], fp16 (or fp32 in the 32-bit mode).
//
// This file is compiled without fast math.
#include "tc05.cuh"
#include "warp_mma.cuh"

using namespace b200;
using namespace b200::tc;

constexpr float kLog2e = 1.4426950408889634f;

// A wait that ran out leaves copies in flight: give them time to land before the shared memory goes to another block.
__device__ __forceinline__ void drain_after_abort() {
  const unsigned long long t0 = globaltimer_ns();
  while (globaltimer_ns() - t0 < 2000000ull) __nanosleep(1000);
}

// ------------------------------------------------------------------ finish of the projections

struct MixedArgs {
  const float* in;         // [T][ld]: H queries of dim columns from column 0 on, G keys from column k_off on
  int ld, k_off;
  const float* bias;       // added to the row's columns, or null
  const float* mix;        // [H][H]
  float q_scale;
  const int* slot;         // physical cache slot (page * page_size + offset); < 0: no cache write
  int H, G, dim, DK, page_size;
  float* q32;              // [T][H][G * DK] or null
  __half* q16;             // the same, or null
};
__device__ __forceinline__ void put8(float* p, const float (&v)[8]) {
  *(float4*)p = make_float4(v[0], v[1], v[2], v[3]);
  *(float4*)(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}
__device__ __forceinline__ void put8(__half* p, const float (&v)[8]) {
  uint4 o;
  __half2* h = (__half2*)&o;
#pragma unroll
  for (int i = 0; i < 4; i++) h[i] = __floats2half2_rn(v[2 * i], v[2 * i + 1]);
  *(uint4*)p = o;
}
// One block per token.  A thread keeps eight columns of one group's queries (REP of them; REP = 0: any number, read again for every head) and
// walks the heads: REP multiply-adds per result, results leave as whole rows.  VEC: rows, heads and bias come in 16-byte pieces.
template <int REP, bool VEC, typename CT>
__global__ void __launch_bounds__(256) mixed_finish_kernel(const MixedArgs a, CT* __restrict__ kc) {
  extern __shared__ __align__(16) float sT[];       // [H][H]
  const int t = blockIdx.x, tid = threadIdx.x, rep = REP ? REP : a.H / a.G;
  for (int i = tid; i < a.H * a.H; i += 256) sT[i] = a.mix[i];
  pdl_trigger();
  pdl_wait();
  const float* row = a.in + (size_t)t * a.ld;
  const int n8 = a.G * a.DK >> 3, d8 = a.DK >> 3;   // pieces of eight columns of a cache row, of one head
  const int shares = max(1, 256 / n8), per = (a.H + shares - 1) / shares;
  auto fetch = [&](int col, int d, float (&v)[8]) {
    if constexpr (VEC) {
      float4 x = make_float4(0.f, 0.f, 0.f, 0.f), y = x;
      if (d < a.dim) {
        x = *(const float4*)(row + col + d);
        y = *(const float4*)(row + col + d + 4);
        if (a.bias) {
          const float4 p = *(const float4*)(a.bias + col + d), q = *(const float4*)(a.bias + col + d + 4);
          x.x += p.x; x.y += p.y; x.z += p.z; x.w += p.w;
          y.x += q.x; y.y += q.y; y.z += q.z; y.w += q.w;
        }
      }
      v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w; v[4] = y.x; v[5] = y.y; v[6] = y.z; v[7] = y.w;
    } else {
#pragma unroll
      for (int i = 0; i < 8; i++) v[i] = d + i < a.dim ? row[col + d + i] + (a.bias ? a.bias[col + d + i] : 0.f) : 0.f;
    }
  };
  const int s = a.slot[t];
  if (s >= 0)
    for (int p = tid; p < n8; p += 256) {
      float v[8];
      fetch(a.k_off + p / d8 * a.dim, (p % d8) << 3, v);
      put8(kc + ((size_t)(s / a.page_size) * a.page_size + s % a.page_size) * n8 * 8 + p * 8, v);
    }
  for (int it = tid; it < n8 * shares || it == tid; it += 256) {
    const bool live = it < n8 * shares;
    const int p = it % n8, c = p / d8, d = (p % d8) << 3, h0 = it / n8 * per, h1 = live ? min(a.H, h0 + per) : 0;
    float q[REP ? REP : 1][8];
    if constexpr (REP > 0) {
      if (live)
#pragma unroll
        for (int r = 0; r < REP; r++) {
          fetch((c * REP + r) * a.dim, d, q[r]);
#pragma unroll
          for (int i = 0; i < 8; i++) q[r][i] *= a.q_scale;
        }
    }
    if (it == tid) __syncthreads();                 // sT; every thread comes here once, its first queries on their way
    for (int h = h0; h < h1; h++) {
      const float* m = sT + h * a.H + c * rep;
      float o[8];
#pragma unroll
      for (int i = 0; i < 8; i++) o[i] = 0.f;
      if constexpr (REP > 0) {
#pragma unroll
        for (int r = 0; r < REP; r++)
#pragma unroll
          for (int i = 0; i < 8; i++) o[i] = fmaf(m[r], q[r][i], o[i]);
      } else {
        for (int r = 0; r < rep; r++) {
          fetch((c * rep + r) * a.dim, d, q[0]);
#pragma unroll
          for (int i = 0; i < 8; i++) o[i] = fmaf(m[r], q[0][i] * a.q_scale, o[i]);
        }
      }
      const size_t at = ((size_t)t * a.H + h) * n8 * 8 + p * 8;
      if (a.q32) put8(a.q32 + at, o);
      if (a.q16) put8(a.q16 + at, o);
    }
  }
}
template <bool VEC, typename CT>
static int launch_mixed_finish(int T, const MixedArgs& a, CT* kc, cudaStream_t st) {
  const size_t smem = (size_t)a.H * a.H * 4;
  auto kern = mixed_finish_kernel<0, VEC, CT>;
  switch (a.H / a.G) {
    case 1: kern = mixed_finish_kernel<1, VEC, CT>; break;
    case 2: kern = mixed_finish_kernel<2, VEC, CT>; break;
    case 4: kern = mixed_finish_kernel<4, VEC, CT>; break;
    case 8: kern = mixed_finish_kernel<8, VEC, CT>; break;
  }
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  return launch_pdl(kern, dim3(T), dim3(256), smem, st, a, kc);
}
// kc [page][page_size][G * DK], fp32 (cache_f32) or fp16; DK a multiple of 8, at most 224 query heads.
B200_API int b200_mixed_finish(const float* in, int ld, int T, int k_off, const float* bias, const float* mix, float q_scale, const int* slot,
                               int H, int G, int dim, int DK, int page_size, float* q32, void* q16, void* kc, int cache_f32, cudaStream_t st) {
  if (T < 1 || G < 1 || H < 1 || H % G || H > 224 || dim < 1 || DK < dim || DK % 8 || page_size < 1 || (!q32 && !q16) || !kc || !mix || !slot ||
      k_off < H * dim || ld < k_off + G * dim || ((uintptr_t)q32 | (uintptr_t)q16 | (uintptr_t)kc) & 15)
    return B200_ERR_BAD_ARG;
  MixedArgs a;
  a.in = in; a.ld = ld; a.k_off = k_off; a.bias = bias; a.mix = mix; a.q_scale = q_scale; a.slot = slot; a.H = H; a.G = G; a.dim = dim; a.DK = DK;
  a.page_size = page_size; a.q32 = q32; a.q16 = (__half*)q16;
  const bool vec = ((ld | k_off | dim) & 7) == 0 && (((uintptr_t)in | (uintptr_t)bias) & 15) == 0;
  if (vec) return cache_f32 ? launch_mixed_finish<true>(T, a, (float*)kc, st) : launch_mixed_finish<true>(T, a, (__half*)kc, st);
  return cache_f32 ? launch_mixed_finish<false>(T, a, (float*)kc, st) : launch_mixed_finish<false>(T, a, (__half*)kc, st);
}

// ------------------------------------------------------------------ decoding: one query token per sequence

// Grid (shares of the keys, sequences).  Pages come whole, all key heads of 16 tokens, in one TMA copy each: [2][W / 64][8 rows][128 bytes], swizzled,
// into a ring.  Two warps work on a page, each for half of the query heads (a slot of the ring is always the same pair's):
//   raw scores      S^T = K Q^T per key head, 16 keys x 8 query heads a tile; the two warps swap theirs through shared memory
//   mixture         S^T T^T on bf16 products: the scores as three bf16 pieces (24 bits: fp32's own), T is stored in bf16
//   softmax         running, in base 2; a head's offset moves only when its maximum has grown by 2^8
//   output          O^T += K^T P^T, the transposed weights coming from movmatrix
// A group's query heads are padded to RP of 1, 2, 4 or a multiple of 8.  Where a tile's eight heads belong to several groups, the raw product runs
// over all their keys with the other groups' queries as zeros, and the output product puts 8 keys of two groups into one step of 16.
struct MixedDecArgs {
  const float* q;          // [B][H * DK], scaled
  const uint2* mix;        // the mixture as B operand (see mixed_prepare_kernel), then the padded heads' slopes
  const float* sinks;      // [H] or null
  const int* page_table;
  const int* seq_lens;
  int max_pages, H, G, rp, window, S, nslot;
  float* out_f32;          // [B][H * DK]
  __nv_bfloat16* out_bf16;
  float* part_acc;         // [B][S][8 NT][DK]
  float* part_ml;          // [B][S][8 NT][2]
  int* status;
};
__device__ __forceinline__ float2 split_bf16(float x, float y, uint32_t& packed) {      // the pair's bf16 values, and what they leave
  const __nv_bfloat162 p = __floats2bfloat162_rn(x, y);
  packed = *(const uint32_t*)&p;
  const float2 f = __bfloat1622float2(p);
  return make_float2(x - f.x, y - f.y);
}
__device__ __forceinline__ void pair_barrier(int pair) { asm volatile("bar.sync %0, 64;" ::"r"(pair + 1) : "memory"); }

// Once per layer, at load: out [NT / 2][NT][32 lanes] = the fragments of T^T (rows the raw slots, columns the mixed ones), and [8 NT] slopes in base 2.
__global__ void mixed_prepare_kernel(const float* __restrict__ mix, const float* __restrict__ slopes, int H, int G, int rp, int NT, uint2* __restrict__ out) {
  const int rep = H / G, n = NT / 2 * NT * 32;
  auto head_of = [&](int slot) { return slot < G * rp && slot % rp < rep ? slot / rp * rep + slot % rp : -1; };
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    const int l = i & 31, nt = (i >> 5) % NT, kk = (i >> 5) / NT, ho = head_of(nt * 8 + (l >> 2));
    uint32_t w[2];
    for (int e = 0; e < 2; e++) {
      const int k = kk * 16 + e * 8 + (l & 3) * 2, h0 = head_of(k), h1 = head_of(k + 1);
      const __nv_bfloat162 v = __floats2bfloat162_rn(ho >= 0 && h0 >= 0 ? mix[ho * H + h0] : 0.f, ho >= 0 && h1 >= 0 ? mix[ho * H + h1] : 0.f);
      w[e] = *(const uint32_t*)&v;
    }
    out[i] = make_uint2(w[0], w[1]);
  }
  for (int i = threadIdx.x; i < 8 * NT; i += blockDim.x) {
    const int h = head_of(i);
    ((float*)(out + n))[i] = h >= 0 && slopes ? slopes[h] * kLog2e : 0.f;
  }
}

// NT: tiles of eight (padded) query heads, an even number; THREADS: at most that many (registers).
template <int DK, int NT, int THREADS>
__global__ void __launch_bounds__(THREADS, 1) mixed_decode_kernel(const __grid_constant__ CUtensorMap tm, const MixedDecArgs a) {
  constexpr int QLD = DK + 8, KB = DK / 64, NW = NT / 2, SLOTS = 8 * NT;       // NW: tiles of a warp
  extern __shared__ uint8_t dyn_raw[];
  __shared__ float s_ml[THREADS / 64][SLOTS][2];
  __shared__ int s_fail[THREADS / 64];
  __shared__ int s_abort;
  uint8_t* ring = (uint8_t*)(((uintptr_t)dyn_raw + 1023) & ~(uintptr_t)1023);
  const int W = a.G * DK, page_bytes = 32 * W, NB = W / 64, pairs = blockDim.x >> 6;
  float* s_acc = (float*)ring;                                           // [pairs][SLOTS][DK], once the pages are done with
  const size_t ring_bytes = max((size_t)a.nslot * page_bytes, (size_t)pairs * SLOTS * DK * 4);
  uint64_t* bars = (uint64_t*)(ring + ring_bytes);
  float4* sX = (float4*)(bars + ((a.nslot + 1) & ~1));                   // [pairs][2][NW][32] raw scores on their way to the partner
  uint2* sT = (uint2*)(sX + pairs * NT * 32);                            // [NT / 2][NT][32]
  __half* sQ = (__half*)(sT + NT / 2 * NT * 32);                         // [SLOTS + 1][QLD], the last row zeros
  int* s_pid = (int*)(sQ + (SLOTS + 1) * QLD);

  const int split = blockIdx.x, b = blockIdx.y;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g4 = lane >> 2, t4 = lane & 3;
  const int pair = warp >> 1, hf = warp & 1, T0 = hf * NW;               // this warp's first tile
  const int rp = a.rp, rep = a.H / a.G, nsub = rp < 8 ? 8 / rp : 1;
  if (tid == 0) {
    for (int s = 0; s < a.nslot; s++) mbar_init(smem_u32(bars + s), 1);
    s_abort = 0;
    fence_barrier_init();
    tma_prefetch_desc(&tm);
  }
  if (tid < pairs) s_fail[tid] = 0;
  for (int i = tid; i < (SLOTS + 1) * QLD / 8; i += blockDim.x) ((uint4*)sQ)[i] = make_uint4(0u, 0u, 0u, 0u);
  for (int i = tid; i < NT * NT * 8; i += blockDim.x) ((uint4*)sT)[i] = ((const uint4*)a.mix)[i];           // weights: nothing to wait for
  float sl[NW][2];
#pragma unroll
  for (int nt = 0; nt < NW; nt++)
#pragma unroll
    for (int e = 0; e < 2; e++) sl[nt][e] = ((const float*)(a.mix + NT * NT * 16))[(T0 + nt) * 8 + 2 * t4 + e];
  pdl_trigger();
  pdl_wait();
  const int len = a.seq_lens[b];
  const int first = a.window > 0 && len > a.window ? len - a.window : 0;
  const int p_first = first >> 4, p_last = (len + 15) >> 4;
  const int per = (p_last - p_first + a.S - 1) / a.S;
  const int pa = p_first + split * per, np = max(0, min(p_last, pa + per) - pa);
  const int* pt = a.page_table + (size_t)b * a.max_pages;
  auto issue = [&](int i, int page) {   // one lane: page i of the share into its slot
    const uint32_t bar = smem_u32(bars + i % a.nslot);
    mbar_expect_tx(bar, page_bytes);
    tma_load_4d(smem_u32(ring + (size_t)(i % a.nslot) * page_bytes), &tm, bar, 0, 0, 0, page * 2);
  };
  __syncthreads();
  if (lane == 0 && hf == 0)
    for (int i = pair; i < min(np, a.nslot); i += pairs) issue(i, pt[pa + i]);
  for (int i = tid; i < np; i += blockDim.x) s_pid[i] = pt[pa + i];
  for (int i = tid; i < a.H * (DK / 4); i += blockDim.x) {
    const int h = i / (DK / 4), c = i % (DK / 4) * 4;
    const float4 v = ((const float4*)(a.q + (size_t)b * a.H * DK))[i];
    *(uint2*)(sQ + (h / rep * rp + h % rep) * QLD + c) = make_uint2(pack_h2(v.x, v.y), pack_h2(v.z, v.w));
  }
  __syncthreads();

  float o[NW][DK / 16][4], mu[NW][2], l[NW][2];
#pragma unroll
  for (int nt = 0; nt < NW; nt++) {
#pragma unroll
    for (int m = 0; m < DK / 16; m++) o[nt][m][0] = o[nt][m][1] = o[nt][m][2] = o[nt][m][3] = 0.f;
    mu[nt][0] = mu[nt][1] = -INFINITY;
    l[nt][0] = l[nt][1] = 0.f;
  }
  const int mi = lane >> 3, r8 = lane & 7;              // ldmatrix: tile and row of this lane's address
  float4* xs = sX + (size_t)pair * NT * 32 + lane;      // [2][NW], 32 apart
  for (int i = pair; i < np; i += pairs) {
    const int s = i % a.nslot;
    bool ok = mbar_wait(smem_u32(bars + s), (uint32_t)((i / a.nslot) & 1), &s_abort);
    ok = __all_sync(0xffffffffu, ok);
    if (!ok) s_fail[pair] = 1;                           // both warps meet at the barrier below and leave together
    const uint32_t page = smem_u32(ring) + (uint32_t)(s * page_bytes);
    // key row `row` of the page at key head c, and 16-byte piece `ch` of it (r8: the row's place among its eight)
    auto row_at = [&](int row, int c) { return page + (uint32_t)((row >> 3) * NB + c * KB) * 1024u + (uint32_t)r8 * 128u; };
    auto piece_at = [&](int ch) { return (uint32_t)(ch >> 3) * 1024u + (uint32_t)(((ch & 7) ^ r8) << 4); };
    float sc[NW][4];
#pragma unroll
    for (int j = 0; j < NW; j++) sc[j][0] = sc[j][1] = sc[j][2] = sc[j][3] = 0.f;
#pragma unroll 1
    for (int u = 0; u < nsub; u++) {
      uint32_t ka[NW], qa[NW];                            // tile j: this lane's key row of the u-th head the tile meets, its query row
#pragma unroll
      for (int j = 0; j < NW; j++) {
        const int c = rp < 8 ? (T0 + j) * nsub + u : (T0 + j) * 8 / rp;
        ka[j] = row_at(r8 + (mi & 1) * 8, min(c, a.G - 1));       // (a head that is not there meets zero queries)
        qa[j] = smem_u32(sQ + ((rp >= 8 || r8 / rp == u) ? (T0 + j) * 8 + r8 : SLOTS) * QLD + mi * 8);
      }
#pragma unroll
      for (int kk = 0; kk < DK / 32; kk++)
#pragma unroll
        for (int j = 0; j < NW; j++) {
          uint32_t k0[4], k1[4], q[4];
          ldsm_x4(ka[j] + piece_at(kk * 4 + (mi >> 1)), k0[0], k0[1], k0[2], k0[3]);
          ldsm_x4(ka[j] + piece_at(kk * 4 + 2 + (mi >> 1)), k1[0], k1[1], k1[2], k1[3]);
          ldsm_x4(qa[j] + kk * 64, q[0], q[1], q[2], q[3]);
          mma16816(sc[j], k0, q[0], q[1]);
          mma16816(sc[j], k1, q[2], q[3]);
        }
    }
    // the partner's tiles
    float ot[NW][4];
#pragma unroll
    for (int j = 0; j < NW; j++) xs[(hf * NW + j) * 32] = make_float4(sc[j][0], sc[j][1], sc[j][2], sc[j][3]);
    pair_barrier(pair);
    if (*(volatile int*)&s_fail[pair]) break;
#pragma unroll
    for (int j = 0; j < NW; j++) {
      const float4 v = xs[((hf ^ 1) * NW + j) * 32];
      ot[j][0] = v.x; ot[j][1] = v.y; ot[j][2] = v.z; ot[j][3] = v.w;
    }
    float d[NW][4];
#pragma unroll
    for (int nt = 0; nt < NW; nt++) d[nt][0] = d[nt][1] = d[nt][2] = d[nt][3] = 0.f;
    auto mix_step = [&](int kk, const float (&x)[4], const float (&y)[4]) {      // raw slots 16 kk .. 16 kk + 15
      uint32_t hi[4], md[4], lo[4];
#pragma unroll
      for (int p = 0; p < 4; p++) {
        const float* v = (p < 2 ? x : y) + (p & 1) * 2;
        float2 r = split_bf16(v[0], v[1], hi[p]);
        r = split_bf16(r.x, r.y, md[p]);
        split_bf16(r.x, r.y, lo[p]);
      }
      uint2 w[NW];
#pragma unroll
      for (int nt = 0; nt < NW; nt++) w[nt] = sT[(kk * NT + T0 + nt) * 32 + lane];
#pragma unroll
      for (int nt = 0; nt < NW; nt++) mma16816_bf16(d[nt], lo, w[nt].x, w[nt].y);
#pragma unroll
      for (int nt = 0; nt < NW; nt++) mma16816_bf16(d[nt], md, w[nt].x, w[nt].y);
#pragma unroll
      for (int nt = 0; nt < NW; nt++) mma16816_bf16(d[nt], hi, w[nt].x, w[nt].y);
    };
    if constexpr (NW == 1) {
      if (hf == 0) mix_step(0, sc[0], ot[0]);
      else mix_step(0, ot[0], sc[0]);
    } else {
#pragma unroll
      for (int k = 0; k < NW / 2; k++) mix_step(hf * (NW / 2) + k, sc[2 * k], sc[2 * k + 1]);
#pragma unroll
      for (int k = 0; k < NW / 2; k++) mix_step((hf ^ 1) * (NW / 2) + k, ot[2 * k], ot[2 * k + 1]);
    }
    const int t0 = (pa + i) * 16 + g4, t1 = t0 + 8;
    const bool in0 = t0 >= first && t0 < len, in1 = t1 >= first && t1 < len;
    const float f0 = (float)(len - 1 - t0), f1 = (float)(len - 1 - t1);
    bool grown = false;
#pragma unroll
    for (int nt = 0; nt < NW; nt++)
#pragma unroll
      for (int e = 0; e < 2; e++) {
        d[nt][e] = in0 ? fmaf(d[nt][e], kLog2e, -sl[nt][e] * f0) : -INFINITY;
        d[nt][e + 2] = in1 ? fmaf(d[nt][e + 2], kLog2e, -sl[nt][e] * f1) : -INFINITY;
        grown |= fmaxf(d[nt][e], d[nt][e + 2]) > mu[nt][e] + 8.f;
      }
    if (__any_sync(0xffffffffu, grown)) {
#pragma unroll
      for (int nt = 0; nt < NW; nt++)
#pragma unroll
        for (int e = 0; e < 2; e++) {
          float mx = fmaxf(d[nt][e], d[nt][e + 2]);
          mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 4));
          mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 8));
          mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 16));
          mx = fmaxf(mx, mu[nt][e]);
          const float c = mu[nt][e] == -INFINITY ? 0.f : ex2_approx(mu[nt][e] - mx);
          mu[nt][e] = mx;
          l[nt][e] *= c;
#pragma unroll
          for (int m = 0; m < DK / 16; m++) {
            o[nt][m][e] *= c;
            o[nt][m][e + 2] *= c;
          }
        }
    }
#pragma unroll
    for (int nt = 0; nt < NW; nt++) {
      float p[4];
#pragma unroll
      for (int e = 0; e < 2; e++) {
        const float off = mu[nt][e] == -INFINITY ? 0.f : mu[nt][e];
        p[e] = ex2_approx(d[nt][e] - off);
        p[e + 2] = ex2_approx(d[nt][e + 2] - off);
        l[nt][e] += p[e] + p[e + 2];
      }
      const uint32_t w[2] = {transpose_8x8(pack_h2(p[0], p[1])), transpose_8x8(pack_h2(p[2], p[3]))};      // keys 0..7, 8..15 of head g4
      const int tile = T0 + nt;
      if (rp >= 8) {
        const uint32_t at = row_at(r8 + (mi >> 1) * 8, min(tile * 8 / rp, a.G - 1));
#pragma unroll
        for (int m = 0; m < DK / 16; m++) {
          uint32_t k[4];
          ldsm_x4_t(at + piece_at(m * 2 + (mi & 1)), k[0], k[1], k[2], k[3]);
          mma16816(o[nt][m], k, w[0], w[1]);
        }
      } else {
#pragma unroll 1
        for (int pr = 0; pr < nsub >> 1; pr++) {
          const int c = min(tile * nsub + 2 * pr + (mi >> 1), a.G - 1), sub = g4 / rp - 2 * pr;
          const uint32_t at = row_at(r8, c);
#pragma unroll
          for (int kg = 0; kg < 2; kg++) {
            const uint32_t b0 = sub == 0 ? w[kg] : 0u, b1 = sub == 1 ? w[kg] : 0u;
#pragma unroll
            for (int m = 0; m < DK / 16; m++) {
              uint32_t k[4];
              ldsm_x4_t(at + (uint32_t)(kg * NB) * 1024u + piece_at(m * 2 + (mi & 1)), k[0], k[1], k[2], k[3]);
              mma16816(o[nt][m], k, b0, b1);
            }
          }
        }
      }
    }
    pair_barrier(pair);                                  // both are done with the page, and with each other's scores
    if (lane == 0 && hf == 0 && i + a.nslot < np) issue(i + a.nslot, s_pid[i + a.nslot]);
  }
  __syncthreads();                                      // every page has been read: the ring becomes the partial outputs
  if (tid == 0 && s_abort && a.status) atomicExch(a.status, (int)B200_ERR_TIMEOUT_TMA);
  if (s_abort) drain_after_abort();
  __syncthreads();
#pragma unroll
  for (int nt = 0; nt < NW; nt++)
#pragma unroll
    for (int e = 0; e < 2; e++) {
      float v = l[nt][e];
      v += __shfl_xor_sync(0xffffffffu, v, 4);
      v += __shfl_xor_sync(0xffffffffu, v, 8);
      v += __shfl_xor_sync(0xffffffffu, v, 16);
      const int slot = (T0 + nt) * 8 + 2 * t4 + e;
      if (g4 == 0) {
        s_ml[pair][slot][0] = mu[nt][e];
        s_ml[pair][slot][1] = v;
      }
      float* acc = s_acc + ((size_t)pair * SLOTS + slot) * DK;
#pragma unroll
      for (int m = 0; m < DK / 16; m++) {
        acc[m * 16 + g4] = o[nt][m][e];
        acc[m * 16 + g4 + 8] = o[nt][m][e + 2];
      }
    }
  __syncthreads();
  // the pairs' shares: each one's factor per head takes the place of its maximum
  const size_t row = ((size_t)b * a.S + split) * SLOTS;
  for (int slot = tid; slot < SLOTS; slot += blockDim.x) {
    const int h = slot % rp < rep && slot < a.G * rp ? slot / rp * rep + slot % rp : -1;
    float M = -INFINITY, L = 0.f;
    for (int w = 0; w < pairs; w++) M = fmaxf(M, s_ml[w][slot][0]);
    const bool last = a.S == 1;
    const float sk = last && a.sinks && h >= 0 ? a.sinks[h] * kLog2e : -INFINITY, M2 = fmaxf(M, sk);
    for (int w = 0; w < pairs; w++) {
      const float c = s_ml[w][slot][0] == -INFINITY ? 0.f : ex2_approx(s_ml[w][slot][0] - M2);
      L += s_ml[w][slot][1] * c;
      s_ml[w][slot][0] = c;
    }
    if (last) {
      if (sk != -INFINITY) L += ex2_approx(sk - M2);
      const float inv = L > 0.f ? 1.f / L : 0.f;
      for (int w = 0; w < pairs; w++) s_ml[w][slot][0] *= inv;
    } else {
      a.part_ml[(row + slot) * 2] = M;
      a.part_ml[(row + slot) * 2 + 1] = L;
    }
  }
  __syncthreads();
  for (int x = tid; x < SLOTS * (DK / 4); x += blockDim.x) {
    const int slot = x / (DK / 4), e = x % (DK / 4) * 4;
    float4 A = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int w = 0; w < pairs; w++) {
      const float4 v = *(const float4*)(s_acc + ((size_t)w * SLOTS + slot) * DK + e);
      const float c = s_ml[w][slot][0];
      A.x = fmaf(v.x, c, A.x); A.y = fmaf(v.y, c, A.y); A.z = fmaf(v.z, c, A.z); A.w = fmaf(v.w, c, A.w);
    }
    if (a.S > 1) {
      *(float4*)(a.part_acc + (row + slot) * DK + e) = A;
    } else if (slot < a.G * rp && slot % rp < rep) {
      const size_t at = ((size_t)b * a.H + slot / rp * rep + slot % rp) * DK + e;
      if (a.out_f32) *(float4*)(a.out_f32 + at) = A;
      if (a.out_bf16) {
        const __nv_bfloat162 p0 = __floats2bfloat162_rn(A.x, A.y), p1 = __floats2bfloat162_rn(A.z, A.w);
        *(uint2*)(a.out_bf16 + at) = make_uint2(*(const uint32_t*)&p0, *(const uint32_t*)&p1);
      }
    }
  }
}
// The shares of one (sequence, head): a thread per output column.
template <int DK>
__global__ void __launch_bounds__(DK) mixed_merge_kernel(const float* __restrict__ acc, const float* __restrict__ ml, const float* __restrict__ sinks,
                                                         int H, int rep, int rp, int n_slots, int S, float* __restrict__ out_f32,
                                                         __nv_bfloat16* __restrict__ out_bf16) {
  pdl_trigger();
  pdl_wait();
  const int h = blockIdx.x, b = blockIdx.y, e = threadIdx.x, slot = h / rep * rp + h % rep, lane = e & 31;
  const size_t row = (size_t)b * S;
  // lane s holds share s (up to 64 shares: two each)
  float m[2], l[2], M = sinks ? sinks[h] * kLog2e : -INFINITY;
#pragma unroll
  for (int k = 0; k < 2; k++) {
    const int s = lane + 32 * k;
    m[k] = s < S ? ml[((row + s) * n_slots + slot) * 2] : -INFINITY;
    l[k] = s < S ? ml[((row + s) * n_slots + slot) * 2 + 1] : 0.f;
  }
  M = fmaxf(M, warp_max(fmaxf(m[0], m[1])));
  float c[2], L = 0.f;
#pragma unroll
  for (int k = 0; k < 2; k++) {
    c[k] = m[k] == -INFINITY ? 0.f : ex2_approx(m[k] - M);
    L += l[k] * c[k];
  }
  L = warp_sum(L);
  if (sinks) L += ex2_approx(sinks[h] * kLog2e - M);
  float A = 0.f;
  for (int s0 = 0; s0 < S; s0 += 8) {
    float v[8];
#pragma unroll
    for (int i = 0; i < 8; i++) v[i] = s0 + i < S ? acc[((row + s0 + i) * n_slots + slot) * DK + e] : 0.f;
#pragma unroll
    for (int i = 0; i < 8; i++) A = fmaf(v[i], __shfl_sync(0xffffffffu, s0 < 32 ? c[0] : c[1], (s0 + i) & 31), A);
  }
  const float v = L > 0.f ? A / L : 0.f;
  const size_t at = ((size_t)b * H + h) * DK + e;
  if (out_f32) out_f32[at] = v;
  if (out_bf16) out_bf16[at] = __float2bfloat16(v);
}

// Padded group size and tiles of eight padded heads (2, 4 or 8); false: sizes the kernel does not take.
static bool mixed_decode_plan(int H, int G, int DK, int& rp, int& nt) {
  if (G < 1 || H < 1 || H % G || (DK != 64 && DK != 128)) return false;
  const int rep = H / G;
  rp = rep <= 1 ? 1 : rep <= 2 ? 2 : rep <= 4 ? 4 : (rep + 7) / 8 * 8;
  const int tiles = (G * rp + 7) / 8;
  nt = tiles <= 2 ? 2 : tiles <= 4 ? 4 : 8;
  return tiles <= 8 && G * DK <= 1536;
}
B200_API int b200_mixed_decode_ok(int H, int G, int DK) {
  int rp, nt;
  return mixed_decode_plan(H, G, DK, rp, nt) ? 1 : 0;
}
B200_API size_t b200_mixed_decode_scratch_floats(int B, int H, int G, int DK, int S) {
  int rp, nt;
  return mixed_decode_plan(H, G, DK, rp, nt) ? (size_t)B * S * nt * 8 * (DK + 2) : 0;
}
// 32-bit words of what b200_mixed_decode_prepare writes.
B200_API size_t b200_mixed_decode_prepared_words(int H, int G, int DK) {
  int rp, nt;
  return mixed_decode_plan(H, G, DK, rp, nt) ? (size_t)nt * nt * 32 + 8 * nt : 0;
}
// mix fp32 [H][H] (bf16 values), slopes [H] of the mixed scores (or null) -> the form the decode kernel reads.
B200_API int b200_mixed_decode_prepare(const float* mix, const float* slopes, int H, int G, int DK, void* out, cudaStream_t st) {
  int rp, nt;
  if (!mix || !out || ((uintptr_t)out & 15) || !mixed_decode_plan(H, G, DK, rp, nt)) return B200_ERR_BAD_ARG;
  mixed_prepare_kernel<<<1, 256, 0, st>>>(mix, slopes, H, G, rp, nt, (uint2*)out);
  return (int)cudaGetLastError();
}
template <int DK, int NT, int THREADS>
static int launch_mixed_decode(MixedDecArgs a, const void* kc, int n_pages, int B, float* scratch, cudaStream_t st) {
  const int W = a.G * DK, page = 32 * W;
  const size_t out = (size_t)NT * 8 * DK * 4;
  const int listed = a.window > 0 ? min(a.max_pages, a.window / 16 + 2) : a.max_pages;      // pages a share can have
  const size_t fixed = 1024 + 20 * 8 + NT * NT * 128 + (8 * NT + 1) * (DK + 8) * 2 + ((size_t)listed + 4) * 4;
  if (fixed > 100 * 1024) return B200_ERR_BAD_ARG;
  const size_t room = 222 * 1024 - fixed;               // (the rest of an SM's: this kernel's static part)
  int pairs = 0;
  for (int p = THREADS / 64; p >= 1 && (!pairs || p > THREADS / 128); p--) {      // the most pages in flight, of many warps
    const size_t left = room - (size_t)p * NT * 512;
    const int cap = (int)(left / page < 18 ? left / page : 18);
    if (cap >= p && p * out <= left && (!pairs || cap / p * p > a.nslot)) {
      pairs = p;
      a.nslot = cap / p * p;
    }
  }
  if (!pairs) return B200_ERR_BAD_ARG;
  a.part_acc = scratch;
  a.part_ml = scratch ? scratch + (size_t)B * a.S * NT * 8 * DK : nullptr;
  const size_t ring = (size_t)a.nslot * page > pairs * out ? (size_t)a.nslot * page : pairs * out, smem = fixed + (size_t)pairs * NT * 512 + ring;
  auto kern = mixed_decode_kernel<DK, NT, THREADS>;
  static size_t configured = 0;
  if (smem > configured) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = smem;
  }
  CUtensorMap tm;
  const int rc = make_tmap_rows8(&tm, kc, (uint64_t)n_pages * 16, W, W / 64);
  if (rc) return rc;
  const int err = launch_pdl(kern, dim3(a.S, B), dim3(64 * pairs), smem, st, tm, a);
  if (err || a.S == 1) return err;
  return launch_pdl(mixed_merge_kernel<DK>, dim3(a.H, B), dim3(DK), 0, st, (const float*)a.part_acc, (const float*)a.part_ml, a.sinks, a.H, a.H / a.G, a.rp, NT * 8,
                    a.S, a.out_f32, a.out_bf16);
}
// q fp32 [B][H][DK], scaled; mix: prepared (above); kc fp16 [n_pages][16][G * DK]; sizes as b200_mixed_decode_ok has them.  S: shares of the keys, at
// most 64 (scratch where there are several).
B200_API int b200_mixed_decode(const float* q, const void* kc, const void* mix, const float* sinks, const int* page_table, int max_pages, int n_pages,
                               const int* seq_lens, int B, int H, int G, int DK, int window, int S, float* out_f32, void* out_bf16, float* scratch,
                               int* status, cudaStream_t st) {
  MixedDecArgs a = {};
  int nt;
  if (B < 1 || S < 1 || S > 64 || window < 0 || max_pages < 1 || !q || !kc || !mix || (!out_f32 && !out_bf16) || (S > 1 && !scratch) ||
      !mixed_decode_plan(H, G, DK, a.rp, nt) || (((uintptr_t)q | (uintptr_t)mix) & 15))
    return B200_ERR_BAD_ARG;
  a.q = q; a.mix = (const uint2*)mix; a.sinks = sinks; a.page_table = page_table; a.seq_lens = seq_lens; a.max_pages = max_pages; a.H = H; a.G = G;
  a.window = window; a.S = S; a.out_f32 = out_f32; a.out_bf16 = (__nv_bfloat16*)out_bf16; a.status = status;
  if (DK == 64) {
    if (nt == 2) return launch_mixed_decode<64, 2, 384>(a, kc, n_pages, B, scratch, st);
    if (nt == 4) return launch_mixed_decode<64, 4, 384>(a, kc, n_pages, B, scratch, st);
    return launch_mixed_decode<64, 8, 384>(a, kc, n_pages, B, scratch, st);
  }
  if (nt == 2) return launch_mixed_decode<128, 2, 384>(a, kc, n_pages, B, scratch, st);
  if (nt == 4) return launch_mixed_decode<128, 4, 384>(a, kc, n_pages, B, scratch, st);
  return launch_mixed_decode<128, 8, 256>(a, kc, n_pages, B, scratch, st);
}

// ------------------------------------------------------------------ prompts: wide queries on the 5th-generation tensor cores

// One CTA = 128 query rows of one head against blocks of 128 keys, in the manner of attn_prefill_tc05.cu: two warps that copy keys, one warp that issues
// the score products, one for the output products, eight softmax warps (two to a tensor-memory quarter, half of a block's keys and of the output
// columns each).  What differs:
//   - a score is a product over G slices (a key head's DK columns each); slices of 128 keys are the entries of the ring.  The head's own slice comes
//     last in a block: it is the value operand too, and its entry is given back by the output product instead of the score product.
//   - a slice is gathered from eight pages.  16-byte asynchronous copies by 64 threads do that in some 500 cycles; TMA copies of a page's part each
//     (4 KB) took 1600.
//   - the wide query row lies in tensor memory as far as that reaches (QT slices), the rest in shared memory, both read as the A operand.
//   - where the slices leave no room for two score accumulators (NS = 1), a block's score product waits for the output product before it.
//   - slopes: one multiply-add per score, the block's part of the distance joins the exponent's offset.
constexpr int QB = 128, KEYS = 128;
constexpr uint32_t kTmemCols = 512;
constexpr float kRescale = 8.f;                   // log2 units

struct MixedPreArgs {
  const __half* q;         // [T_total][H][G * DK], mixed and scaled
  const __half* kc;        // [pages][16][G * DK]
  const float* slopes;     // [H] or null
  const float* sinks;      // [H] or null
  const int* page_table;
  const int* q_start;
  const int* q_len;
  const int* ctx_len;
  int max_pages, H, G, T_total, window, QT, R;    // R: ring entries
  __nv_bfloat16* out;      // [T_total][H * DK]
  float* out_f32;          // instead of out where given
  int* status;
};

template <int DK, int NS>
__global__ void __launch_bounds__(384, 1) mixed_prefill_kernel(const __grid_constant__ CUtensorMap tmQ, const MixedPreArgs a) {
  constexpr int CB = DK / 64, SLICE = KEYS * DK * 2, BOX = KEYS * 128;        // BOX: 64 columns of a slice, [128 rows][128 bytes]
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  const int QS = a.G - a.QT, R = a.R;
  uint8_t* sQ = smem;                                     // QS slices of the queries, [CB][128 rows][128 bytes] each
  uint8_t* sK = sQ + (size_t)QS * SLICE;                  // R ring entries
  uint64_t* bars = (uint64_t*)(sK + (size_t)R * SLICE);
  uint64_t* q_full = bars;                                // [1] the part in tensor memory
  uint64_t* qs_full = bars + 1;                           // [1] the part in shared memory
  uint64_t* s_full = bars + 2;                            // [2]
  uint64_t* s_empty = bars + 4;                           // [2]
  uint64_t* p_full = bars + 6;                            // [2]
  uint64_t* pv_done = bars + 8;                           // [2]
  uint64_t* x_full = bars + 10;                           // [4 quarters][2]
  uint64_t* qt_full = bars + 18;                          // [1] queries on their way to tensor memory have landed in the ring
  uint64_t* qt_empty = bars + 19;                         // [1] and have been read from it
  uint32_t* tmem_holder = (uint32_t*)(bars + 20);
  volatile int* abort_flag = (volatile int*)(tmem_holder + 1);
  uint64_t* k_full = bars + 22;                           // [R]
  uint64_t* k_empty = k_full + R;                         // [R]
  float* xch = (float*)(bars + 22 + 2 * R);               // [NS][2 (half)][128 rows]

  const int seq = blockIdx.z, h = blockIdx.x, qb = gridDim.y - 1 - blockIdx.y;   // every head's longest (latest) query blocks first
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    mbar_init(smem_u32(q_full), 8);
    mbar_init(smem_u32(qs_full), 1);
    mbar_init(smem_u32(qt_full), 1);
    mbar_init(smem_u32(qt_empty), 8);
    for (int s = 0; s < R; s++) {
      mbar_init(smem_u32(k_full + s), 64);
      mbar_init(smem_u32(k_empty + s), 1);
    }
    for (int s = 0; s < 2; s++) {
      mbar_init(smem_u32(s_full + s), 1);
      mbar_init(smem_u32(s_empty + s), 8);
      mbar_init(smem_u32(p_full + s), 8);
      mbar_init(smem_u32(pv_done + s), 1);
    }
    for (int s = 0; s < 8; s++) mbar_init(smem_u32(x_full + s), 2);
    *abort_flag = 0;
    fence_barrier_init();
    tma_prefetch_desc(&tmQ);
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(tmem_holder), kTmemCols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_holder;
  pdl_trigger();
  pdl_wait();

  const int qlen = a.q_len[seq], q0 = qb * QB;
  const bool live = q0 < qlen;            // a dead CTA still goes through the common exit (it holds tensor memory)
  const int ctx = a.ctx_len[seq], qs = a.q_start[seq], G = a.G, W = G * DK;
  const int own = h / (a.H / G);
  const int pos0 = ctx - qlen + q0;       // absolute position of this CTA's first query row
  const int k_hi = min(ctx, pos0 + QB), k_lo = a.window > 0 ? max(0, pos0 - a.window + 1) : 0;
  const int jb0 = k_lo / KEYS, nb = live ? (k_hi + KEYS - 1) / KEYS - jb0 : 0;
  const uint32_t S_T = tmem_base, O_T = tmem_base + NS * KEYS, Q_T = O_T + DK;
  // what goes to tensor memory passes through the place of the slices that stay in shared memory, where they are as many, else through the ring
  const bool in_place = QS >= a.QT;
  uint8_t* sStage = in_place ? sQ : sK;
  const int stage = in_place ? a.QT : R;

  if (warp == 0 || warp == 10) {
    // Entries e = j * G + u in order (block j, u-th slice of it), all by both warps: thread x copies 16-byte piece x % 8 of every eighth row.  The
    // barrier counts the threads whose copies have landed; the fence between those writes and the tensor cores' reads is the issuing warps'.
    if (nb > 0) {
      const int* pt = a.page_table + (size_t)seq * a.max_pages;
      bool ok = true;
      // the queries: QT slices by way of shared memory to tensor memory, `stage` at a time, the others to where they stay
      if (warp == 0 && lane == 0) {
        auto fetch = [&](uint8_t* to, int u, uint32_t bar) {
          for (int c = 0; c < CB; c++) tma_load_2d(smem_u32(to + c * BOX), &tmQ, bar, h * W + (own + 1 + u) % G * DK + c * 64, qs + q0);
        };
        for (int u0 = 0; u0 < a.QT && ok; u0 += stage) {
          const int n = min(stage, a.QT - u0);
          if (u0 > 0) ok = mbar_wait(smem_u32(qt_empty), (uint32_t)(u0 / stage - 1) & 1, abort_flag);
          if (!ok) break;
          mbar_expect_tx(smem_u32(qt_full), n * SLICE);
          for (int i = 0; i < n; i++) fetch(sStage + (size_t)i * SLICE, u0 + i, smem_u32(qt_full));
        }
      }
      ok = __all_sync(0xffffffffu, ok);
      if (!in_place && ok) ok = mbar_wait(smem_u32(q_full), 0, abort_flag);      // the ring is free for keys
      ok = __all_sync(0xffffffffu, ok);
      const int x = (warp == 0 ? 0 : 32) + lane, r0 = x >> 3, c0 = x & 7;
      const uint32_t dst0 = smem_u32(sK) + (uint32_t)(r0 * 128 + ((c0 ^ r0) << 4));
      const __half* src0 = a.kc + (size_t)r0 * W + c0 * 8;
      int s = 0, ph = 1;                           // slot of the entry and the parity of its being free
      auto fetch_rest = [&]() {                    // the slices that stay in shared memory, once nothing passes through there any more
        if (QS == 0 || !ok || warp != 0) return;
        if (in_place) ok = __all_sync(0xffffffffu, mbar_wait(smem_u32(q_full), 0, abort_flag));
        if (ok && lane == 0) {
          mbar_expect_tx(smem_u32(qs_full), QS * SLICE);
          for (int u = a.QT; u < G; u++)
            for (int c = 0; c < CB; c++)
              tma_load_2d(smem_u32(sQ + (size_t)(u - a.QT) * SLICE + c * BOX), &tmQ, smem_u32(qs_full), h * W + (own + 1 + u) % G * DK + c * 64, qs + q0);
        }
        __syncwarp();
      };
      if (!in_place) fetch_rest();
      for (int j = 0; j < nb && ok; j++) {
        const __half* page[KEYS / 16];             // read together: one at a time, their latency would bound the copies
#pragma unroll
        for (int p = 0; p < KEYS / 16; p++) {
          const int pi = (jb0 + j) * (KEYS / 16) + p;
          page[p] = src0 + (size_t)(pi * 16 < ctx ? pt[pi] : 0) * 16 * W;         // pages past the context are masked anyway
        }
        int sl = own;
        for (int u = 0; u < G; u++) {
          sl = sl + 1 == G ? 0 : sl + 1;
          ok = mbar_wait(smem_u32(k_empty + s), ph, abort_flag);
          ok = __all_sync(0xffffffffu, ok);
          if (!ok) break;
          const uint32_t dst = dst0 + (uint32_t)(s * SLICE);
#pragma unroll
          for (int p = 0; p < KEYS / 16; p++)
#pragma unroll
            for (int i = 0; i < 2; i++)
#pragma unroll
              for (int c = 0; c < CB; c++) cp_async16(dst + c * BOX + (p * 2 + i) * 1024, page[p] + sl * DK + c * 64 + (size_t)i * 8 * W);
          cp_async_arrive(smem_u32(k_full + s));
          if (++s == R) { s = 0; ph ^= 1; }
          if (in_place && j == 0 && u == min(a.QT, R) - 1) fetch_rest();      // behind the first keys, which need no more than tensor memory's part
        }
      }
      cp_async_wait_all();
    }
  } else if (warp == 1) {
    if (nb > 0) {                                  // the whole warp walks the loop, one lane issues: operands stay warp-uniform
      constexpr uint32_t idesc = idesc_f16(QB, KEYS, false);
      const bool issuer = elect_one();
      const uint64_t k0 = smem_desc_sw128(smem_u32(sK)), q0d = smem_desc_sw128(smem_u32(sQ));
      bool ok = mbar_wait(smem_u32(q_full), 0, abort_flag);
      int s = 0, ph = 0;                           // slot and parity of the entry
      for (int j = 0; j < nb && ok; j++) {
        const int b = j % NS, use = j / NS;
        if (!mbar_wait(smem_u32(s_empty + b), (uint32_t)(use & 1) ^ 1, abort_flag)) break;
        if (j >= NS && !mbar_wait(smem_u32(pv_done + b), (uint32_t)(use - 1) & 1, abort_flag)) break;      // the weights before lie in this accumulator
        const uint32_t acc = S_T + b * KEYS;
        for (int u = 0; u < G; u++) {
          ok = mbar_wait(smem_u32(k_full + s), (uint32_t)ph, abort_flag) && (j > 0 || u != a.QT || mbar_wait(smem_u32(qs_full), 0, abort_flag));
          if (!ok) break;
          fence_proxy_async_smem();
          tc_fence_after();
          const uint64_t kd = k0 + (uint64_t)(s * (SLICE >> 4));
          if (issuer) {
            if (u < a.QT) {
              const uint32_t qt = Q_T + u * (DK / 2);
              umma_ts(acc, qt, kd, idesc, u != 0 ? 1u : 0u);
#pragma unroll
              for (int kk = 1; kk < DK / 16; kk++) umma_ts(acc, qt + 8 * kk, kd + ((kk >> 2) * (BOX >> 4) + 2 * (kk & 3)), idesc, 1u);
            } else {
              const uint64_t qd = q0d + (uint64_t)((u - a.QT) * (SLICE >> 4));
#pragma unroll
              for (int kk = 0; kk < DK / 16; kk++)
                umma_bf16(acc, qd + ((kk >> 2) * (BOX >> 4) + 2 * (kk & 3)), kd + ((kk >> 2) * (BOX >> 4) + 2 * (kk & 3)), idesc, 1u);
            }
            umma_commit(smem_u32(u != G - 1 ? k_empty + s : s_full + b));
          }
          __syncwarp();
          if (++s == R) { s = 0; ph ^= 1; }
        }
      }
    }
  } else if (warp == 11) {
    if (nb > 0) {
      constexpr uint32_t idesc = idesc_f16(QB, DK, true);
      const bool issuer = elect_one();
      const uint64_t v0 = smem_desc_sw128_mn(smem_u32(sK), BOX);
      for (int j = 0; j < nb; j++) {
        const int b = j % NS, e = j * G + G - 1, s = e % R;
        if (!mbar_wait(smem_u32(p_full + b), (uint32_t)(j / NS) & 1, abort_flag)) break;      // weights written, output rows rescaled if needed
        if (!mbar_wait(smem_u32(k_full + s), (uint32_t)(e / R) & 1, abort_flag)) break;       // (landed long ago: the scores needed it; only now is the parity its own)
        fence_proxy_async_smem();
        tc_fence_after();
        const uint64_t vd = v0 + (uint64_t)(s * (SLICE >> 4));
        if (issuer) {
          umma_ts(O_T, S_T + b * KEYS, vd, idesc, j != 0 ? 1u : 0u);
#pragma unroll
          for (int kk = 1; kk < KEYS / 16; kk++) umma_ts(O_T, S_T + b * KEYS + (kk >> 2) * 64 + 8 * (kk & 3), vd + 128 * kk, idesc, 1u);
          umma_commit(smem_u32(pv_done + b));
          umma_commit(smem_u32(k_empty + s));
        }
        __syncwarp();
      }
    }
  } else if (warp < 10 && nb > 0) {
    const int q = warp & 3;                      // tensor-memory lane quarter this warp may read
    const int hsel = (warp - 2) >> 2;            // which half of a block's keys and of the output columns
    const int row = q * 32 + lane, qpos = pos0 + row;
    const int row_lo = a.window > 0 ? qpos - a.window + 1 : 0, lo_max = a.window > 0 ? pos0 + QB - a.window : 0;      // first key of this row, of the last row
    const uint32_t lane_addr = (uint32_t)(q * 32) << 16;
    constexpr int HK = KEYS / 2, HO = DK / 2;
    const float slope = a.slopes ? a.slopes[h] : 0.f;
    float m_used = -INFINITY, l = 0.f;           // exponent offset of this row (log2 units), this warp's part of the row sum
    bool ok = true;
    for (int u0 = 0; u0 < a.QT && ok; u0 += stage) {   // this row's queries to tensor memory, every other box by the partner warp
      ok = mbar_wait(smem_u32(qt_full), (uint32_t)(u0 / stage) & 1, abort_flag);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      const int n = min(stage, a.QT - u0) * CB;
      for (int i = hsel; i < n; i += 2) {
        const uint8_t* src = sStage + (size_t)i * BOX + row * 128;
        uint32_t r[32];
#pragma unroll
        for (int c = 0; c < 8; c++) {
          const uint4 v = *(const uint4*)(src + ((c ^ (row & 7)) << 4));
          r[4 * c] = v.x; r[4 * c + 1] = v.y; r[4 * c + 2] = v.z; r[4 * c + 3] = v.w;
        }
        tmem_st32(Q_T + lane_addr + (u0 * CB + i) * 32, r);
      }
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(u0 + stage < a.QT ? qt_empty : q_full));
    }
    // both warps of a pair have written their half to xch; `n`: how many times barrier bb has been used
    auto pair_sync = [&](int bb, int n) -> bool {
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(x_full + q * 2 + bb));
      const bool k = mbar_wait(smem_u32(x_full + q * 2 + bb), (uint32_t)n & 1, abort_flag);
      return __all_sync(0xffffffffu, k && !*abort_flag);
    };
    for (int j = 0; j < nb && ok; j++) {
      const int b = j % NS, use = j / NS;
      ok = mbar_wait(smem_u32(s_full + b), (uint32_t)use & 1, abort_flag);
      ok = __all_sync(0xffffffffu, ok && !*abort_flag);
      if (!ok) break;
      tc_fence_after();
      float sv[HK];
      {
        uint32_t r0[32], r1[32];
        tmem_ld32(S_T + b * KEYS + lane_addr + hsel * HK, r0);
        tmem_ld32(S_T + b * KEYS + lane_addr + hsel * HK + 32, r1);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; i++) {
          sv[i] = fmaf(slope, (float)i, __uint_as_float(r0[i]));
          sv[32 + i] = fmaf(slope, (float)(32 + i), __uint_as_float(r1[i]));
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(s_empty + b));
      const int kb0 = (jb0 + j) * KEYS;
      const float base = slope * (float)(kb0 + hsel * HK - qpos);      // the distance's part that all of this warp's keys of the block share
      if (kb0 + KEYS - 1 > pos0 || kb0 + KEYS > ctx || kb0 < lo_max) {
        const int lo = row_lo - kb0 - hsel * HK, hi = min(qpos, ctx - 1) - kb0 - hsel * HK;
#pragma unroll
        for (int i = 0; i < HK; i++)
          if (i < lo || i > hi) sv[i] = -INFINITY;
      }
      float mx0 = fmaxf(sv[0], sv[1]), mx1 = fmaxf(sv[2], sv[3]);
#pragma unroll
      for (int i = 4; i < HK; i += 4) {
        mx0 = max3(mx0, sv[i], sv[i + 1]);
        mx1 = max3(mx1, sv[i + 2], sv[i + 3]);
      }
      const float mine = fmaxf(mx0, mx1) + base;
      float* xb = xch + b * 256;
      xb[hsel * 128 + row] = mine;
      ok = pair_sync(b, use);
      if (!ok) break;
      const float bmax = fmaxf(mine, xb[(hsel ^ 1) * 128 + row]) * kLog2e;
      const bool unset = m_used == -INFINITY;
      const bool behind = bmax > m_used + kRescale;
      if (j > 0 && __any_sync(0xffffffffu, behind && !unset)) {
        const float m_new = fmaxf(m_used, bmax);
        const float scale = (m_new == -INFINITY) ? 1.f : ex2_approx(m_used - m_new);
        ok = mbar_wait(smem_u32(pv_done + (j - 1) % NS), (uint32_t)((j - 1) / NS) & 1, abort_flag);       // the output product before has finished
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
        m_used = bmax;                             // nothing accumulated yet under the old offset
      }
      const float off = (m_used == -INFINITY) ? 0.f : fmaf(base, kLog2e, -m_used);
      float sum0 = 0.f, sum1 = 0.f, sum2 = 0.f, sum3 = 0.f;
      uint32_t pw[HK / 2];
#pragma unroll
      for (int i = 0; i < HK / 2; i++) {
        const float p0 = ex2_approx(fmaf(sv[2 * i], kLog2e, off)), p1 = ex2_approx(fmaf(sv[2 * i + 1], kLog2e, off));
        if (i & 1) { sum2 += p0; sum3 += p1; } else { sum0 += p0; sum1 += p1; }
        const __half2 hh = __floats2half2_rn(p0, p1);
        pw[i] = *(const uint32_t*)&hh;
      }
      tmem_st32(S_T + b * KEYS + lane_addr + hsel * HK, pw);
      tmem_st_wait();
      l += (sum0 + sum1) + (sum2 + sum3);
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(p_full + b));
    }
    if (ok) {
      ok = mbar_wait(smem_u32(pv_done + (nb - 1) % NS), (uint32_t)((nb - 1) / NS) & 1, abort_flag);          // the last output product
      ok = __all_sync(0xffffffffu, ok && !*abort_flag);
    }
    if (__all_sync(0xffffffffu, ok)) {
      const int b = nb % NS;                       // the buffer the last block did not use (or the only one, whose readers are done)
      float* xl = xch + b * 256;
      xl[hsel * 128 + row] = l;
      ok = pair_sync(b, nb / NS);
      l += xl[(hsel ^ 1) * 128 + row];
      tc_fence_after();
      if (a.sinks) l += (m_used == -INFINITY) ? 1.f : ex2_approx(a.sinks[h] * kLog2e - m_used);
      const float inv = l > 0.f ? 1.f / l : 0.f;
      // 32 rows of HO columns per warp go through shared memory (the ring, whose last reader has finished), so that whole lines leave
      const int rows = ok ? min(32, qlen - q0 - q * 32) : 0;
      float* stg = (float*)sK + (size_t)(warp - 2) * 32 * 32;
#pragma unroll
      for (int c = 0; c < HO / 32; c++) {
        uint32_t r[32];
        tmem_ld32(O_T + lane_addr + hsel * HO + c * 32, r);
        tmem_ld_wait();
        __syncwarp();
#pragma unroll
        for (int i = 0; i < 8; i++)
          *(float4*)(stg + lane * 32 + ((i ^ (lane & 7)) << 2)) = make_float4(__uint_as_float(r[4 * i]) * inv, __uint_as_float(r[4 * i + 1]) * inv,
                                                                             __uint_as_float(r[4 * i + 2]) * inv, __uint_as_float(r[4 * i + 3]) * inv);
        __syncwarp();
#pragma unroll
        for (int i = 0; i < 8; i++) {
          const int rr = i * 4 + (lane >> 3), p = lane & 7;
          if (rr >= rows) continue;
          const float4 v = *(const float4*)(stg + rr * 32 + ((p ^ (rr & 7)) << 2));
          const size_t at = ((size_t)(qs + q0 + q * 32 + rr) * a.H + h) * DK + hsel * HO + c * 32 + p * 4;
          if (a.out_f32) {
            *(float4*)(a.out_f32 + at) = v;
          } else {
            const __nv_bfloat162 x = __floats2bfloat162_rn(v.x, v.y), y = __floats2bfloat162_rn(v.z, v.w);
            *(uint2*)(a.out + at) = make_uint2(*(const uint32_t*)&x, *(const uint32_t*)&y);
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (*abort_flag) drain_after_abort();
  if (warp == 1) tmem_dealloc(tmem_base, kTmemCols);
  if (threadIdx.x == 0 && *abort_flag && a.status) atomicExch(a.status, (int)B200_ERR_TIMEOUT_MMA);
}

// Score accumulators, slices of the queries in tensor memory, ring entries; false: sizes the kernel does not take.
static bool mixed_prefill_plan(int G, int DK, int& ns, int& qt, int& r) {
  if (G < 1 || (DK != 64 && DK != 128)) return false;
  const int slice = KEYS * DK * 2;
  for (ns = 2; ns >= 1; ns--) {
    const int most = (232448 - 1024 - 38 * 8 - ns * 1024) / slice;
    qt = (512 - ns * KEYS - DK) / (DK / 2);
    if (qt > G) qt = G;
    r = most - (G - qt);
    if (r > 8) r = 8;
    if (r >= 3) return true;
  }
  return false;
}
B200_API int b200_mixed_prefill_ok(int G, int DK) {
  int ns, qt, r;
  return mixed_prefill_plan(G, DK, ns, qt, r) ? 1 : 0;
}
template <int DK, int NS>
static int launch_mixed_prefill(const CUtensorMap& tq, const MixedPreArgs& a, int n_seqs, int max_q, cudaStream_t st) {
  const size_t smem = 1024 + (size_t)(a.G - a.QT + a.R) * KEYS * DK * 2 + (22 + 2 * a.R) * 8 + NS * 1024;
  if (smem > 232448) return B200_ERR_BAD_ARG;
  auto kern = mixed_prefill_kernel<DK, NS>;
  static size_t configured = 0;
  if (smem > configured) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = smem;
  }
  return launch_pdl(kern, dim3(a.H, (max_q + QB - 1) / QB, n_seqs), dim3(384), smem, st, tq, a);
}
// q fp16 [T_total][H][G * DK] (mixed, scaled); kc fp16 [n_pages][16][G * DK], whole pages of finite numbers; out bf16 [T_total][H * DK], or the same
// in fp32 to out_f32.  max_q: the longest portion.
B200_API int b200_mixed_prefill(const void* q, const void* kc, const float* slopes, const float* sinks, const int* page_table, int max_pages,
                                const int* q_start, const int* q_len, const int* ctx_len, int n_seqs, int max_q, int T_total, int H, int G, int DK,
                                int window, void* out, float* out_f32, int* status, cudaStream_t st) {
  int ns, qt, r;
  if (n_seqs < 1 || max_q < 1 || T_total < 1 || H < 1 || window < 0 || !q || !kc || ((uintptr_t)kc & 15) || !page_table || (!out && !out_f32) || G < 1 || H % G ||
      !mixed_prefill_plan(G, DK, ns, qt, r))
    return B200_ERR_BAD_ARG;
  MixedPreArgs a = {};
  a.q = (const __half*)q; a.kc = (const __half*)kc; a.slopes = slopes; a.sinks = sinks; a.page_table = page_table; a.q_start = q_start; a.q_len = q_len; a.ctx_len = ctx_len;
  a.max_pages = max_pages; a.H = H; a.G = G; a.T_total = T_total; a.window = window; a.QT = qt; a.R = r; a.out = (__nv_bfloat16*)out; a.out_f32 = out_f32;
  a.status = status;
  CUtensorMap tq;
  const int rc = make_tmap_2d(&tq, q, 2, (uint64_t)T_total, (uint64_t)H * G * DK, (uint64_t)H * G * DK * 2, QB, 64, true);
  if (rc) return rc;
  if (DK == 64) return ns == 2 ? launch_mixed_prefill<64, 2>(tq, a, n_seqs, max_q, st) : launch_mixed_prefill<64, 1>(tq, a, n_seqs, max_q, st);
  return ns == 2 ? launch_mixed_prefill<128, 2>(tq, a, n_seqs, max_q, st) : launch_mixed_prefill<128, 1>(tq, a, n_seqs, max_q, st);
}
