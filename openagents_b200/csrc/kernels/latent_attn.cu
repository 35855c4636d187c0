// Latent attention: keys and values of all heads are projections of one cached latent per token, beside one rotated key part that the
// heads share.  The cache holds [latent (CR columns), rotated part (RR columns)] per token, padded with zeros.
//
// Prompts expand the latents of the context into keys and values and run the ordinary attention kernel on them.  Decoding works in the
// latent space instead: a query is multiplied by its head's key projection first, so that every head reads the cached row itself, as key and as
// value (the value projection follows the softmax).  This file holds the steps around both forms and the decode kernel.
//
// Compiled without fast math: the norms and rotations here are required in 32-bit.
#include "tc05.cuh"

using namespace b200;
using namespace b200::tc;

namespace {

constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float2 angle(const float2* tab, int tab_len, double base, int dims, int p, int j) {
  if (tab && p >= 0 && p < tab_len) return tab[(size_t)p * (dims >> 1) + j];
  double sn, cs;
  sincos((double)p * exp2(-2.0 * (double)j / (double)dims * log2(base)), &sn, &cs);
  return make_float2((float)cs, (float)sn);
}
// Element e of a vector whose first `dims` elements rotate (style 0: adjacent pairs, 1: half-split).
__device__ __forceinline__ float rotated(const float* in, int e, int dims, int style, const float2* tab, int tab_len, double base, int p) {
  if (e >= dims) return in[e];
  const int half = dims >> 1, j = style == 1 ? (e < half ? e : e - half) : e >> 1;
  const bool first = style == 1 ? e < half : !(e & 1);
  const float2 c = angle(tab, tab_len, base, dims, p, j);
  const float u = in[style == 1 ? j : 2 * j], v = in[style == 1 ? j + half : 2 * j + 1];
  return first ? u * c.x - v * c.y : v * c.x + u * c.y;
}
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(__half* p, float v) { *p = __float2half(v); }

}  // namespace

// ------------------------------------------------------------------ finish of the down projections

// One block per token of a fused projection row: the query latent is RMS-normed into cq, the key/value latent is RMS-normed and the shared key
// part rotated into the token's cache row.
struct LatentFinishArgs {
  const float* in;         // [T][ld]
  int ld, q_off, c_off, r_off, q_rank, rank, rot_dim, rot, style;
  const float* q_w;        // [q_rank]
  const float* c_w;        // [rank]
  float eps;
  const int* pos;
  const int* slot;         // physical cache slot (page * page_size + offset); < 0: no cache write
  const float2* tab;
  int tab_len;
  double base;
  float* cq32;             // [T][ldq] or null, padding columns zero
  __nv_bfloat16* cq16;
  int ldq, CR, RR;
};
constexpr int kFinishQ = 6, kFinishC = 3;
template <typename CT>
__global__ void __launch_bounds__(256) latent_finish_kernel(const LatentFinishArgs a, CT* __restrict__ cache) {
  __shared__ float2 red[8];
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, nt = blockDim.x;
  const float* row = a.in + (size_t)t * a.ld;
  // both latents are held in registers (the first kFinishQ / kFinishC columns per thread; longer ones are read again)
  float vq[kFinishQ], vc[kFinishC];
  const int s = a.slot[t], p = a.pos[t];
#pragma unroll
  for (int k = 0; k < kFinishQ; k++) {
    const int i = threadIdx.x + k * nt;
    vq[k] = i < a.q_rank ? row[a.q_off + i] : 0.f;
  }
#pragma unroll
  for (int k = 0; k < kFinishC; k++) {
    const int i = threadIdx.x + k * nt;
    vc[k] = i < a.rank ? row[a.c_off + i] : 0.f;
  }
  float sq = 0.f, sc = 0.f;
#pragma unroll
  for (int k = 0; k < kFinishQ; k++) sq += vq[k] * vq[k];
#pragma unroll
  for (int k = 0; k < kFinishC; k++) sc += vc[k] * vc[k];
  for (int i = threadIdx.x + kFinishQ * nt; i < a.q_rank; i += nt) { const float v = row[a.q_off + i]; sq += v * v; }
  for (int i = threadIdx.x + kFinishC * nt; i < a.rank; i += nt) { const float v = row[a.c_off + i]; sc += v * v; }
  sq = warp_sum(sq);
  sc = warp_sum(sc);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = make_float2(sq, sc);
  __syncthreads();
  sq = sc = 0.f;
#pragma unroll
  for (int w = 0; w < 8; w++) {
    const float2 e = red[w];
    sq += e.x;
    sc += e.y;
  }
  const float rq = 1.f / sqrtf(sq / (float)a.q_rank + a.eps), rc = 1.f / sqrtf(sc / (float)a.rank + a.eps);
  auto put_q = [&](int i, float v) {
    if (a.cq32) a.cq32[(size_t)t * a.ldq + i] = v;
    if (a.cq16) a.cq16[(size_t)t * a.ldq + i] = __float2bfloat16(v);
  };
#pragma unroll
  for (int k = 0; k < kFinishQ; k++) {
    const int i = threadIdx.x + k * nt;
    if (i < a.ldq) put_q(i, i < a.q_rank ? vq[k] * rq * a.q_w[i] : 0.f);
  }
  for (int i = threadIdx.x + kFinishQ * nt; i < a.ldq; i += nt) put_q(i, i < a.q_rank ? row[a.q_off + i] * rq * a.q_w[i] : 0.f);
  if (s < 0) return;
  CT* dst = cache + (size_t)s * (a.CR + a.RR);
#pragma unroll
  for (int k = 0; k < kFinishC; k++) {
    const int i = threadIdx.x + k * nt;
    if (i < a.CR) put(dst + i, i < a.rank ? vc[k] * rc * a.c_w[i] : 0.f);
  }
  for (int i = threadIdx.x + kFinishC * nt; i < a.CR; i += nt) put(dst + i, i < a.rank ? row[a.c_off + i] * rc * a.c_w[i] : 0.f);
  for (int i = threadIdx.x; i < a.RR; i += nt)
    put(dst + a.CR + i, i < a.rot_dim ? rotated(row + a.r_off, i, a.rot, a.style, a.tab, a.tab_len, a.base, p) : 0.f);
}
// cache [slots][CR + RR], fp32 when cache_f32 else fp16.
B200_API int b200_latent_finish(const float* in, int ld, int T, int q_off, int c_off, int r_off, int q_rank, int rank, int rot_dim, int rot,
                                int style, const float* q_w, const float* c_w, float eps, const int* pos, const int* slot, const void* tab,
                                int tab_len, double base, float* cq32, void* cq16, int ldq, int CR, int RR, void* cache, int cache_f32,
                                cudaStream_t st) {
  if (T < 1 || q_rank < 1 || rank < 1 || q_rank > ldq || rank > CR || rot_dim > RR || rot < 0 || rot > rot_dim || (rot & 1) || !cache ||
      (!cq32 && !cq16))
    return B200_ERR_BAD_ARG;
  LatentFinishArgs a;
  a.in = in; a.ld = ld; a.q_off = q_off; a.c_off = c_off; a.r_off = r_off; a.q_rank = q_rank; a.rank = rank; a.rot_dim = rot_dim; a.rot = rot;
  a.style = style; a.q_w = q_w; a.c_w = c_w; a.eps = eps; a.pos = pos; a.slot = slot; a.tab = (const float2*)tab; a.tab_len = tab ? tab_len : 0;
  a.base = base; a.cq32 = cq32; a.cq16 = (__nv_bfloat16*)cq16; a.ldq = ldq; a.CR = CR; a.RR = RR;
  if (cache_f32) return launch_pdl(latent_finish_kernel<float>, dim3(T), dim3(256), 0, st, a, (float*)cache);
  return launch_pdl(latent_finish_kernel<__half>, dim3(T), dim3(256), 0, st, a, (__half*)cache);
}

// ------------------------------------------------------------------ finish of the queries

// One warp per (token, head): the unrotated part (scaled) to columns [0, NC) of the head's output row, the rotated part (rotated, scaled) to columns
// [r_col, r_col + RR), padding zero.  NC = 0 leaves the unrotated part to whoever projects it into the latent space.
struct LatentQArgs {
  const float* in;         // [T][ld], head h at h * hs: [dim unrotated, rot_dim rotated]
  int ld, hs, H, dim, rot_dim, rot, style, NC, r_col, RR, width;
  const int* pos;
  const float2* tab;
  int tab_len;
  double base;
  float scale;
  float* q32;              // [T][H][width] or null
  __half* q16;
};
__global__ void __launch_bounds__(128) latent_q_kernel(const LatentQArgs a) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, h = blockIdx.y * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (h >= a.H) return;
  const float* in = a.in + (size_t)t * a.ld + (size_t)h * a.hs;
  const size_t at = ((size_t)t * a.H + h) * a.width;
  const int p = a.pos[t];
  for (int i = lane; i < a.NC + a.RR; i += 32) {
    const int e = i - a.NC, col = e < 0 ? i : a.r_col + e;
    float v = 0.f;
    if (e < 0) {
      if (i < a.dim) v = in[i] * a.scale;
    } else if (e < a.rot_dim) {
      v = rotated(in + a.dim, e, a.rot, a.style, a.tab, a.tab_len, a.base, p) * a.scale;
    }
    if (a.q32) a.q32[at + col] = v;
    if (a.q16) a.q16[at + col] = __float2half(v);
  }
}
B200_API int b200_latent_q(const float* in, int ld, int hs, int T, int H, int dim, int rot_dim, int rot, int style, int NC, int r_col, int RR,
                           int width, const int* pos, const void* tab, int tab_len, double base, float scale, float* q32, void* q16,
                           cudaStream_t st) {
  if (T < 1 || H < 1 || dim < 1 || rot_dim > RR || rot < 0 || rot > rot_dim || (rot & 1) || (NC && NC < dim) || r_col < NC || r_col + RR > width ||
      (!q32 && !q16))
    return B200_ERR_BAD_ARG;
  LatentQArgs a;
  a.in = in; a.ld = ld; a.hs = hs; a.H = H; a.dim = dim; a.rot_dim = rot_dim; a.rot = rot; a.style = style; a.NC = NC; a.r_col = r_col; a.RR = RR;
  a.width = width; a.pos = pos; a.tab = (const float2*)tab; a.tab_len = tab ? tab_len : 0; a.base = base; a.scale = scale; a.q32 = q32;
  a.q16 = (__half*)q16;
  return launch_pdl(latent_q_kernel, dim3(T, (H + 3) / 4), dim3(128), 0, st, a);
}

// ------------------------------------------------------------------ latents of the context, for their expansion

// Rows [base[b], base[b] + ctx_len[b]) of out (bf16 [rows][CR]) = the cached latents of sequence b.
__global__ void __launch_bounds__(256) latent_gather_kernel(const __half* __restrict__ cache, int KS, int CR, const int* __restrict__ page_table,
                                                            int max_pages, const int* __restrict__ ctx_len, const int* __restrict__ base,
                                                            __nv_bfloat16* __restrict__ out) {
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.y, len = ctx_len[b], c8 = CR >> 3;
  const int* pt = page_table + (size_t)b * max_pages;
  for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < len * c8; i += gridDim.x * blockDim.x) {
    const int key = i / c8, c = i % c8;
    const uint4 v = *(const uint4*)(cache + ((size_t)pt[key >> 4] * 16 + (key & 15)) * KS + c * 8);
    const __half2* h = (const __half2*)&v;
    uint4 o;
    __nv_bfloat162* p = (__nv_bfloat162*)&o;
#pragma unroll
    for (int k = 0; k < 4; k++) {
      const float2 f = __half22float2(h[k]);
      p[k] = __floats2bfloat162_rn(f.x, f.y);
    }
    *(uint4*)(out + (size_t)(base[b] + key) * CR + c * 8) = o;
  }
}
B200_API int b200_latent_gather(const void* cache, int KS, int CR, const int* page_table, int max_pages, const int* ctx_len, const int* base,
                                int n_seqs, int max_ctx, void* out, cudaStream_t st) {
  if (n_seqs < 1 || max_ctx < 1 || CR < 8 || CR % 8 || KS % 8 || CR > KS) return B200_ERR_BAD_ARG;
  const long work = (long)max_ctx * (CR / 8);
  const int gx = (int)min((work + 1023) / 1024, (long)2048);
  return launch_pdl(latent_gather_kernel, dim3(gx, n_seqs), dim3(256), 0, st, (const __half*)cache, KS, CR, page_table, max_pages, ctx_len, base,
                    (__nv_bfloat16*)out);
}

// ------------------------------------------------------------------ decoding in the latent space

// One CTA = (share of the keys, group of N heads, query row).  The cached rows are the 128-row operand of both products and the heads the narrow
// one, so a product costs what its heads need:
//   S^T [keys][N]  = C [128 keys][CR + RR] Q'^T         (K-major A)
//   O^T [dims][N] += C^T [128 dims][128 keys] P^T       per 128 latent dimensions (MN-major A: the same bytes, read the other way)
// Roles: warps 0..7 softmax, rescale and output; warps 8..11 fetch two 16-token pages of a 128-key block each; warp 12 issues the first product, warp 13
// the second.  A block is 147 KB at 512 + 64 columns, so shared memory holds little more than one: it is handed over in pairs of 64-column boxes, the
// first product follows the copies pair by pair, and the second gives each pair back as soon as it is done with it.  Scores, weights and sums are fp32; P is fp16.  A head's exponent offset moves only when its maximum has grown by more than 8 (log2).
// Every wait is bounded; one that runs out sets the status word and the CTA leaves through the common exit.
namespace {

constexpr int kLPairs = 8;                             // pairs of boxes in shared memory at most
constexpr int kLKeys = 128, kLBox = kLKeys * 128, kLThreads = 448;
constexpr float kRescaleStep = 8.f;

struct LatentDecArgs {
  const float* q;          // [R][H][CR + RR]: projected into the latent space, rotated, scaled
  const int* page_table;   // [n_seqs][max_pages]
  const int* row_seq;      // [R] sequence of each row, or null: row r is sequence r
  const int* pos;          // [R] position of each row: it sees keys 0..pos
  const float* sinks;      // [H] or null
  int max_pages, H, CR, RR, S, pairs;      // pairs: slots of the ring
  float* part;             // S > 1: [R][S][H][CR], then [R][S][H][2] (offset, sum)
  float* part_ml;
  float* out_f32;          // [R][ldo], head h at column h * CR
  __nv_bfloat16* out_bf16;
  int ldo;
  int* status;
};

// fp16 x fp16 -> fp32, 128 x N; a_mn: the A operand is MN-major.
__host__ __device__ constexpr uint32_t idesc_lat(int N, bool a_mn) {
  return (1u << 4) | ((a_mn ? 1u : 0u) << 15) | ((uint32_t)(N >> 3) << 17) | ((uint32_t)(128 >> 4) << 24);
}
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
template <int NC>
__device__ __forceinline__ void tmem_ld(uint32_t taddr, uint32_t (&r)[NC]) {
  static_assert(NC == 8 || NC == 16, "columns");
  if constexpr (NC == 8)
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x8.b32 {%0, %1, %2, %3, %4, %5, %6, %7}, [%8];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]) : "r"(taddr) : "memory");
  else
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15}, [%16];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]),
                   "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]) : "r"(taddr) : "memory");
}
template <int NC>
__device__ __forceinline__ void tmem_st(uint32_t taddr, const uint32_t (&r)[NC]) {
  if constexpr (NC == 8)
    asm volatile("tcgen05.st.sync.aligned.32x32b.x8.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8};"
                 ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]) : "memory");
  else
    asm volatile("tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};"
                 ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]),
                   "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]) : "memory");
}
// The 256 softmax threads meet, and all learn whether every one of them is fine.
__device__ __forceinline__ bool meet(bool ok) {
  uint32_t r;
  asm volatile("{\n\t.reg .pred p, q;\n\tsetp.ne.b32 p, %1, 0;\n\tbarrier.cta.red.and.pred q, 1, 256, p;\n\tselp.u32 %0, 1, 0, q;\n\t}"
               : "=r"(r) : "r"((uint32_t)ok) : "memory");
  return r != 0;
}
__device__ __forceinline__ float lanes_max(float v) {
  float r;
  asm("redux.sync.max.f32 %0, %1, 0xffffffff;" : "=f"(r) : "f"(v));
  return r;
}
// NC values per lane -> the sum over the 32 lanes of column `col` (returned).  Halves are exchanged, so it takes about NC shuffles.
template <int NC>
__device__ __forceinline__ float sum_columns(const float (&in)[NC], int lane, int& col) {
  float v[NC];
#pragma unroll
  for (int i = 0; i < NC; i++) v[i] = in[i];
  col = 0;
  int n = NC, off = 16;
#pragma unroll
  for (; n > 1; n >>= 1, off >>= 1) {
    const bool up = lane & off;
    const int h = n >> 1;
    col += up ? h : 0;
#pragma unroll
    for (int i = 0; i < NC / 2; i++) {
      if (i >= h) continue;
      const float keep = up ? v[i + h] : v[i], give = up ? v[i] : v[i + h];
      v[i] = keep + __shfl_xor_sync(0xffffffffu, give, off);
    }
  }
#pragma unroll
  for (; off > 0; off >>= 1) v[0] += __shfl_xor_sync(0xffffffffu, v[0], off);
  return v[0];
}

template <int N>
__global__ void __launch_bounds__(kLThreads, 1) latent_decode_kernel(const __grid_constant__ CUtensorMap tm, const LatentDecArgs a) {
  constexpr int NC = N / 2;                            // head columns per softmax warp
  constexpr uint32_t TMEM_COLS = 256;                  // S: 2 x N, O: up to 5 x N
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  const int boxes = (a.CR + a.RR) >> 6, c_boxes = a.CR >> 6, W = a.CR + a.RR;
  const int nt = (a.CR + 127) >> 7;                    // 128-dimension tiles of the output = pairs of a block (the last may be half)
  uint8_t* sC = smem;                                  // pairs x 2 x [128 keys][128 bytes]
  uint8_t* sR = sC + a.pairs * 2 * kLBox;              // the rotated parts' boxes, one block of them
  uint8_t* sQ = sR + (boxes - c_boxes) * kLBox;        // boxes x [N][128 bytes]
  uint8_t* sP = sQ + boxes * N * 128;                  // 2 key halves x [N][64 keys]
  uint64_t* bars = (uint64_t*)(sP + 2 * N * 128);
  uint64_t* c_full = bars;                             // [pairs]
  uint64_t* c_empty = bars + kLPairs;                  // [pairs]
  uint64_t* r_full = bars + 2 * kLPairs;
  uint64_t* r_empty = r_full + 1;
  uint64_t* s_full = r_full + 2;                       // [2]
  uint64_t* s_empty = r_full + 4;                      // [2]
  uint64_t* p_full = r_full + 6;
  uint64_t* pv_done = r_full + 7;
  uint32_t* tmem_holder = (uint32_t*)(r_full + 8);
  volatile int* abort_flag = (volatile int*)(tmem_holder + 1);
  float* s_part = (float*)(r_full + 10);               // [2 (block parity)][4 quarters][N] maxima, then sums
  float* s_inv = s_part + 8 * N;                       // [N] 1 / sum

  const int split = blockIdx.x, h0 = blockIdx.y * N, row = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if (tid == 0) {
    for (int s = 0; s < kLPairs; s++) {
      mbar_init(smem_u32(c_full + s), 4);
      mbar_init(smem_u32(c_empty + s), 1);
    }
    mbar_init(smem_u32(r_full), 4);
    mbar_init(smem_u32(r_empty), 1);
    for (int s = 0; s < 2; s++) {
      mbar_init(smem_u32(s_full + s), 1);
      mbar_init(smem_u32(s_empty + s), 8);
    }
    mbar_init(smem_u32(p_full), 8);
    mbar_init(smem_u32(pv_done), 1);
    *abort_flag = 0;
    fence_barrier_init();
    tma_prefetch_desc(&tm);
  }
  if (warp == 12) {
    tmem_alloc(smem_u32(tmem_holder), TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_holder, S_T = tmem, O_T = tmem + 2 * N;
  pdl_trigger();
  pdl_wait();

  const int len = a.pos[row] + 1;
  const int blocks = (len + kLKeys - 1) / kLKeys, per = (blocks + a.S - 1) / a.S;
  const int j0 = split * per, nb = max(0, min(blocks, j0 + per) - j0);
  const int* pt = a.page_table + (size_t)(a.row_seq ? a.row_seq[row] : row) * a.max_pages;

  // one lane of warps 8..11: this warp's two pages of one part of block j (i = -1: the rotated boxes, else pair i)
  auto fetch = [&](int j, int i) {
    const int slot = i < 0 ? 0 : (j * nt + i) % a.pairs, b0 = i < 0 ? c_boxes : 2 * i, n_box = (i < 0 ? boxes : min(2 * i + 2, c_boxes)) - b0;
    const uint32_t bar = smem_u32(i < 0 ? r_full : c_full + slot);
    uint8_t* dst = i < 0 ? sR : sC + (size_t)slot * 2 * kLBox;
    mbar_expect_tx(bar, n_box * 4096);
#pragma unroll
    for (int h = 0; h < 2; h++) {
      const int p = (warp - 8) * 2 + h, pi = (j0 + j) * (kLKeys / 16) + p;
      const int r = (pi * 16 < len ? pt[pi] : 0) * 16;                    // pages past the context are masked
      for (int c = 0; c < n_box; c++) tma_load_2d(smem_u32(dst + c * kLBox + p * 2048), &tm, bar, (b0 + c) * 64, r);
    }
  };
  const bool producer = warp >= 8 && warp < 12;
  if (producer) {
    if (lane == 0)
      for (int i = -1; i < nt && nb > 0; i++) fetch(0, i);               // the first block: the ring is empty and holds all of it
    __syncwarp();
  } else {
    // queries: fp32 -> fp16, 128-byte-swizzled rows of 64 columns; heads past the last are zeros
    const int t = warp < 8 ? tid : tid - 128, n_t = kLThreads - 128, q4 = W >> 2;
#pragma unroll 4
    for (int i = t; i < N * q4; i += n_t) {
      const int n = i / q4, c = (i - n * q4) * 4, cc = c & 63;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (h0 + n < a.H) v = *(const float4*)(a.q + ((size_t)row * a.H + h0 + n) * W + c);
      const __half2 x = __floats2half2_rn(v.x, v.y), y = __floats2half2_rn(v.z, v.w);
      *(uint2*)(sQ + (c >> 6) * (N * 128) + n * 128 + (((cc >> 3) ^ (n & 7)) << 4) + (cc & 7) * 2) =
          make_uint2(*(const uint32_t*)&x, *(const uint32_t*)&y);
    }
    fence_proxy_async_smem();
  }
  __syncthreads();

  if (producer) {
    if (lane == 0) {
      bool ok = true;
      for (int j = 1; j < nb && ok; j++)
        for (int i = -1; i < nt && ok; i++) {          // the rotated parts first: they are given back first
          const int t = j * nt + i;
          ok = i < 0 ? mbar_wait(smem_u32(r_empty), (j & 1) ^ 1, abort_flag)
                     : mbar_wait(smem_u32(c_empty + t % a.pairs), ((t / a.pairs) & 1) ^ 1, abort_flag);
          if (ok) fetch(j, i);
        }
    }
  } else if (warp == 12) {
    if (lane == 0) {
      bool ok = true;
      const uint32_t qa = smem_u32(sQ);
      for (int j = 0; j < nb && ok; j++) {
        const int b = j & 1;
        if (!mbar_wait(smem_u32(s_empty + b), ((j >> 1) & 1) ^ 1, abort_flag)) break;
        for (int i = -1; i < nt && ok; i++) {
          const int t = j * nt + i, slot = i < 0 ? 0 : t % a.pairs, b0 = i < 0 ? c_boxes : 2 * i, b1 = i < 0 ? boxes : min(2 * i + 2, c_boxes);
          ok = i < 0 ? mbar_wait(smem_u32(r_full), j & 1, abort_flag) : mbar_wait(smem_u32(c_full + slot), (t / a.pairs) & 1, abort_flag);
          if (!ok) break;
          tc_fence_after();
          const uint32_t ca = smem_u32(i < 0 ? sR : sC + (size_t)slot * 2 * kLBox);
          for (int c = b0; c < b1; c++) {
            const uint64_t ad = smem_desc_sw128(ca + (c - b0) * kLBox), qd = smem_desc_sw128(qa + c * (N * 128));
#pragma unroll
            for (int k = 0; k < 4; k++) umma_bf16(S_T + b * N, ad + 2 * k, qd + 2 * k, idesc_lat(N, false), (i >= 0 || c > b0 || k) ? 1u : 0u);
          }
          if (i < 0) umma_commit(smem_u32(r_empty));   // the rotated parts are no values: nobody else reads them
        }
        if (ok) umma_commit(smem_u32(s_full + b));
      }
    }
  } else if (warp == 13) {
    if (lane == 0) {
      bool ok = true;
      // the page of the partial results is looked up while there is time
      if (a.S > 1) asm volatile("prefetch.global.L2 [%0];" ::"l"(a.part + (((size_t)row * a.S + split) * a.H + h0) * a.CR));
      for (int j = 0; j < nb && ok; j++) {
        for (int i = 0; i < nt && ok; i++) ok = mbar_wait(smem_u32(c_full + (j * nt + i) % a.pairs), ((j * nt + i) / a.pairs) & 1, abort_flag);
        if (!ok || !mbar_wait(smem_u32(p_full), j & 1, abort_flag)) break;
        tc_fence_after();
        const uint64_t pd = smem_desc_sw128(smem_u32(sP));
        for (int i = 0; i < nt; i++) {
          const int slot = (j * nt + i) % a.pairs;
          const uint64_t ad = smem_desc_sw128_mn(smem_u32(sC + (size_t)slot * 2 * kLBox), kLBox);
#pragma unroll
          for (int k = 0; k < 8; k++)
            umma_bf16(O_T + i * N, ad + 128 * k, pd + (k >> 2) * (N * 8) + 2 * (k & 3), idesc_lat(N, true), (j | k) ? 1u : 0u);
          umma_commit(smem_u32(c_empty + slot));
        }
        umma_commit(smem_u32(pv_done));
      }
    }
  } else {
    const int q = warp & 3, half = warp >> 2, c0 = half * NC;
    const uint32_t lane_addr = (uint32_t)(q * 32) << 16;
    const int key_in = q * 32 + lane;
    float m_used[NC], l[NC];                           // this warp's heads: exponent offset (log2 units, the same in every thread), part of the sum
#pragma unroll
    for (int i = 0; i < NC; i++) {
      m_used[i] = -INFINITY;
      l[i] = 0.f;
    }
    bool ok = true;
    for (int j = 0; j < nb; j++) {
      const int b = j & 1;
      ok = ok && mbar_wait(smem_u32(s_full + b), (j >> 1) & 1, abort_flag);
      if (j > 0) ok = ok && mbar_wait(smem_u32(pv_done), (j - 1) & 1, abort_flag);      // P is free again, O is at rest
      ok = __all_sync(0xffffffffu, ok);
      tc_fence_after();
      float x[NC];
      bool behind = false;
      {
        uint32_t r[NC];
        tmem_ld<NC>(S_T + b * N + lane_addr + c0, r);
        tmem_ld_wait();
        const bool seen = (j0 + j) * kLKeys + key_in < len;
#pragma unroll
        for (int i = 0; i < NC; i++) x[i] = seen ? __uint_as_float(r[i]) * kLog2e : -INFINITY;
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(smem_u32(s_empty + b));
#pragma unroll
        for (int i = 0; i < NC; i++) behind |= x[i] > m_used[i] + kRescaleStep;      // also while no offset is set
        behind = __any_sync(0xffffffffu, behind);
      }
      if (!meet(ok && !behind)) {                      // some offset has to move (always in the first block), or something failed
        float* part = s_part + b * 4 * N;
#pragma unroll
        for (int i = 0; i < NC; i++) {
          const float mx = lanes_max(x[i]);            // over this warp's keys
          if (lane == 0) part[q * N + c0 + i] = mx;
        }
        if (!meet(ok)) break;
        float sc[NC];
        bool moved = false;
#pragma unroll
        for (int i = 0; i < NC; i++) {
          const float* p = part + c0 + i;
          const float top = fmaxf(fmaxf(p[0], p[N]), fmaxf(p[2 * N], p[3 * N])), old = m_used[i];
          const bool up = top > old + kRescaleStep;
          m_used[i] = up ? top : old;
          sc[i] = up && old != -INFINITY ? ex2(old - top) : 1.f;
          moved |= sc[i] != 1.f;
        }
        if (moved) {                                   // uniform: every thread of the warp sees the same maxima
          for (int i = 0; i < nt; i++) {
            uint32_t r[NC];
            tmem_ld<NC>(O_T + i * N + lane_addr + c0, r);
            tmem_ld_wait();
#pragma unroll
            for (int k = 0; k < NC; k++) r[k] = __float_as_uint(__uint_as_float(r[k]) * sc[k]);
            tmem_st<NC>(O_T + i * N + lane_addr + c0, r);
          }
          tmem_st_wait();
#pragma unroll
          for (int i = 0; i < NC; i++) l[i] *= sc[i];
        }
      }
      {
        uint8_t* p = sP + (key_in >> 6) * (N * 128) + c0 * 128 + (key_in & 7) * 2;
        const int chunk = (key_in & 63) >> 3;
#pragma unroll
        for (int i = 0; i < NC; i++) {
          const float w = ex2(x[i] - m_used[i]);       // finite: the first block has a visible key
          l[i] += w;
          *(__half*)(p + i * 128 + ((chunk ^ (i & 7)) << 4)) = __float2half(w);      // c0 is a multiple of 8
        }
        fence_proxy_async_smem();
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(p_full));
    }
    if (nb > 0) {
      ok = ok && mbar_wait(smem_u32(pv_done), (nb - 1) & 1, abort_flag);
      ok = __all_sync(0xffffffffu, ok);
    }
    // the sums of the four lane quarters, then the offsets, to shared memory (the buffer the last block did not use, then the other one)
    float* part = s_part + (nb & 1) * 4 * N;
    float* offs = s_part + ((nb & 1) ^ 1) * 4 * N;
    {
      int col;
      const float sum = sum_columns<NC>(l, lane, col);
      part[q * N + c0 + col] = sum;                    // the lanes of a column hold the same value
    }
    if (meet(ok)) {
      if (q == 0 && lane == 0) {
#pragma unroll
        for (int i = 0; i < NC; i++) offs[c0 + i] = m_used[i];
      }
      meet(true);
      tc_fence_after();
      const size_t p_row = ((size_t)row * a.S + split) * a.H;
      if (tid < N && h0 + tid < a.H) {
        const float sum = (part[tid] + part[N + tid]) + (part[2 * N + tid] + part[3 * N + tid]), m = offs[tid];
        if (a.S > 1) {
          *(float2*)(a.part_ml + (p_row + h0 + tid) * 2) = make_float2(m, sum);
        } else if (a.sinks) {
          const float sk = a.sinks[h0 + tid] * kLog2e, mx = fmaxf(m, sk), c = ex2(m - mx);
          s_inv[tid] = c / (sum * c + ex2(sk - mx));
        } else {
          s_inv[tid] = sum > 0.f ? 1.f / sum : 0.f;
        }
      }
      meet(true);
      for (int i = 0; i < nt && nb > 0; i++) {
        uint32_t r[NC];
        tmem_ld<NC>(O_T + i * N + lane_addr + c0, r);
        tmem_ld_wait();
        const int d = i * 128 + q * 32 + lane;
        if (d >= a.CR) continue;
#pragma unroll
        for (int k = 0; k < NC; k++) {
          const int h = h0 + c0 + k;
          if (h >= a.H) continue;
          const float v = __uint_as_float(r[k]);
          if (a.S > 1) {
            a.part[(p_row + h) * a.CR + d] = v;
          } else {
            const size_t at = (size_t)row * a.ldo + (size_t)h * a.CR + d;
            if (a.out_f32) a.out_f32[at] = v * s_inv[c0 + k];
            if (a.out_bf16) a.out_bf16[at] = __float2bfloat16(v * s_inv[c0 + k]);
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 12) tmem_dealloc(tmem, TMEM_COLS);
  if (tid == 0 && *abort_flag && a.status) atomicExch(a.status, (int)B200_ERR_TIMEOUT_MMA);
}

// Shares of the keys -> one output row per (row, head), with the sink's term.
constexpr int kLShares = 64;
__global__ void __launch_bounds__(128) latent_merge_kernel(const LatentDecArgs a) {
  __shared__ float s_w[kLShares];
  pdl_trigger();
  pdl_wait();
  const int h = blockIdx.x, row = blockIdx.y, lane = threadIdx.x & 31;
  const size_t p0 = (size_t)row * a.S * a.H + h;
  // every warp reads the shares' offsets and sums: one or two per lane
  float2 ml[kLShares / 32];
  float M = a.sinks ? a.sinks[h] * kLog2e : -INFINITY;
#pragma unroll
  for (int k = 0; k < kLShares / 32; k++) {
    const int s = lane + 32 * k;
    ml[k] = s < a.S ? *(const float2*)(a.part_ml + (p0 + (size_t)s * a.H) * 2) : make_float2(-INFINITY, 0.f);
  }
#pragma unroll
  for (int k = 0; k < kLShares / 32; k++) M = fmaxf(M, ml[k].x);
  M = warp_max(M);
  float L = 0.f, w[kLShares / 32];
#pragma unroll
  for (int k = 0; k < kLShares / 32; k++) {
    w[k] = ml[k].x == -INFINITY ? 0.f : ex2(ml[k].x - M);
    L += ml[k].y * w[k];
  }
  L = warp_sum(L);
  if (a.sinks) L += ex2(a.sinks[h] * kLog2e - M);
  const float inv = L > 0.f ? 1.f / L : 0.f;
  if (threadIdx.x < 32) {
#pragma unroll
    for (int k = 0; k < kLShares / 32; k++) s_w[lane + 32 * k] = w[k] * inv;
  }
  __syncthreads();
  for (int d = threadIdx.x * 4; d < a.CR; d += blockDim.x * 4) {
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int s = 0; s < a.S; s++) {
      const float f = s_w[s];
      if (f == 0.f) continue;                          // a share without keys has written nothing
      const float4 v = *(const float4*)(a.part + (p0 + (size_t)s * a.H) * a.CR + d);
      o.x = fmaf(v.x, f, o.x); o.y = fmaf(v.y, f, o.y); o.z = fmaf(v.z, f, o.z); o.w = fmaf(v.w, f, o.w);
    }
    const size_t at = (size_t)row * a.ldo + (size_t)h * a.CR + d;
    if (a.out_f32) *(float4*)(a.out_f32 + at) = o;
    if (a.out_bf16) {
      const __nv_bfloat162 x = __floats2bfloat162_rn(o.x, o.y), y = __floats2bfloat162_rn(o.z, o.w);
      *(uint2*)(a.out_bf16 + at) = make_uint2(*(const uint32_t*)&x, *(const uint32_t*)&y);
    }
  }
}

size_t latent_smem(int N, int CR, int RR, int pairs) {
  const size_t boxes = (CR + RR) / 64;
  return 1024 + (size_t)pairs * 2 * kLBox + (RR / 64) * kLBox + boxes * N * 128 + 2 * N * 128 + (2 * kLPairs + 12) * 8 + 9 * N * 4;
}
// Slots of the ring of pairs: as many as fit, 0 where not even one block does.
int latent_pairs(int N, int CR, int RR) {
  int p = kLPairs;
  while (p > 0 && latent_smem(N, CR, RR, p) > 226 * 1024) p--;
  return p >= (CR + 127) / 128 ? p : 0;
}

template <int N>
int launch_latent(const CUtensorMap& tm, LatentDecArgs& a, int R, cudaStream_t st) {
  a.pairs = latent_pairs(N, a.CR, a.RR);
  const size_t smem = latent_smem(N, a.CR, a.RR, a.pairs);
  auto kern = latent_decode_kernel<N>;
  static size_t configured = 48 * 1024;
  if (smem > configured) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = smem;
  }
  const int rc = launch_pdl(kern, dim3(a.S, (a.H + N - 1) / N, R), dim3(kLThreads), smem, st, tm, a);
  if (rc || a.S == 1) return rc;
  return launch_pdl(latent_merge_kernel, dim3(a.H, R), dim3(128), 0, st, a);
}

}  // namespace

// Whether the tensor-core decode kernel takes these (padded) sizes.
B200_API int b200_latent_decode_ok(int H, int CR, int RR) {
  return CR >= 64 && CR % 64 == 0 && RR >= 64 && RR % 64 == 0 && CR <= 512 && latent_pairs(H <= 16 ? 16 : 32, CR, RR) > 0;
}
B200_API size_t b200_latent_decode_scratch_floats(int R, int H, int CR, int S) { return S > 1 ? (size_t)R * S * H * (CR + 2) : 0; }

// q fp32 [R][H][CR + RR]; cache fp16 [n_pages][16][CR + RR]; outputs [R][ldo], head h at column h * CR.  S: shares of the keys (one CTA each).
B200_API int b200_latent_decode(const float* q, const void* cache, const int* page_table, int max_pages, int n_pages, const int* row_seq,
                                const int* pos, const float* sinks, int R, int H, int CR, int RR, int S, float* scratch, float* out_f32,
                                void* out_bf16, int ldo, int* status, cudaStream_t st) {
  if (R < 1 || H < 1 || S < 1 || S > kLShares || ldo % 4 || !b200_latent_decode_ok(H, CR, RR) || (S > 1 && !scratch) || ldo < H * CR || (!out_f32 && !out_bf16))
    return B200_ERR_BAD_ARG;
  CUtensorMap tm;
  const int rc = make_tmap_2d(&tm, cache, 2, (uint64_t)n_pages * 16, (uint64_t)(CR + RR), (uint64_t)(CR + RR) * 2, 16, 64, true);
  if (rc) return rc;
  LatentDecArgs a;
  a.q = q; a.page_table = page_table; a.row_seq = row_seq; a.pos = pos; a.sinks = sinks; a.max_pages = max_pages; a.H = H; a.CR = CR; a.RR = RR;
  a.S = S; a.part = scratch; a.part_ml = scratch ? scratch + (size_t)R * S * H * CR : nullptr; a.out_f32 = out_f32;
  a.out_bf16 = (__nv_bfloat16*)out_bf16; a.ldo = ldo; a.status = status;
  return H <= 16 ? launch_latent<16>(tm, a, R, st) : launch_latent<32>(tm, a, R, st);
}
