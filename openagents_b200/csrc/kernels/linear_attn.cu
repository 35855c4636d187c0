// Gated linear attention with a decay per key channel.  Per head, with state S [dim][vdim] (fp32, zero at a sequence's start):
//   S_t = diag(alpha_t) S_(t-1) + k_t v_t^T        o_t = S_t^T q_t / sqrt(dim)
//   alpha = sigmoid(z)^(1/tau),  z = A2 a + b2     (a = the low-rank projection of the layer's input)
//   out   = o / rms(o) * w * silu(g)               (rms over a head's vdim)
// Every sequence owns a slot of the state tensor; a chunk whose first token is at position 0 starts from zero without
// reading it.
//
// This file is compiled without fast math; decays, their logarithms and exponentials, the state and the norms are fp32.
#include "common.cuh"

using namespace b200;

struct GlaArgs {
  const float* in;         // [T][ld] fused projections
  int ld, q_off, k_off, v_off, g_off, a_off, rank;
  const float* a2;         // [rank][H * dim]
  const float* b2;         // [H * dim]
  const float* w;          // [vdim]
  float* state;            // [slots][H][dim][VP]
  const int* q_start;
  const int* q_len;
  const int* ctx_len;      // tokens of the sequence after this chunk
  const int* slot;         // state slot per sequence; < 0: start from zero, keep nothing
  int H, dim, vdim, VP;
  float inv_tau, q_scale, eps;
  float* out_f32;          // [T][ldo], head h at column h * VP, columns vdim..VP zero
  __nv_bfloat16* out_bf16;
  int ldo;
};

// log of the decay: log sigmoid(z) / tau, without cancellation on either side
__device__ __forceinline__ float log_decay(float z, float inv_tau) {
  return -(fmaxf(-z, 0.f) + log1pf(expf(-fabsf(z)))) * inv_tau;
}

// Token by token: decoding (one token per sequence) and the 32-bit mode's prompts.  One CTA per (head, sequence); a thread
// owns the same float4 columns of the same state rows at every token, so the state needs no barrier of its own.
__global__ void __launch_bounds__(256) gla_recurrent_kernel(const GlaArgs a) {
  extern __shared__ __align__(16) float sm[];
  float* s_al = sm;                        // [dim] each
  float* s_q = s_al + a.dim;
  float* s_k = s_q + a.dim;
  float* s_v = s_k + a.dim + ((4 - ((3 * a.dim) & 3)) & 3);      // [VP], 16-byte aligned
  float* s_o = s_v + a.VP;                 // [groups][VP]
  __shared__ float red[32];
  pdl_trigger();
  pdl_wait();
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  const int n = a.q_len[b], t0 = a.q_start[b], slot = a.slot[b];
  bool fresh = a.ctx_len[b] - n == 0 || slot < 0;
  const int nv = a.VP >> 2, groups = 256 / nv, grp = tid / nv, col = tid % nv;
  float4* S = (float4*)(a.state + ((size_t)max(slot, 0) * a.H + h) * a.dim * a.VP);
  const bool keep = slot >= 0;
  for (int i = 0; i < n; i++) {
    const float* row = a.in + (size_t)(t0 + i) * a.ld;
    for (int d = tid; d < a.dim; d += 256) {
      const int c = h * a.dim + d;
      float z = a.b2[c];
      for (int r = 0; r < a.rank; r++) z = fmaf(a.a2[(size_t)r * a.H * a.dim + c], row[a.a_off + r], z);
      s_al[d] = expf(log_decay(z, a.inv_tau));
      s_q[d] = row[a.q_off + c] * a.q_scale;
      s_k[d] = row[a.k_off + c];
    }
    for (int e = tid; e < a.VP; e += 256) s_v[e] = e < a.vdim ? row[a.v_off + h * a.vdim + e] : 0.f;
    __syncthreads();
    if (grp < groups) {
      const float4 v = *(const float4*)(s_v + 4 * col);
      float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
      for (int d = grp; d < a.dim; d += groups) {
        float4 x = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : S[(size_t)d * nv + col];
        const float al = s_al[d], k = s_k[d], q = s_q[d];
        x.x = fmaf(al, x.x, k * v.x);
        x.y = fmaf(al, x.y, k * v.y);
        x.z = fmaf(al, x.z, k * v.z);
        x.w = fmaf(al, x.w, k * v.w);
        if (keep) S[(size_t)d * nv + col] = x;
        o.x = fmaf(q, x.x, o.x);
        o.y = fmaf(q, x.y, o.y);
        o.z = fmaf(q, x.z, o.z);
        o.w = fmaf(q, x.w, o.w);
      }
      *(float4*)(s_o + grp * a.VP + 4 * col) = o;
    }
    __syncthreads();
    float ss = 0.f;
    for (int e = tid; e < a.VP; e += 256) {
      float o = 0.f;
      for (int g = 0; g < groups; g++) o += s_o[g * a.VP + e];
      s_o[e] = o;
      ss += o * o;                         // padding columns are zero
    }
    const float r = 1.f / sqrtf(block_sum(ss, red) / (float)a.vdim + a.eps);
    for (int e = tid; e < a.VP; e += 256) {
      float o = 0.f;
      if (e < a.vdim) {
        const float g = row[a.g_off + h * a.vdim + e];
        o = s_o[e] * r * a.w[e] * (g / (1.f + expf(-g)));
      }
      const size_t at = (size_t)(t0 + i) * a.ldo + (size_t)h * a.VP + e;
      if (a.out_f32) a.out_f32[at] = o;
      if (a.out_bf16) a.out_bf16[at] = __float2bfloat16(o);
    }
    fresh = false;
    __syncthreads();
  }
}

static int gla_fill(GlaArgs& a, const float* in, int ld, int q_off, int k_off, int v_off, int g_off, int a_off, int rank,
                    const float* a2, const float* b2, const float* w, float* state, const int* q_start, const int* q_len,
                    const int* ctx_len, const int* slot, int n_seqs, int H, int dim, int vdim, int VP, float tau, float q_scale,
                    float eps, float* out_f32, void* out_bf16, int ldo) {
  if (n_seqs < 1 || H < 1 || dim < 1 || vdim < 1 || VP < vdim || VP % 4 || VP > 1024 || dim > 1024 || rank < 1 || tau == 0.f ||
      ldo < H * VP || ((uintptr_t)state % 16) || !slot)
    return B200_ERR_BAD_ARG;
  a.in = in; a.ld = ld; a.q_off = q_off; a.k_off = k_off; a.v_off = v_off; a.g_off = g_off; a.a_off = a_off; a.rank = rank;
  a.a2 = a2; a.b2 = b2; a.w = w; a.state = state; a.q_start = q_start; a.q_len = q_len; a.ctx_len = ctx_len; a.slot = slot;
  a.H = H; a.dim = dim; a.vdim = vdim; a.VP = VP; a.inv_tau = 1.f / tau; a.q_scale = q_scale; a.eps = eps; a.out_f32 = out_f32;
  a.out_bf16 = (__nv_bfloat16*)out_bf16; a.ldo = ldo;
  return 0;
}

B200_API int b200_gla_recurrent(const float* in, int ld, int q_off, int k_off, int v_off, int g_off, int a_off, int rank,
                                const float* a2, const float* b2, const float* w, float* state, const int* q_start,
                                const int* q_len, const int* ctx_len, const int* slot, int n_seqs, int H, int dim, int vdim,
                                int VP, float tau, float q_scale, float eps, float* out_f32, void* out_bf16, int ldo,
                                cudaStream_t st) {
  GlaArgs a;
  int rc = gla_fill(a, in, ld, q_off, k_off, v_off, g_off, a_off, rank, a2, b2, w, state, q_start, q_len, ctx_len, slot, n_seqs, H,
                    dim, vdim, VP, tau, q_scale, eps, out_f32, out_bf16, ldo);
  if (rc) return rc;
  const int nv = VP / 4, groups = 256 / nv;
  const size_t smem = 4 * ((size_t)3 * dim + 8 + VP + (size_t)groups * VP);      // at most 12 + 4 + 4 KB
  return launch_pdl(gla_recurrent_kernel, dim3(H, n_seqs), dim3(256), smem, st, a);
}

// ------------------------------------------------------------------ prompts: 64-token chunks on the tensor cores
//
// With b_t the running sum of log decays from the chunk's start and C its last token:
//   o_t = (q_t e^{b_t}) S + sum_{s<=t} A[t][s] v_s,   A[t][s] = sum_d q_td k_sd e^{b_td - b_sd}
//   S'  = diag(e^{b_C}) S + sum_s (k_s e^{b_C - b_s}) v_s^T
// gla_prepare_kernel computes the decays, the decayed queries and keys and A for every chunk and head in parallel;
// gla_scan_kernel walks a sequence's chunks with S in registers; gla_out_kernel norms and gates.
//
// The operands that hold decays or the state enter the tensor cores as two bf16 numbers each (value and remainder, about 16
// bits of mantissa), products accumulate in fp32, and the state stays fp32 between chunks; only v, a plain projection, is
// rounded to bf16 once.  A as a product of q e^{b} and k e^{-b} is exact in relative terms but the second factor grows with the
// decay; a chunk whose decay passes e^-60 in some channel takes the direct sum, whose exponents are never positive.

constexpr int GC = 64;                 // tokens per chunk
constexpr float kFactorLimit = 60.f;
constexpr int kMaxRank = 64;

struct GlaChunkWs {
  __nv_bfloat16 *qh, *ql, *kh, *kl;    // [T][H][DP] decayed queries / keys, value and remainder
  __nv_bfloat16 *ah, *al;              // [T][H][GC]
  __nv_bfloat16* v;                    // [T][H][VP]
  float* dec;                          // [chunk slots][H][DP]  e^{b_C}
  float* o;                            // [T][H][VP]
};

// Chunk c of a sequence whose tokens start at row q_start owns slot q_start / 64 + seq + c: no two chunks of a batch share one.
__device__ __forceinline__ size_t chunk_slot(int q_start, int seq, int c) { return (size_t)(q_start / GC) + seq + c; }

__device__ __forceinline__ void split_bf16(float x, __nv_bfloat16& hi, __nv_bfloat16& lo) {
  hi = __float2bfloat16(x);
  lo = __float2bfloat16(x - __bfloat162float(hi));
}
__device__ __forceinline__ uint32_t pack_bf2(__nv_bfloat16 a, __nv_bfloat16 b) {
  __nv_bfloat162 p = __halves2bfloat162(a, b);
  return *(uint32_t*)&p;
}
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  __nv_bfloat16 xh, xl, yh, yl;
  split_bf16(x, xh, xl);
  split_bf16(y, yh, yl);
  hi = pack_bf2(xh, yh);
  lo = pack_bf2(xl, yl);
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t s32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ldsm4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}

template <int DP>
__global__ void __launch_bounds__(256) gla_prepare_kernel(const GlaArgs a, const GlaChunkWs ws) {
  constexpr int LD = DP + 8;           // fp32 row stride: conflict-free fragment reads
  extern __shared__ __align__(16) float sm[];
  float* sq = sm;                      // [GC][LD]
  float* sk = sq + GC * LD;
  float* sb = sk + GC * LD;            // log decays, then their running sums
  float* sa = sb + GC * LD;            // [GC][rank]
  __shared__ float red[32];
  pdl_trigger();
  pdl_wait();
  const int c = blockIdx.x, h = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x;
  const int len = a.q_len[seq], qs = a.q_start[seq];
  if (c * GC >= len) return;
  const int n = min(GC, len - c * GC), t0 = qs + c * GC;
  const float* in = a.in + (size_t)t0 * a.ld;
  for (int i = tid; i < GC * DP; i += 256) {
    const int t = i / DP, d = i % DP;
    const bool live = t < n && d < a.dim;
    const float* row = in + (size_t)t * a.ld;
    sq[t * LD + d] = live ? row[a.q_off + h * a.dim + d] * a.q_scale : 0.f;
    sk[t * LD + d] = live ? row[a.k_off + h * a.dim + d] : 0.f;
  }
  for (int i = tid; i < n * a.rank; i += 256) sa[i] = in[(size_t)(i / a.rank) * a.ld + a.a_off + i % a.rank];
  for (int i = tid; i < n * a.VP; i += 256) {
    const int t = i / a.VP, e = i % a.VP;
    ws.v[((size_t)(t0 + t) * a.H + h) * a.VP + e] = __float2bfloat16(e < a.vdim ? in[(size_t)t * a.ld + a.v_off + h * a.vdim + e] : 0.f);
  }
  __syncthreads();
  {  // z, sixteen ranks at a time with this channel's weights in registers, then the log decay (rows past the end: no decay)
    const int d = tid % DP;
    const bool live = d < a.dim;
    const int ch = h * a.dim + d;
    for (int r0 = 0; r0 < a.rank; r0 += 16) {
      float w[16];
#pragma unroll
      for (int r = 0; r < 16; r++) w[r] = (live && r0 + r < a.rank) ? a.a2[(size_t)(r0 + r) * a.H * a.dim + ch] : 0.f;
      for (int t = tid / DP; t < n; t += 256 / DP) {
        float z = r0 ? sb[t * LD + d] : (live ? a.b2[ch] : 0.f);
#pragma unroll
        for (int r = 0; r < 16; r++)
          if (r0 + r < a.rank) z = fmaf(w[r], sa[t * a.rank + r0 + r], z);
        sb[t * LD + d] = z;
      }
    }
    for (int t = tid / DP; t < GC; t += 256 / DP) sb[t * LD + d] = (live && t < n) ? log_decay(sb[t * LD + d], a.inv_tau) : 0.f;
  }
  __syncthreads();
  float total = 0.f;
  if (tid < DP) {
    float b = 0.f;
    for (int t = 0; t < GC; t++) {
      b += sb[t * LD + tid];
      sb[t * LD + tid] = b;
    }
    total = -b;
    ws.dec[(chunk_slot(qs, seq, c) * a.H + h) * DP + tid] = expf(b);
  }
  const bool factored = block_max(total, red) < kFactorLimit;      // ends with every running sum visible
  __syncthreads();
  for (int i = tid; i < n * DP; i += 256) {
    const int t = i / DP, d = i % DP;
    const float b = sb[t * LD + d], q = sq[t * LD + d], k = sk[t * LD + d];
    const float eb = expf(b), qd = q * eb;
    const size_t at = ((size_t)(t0 + t) * a.H + h) * DP + d;
    split_bf16(qd, ws.qh[at], ws.ql[at]);
    split_bf16(k * expf(sb[(GC - 1) * LD + d] - b), ws.kh[at], ws.kl[at]);
    if (factored) {
      sq[t * LD + d] = qd;
      sk[t * LD + d] = k * expf(-b);
    }
  }
  __syncthreads();
  const int warp = tid >> 5, lane = tid & 31, g4 = lane >> 2, t4 = lane & 3;
  if (factored) {
    // warp = 16 rows x 32 columns of the lower triangle
    const int m0 = (warp >> 1) * 16, n0 = (warp & 1) * 32;
    float acc[4][4] = {};
    if (n0 <= m0 + 15) {
      for (int k0 = 0; k0 < DP; k0 += 16) {
        uint32_t ah[4], al[4];
#pragma unroll
        for (int i = 0; i < 4; i++) {
          const float2 x = *(const float2*)(sq + (m0 + g4 + 8 * (i & 1)) * LD + k0 + 2 * t4 + 8 * (i >> 1));
          split2(x.x, x.y, ah[i], al[i]);
        }
#pragma unroll
        for (int j = 0; j < 4; j++) {
          uint32_t bh[2], bl[2];
#pragma unroll
          for (int i = 0; i < 2; i++) {
            const float2 x = *(const float2*)(sk + (n0 + 8 * j + g4) * LD + k0 + 2 * t4 + 8 * i);
            split2(x.x, x.y, bh[i], bl[i]);
          }
          mma_bf16(acc[j], ah, bh[0], bh[1]);
          mma_bf16(acc[j], ah, bl[0], bl[1]);
          mma_bf16(acc[j], al, bh[0], bh[1]);
        }
      }
    }
#pragma unroll
    for (int j = 0; j < 4; j++)
#pragma unroll
      for (int hf = 0; hf < 2; hf++) {
        const int t = m0 + g4 + 8 * hf, s = n0 + 8 * j + 2 * t4;
        if (t >= n) continue;
        uint32_t hi, lo;
        split2(s <= t ? acc[j][2 * hf] : 0.f, s + 1 <= t ? acc[j][2 * hf + 1] : 0.f, hi, lo);
        const size_t at = ((size_t)(t0 + t) * a.H + h) * GC + s;
        *(uint32_t*)(ws.ah + at) = hi;
        *(uint32_t*)(ws.al + at) = lo;
      }
  } else {
    for (int i = tid; i < n * GC; i += 256) {
      const int t = i / GC, s = i % GC;
      float x = 0.f;
      if (s <= t)
        for (int d = 0; d < a.dim; d++) x = fmaf(sq[t * LD + d] * sk[s * LD + d], expf(sb[t * LD + d] - sb[s * LD + d]), x);
      const size_t at = ((size_t)(t0 + t) * a.H + h) * GC + s;
      split_bf16(x, ws.ah[at], ws.al[at]);
    }
  }
}

// One CTA = 64 value columns of one head of one sequence; a warp owns 16 of them.  Everything is kept transposed (value columns as
// the rows of the MMA), so that the state's accumulator registers are the A operand of the query product as they lie.
template <int DP>
__global__ void __launch_bounds__(128) gla_scan_kernel(const GlaArgs a, const GlaChunkWs ws) {
  constexpr int STAGES = DP <= 128 ? 2 : 1;
  constexpr int LQ = DP + 8, LA = GC + 8;                     // bf16 row strides: 16 bytes past a multiple of 128
  constexpr int STAGE = 4 * GC * LQ + 2 * GC * LA + GC * LA;  // qh ql kh kl | ah al | v
  extern __shared__ __align__(16) __nv_bfloat16 sb16[];
  float* sdec = (float*)(sb16 + STAGES * STAGE);              // [STAGES][DP]
  pdl_trigger();
  pdl_wait();
  const int v0 = blockIdx.x * 64, h = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x;
  const int warp = tid >> 5, lane = tid & 31, g4 = lane >> 2, t4 = lane & 3;
  const int len = a.q_len[seq], qs = a.q_start[seq], slot = a.slot[seq];
  const bool fresh = a.ctx_len[seq] - len == 0 || slot < 0;
  const int nc = (len + GC - 1) / GC;
  float* S = a.state + ((size_t)max(slot, 0) * a.H + h) * a.dim * a.VP;

  auto cp16 = [](void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(s32(dst)), "l"(src));
  };
  auto load = [&](int c) {
    __nv_bfloat16* st = sb16 + (c % STAGES) * STAGE;
    const int n = min(GC, len - c * GC);
    const size_t row0 = (size_t)(qs + c * GC);
    constexpr int CQ = DP / 8;
    for (int i = tid; i < 4 * GC * CQ; i += 128) {
      const int p = i / (GC * CQ), t = (i / CQ) % GC, x = i % CQ;
      const __nv_bfloat16* src = p == 0 ? ws.qh : p == 1 ? ws.ql : p == 2 ? ws.kh : ws.kl;
      __nv_bfloat16* dst = st + p * GC * LQ + t * LQ + x * 8;
      if (t < n) cp16(dst, src + ((row0 + t) * a.H + h) * DP + x * 8);
      else *(uint4*)dst = make_uint4(0u, 0u, 0u, 0u);
    }
    __nv_bfloat16* sA = st + 4 * GC * LQ;
    for (int i = tid; i < 2 * GC * 8; i += 128) {
      const int p = i / (GC * 8), t = (i / 8) % GC, x = i % 8;
      __nv_bfloat16* dst = sA + p * GC * LA + t * LA + x * 8;
      if (t < n) cp16(dst, (p ? ws.al : ws.ah) + ((row0 + t) * a.H + h) * GC + x * 8);
      else *(uint4*)dst = make_uint4(0u, 0u, 0u, 0u);
    }
    __nv_bfloat16* sV = sA + 2 * GC * LA;
    for (int i = tid; i < GC * 8; i += 128) {
      const int t = i / 8, x = i % 8;
      __nv_bfloat16* dst = sV + t * LA + x * 8;
      if (t < n && v0 + x * 8 < a.VP) cp16(dst, ws.v + ((row0 + t) * a.H + h) * a.VP + v0 + x * 8);
      else *(uint4*)dst = make_uint4(0u, 0u, 0u, 0u);
    }
    for (int i = tid; i < DP / 4; i += 128) cp16(sdec + (c % STAGES) * DP + i * 4, ws.dec + (chunk_slot(qs, seq, c) * a.H + h) * DP + i * 4);
    asm volatile("cp.async.commit_group;");
  };

  load(0);
  // state (transposed): sacc[j] = rows v0 + 16 warp + g4 (+ 8), columns d = 8 j + 2 t4 (+ 1)
  float sacc[DP / 8][4];
#pragma unroll
  for (int j = 0; j < DP / 8; j++)
#pragma unroll
    for (int e = 0; e < 4; e++) {
      const int v = v0 + warp * 16 + g4 + 8 * (e >> 1), d = 8 * j + 2 * t4 + (e & 1);
      sacc[j][e] = (!fresh && v < a.VP && d < a.dim) ? S[(size_t)d * a.VP + v] : 0.f;
    }
  bool zero_state = fresh;

  for (int c = 0; c < nc; c++) {
    if (STAGES == 2 && c + 1 < nc) {
      load(c + 1);
      asm volatile("cp.async.wait_group 1;");
    } else {
      asm volatile("cp.async.wait_group 0;");
    }
    __syncthreads();
    const __nv_bfloat16* st = sb16 + (c % STAGES) * STAGE;
    const __nv_bfloat16 *sQh = st, *sQl = st + GC * LQ, *sKh = st + 2 * GC * LQ, *sKl = st + 3 * GC * LQ;
    const __nv_bfloat16 *sAh = st + 4 * GC * LQ, *sAl = sAh + GC * LA, *sV = sAl + GC * LA;
    const float* dec = sdec + (c % STAGES) * DP;
    float oacc[8][4];
#pragma unroll
    for (int j = 0; j < 8; j++) oacc[j][0] = oacc[j][1] = oacc[j][2] = oacc[j][3] = 0.f;
    if (!zero_state) {                 // O^T = S^T (q e^b)^T
#pragma unroll
      for (int kd = 0; kd < DP / 16; kd++) {
        uint32_t ah[4], al[4];
        split2(sacc[2 * kd][0], sacc[2 * kd][1], ah[0], al[0]);
        split2(sacc[2 * kd][2], sacc[2 * kd][3], ah[1], al[1]);
        split2(sacc[2 * kd + 1][0], sacc[2 * kd + 1][1], ah[2], al[2]);
        split2(sacc[2 * kd + 1][2], sacc[2 * kd + 1][3], ah[3], al[3]);
#pragma unroll
        for (int j = 0; j < 8; j += 2) {
          const int r = (j + (lane >> 4)) * 8 + (lane & 7), x = kd * 16 + ((lane >> 3) & 1) * 8;
          uint32_t bh[4], bl[4];
          ldsm4(s32(sQh + r * LQ + x), bh);
          ldsm4(s32(sQl + r * LQ + x), bl);
          mma_bf16(oacc[j], ah, bh[0], bh[1]);
          mma_bf16(oacc[j], ah, bl[0], bl[1]);
          mma_bf16(oacc[j], al, bh[0], bh[1]);
          mma_bf16(oacc[j + 1], ah, bh[2], bh[3]);
          mma_bf16(oacc[j + 1], ah, bl[2], bl[3]);
          mma_bf16(oacc[j + 1], al, bh[2], bh[3]);
        }
      }
#pragma unroll
      for (int j = 0; j < DP / 8; j++) {
        const float2 f = *(const float2*)(dec + 8 * j + 2 * t4);
        sacc[j][0] *= f.x;
        sacc[j][1] *= f.y;
        sacc[j][2] *= f.x;
        sacc[j][3] *= f.y;
      }
    }
    zero_state = false;
#pragma unroll
    for (int kt = 0; kt < GC / 16; kt++) {
      uint32_t va[4];                  // V^T: 16 value columns x 16 tokens
      ldsm4t(s32(sV + (kt * 16 + (lane >> 4) * 8 + (lane & 7)) * LA + warp * 16 + ((lane >> 3) & 1) * 8), va);
#pragma unroll
      for (int j = 2 * kt; j < 8; j += 2) {          // O^T += V^T A^T: output tokens 8 j.. see tokens up to their own
        const int r = (j + (lane >> 4)) * 8 + (lane & 7), x = kt * 16 + ((lane >> 3) & 1) * 8;
        uint32_t bh[4], bl[4];
        ldsm4(s32(sAh + r * LA + x), bh);
        ldsm4(s32(sAl + r * LA + x), bl);
        mma_bf16(oacc[j], va, bh[0], bh[1]);
        mma_bf16(oacc[j], va, bl[0], bl[1]);
        mma_bf16(oacc[j + 1], va, bh[2], bh[3]);
        mma_bf16(oacc[j + 1], va, bl[2], bl[3]);
      }
      const int r = kt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8;
#pragma unroll
      for (int j = 0; j < DP / 8; j += 2) {          // S^T += V^T (k e^{b_C - b})
        uint32_t bh[4], bl[4];
        ldsm4t(s32(sKh + r * LQ + (j + (lane >> 4)) * 8), bh);
        ldsm4t(s32(sKl + r * LQ + (j + (lane >> 4)) * 8), bl);
        mma_bf16(sacc[j], va, bh[0], bh[1]);
        mma_bf16(sacc[j], va, bl[0], bl[1]);
        mma_bf16(sacc[j + 1], va, bh[2], bh[3]);
        mma_bf16(sacc[j + 1], va, bl[2], bl[3]);
      }
    }
    const int n = min(GC, len - c * GC);
#pragma unroll
    for (int j = 0; j < 8; j++)
#pragma unroll
      for (int e = 0; e < 4; e++) {
        const int v = v0 + warp * 16 + g4 + 8 * (e >> 1), t = 8 * j + 2 * t4 + (e & 1);
        if (t < n && v < a.VP) ws.o[((size_t)(qs + c * GC + t) * a.H + h) * a.VP + v] = oacc[j][e];
      }
    __syncthreads();
    if (STAGES == 1 && c + 1 < nc) load(c + 1);
  }
  if (slot >= 0) {
#pragma unroll
    for (int j = 0; j < DP / 8; j++)
#pragma unroll
      for (int e = 0; e < 4; e++) {
        const int v = v0 + warp * 16 + g4 + 8 * (e >> 1), d = 8 * j + 2 * t4 + (e & 1);
        if (v < a.VP && d < a.dim) S[(size_t)d * a.VP + v] = sacc[j][e];
      }
  }
}

// out = o / rms(o) * w * silu(g), one warp per (token, head).
__global__ void __launch_bounds__(128) gla_out_kernel(const GlaArgs a, const float* __restrict__ o) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, h = blockIdx.y * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (h >= a.H) return;
  const float* src = o + ((size_t)t * a.H + h) * a.VP;
  const float* g = a.in + (size_t)t * a.ld + a.g_off + h * a.vdim;
  float ss = 0.f;
  for (int e = lane; e < a.vdim; e += 32) {
    const float x = src[e];
    ss = fmaf(x, x, ss);
  }
  const float r = 1.f / sqrtf(warp_sum(ss) / (float)a.vdim + a.eps);
  for (int e = lane; e < a.VP; e += 32) {
    float x = 0.f;
    if (e < a.vdim) {
      const float y = g[e];
      x = src[e] * r * a.w[e] * (y / (1.f + expf(-y)));
    }
    const size_t at = (size_t)t * a.ldo + (size_t)h * a.VP + e;
    if (a.out_f32) a.out_f32[at] = x;
    if (a.out_bf16) a.out_bf16[at] = __float2bfloat16(x);
  }
}

static int chunk_dp(int dim) { return dim <= 32 ? 32 : dim <= 64 ? 64 : dim <= 128 ? 128 : dim <= 256 ? 256 : 0; }
static size_t align256(size_t n) { return (n + 255) & ~(size_t)255; }

// Bytes of workspace for b200_gla_chunked; 0: sizes it does not take (the caller then uses b200_gla_recurrent).
B200_API size_t b200_gla_chunk_bytes(int T, int n_seqs, int H, int dim, int VP, int rank) {
  const int DP = chunk_dp(dim);
  if (!DP || rank > kMaxRank || VP % 8) return 0;
  const size_t th = (size_t)T * H;
  return 4 * align256(th * DP * 2) + 2 * align256(th * GC * 2) + align256(th * VP * 2) +
         align256(((size_t)T / GC + n_seqs + 1) * H * DP * 4) + align256(th * VP * 4);
}

template <int DP>
static int launch_chunked(const GlaArgs& a, const GlaChunkWs& w, int T, int n_seqs, int max_q, cudaStream_t st) {
  const size_t s1 = 4 * (size_t)(3 * GC * (DP + 8) + GC * a.rank);
  constexpr int stages = DP <= 128 ? 2 : 1;
  constexpr size_t s2 = (size_t)stages * 2 * (4 * GC * (DP + 8) + 3 * GC * (GC + 8)) + (size_t)stages * DP * 4;
  static_assert(s2 <= 232448, "shared memory per CTA");
  if (s1 > 231 * 1024 - 4096) return B200_ERR_BAD_ARG;
  static size_t configured = 0;
  if (s1 > configured) {
    cudaError_t e = cudaFuncSetAttribute(gla_prepare_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s1);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(gla_scan_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s2);
    if (e != cudaSuccess) return (int)e;
    configured = s1;
  }
  int rc = launch_pdl(gla_prepare_kernel<DP>, dim3((max_q + GC - 1) / GC, a.H, n_seqs), dim3(256), s1, st, a, w);
  if (rc) return rc;
  rc = launch_pdl(gla_scan_kernel<DP>, dim3((a.VP + 63) / 64, a.H, n_seqs), dim3(128), s2, st, a, w);
  if (rc) return rc;
  return launch_pdl(gla_out_kernel, dim3(T, (a.H + 3) / 4), dim3(128), 0, st, a, (const float*)w.o);
}

// As b200_gla_recurrent, for prompts: T rows in all, max_q = longest chunk of a sequence; ws: b200_gla_chunk_bytes bytes, 256-byte
// aligned.
B200_API int b200_gla_chunked(const float* in, int ld, int q_off, int k_off, int v_off, int g_off, int a_off, int rank,
                              const float* a2, const float* b2, const float* w, float* state, const int* q_start,
                              const int* q_len, const int* ctx_len, const int* slot, int n_seqs, int H, int dim, int vdim, int VP,
                              float tau, float q_scale, float eps, float* out_f32, void* out_bf16, int ldo, int T, int max_q,
                              void* ws, size_t ws_bytes, cudaStream_t st) {
  GlaArgs a;
  int rc = gla_fill(a, in, ld, q_off, k_off, v_off, g_off, a_off, rank, a2, b2, w, state, q_start, q_len, ctx_len, slot, n_seqs, H,
                    dim, vdim, VP, tau, q_scale, eps, out_f32, out_bf16, ldo);
  if (rc) return rc;
  const size_t need = b200_gla_chunk_bytes(T, n_seqs, H, dim, VP, rank);
  if (!need || ws_bytes < need || T < 1 || max_q < 1 || ((uintptr_t)ws % 256)) return B200_ERR_BAD_ARG;
  const int DP = chunk_dp(dim);
  const size_t th = (size_t)T * H;
  char* p = (char*)ws;
  auto take = [&](size_t n) { char* q = p; p += align256(n); return q; };
  GlaChunkWs g;
  g.qh = (__nv_bfloat16*)take(th * DP * 2); g.ql = (__nv_bfloat16*)take(th * DP * 2);
  g.kh = (__nv_bfloat16*)take(th * DP * 2); g.kl = (__nv_bfloat16*)take(th * DP * 2);
  g.ah = (__nv_bfloat16*)take(th * GC * 2); g.al = (__nv_bfloat16*)take(th * GC * 2);
  g.v = (__nv_bfloat16*)take(th * VP * 2);
  g.dec = (float*)take(((size_t)T / GC + n_seqs + 1) * H * DP * 4);
  g.o = (float*)take(th * VP * 4);
  switch (DP) {
    case 32: return launch_chunked<32>(a, g, T, n_seqs, max_q, st);
    case 64: return launch_chunked<64>(a, g, T, n_seqs, max_q, st);
    case 128: return launch_chunked<128>(a, g, T, n_seqs, max_q, st);
    case 256: return launch_chunked<256>(a, g, T, n_seqs, max_q, st);
  }
  return B200_ERR_BAD_ARG;
}
