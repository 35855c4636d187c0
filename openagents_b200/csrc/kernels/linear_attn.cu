// Gated linear attention with a decay per key channel.  Per head, with state S [dim][vdim] (fp32, zero at a sequence's start):
//   S_t = diag(alpha_t) S_(t-1) + k_t v_t^T        o_t = S_t^T q_t / sqrt(dim)
//   alpha = sigmoid(z)^(1/tau),  z = A2 a + b2     (a = the low-rank projection of the layer's input)
//   out   = o / rms(o) * w * silu(g)               (rms over a head's vdim)
// Every sequence owns a slot of the state tensor; a chunk whose first token is at position 0 starts from zero without
// reading it.
//
// This file is compiled without fast math; decays, their logarithms and exponentials, the state and the norms are fp32.
#include <cooperative_groups.h>

#include "chunk_mma.cuh"

namespace cg = cooperative_groups;
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

// Token by token: decoding (one token per sequence) and the 32-bit mode's prompts.  One cluster per (head, sequence), whose CTAs
// share the value columns (few sequences: more SMs on the state's bytes); a thread owns the same float4 columns of the same state rows
// at every token, so the state needs no barrier of its own.  The rows are read eight at a time, the next eight in flight.
constexpr int kGlaRows = 8;
__global__ void __launch_bounds__(256) gla_recurrent_kernel(const GlaArgs a) {
  extern __shared__ __align__(16) float sm[];
  cg::cluster_group cluster = cg::this_cluster();
  const int CL = cluster.num_blocks(), part = cluster.block_rank();
  const int nv_all = a.VP >> 2, nv = nv_all / CL, W = nv * 4, e0 = part * W;     // this CTA's columns [e0, e0 + W)
  float* s_al = sm;                        // [dim] each
  float* s_q = s_al + a.dim;
  float* s_k = s_q + a.dim;
  float* s_v = s_k + a.dim + ((4 - ((3 * a.dim) & 3)) & 3);      // [W], 16-byte aligned
  float* s_o = s_v + W;                    // [groups][W]
  __shared__ float red[32];
  __shared__ float s_part[2];              // this CTA's sum of squares, by token parity
  pdl_trigger();
  const int h = blockIdx.x / CL, b = blockIdx.y, tid = threadIdx.x;
  // One channel per thread (heads of up to 256) and up to 16 ranks: the decay's weights are read while the projection still runs.
  const bool held = a.dim <= 256 && a.rank <= 16;
  float wz[16], bz = 0.f;
  if (held && tid < a.dim) {
    bz = a.b2[h * a.dim + tid];
#pragma unroll
    for (int r = 0; r < 16; r++) wz[r] = r < a.rank ? a.a2[(size_t)r * a.H * a.dim + h * a.dim + tid] : 0.f;
  }
  const float wo = (tid < W && e0 + tid < a.vdim) ? a.w[e0 + tid] : 0.f;
  pdl_wait();
  const int n = a.q_len[b], t0 = a.q_start[b], slot = a.slot[b];
  bool fresh = a.ctx_len[b] - n == 0 || slot < 0;
  const int groups = 256 / nv, grp = tid / nv, col = tid % nv;
  const bool active = grp < groups, keep = slot >= 0;
  float4* S = (float4*)(a.state + ((size_t)max(slot, 0) * a.H + h) * a.dim * a.VP) + part * nv + col;
  auto fetch = [&](float4 (&x)[kGlaRows], int d0) {
#pragma unroll
    for (int k = 0; k < kGlaRows; k++) {
      const int d = d0 + k * groups;
      x[k] = (active && !fresh && d < a.dim) ? S[(size_t)d * nv_all] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  for (int i = 0; i < n; i++) {
    float4 cur[kGlaRows], nxt[kGlaRows];
    fetch(cur, grp);                       // in flight while the decays are computed
    const float* row = a.in + (size_t)(t0 + i) * a.ld;
    const float gate = (tid < W && e0 + tid < a.vdim) ? row[a.g_off + h * a.vdim + e0 + tid] : 0.f;      // used at the end
    if (held && tid < a.dim) {
      const int c = h * a.dim + tid;
      const float q = row[a.q_off + c], k = row[a.k_off + c];
      float x[16];
#pragma unroll
      for (int r = 0; r < 16; r++) x[r] = r < a.rank ? row[a.a_off + r] : 0.f;
      float z = bz;
#pragma unroll
      for (int r = 0; r < 16; r++) z = fmaf(wz[r], x[r], z);
      s_q[tid] = q * a.q_scale;
      s_k[tid] = k;
      s_al[tid] = expf(log_decay(z, a.inv_tau));
    }
    for (int d = held ? a.dim : tid; d < a.dim; d += 256) {
      const int c = h * a.dim + d;
      float z = a.b2[c];
#pragma unroll 8
      for (int r = 0; r < a.rank; r++) z = fmaf(a.a2[(size_t)r * a.H * a.dim + c], row[a.a_off + r], z);
      s_q[d] = row[a.q_off + c] * a.q_scale;
      s_k[d] = row[a.k_off + c];
      s_al[d] = expf(log_decay(z, a.inv_tau));
    }
    for (int e = tid; e < W; e += 256) s_v[e] = e0 + e < a.vdim ? row[a.v_off + h * a.vdim + e0 + e] : 0.f;
    __syncthreads();
    if (active) {
      const float4 v = *(const float4*)(s_v + 4 * col);
      float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int d0 = grp; d0 < a.dim; d0 += kGlaRows * groups) {
        fetch(nxt, d0 + kGlaRows * groups);
#pragma unroll
        for (int k = 0; k < kGlaRows; k++) {
          const int d = d0 + k * groups;
          if (d >= a.dim) break;
          const float al = s_al[d], kk = s_k[d], q = s_q[d];
          float4 x = cur[k];
          x.x = fmaf(al, x.x, kk * v.x);
          x.y = fmaf(al, x.y, kk * v.y);
          x.z = fmaf(al, x.z, kk * v.z);
          x.w = fmaf(al, x.w, kk * v.w);
          if (keep) S[(size_t)d * nv_all] = x;
          o.x = fmaf(q, x.x, o.x);
          o.y = fmaf(q, x.y, o.y);
          o.z = fmaf(q, x.z, o.z);
          o.w = fmaf(q, x.w, o.w);
        }
#pragma unroll
        for (int k = 0; k < kGlaRows; k++) cur[k] = nxt[k];
      }
      *(float4*)(s_o + grp * W + 4 * col) = o;
    }
    __syncthreads();
    float ss = 0.f;
    for (int e = tid; e < W; e += 256) {
      float o = 0.f;
      for (int g = 0; g < groups; g++) o += s_o[g * W + e];
      s_o[e] = o;
      ss += o * o;                         // padding columns are zero
    }
    ss = block_sum(ss, red);
    if (CL > 1) {
      if (tid == 0) s_part[i & 1] = ss;
      cluster.sync();
      ss = 0.f;
      for (int p = 0; p < CL; p++) ss += *cluster.map_shared_rank(&s_part[i & 1], p);
    }
    const float r = 1.f / sqrtf(ss / (float)a.vdim + a.eps);
    for (int e = tid; e < W; e += 256) {
      float o = 0.f;
      if (e0 + e < a.vdim) {
        const float g = e < 256 ? gate : row[a.g_off + h * a.vdim + e0 + e];
        o = s_o[e] * r * (e < 256 ? wo : a.w[e0 + e]) * (g / (1.f + expf(-g)));
      }
      const size_t at = (size_t)(t0 + i) * a.ldo + (size_t)h * a.VP + e0 + e;
      if (a.out_f32) a.out_f32[at] = o;
      if (a.out_bf16) a.out_bf16[at] = __float2bfloat16(o);
    }
    fresh = !keep;
    __syncthreads();
  }
  if (CL > 1) cluster.sync();              // peers may still be reading this CTA's sum
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
  int CL = 1;                            // CTAs per head: until the SMs are covered, eight float4 columns each at least
  while (CL < 8 && (long)H * n_seqs * CL < 148 && (VP / 4) % (2 * CL) == 0 && VP / 4 / (2 * CL) >= 8) CL *= 2;
  const int nv = VP / 4 / CL, groups = 256 / nv;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(H * CL, n_seqs);
  cfg.blockDim = dim3(256);
  cfg.dynamicSmemBytes = 4 * ((size_t)3 * dim + 8 + 4 * nv + (size_t)groups * 4 * nv);      // at most 12 + 4 + 4 KB
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = CL;
  attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = b200_pdl_enabled() ? 2 : 1;
  return (int)cudaLaunchKernelEx(&cfg, gla_recurrent_kernel, a);
}

// ------------------------------------------------------------------ prompts: 64-token chunks on the tensor cores
//
// With b_t the running sum of log decays from the chunk's start and C its last token:
//   o_t = (q_t e^{b_t}) S + sum_{s<=t} A[t][s] v_s,   A[t][s] = sum_d q_td k_sd e^{b_td - b_sd}
//   S'  = diag(e^{b_C}) S + sum_s (k_s e^{b_C - b_s}) v_s^T
// gla_prepare_kernel computes the decays, the decayed queries and keys and A, all chunks and heads in parallel;
// gla_state_kernel walks a sequence's chunks with S in registers and leaves every chunk's starting state behind;
// gla_output_kernel forms the outputs, norms and gates them, again in parallel.
//
// The operands that hold decays or the state enter the tensor cores as two bf16 numbers each (value and remainder, about 16
// bits of mantissa), products accumulate in fp32, and the state stays fp32 between chunks; only v, a plain projection, is
// rounded to bf16 once.  A as a product of q e^{b} and k e^{-b} is exact in relative terms but the second factor grows with the
// decay; a chunk whose decay passes e^-60 in some channel takes the direct sum, whose exponents are never positive.

constexpr float kFactorLimit = 60.f;
constexpr int kMaxRank = 64;

struct GlaChunkWs {
  __nv_bfloat16 *qh, *ql, *kh, *kl;    // [T][H][DP] decayed queries / keys, value and remainder
  __nv_bfloat16 *ah, *al;              // [T][H][GC]
  __nv_bfloat16* v;                    // [T][H][VP]
  float* dec;                          // [chunk slots][H][DP]  e^{b_C}
  uint4* s;                            // [chunk slots][H][value tile of 16][DP / 16][lane][2]: the state at the chunk's start as MMA
                                       // operand registers (value columns as rows), four of values, four of remainders
  int nvt;                             // value tiles, a multiple of 4
};

constexpr int prep_threads(int dp) { return dp >= 64 ? 512 : 256; }

template <int DP>
__global__ void __launch_bounds__(prep_threads(DP), DP <= 128 ? 2 : 1) gla_prepare_kernel(const GlaArgs a, const GlaChunkWs ws) {
  constexpr int LQ = DP + 8;           // bf16 row stride: 16 bytes past a multiple of 128 (or 64)
  constexpr int NT = prep_threads(DP), NG = NT / (DP / 2), TPT = GC / NG, LB = TPT < 8 ? TPT : 8;      // a thread owns two channels of TPT consecutive tokens
  extern __shared__ __align__(16) __nv_bfloat16 p16[];
  __nv_bfloat16 *sqh = p16, *sql = sqh + GC * LQ;              // q e^b
  __nv_bfloat16 *sxh = sql + GC * LQ, *sxl = sxh + GC * LQ;    // k e^-b  (direct path: b itself, as fp32)
  __nv_bfloat16 *skh = sxl + GC * LQ, *skl = skh + GC * LQ;    // k e^(b_C - b)
  float* sa = (float*)(skl + GC * LQ);                         // [GC][rank rounded up to 16]
  float* stot = sa + GC * ((a.rank + 15) & ~15);               // [NG][DP]
  __shared__ float red[32];
  pdl_trigger();
  const int c = blockIdx.x, h = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x;
  const int d = tid % (DP / 2) * 2, grp = tid / (DP / 2), ch = h * a.dim + d, LR = (a.rank + 15) & ~15;
  const bool c0 = d < a.dim, c1 = d + 1 < a.dim;
  float w0[16], w1[16];                // weights: read while the projection still runs
  auto weights = [&](int r0) {
#pragma unroll
    for (int r = 0; r < 16; r++) {
      const float* p = a.a2 + (size_t)(r0 + r) * a.H * a.dim + ch;
      w0[r] = (c0 && r0 + r < a.rank) ? p[0] : 0.f;
      w1[r] = (c1 && r0 + r < a.rank) ? p[1] : 0.f;
    }
  };
  weights(0);
  const float2 bias = make_float2(c0 ? a.b2[ch] : 0.f, c1 ? a.b2[ch + 1] : 0.f);
  pdl_wait();
  const int len = a.q_len[seq], qs = a.q_start[seq];
  if (c * GC >= len) return;
  const int n = min(GC, len - c * GC), t0 = qs + c * GC;
  const float* in = a.in + (size_t)t0 * a.ld;
  if (((a.vdim | a.dim | a.v_off | a.q_off | a.k_off | a.ld) & 3) == 0 && tid < 3 * GC && tid % GC < n) {     // rows read later, into L2 now
    const int w3 = tid / GC;
    const float* p = in + (size_t)(tid % GC) * a.ld + (w3 == 0 ? a.q_off + h * a.dim : w3 == 1 ? a.k_off + h * a.dim : a.v_off + h * a.vdim);
    prefetch_l2(p, (w3 == 2 ? a.vdim : a.dim) * 4);
  }
  for (int i = tid; i < GC * LR; i += NT) {
    const int t = i / LR, r = i % LR;
    sa[i] = (t < n && r < a.rank) ? in[(size_t)t * a.ld + a.a_off + r] : 0.f;
  }
  if (((a.vdim | a.v_off | a.ld | a.VP) & 3) == 0) {
    GridWalk g(tid, NT, a.VP / 4);
#pragma unroll 4
    for (; g.r < n; g.next()) {
      const int t = g.r, e = g.c * 4;
      float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
      if (e < a.vdim) x = __ldg((const float4*)(in + (size_t)t * a.ld + a.v_off + h * a.vdim + e));
      *(uint2*)(ws.v + ((size_t)(t0 + t) * a.H + h) * a.VP + e) =
          make_uint2(pack_bf2(__float2bfloat16(x.x), __float2bfloat16(x.y)), pack_bf2(__float2bfloat16(x.z), __float2bfloat16(x.w)));
    }
  } else {
    for (int i = tid; i < n * a.VP; i += NT) {
      const int t = i / a.VP, e = i % a.VP;
      ws.v[((size_t)(t0 + t) * a.H + h) * a.VP + e] = __float2bfloat16(e < a.vdim ? in[(size_t)t * a.ld + a.v_off + h * a.vdim + e] : 0.f);
    }
  }
  __syncthreads();
  // log decays of this thread's tokens, sixteen ranks at a time, then their running sums
  float2 b[TPT];
#pragma unroll
  for (int i = 0; i < TPT; i++) b[i] = bias;
  for (int r0 = 0; r0 < LR; r0 += 16) {
    if (r0) weights(r0);
#pragma unroll
    for (int i = 0; i < TPT; i++) {
      const float4* x = (const float4*)(sa + (grp * TPT + i) * LR + r0);
#pragma unroll
      for (int r = 0; r < 4; r++) {
        const float4 y = x[r];
        b[i].x = fmaf(w0[4 * r], y.x, fmaf(w0[4 * r + 1], y.y, fmaf(w0[4 * r + 2], y.z, fmaf(w0[4 * r + 3], y.w, b[i].x))));
        b[i].y = fmaf(w1[4 * r], y.x, fmaf(w1[4 * r + 1], y.y, fmaf(w1[4 * r + 2], y.z, fmaf(w1[4 * r + 3], y.w, b[i].y))));
      }
    }
  }
  float2 sum = make_float2(0.f, 0.f);
#pragma unroll
  for (int i = 0; i < TPT; i++) {
    if (grp * TPT + i < n) {
      if (c0) sum.x += log_decay(b[i].x, a.inv_tau);
      if (c1) sum.y += log_decay(b[i].y, a.inv_tau);
    }
    b[i] = sum;
  }
  *(float2*)(stot + grp * DP + d) = sum;
  __syncthreads();
  float2 before = make_float2(0.f, 0.f), total = before;
#pragma unroll
  for (int g = 0; g < NG; g++) {
    const float2 x = *(const float2*)(stot + g * DP + d);
    if (g < grp) {
      before.x += x.x;
      before.y += x.y;
    }
    total.x += x.x;
    total.y += x.y;
  }
  const float2 etot = make_float2(expf(total.x), expf(total.y));
  if (grp == 0) *(float2*)(ws.dec + (chunk_slot(qs, seq, c) * a.H + h) * DP + d) = etot;
  const bool factored = block_max(fmaxf(-total.x, -total.y), red) < kFactorLimit;
  float* sb = (float*)sxh;             // [GC][LQ]
  const bool even = ((a.dim | a.q_off | a.k_off | a.ld) & 1) == 0;
  auto pair = [&](const float* p, bool row) -> float2 {
    if (!row || !c0) return make_float2(0.f, 0.f);
    if (even) return __ldg((const float2*)p);          // an even head size: both channels exist
    return make_float2(__ldg(p), c1 ? __ldg(p + 1) : 0.f);
  };
  auto put2 = [&](__nv_bfloat16* hi, __nv_bfloat16* lo, int at, float x, float y) {
    uint32_t u, v;
    split2(x, y, u, v);
    *(uint32_t*)(hi + at) = u;
    *(uint32_t*)(lo + at) = v;
  };
#pragma unroll
  for (int i0 = 0; i0 < TPT; i0 += LB) {
    float2 q[LB], k[LB];               // LB tokens' loads in flight
#pragma unroll
    for (int i = 0; i < LB; i++) {
      const int t = grp * TPT + i0 + i;
      q[i] = pair(in + (size_t)t * a.ld + a.q_off + ch, t < n);
      k[i] = pair(in + (size_t)t * a.ld + a.k_off + ch, t < n);
    }
#pragma unroll
    for (int i = 0; i < LB; i++) {
      const int at = (grp * TPT + i0 + i) * LQ + d;
      const float bx = b[i0 + i].x + before.x, by = b[i0 + i].y + before.y;
      const float ex = expf(bx), ey = expf(by);
      put2(sqh, sql, at, q[i].x * a.q_scale * ex, q[i].y * a.q_scale * ey);
      if (factored) {                  // e^b stays above e^-60: its reciprocal and e^b_C times that are as exact as their exponentials
        const float kx = k[i].x / ex, ky = k[i].y / ey;
        put2(sxh, sxl, at, kx, ky);
        put2(skh, skl, at, kx * etot.x, ky * etot.y);
      } else {
        put2(skh, skl, at, k[i].x * expf(total.x - bx), k[i].y * expf(total.y - by));
        *(float2*)(sb + at) = make_float2(bx, by);
      }
    }
  }
  __syncthreads();
  for (int i = tid; i < n * (DP / 8); i += NT) {          // 16 bytes a time
    const int t = i / (DP / 8), x = i % (DP / 8) * 8;
    const size_t at = ((size_t)(t0 + t) * a.H + h) * DP + x;
    *(uint4*)(ws.qh + at) = *(const uint4*)(sqh + t * LQ + x);
    *(uint4*)(ws.ql + at) = *(const uint4*)(sql + t * LQ + x);
    *(uint4*)(ws.kh + at) = *(const uint4*)(skh + t * LQ + x);
    *(uint4*)(ws.kl + at) = *(const uint4*)(skl + t * LQ + x);
  }
  const int warp = tid >> 5, lane = tid & 31, g4 = lane >> 2, t4 = lane & 3;
  if (factored) {
    // warp = 16 rows x 8 NJ columns of the lower triangle
    constexpr int WN = NT / 128, NJ = 8 / WN;
    const int m0 = (warp / WN) * 16, n0 = (warp % WN) * 8 * NJ;
    float acc[NJ][4] = {};
    if (n0 <= m0 + 15) {
#pragma unroll
      for (int k0 = 0; k0 < DP; k0 += 16) {
        uint32_t ah[4], al[4];
        const int ra = (m0 + (lane & 15)) * LQ + k0 + (lane >> 4) * 8;
        ldsm4(s32(sqh + ra), ah);
        ldsm4(s32(sql + ra), al);
#pragma unroll
        for (int j = 0; j < NJ; j += 2) {
          const int rb = (n0 + (j + (lane >> 4)) * 8 + (lane & 7)) * LQ + k0 + ((lane >> 3) & 1) * 8;
          uint32_t bh[4], bl[4];
          ldsm4(s32(sxh + rb), bh);
          ldsm4(s32(sxl + rb), bl);
          mma_bf16(acc[j], ah, bh[0], bh[1]);
          mma_bf16(acc[j], ah, bl[0], bl[1]);
          mma_bf16(acc[j], al, bh[0], bh[1]);
          mma_bf16(acc[j + 1], ah, bh[2], bh[3]);
          mma_bf16(acc[j + 1], ah, bl[2], bl[3]);
          mma_bf16(acc[j + 1], al, bh[2], bh[3]);
        }
      }
    }
#pragma unroll
    for (int j = 0; j < NJ; j++)
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
    for (int i = tid; i < n * GC; i += NT) {
      const int t = i / GC, s = i % GC;
      float x = 0.f;
      if (s <= t) {
        const float *q = in + (size_t)t * a.ld + a.q_off + h * a.dim, *k = in + (size_t)s * a.ld + a.k_off + h * a.dim;
        for (int e = 0; e < a.dim; e++) x = fmaf(q[e] * a.q_scale * k[e], expf(sb[t * LQ + e] - sb[s * LQ + e]), x);
      }
      const size_t at = ((size_t)(t0 + t) * a.H + h) * GC + s;
      split_bf16(x, ws.ah[at], ws.al[at]);
    }
  }
}

constexpr int kStateStages = 3;
constexpr int state_slice(int dp) { return dp < 64 ? dp : 64; }

// One CTA = 64 value columns x DS key channels of one head of one sequence (no entry of the state meets another before the output
// product); a warp owns 16 value columns and half of the channels.  The state is kept transposed (value columns as the
// rows of the MMA): its accumulator registers, split into values and remainders, are the A operand of the output product as they lie,
// and that is the form a chunk's starting state is stored in.
template <int DP>
__global__ void __launch_bounds__(256) gla_state_kernel(const GlaArgs a, const GlaChunkWs ws) {
  constexpr int DS = state_slice(DP), DW = DS / 2, LQ = DS + 8, LV = 72;
  constexpr int STAGE = 2 * GC * LQ + GC * LV;                // kh kl | v
  extern __shared__ __align__(16) __nv_bfloat16 sb16[];
  float* sdec = (float*)(sb16 + kStateStages * STAGE);        // [stages][DS]
  pdl_trigger();
  pdl_wait();
  const int vs = blockIdx.x / (DP / DS), d0 = blockIdx.x % (DP / DS) * DS, v0 = vs * 64, h = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x;
  const int warp = (tid >> 5) & 3, dw = (tid >> 7) * DW, lane = tid & 31, g4 = lane >> 2, t4 = lane & 3;
  const int len = a.q_len[seq], qs = a.q_start[seq], slot = a.slot[seq];
  const bool fresh = a.ctx_len[seq] - len == 0 || slot < 0;
  const int nc = (len + GC - 1) / GC;
  float* S = a.state + ((size_t)max(slot, 0) * a.H + h) * a.dim * a.VP;

  auto cp16 = [](void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(s32(dst)), "l"(src));
  };
  // this thread's 16-byte pieces of a chunk: KP of the keys (values, then remainders), two of V, and one of the decays for some
  constexpr int CQ = DS / 8, KP = 2 * GC * CQ / 256;
  const __nv_bfloat16 *ksrc[KP], *vsrc[2];
  int kt0[KP], kdst[KP];
#pragma unroll
  for (int m = 0; m < KP; m++) {
    const int i = tid + 256 * m, p = i / (GC * CQ), t = (i / CQ) % GC, x = i % CQ;
    kt0[m] = t;
    kdst[m] = p * GC * LQ + t * LQ + x * 8;
    ksrc[m] = (p ? ws.kl : ws.kh) + ((size_t)(qs + t) * a.H + h) * DP + d0 + x * 8;
  }
  const int vt0 = tid / 8, vx = (tid % 8) * 8;
  const bool vlive = v0 + vx < a.VP;
#pragma unroll
  for (int m = 0; m < 2; m++) vsrc[m] = ws.v + ((size_t)(qs + vt0 + 32 * m) * a.H + h) * a.VP + v0 + vx;
  const float* dsrc = ws.dec + (chunk_slot(qs, seq, 0) * a.H + h) * DP + d0 + tid * 4;
  const size_t kstep = (size_t)GC * a.H * DP, vstep = (size_t)GC * a.H * a.VP, dstep = (size_t)a.H * DP;
  auto load = [&](int c) {
    if (c < nc) {
      __nv_bfloat16* st = sb16 + (c % kStateStages) * STAGE;
      const int n = len - c * GC;
#pragma unroll
      for (int m = 0; m < KP; m++) {
        if (kt0[m] < n) cp16(st + kdst[m], ksrc[m] + c * kstep);
        else *(uint4*)(st + kdst[m]) = make_uint4(0u, 0u, 0u, 0u);
      }
#pragma unroll
      for (int m = 0; m < 2; m++) {
        __nv_bfloat16* dst = st + 2 * GC * LQ + (vt0 + 32 * m) * LV + vx;
        if (vlive && vt0 + 32 * m < n) cp16(dst, vsrc[m] + c * vstep);
        else *(uint4*)dst = make_uint4(0u, 0u, 0u, 0u);
      }
      if (tid < DS / 4) cp16(sdec + (c % kStateStages) * DS + tid * 4, dsrc + c * dstep);
    }
    asm volatile("cp.async.commit_group;");      // empty past the end: keeps the count of groups in flight
  };

#pragma unroll
  for (int c = 0; c < kStateStages - 1; c++) load(c);
  // sacc[j] = rows v0 + 16 warp + g4 (+ 8), columns d = d0 + 8 j + 2 t4 (+ 1)
  float sacc[DW / 8][4];
#pragma unroll
  for (int j = 0; j < DW / 8; j++)
#pragma unroll
    for (int e = 0; e < 4; e++) {
      const int v = v0 + warp * 16 + g4 + 8 * (e >> 1), d = d0 + dw + 8 * j + 2 * t4 + (e & 1);
      sacc[j][e] = (!fresh && v < a.VP && d < a.dim) ? S[(size_t)d * a.VP + v] : 0.f;
    }
  for (int c = 0; c < nc; c++) {
    asm volatile("cp.async.wait_group %0;" ::"n"(kStateStages - 2));
    __syncthreads();                   // chunk c has landed, and everyone is done with the stage that is refilled now
    load(c + kStateStages - 1);
    const __nv_bfloat16* st = sb16 + (c % kStateStages) * STAGE;
    const __nv_bfloat16 *sKh = st, *sKl = st + GC * LQ, *sV = st + 2 * GC * LQ;
    const float* dec = sdec + (c % kStateStages) * DS;
    if (c > 0 || !fresh) {
      uint4* frag = ws.s + (((chunk_slot(qs, seq, c) * a.H + h) * ws.nvt + vs * 4 + warp) * (DP / 16) * 32 + (d0 + dw) * 2 + lane) * 2;
#pragma unroll
      for (int kd = 0; kd < DW / 16; kd++) {
        uint4 hi, lo;
        split2(sacc[2 * kd][0], sacc[2 * kd][1], hi.x, lo.x);
        split2(sacc[2 * kd][2], sacc[2 * kd][3], hi.y, lo.y);
        split2(sacc[2 * kd + 1][0], sacc[2 * kd + 1][1], hi.z, lo.z);
        split2(sacc[2 * kd + 1][2], sacc[2 * kd + 1][3], hi.w, lo.w);
        frag[kd * 64] = hi;
        frag[kd * 64 + 1] = lo;
      }
#pragma unroll
      for (int j = 0; j < DW / 8; j++) {
        const float2 f = *(const float2*)(dec + dw + 8 * j + 2 * t4);
        sacc[j][0] *= f.x;
        sacc[j][1] *= f.y;
        sacc[j][2] *= f.x;
        sacc[j][3] *= f.y;
      }
    }
#pragma unroll
    for (int kt = 0; kt < GC / 16; kt++) {
      uint32_t va[4];                  // V^T: 16 value columns x 16 tokens
      ldsm4t(s32(sV + (kt * 16 + (lane >> 4) * 8 + (lane & 7)) * LV + warp * 16 + ((lane >> 3) & 1) * 8), va);
      const int r = kt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8;
#pragma unroll
      for (int j = 0; j < DW / 8; j += 2) {          // S^T += V^T (k e^{b_C - b})
        uint32_t bh[4], bl[4];
        ldsm4t(s32(sKh + r * LQ + dw + (j + (lane >> 4)) * 8), bh);
        ldsm4t(s32(sKl + r * LQ + dw + (j + (lane >> 4)) * 8), bl);
        mma_bf16(sacc[j], va, bh[0], bh[1]);
        mma_bf16(sacc[j + 1], va, bh[2], bh[3]);
        mma_bf16(sacc[j], va, bl[0], bl[1]);
        mma_bf16(sacc[j + 1], va, bl[2], bl[3]);
      }
    }
  }
  if (slot >= 0) {
#pragma unroll
    for (int j = 0; j < DW / 8; j++)
#pragma unroll
      for (int e = 0; e < 4; e++) {
        const int v = v0 + warp * 16 + g4 + 8 * (e >> 1), d = d0 + dw + 8 * j + 2 * t4 + (e & 1);
        if (v < a.VP && d < a.dim) S[(size_t)d * a.VP + v] = sacc[j][e];
      }
  }
}

// Outputs of one chunk and head over all its value columns (NV tiles of 16 per warp):
//   O^T = S^T (q e^b)^T + V^T A^T,   then  out = o / rms(o) * w * silu(g).
template <int DP, int NV>
__global__ void __launch_bounds__(256, NV <= 2 ? 2 : 1) gla_output_kernel(const GlaArgs a, const GlaChunkWs ws) {
  constexpr int LQ = DP + 8, LA = GC + 8;
  extern __shared__ __align__(16) __nv_bfloat16 o16[];
  const int LV = ws.nvt * 16 + 8;                              // bf16 row stride of V
  __nv_bfloat16 *sQh = o16, *sQl = sQh + GC * LQ, *sAh = sQl + GC * LQ, *sAl = sAh + GC * LA, *sV = sAl + GC * LA;
  float* so = (float*)o16;                                     // [GC][nvt * 16 + 4], over the operands once they are used
  const int LO = ws.nvt * 16 + 4;
  __shared__ float s_ss[8][GC];
  pdl_trigger();
  pdl_wait();
  const int c = blockIdx.x, h = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x;
  const int warp = tid >> 5, lane = tid & 31, g4 = lane >> 2, t4 = lane & 3;
  const int len = a.q_len[seq], qs = a.q_start[seq];
  if (c * GC >= len) return;
  const bool with_state = c > 0 || !(a.ctx_len[seq] - len == 0 || a.slot[seq] < 0);
  const int n = min(GC, len - c * GC), t0 = qs + c * GC;
  auto cp16 = [](void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(s32(dst)), "l"(src));
  };
  for (int i = tid; i < 2 * GC * 8; i += 256) {
    const int p = i / (GC * 8), t = (i / 8) % GC, x = i % 8;
    __nv_bfloat16* dst = sAh + p * GC * LA + t * LA + x * 8;
    if (t < n) cp16(dst, (p ? ws.al : ws.ah) + ((size_t)(t0 + t) * a.H + h) * GC + x * 8);
    else *(uint4*)dst = make_uint4(0u, 0u, 0u, 0u);
  }
  for (GridWalk g(tid, 256, ws.nvt * 2); g.r < GC; g.next()) {
    const int t = g.r, x = g.c;
    __nv_bfloat16* dst = sV + t * LV + x * 8;
    if (t < n && x * 8 < a.VP) cp16(dst, ws.v + ((size_t)(t0 + t) * a.H + h) * a.VP + x * 8);
    else *(uint4*)dst = make_uint4(0u, 0u, 0u, 0u);
  }
  asm volatile("cp.async.commit_group;");                     // A and V first: their product needs no state
  constexpr int CQ = DP / 8;
  for (int i = tid; i < 2 * GC * CQ; i += 256) {
    const int p = i / (GC * CQ), t = (i / CQ) % GC, x = i % CQ;
    __nv_bfloat16* dst = sQh + p * GC * LQ + t * LQ + x * 8;
    if (t < n) cp16(dst, (p ? ws.ql : ws.qh) + ((size_t)(t0 + t) * a.H + h) * DP + x * 8);
    else *(uint4*)dst = make_uint4(0u, 0u, 0u, 0u);
  }
  asm volatile("cp.async.commit_group;");
  const bool vec = ((a.vdim | a.g_off | a.ld | a.ldo) & 3) == 0 && ((uintptr_t)a.w & 15) == 0;
  if (vec && tid < n) prefetch_l2(a.in + (size_t)(t0 + tid) * a.ld + a.g_off + h * a.vdim, a.vdim * 4);      // gates, read at the end
  const uint4* frag = ws.s + ((chunk_slot(qs, seq, c) * a.H + h) * ws.nvt * (DP / 16) * 32 + lane) * 2;
  uint4 nx[NV][2];                     // the next step's state operands, in flight
  auto fetch = [&](int kd) {
#pragma unroll
    for (int i = 0; i < NV; i++) {
      const uint4* p = frag + ((size_t)min(warp + 8 * i, ws.nvt - 1) * (DP / 16) + kd) * 64;
      nx[i][0] = __ldg(p);
      nx[i][1] = __ldg(p + 1);
    }
  };
  if (with_state) fetch(0);
  asm volatile("cp.async.wait_group 1;");
  __syncthreads();

  float oacc[NV][8][4];                // value tile warp + 8 i; columns = tokens 8 j + 2 t4 (+ 1)
#pragma unroll
  for (int i = 0; i < NV; i++)
#pragma unroll
    for (int j = 0; j < 8; j++) oacc[i][j][0] = oacc[i][j][1] = oacc[i][j][2] = oacc[i][j][3] = 0.f;
#pragma unroll
  for (int kt = 0; kt < GC / 16; kt++) {
    uint32_t va[NV][4];                // V^T: 16 value columns x 16 tokens
#pragma unroll
    for (int i = 0; i < NV; i++)
      ldsm4t(s32(sV + (kt * 16 + (lane >> 4) * 8 + (lane & 7)) * LV + min(warp + 8 * i, ws.nvt - 1) * 16 + ((lane >> 3) & 1) * 8), va[i]);
#pragma unroll
    for (int j = 2 * kt; j < 8; j += 2) {            // output tokens see tokens up to their own
      const int r = (j + (lane >> 4)) * 8 + (lane & 7), x = kt * 16 + ((lane >> 3) & 1) * 8;
      uint32_t bh[4], bl[4];
      ldsm4(s32(sAh + r * LA + x), bh);
      ldsm4(s32(sAl + r * LA + x), bl);
#pragma unroll
      for (int i = 0; i < NV; i++) {
        mma_bf16(oacc[i][j], va[i], bh[0], bh[1]);
        mma_bf16(oacc[i][j + 1], va[i], bh[2], bh[3]);
        mma_bf16(oacc[i][j], va[i], bl[0], bl[1]);
        mma_bf16(oacc[i][j + 1], va[i], bl[2], bl[3]);
      }
    }
  }
  asm volatile("cp.async.wait_group 0;");
  __syncthreads();
  if (with_state) {
#pragma unroll
    for (int kd = 0; kd < DP / 16; kd++) {
      uint32_t sh[NV][4], sl[NV][4];
#pragma unroll
      for (int i = 0; i < NV; i++) {
        sh[i][0] = nx[i][0].x; sh[i][1] = nx[i][0].y; sh[i][2] = nx[i][0].z; sh[i][3] = nx[i][0].w;
        sl[i][0] = nx[i][1].x; sl[i][1] = nx[i][1].y; sl[i][2] = nx[i][1].z; sl[i][3] = nx[i][1].w;
      }
      if (kd + 1 < DP / 16) fetch(kd + 1);
#pragma unroll
      for (int j = 0; j < 8; j += 2) {
        const int r = (j + (lane >> 4)) * 8 + (lane & 7), x = kd * 16 + ((lane >> 3) & 1) * 8;
        uint32_t bh[4], bl[4];
        ldsm4(s32(sQh + r * LQ + x), bh);
        ldsm4(s32(sQl + r * LQ + x), bl);
#pragma unroll
        for (int i = 0; i < NV; i++) {
          mma_bf16(oacc[i][j], sh[i], bh[0], bh[1]);
          mma_bf16(oacc[i][j + 1], sh[i], bh[2], bh[3]);
          mma_bf16(oacc[i][j], sh[i], bl[0], bl[1]);
          mma_bf16(oacc[i][j + 1], sh[i], bl[2], bl[3]);
          mma_bf16(oacc[i][j], sl[i], bh[0], bh[1]);
          mma_bf16(oacc[i][j + 1], sl[i], bh[2], bh[3]);
        }
      }
    }
  }
  // sums of squares per token (value columns past vdim hold zeros), then the tile through shared memory for whole-line stores
#pragma unroll
  for (int j = 0; j < 8; j++)
#pragma unroll
    for (int e = 0; e < 2; e++) {
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < NV; i++)
        if (warp + 8 * i < ws.nvt) ss += oacc[i][j][e] * oacc[i][j][e] + oacc[i][j][e + 2] * oacc[i][j][e + 2];
      ss += __shfl_xor_sync(0xffffffffu, ss, 4);
      ss += __shfl_xor_sync(0xffffffffu, ss, 8);
      ss += __shfl_xor_sync(0xffffffffu, ss, 16);
      if (g4 == 0) s_ss[warp][8 * j + 2 * t4 + e] = ss;
    }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < NV; i++)
    if (warp + 8 * i < ws.nvt) {
#pragma unroll
      for (int j = 0; j < 8; j++)
#pragma unroll
        for (int e = 0; e < 4; e++) so[(8 * j + 2 * t4 + (e & 1)) * LO + (warp + 8 * i) * 16 + g4 + 8 * (e >> 1)] = oacc[i][j][e];
    }
  __syncthreads();
  if (tid < GC) {
    float ss = 0.f;
#pragma unroll
    for (int w = 0; w < 8; w++) ss += s_ss[w][tid];
    s_ss[0][tid] = 1.f / sqrtf(ss / (float)a.vdim + a.eps);
  }
  __syncthreads();
  GridWalk gw(tid, 256, a.VP / 4);
#pragma unroll 4
  for (; gw.r < n; gw.next()) {
    const int t = gw.r, e = gw.c * 4;
    const float r = s_ss[0][t];
    const float* g = a.in + (size_t)(t0 + t) * a.ld + a.g_off + h * a.vdim + e;
    const float4 o = *(const float4*)(so + t * LO + e);
    float y[4] = {o.x, o.y, o.z, o.w}, x[4] = {0.f, 0.f, 0.f, 0.f}, w[4] = {0.f, 0.f, 0.f, 0.f};
    if (vec && e < a.vdim) {
      *(float4*)x = __ldg((const float4*)g);
      *(float4*)w = __ldg((const float4*)(a.w + e));
    } else {
#pragma unroll
      for (int k = 0; k < 4; k++)
        if (e + k < a.vdim) {
          x[k] = __ldg(g + k);
          w[k] = __ldg(a.w + e + k);
        }
    }
#pragma unroll
    for (int k = 0; k < 4; k++) y[k] *= r * w[k] * __fdividef(x[k], 1.f + __expf(-x[k]));      // the output gate: no part of the recurrence
    const size_t at = (size_t)(t0 + t) * a.ldo + (size_t)h * a.VP + e;
    if (a.out_f32) *(float4*)(a.out_f32 + at) = make_float4(y[0], y[1], y[2], y[3]);
    if (a.out_bf16)
      *(uint2*)(a.out_bf16 + at) = make_uint2(pack_bf2(__float2bfloat16(y[0]), __float2bfloat16(y[1])), pack_bf2(__float2bfloat16(y[2]), __float2bfloat16(y[3])));
  }
}

static int chunk_dp(int dim) { return dim <= 32 ? 32 : dim <= 64 ? 64 : dim <= 128 ? 128 : dim <= 256 ? 256 : 0; }
static int value_tiles(int VP) { return (VP + 63) / 64 * 4; }

// Bytes of workspace for b200_gla_chunked; 0: sizes it does not take (the caller then uses b200_gla_recurrent).
B200_API size_t b200_gla_chunk_bytes(int T, int n_seqs, int H, int dim, int VP, int rank) {
  const int DP = chunk_dp(dim);
  if (!DP || rank > kMaxRank || VP % 8 || VP > 512) return 0;
  const size_t th = (size_t)T * H, slots = (size_t)T / GC + n_seqs + 1;
  return 4 * align256(th * DP * 2) + 2 * align256(th * GC * 2) + align256(th * VP * 2) + align256(slots * H * DP * 4) +
         align256(slots * H * value_tiles(VP) * DP * 64);
}

template <int DP, int NV>
static int launch_output(const GlaArgs& a, const GlaChunkWs& w, int n_seqs, int max_q, cudaStream_t st) {
  const size_t operands = 2 * ((size_t)2 * GC * (DP + 8) + 2 * GC * (GC + 8) + (size_t)GC * (w.nvt * 16 + 8));
  const size_t tile = (size_t)GC * (w.nvt * 16 + 4) * 4, smem = operands > tile ? operands : tile;
  if (smem > 220 * 1024) return B200_ERR_BAD_ARG;
  static size_t configured = 0;
  if (smem > configured) {
    cudaError_t e = cudaFuncSetAttribute(gla_output_kernel<DP, NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = smem;
  }
  return launch_pdl(gla_output_kernel<DP, NV>, dim3((max_q + GC - 1) / GC, a.H, n_seqs), dim3(256), smem, st, a, w);
}

template <int DP>
static int launch_chunked(const GlaArgs& a, const GlaChunkWs& w, int n_seqs, int max_q, cudaStream_t st) {
  const size_t s1 = (size_t)6 * GC * (DP + 8) * 2 + 4 * (size_t)(GC * ((a.rank + 15) & ~15) + 2 * prep_threads(DP));
  constexpr int DS = state_slice(DP);
  constexpr size_t s2 = (size_t)kStateStages * (2 * (2 * GC * (DS + 8) + GC * 72) + DS * 4);
  if (s1 > 225 * 1024) return B200_ERR_BAD_ARG;
  static size_t configured = 0;
  if (s1 > configured) {
    cudaError_t e = cudaFuncSetAttribute(gla_prepare_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s1);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(gla_state_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s2);
    if (e != cudaSuccess) return (int)e;
    configured = s1;
  }
  int rc = launch_pdl(gla_prepare_kernel<DP>, dim3((max_q + GC - 1) / GC, a.H, n_seqs), dim3(prep_threads(DP)), s1, st, a, w);
  if (rc) return rc;
  rc = launch_pdl(gla_state_kernel<DP>, dim3(w.nvt / 4 * (DP / DS), a.H, n_seqs), dim3(256), s2, st, a, w);
  if (rc) return rc;
  if (w.nvt <= 8) return launch_output<DP, 1>(a, w, n_seqs, max_q, st);
  if (w.nvt <= 16) return launch_output<DP, 2>(a, w, n_seqs, max_q, st);
  return launch_output<DP, 4>(a, w, n_seqs, max_q, st);
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
  if (!need || ws_bytes < need || T < 1 || max_q < 1 || (ldo & 3) || ((uintptr_t)out_f32 % 16) || ((uintptr_t)out_bf16 % 8) || ((uintptr_t)ws % 256) || ((uintptr_t)in % 16)) return B200_ERR_BAD_ARG;
  const int DP = chunk_dp(dim);
  const size_t th = (size_t)T * H, slots = (size_t)T / GC + n_seqs + 1;
  char* p = (char*)ws;
  auto take = [&](size_t n) { char* q = p; p += align256(n); return q; };
  GlaChunkWs g;
  g.nvt = value_tiles(VP);
  g.qh = (__nv_bfloat16*)take(th * DP * 2); g.ql = (__nv_bfloat16*)take(th * DP * 2);
  g.kh = (__nv_bfloat16*)take(th * DP * 2); g.kl = (__nv_bfloat16*)take(th * DP * 2);
  g.ah = (__nv_bfloat16*)take(th * GC * 2); g.al = (__nv_bfloat16*)take(th * GC * 2);
  g.v = (__nv_bfloat16*)take(th * VP * 2);
  g.dec = (float*)take(slots * H * DP * 4);
  g.s = (uint4*)take(slots * H * g.nvt * DP * 64);
  switch (DP) {
    case 32: return launch_chunked<32>(a, g, n_seqs, max_q, st);
    case 64: return launch_chunked<64>(a, g, n_seqs, max_q, st);
    case 128: return launch_chunked<128>(a, g, n_seqs, max_q, st);
    case 256: return launch_chunked<256>(a, g, n_seqs, max_q, st);
  }
  return B200_ERR_BAD_ARG;
}
