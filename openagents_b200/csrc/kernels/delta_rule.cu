// Generalized delta rule: a linear recurrence that decays its state per key channel, takes away what the state holds along a key, and adds a new
// key / value product.  Per head, with state S [dim][vdim] (fp32, zero at a sequence's start), u = k / sqrt(sum k^2 + 1e-6) and c = a u:
//   S_t = diag(w_t) S_(t-1) - c_t (u_t^T S_(t-1)) + k_t v_t^T        o_t = S_t^T r_t
//   w = exp(-decay * sigmoid(W2 tanh(x) + w0)),  a = sigmoid(a' + ab)      (x: the low-rank projection of the layer's input)
//   out = o / rms(o) * norm * sigmoid(g)                                   (rms over a head's vdim; norm per head and column)
// Every sequence owns a slot of the state tensor; a portion whose first token is at position 0 starts from zero without reading it.
//
// This file is compiled without fast math; decays, their logarithms and exponentials, rates, unit keys, states and norms are fp32.
#include <cooperative_groups.h>

#include "chunk_mma.cuh"
#include "warp_mma.cuh"

namespace cg = cooperative_groups;
using namespace b200;

struct DeltaArgs {
  const float* in;              // [T][ld] fused projections
  int ld, r_off, k_off, v_off, g_off, a_off, x_off, rank;
  const __nv_bfloat16* w2;      // [H * dim][rank8], columns rank.. zero
  int rank8;
  const float* w0;              // [H * dim]
  const float* ab;              // [H * dim]
  const float* norm;            // [H * vdim]
  float* state;                 // [slots][H][dim][VP]
  const int* q_start;
  const int* q_len;
  const int* ctx_len;           // tokens of the sequence after this portion
  const int* slot;              // state slot per sequence; < 0: start from zero, keep nothing
  int H, dim, vdim, VP;
  float decay, eps;
  float* out_f32;               // [T][ldo], head h at column h * VP, columns vdim..VP zero
  __nv_bfloat16* out_bf16;
  int ldo;
};
constexpr int kDeltaDim = 256;        // most key channels of a head
constexpr int kDeltaRank = 1024;      // most ranks of the decay's projection
constexpr float kUnitEps = 1e-6f;

__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
// The same on the hardware's exponential and reciprocal (some 1e-7 relative), for operands that are rounded to two bf16 numbers.
__device__ __forceinline__ float sigmoid_fast(float x) { return __fdividef(1.f, 1.f + __expf(-x)); }

// ------------------------------------------------------------------ token by token

// Decoding, and the prompts of the 32-bit mode.  One cluster per head and share of the sequences, whose CTAs share the value columns.  A CTA walks the tokens
// of its sequences one by one.  While the state meets one token, what the next one does to it (decays, rates) is computed from its projections, and the
// projections of the one after, and with a new sequence its state, are on their way.  The state is updated in shared memory.  With n = 1 / (sum k^2 + 1e-6), R = k^T S and p = (r w)^T S, from one pass over the old state,
//   o = p - n (r . a k) R + (r . k) v        S' = diag(w) S - a k (n R) + k v^T
// so a token needs three sums over the channels and one reduction over the state's rows.
__device__ __forceinline__ void cp_async4(void* dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(s32(dst)), "l"(src) : "memory");
}
struct DeltaLayout {                       // floats of shared memory
  int state, row, ch, kr, x, z, read, red, total;      // offsets; of the first buffer (two of state, ch and kr, three of row)
  int state_n, row_n;                      // sizes of one buffer
};
static DeltaLayout delta_layout(int dim, int W, int rank8, int threads) {
  DeltaLayout l;
  const int groups = threads / (W / 4);
  auto up4 = [](int n) { return (n + 3) & ~3; };
  l.state_n = dim * W;
  l.row_n = up4(3 * dim) + 2 * W + rank8;  // r k a | v g | x
  l.state = 0;
  l.row = 2 * l.state_n;
  l.ch = l.row + 3 * l.row_n;
  l.kr = l.ch + 8 * dim;
  l.x = l.kr + up4(4 * dim);
  l.z = l.x + rank8;
  l.read = l.z + up4(dim);
  l.red = l.read + W;
  l.total = l.red + groups * 2 * W;
  return l;
}
constexpr int kRowPieces = 4;              // elements of a projection row that a thread fetches without working out their places again

// DIM, NV: channels and float4 columns of a CTA's share of a head, where they are known (0: not).
// The fewer threads share a token, the less each spends on anything but the state.
template <int DIM, int NV, int NT>
__global__ void __launch_bounds__(NT, NT == 128 ? 3 : 2) delta_recurrent_kernel(const DeltaArgs a, int n_seqs, const DeltaLayout l) {
  extern __shared__ __align__(16) float sm[];
  cg::cluster_group cluster = cg::this_cluster();
  const int CL = cluster.num_blocks(), part = cluster.block_rank(), dim = DIM ? DIM : a.dim;
  const int nv_all = a.VP >> 2, nv = NV ? NV : nv_all / CL, W = nv * 4, e0 = part * W;     // this CTA's columns [e0, e0 + W)
  const int groups = NT / nv;
  float4* s_ch = (float4*)(sm + l.ch);     // [2][dim] (w, a k, k, -)
  float2* s_kr = (float2*)(sm + l.kr);     // [2][dim] (k, r w)
  float *s_x = sm + l.x, *s_z = sm + l.z, *s_read = sm + l.read, *s_red = sm + l.red;
  __shared__ float red[2][3][8], red1[8];
  __shared__ float s_part[2];              // this CTA's sum of squares, by token parity
  pdl_trigger();
  const int h = blockIdx.x / CL, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  // TPC threads share a channel's low-rank product; its weights are read while the projection still runs
  int TPC = 1;
  while (TPC < 8 && dim * TPC * 2 <= NT) TPC *= 2;
  const int ch = tid / TPC, sub = tid % TPC;
  const __nv_bfloat16* wrow = a.w2 + (size_t)(h * dim + (ch < dim ? ch : 0)) * a.rank8;
  constexpr int HELD = 1024 / NT;
  uint4 held[HELD];
#pragma unroll
  for (int i = 0; i < HELD; i++) held[i] = ch < dim && (sub + i * TPC) * 8 < a.rank8 ? ((const uint4*)wrow)[sub + i * TPC] : make_uint4(0u, 0u, 0u, 0u);
  const int cc = NT - 1 - tid;                // the last warps take a channel each, the first ones an output column
  const float w0 = cc < dim ? a.w0[h * dim + cc] : 0.f, ab = cc < dim ? a.ab[h * dim + cc] : 0.f;
  const float wo = (tid < W && e0 + tid < a.vdim) ? a.norm[h * a.vdim + e0 + tid] : 0.f;
  const int grp = tid / nv, col = tid % nv, rka = (3 * dim + 3) & ~3;
  constexpr int ROWS = DIM ? DIM * NV / NT : 0;                // a thread's state rows, where they are known and all threads have as many
  static_assert(DIM == 0 || (NT % NV == 0 && DIM % (NT / NV) == 0), "whole rows for every thread");
  const bool active = DIM || grp < groups;
  auto rows = [&](auto body) {
    if constexpr (ROWS > 0) {
#pragma unroll
      for (int k = 0; k < ROWS; k++) body(grp + k * groups, k);
    } else {
      int k = 0;
#pragma unroll 4
      for (int d = grp; d < dim; d += groups) body(d, k++);
    }
  };
  // element i of a row as kept in shared memory: its column in the projections (< 0: zero)
  const int row_n = rka + 2 * W + a.rank8;
  auto column = [&](int i) {
    if (i < 3 * dim) {
      const int which = (i >= dim) + (i >= 2 * dim);
      return (which == 0 ? a.r_off : which == 1 ? a.k_off : a.a_off) + h * dim + i - which * dim;
    }
    i -= rka;
    if (i < 0) return -1;
    if (i < 2 * W) {
      const int e = i < W ? i : i - W;
      return e0 + e < a.vdim ? (i < W ? a.v_off : a.g_off) + h * a.vdim + e0 + e : -1;
    }
    return i - 2 * W < a.rank ? a.x_off + i - 2 * W : -1;
  };
  const uint32_t with = __ballot_sync(0xffffffffu, ch < dim);      // whole groups of TPC threads
  int piece[kRowPieces];
#pragma unroll
  for (int k = 0; k < kRowPieces; k++) piece[k] = tid + NT * k < row_n ? column(tid + NT * k) : -1;
  for (int i = tid; i < 3 * l.row_n / 4; i += NT) ((float4*)(sm + l.row))[i] = make_float4(0.f, 0.f, 0.f, 0.f);      // what no copy writes stays zero
  __syncthreads();
  pdl_wait();
  // a token: row t0 + i of entry b, whose n tokens start at row t0 (n = 0: nothing to do)
  struct Item { int b, i, n, t0, slot; bool fresh; };
  auto first = [&](int b) {
    Item q = {b, 0, 0, 0, -1, true};
    if (b < n_seqs) {
      q.n = a.q_len[b];
      q.t0 = a.q_start[b];
      q.slot = a.slot[b];
      q.fresh = a.ctx_len[b] - q.n == 0 || q.slot < 0;
    }
    return q;
  };
  auto next = [&](const Item& q) {
    if (q.i + 1 >= q.n) return first(q.b + gridDim.y);
    Item r = q;
    r.i++;
    return r;
  };
  auto state_of = [&](int slot) { return (float4*)(a.state + ((size_t)max(slot, 0) * a.H + h) * dim * a.VP) + part * nv + (size_t)grp * nv_all + col; };
  const int ds = groups * nv;              // from one of a thread's state rows to the next, in shared memory
  const size_t dg = (size_t)groups * nv_all;
  auto fetch_row = [&](const Item& q, int buf) {
    if (q.n < 1) return;
    const float* src = a.in + (size_t)(q.t0 + q.i) * a.ld;
    float* dst = sm + l.row + buf * l.row_n;
#pragma unroll
    for (int k = 0; k < kRowPieces; k++)
      if (piece[k] >= 0) cp_async4(dst + tid + NT * k, src + piece[k]);
    for (int i = tid + NT * kRowPieces; i < row_n; i += NT) {
      const int c = column(i);
      if (c >= 0) cp_async4(dst + i, src + c);
    }
  };
  auto fetch_state = [&](const Item& q, int buf) {
    if (!active || q.n < 1) return;
    float4* dst = (float4*)(sm + l.state + buf * l.state_n) + grp * nv + col;
    const float4* src = state_of(q.slot);
    const uint32_t to = s32(dst);
    if (!q.fresh) rows([&](int, int k) { cp_async16(to + k * ds * 16, src + k * dg); });
    else rows([&](int, int k) { dst[k * ds] = make_float4(0.f, 0.f, 0.f, 0.f); });
  };
  // what a token does to the state, in three steps with a barrier between them
  auto low_rank = [&](const float* row) {
    for (int r = tid; r < a.rank8; r += NT) s_x[r] = tanhf(row[rka + 2 * W + r]);
  };
  auto decay_logits = [&]() {
    if (ch >= dim) return;
    float z = 0.f;
    auto dot = [&](uint4 q, int at) {
      const __nv_bfloat162* p = (const __nv_bfloat162*)&q;
      const float4 x0 = *(const float4*)(s_x + at), x1 = *(const float4*)(s_x + at + 4);
      float2 f;
      f = __bfloat1622float2(p[0]); z = fmaf(f.x, x0.x, z); z = fmaf(f.y, x0.y, z);
      f = __bfloat1622float2(p[1]); z = fmaf(f.x, x0.z, z); z = fmaf(f.y, x0.w, z);
      f = __bfloat1622float2(p[2]); z = fmaf(f.x, x1.x, z); z = fmaf(f.y, x1.y, z);
      f = __bfloat1622float2(p[3]); z = fmaf(f.x, x1.z, z); z = fmaf(f.y, x1.w, z);
    };
#pragma unroll
    for (int j = 0; j < HELD; j++)
      if ((sub + j * TPC) * 8 < a.rank8) dot(held[j], (sub + j * TPC) * 8);
    for (int j = sub + HELD * TPC; j * 8 < a.rank8; j += TPC) dot(((const uint4*)wrow)[j], j * 8);
    for (int o = 1; o < TPC; o <<= 1) z += __shfl_xor_sync(with, z, o);
    if (sub == 0) s_z[ch] = z;
  };
  auto channels = [&](const float* row, int buf) {
    if (NT - 1 - (warp * 32 + 31) >= dim) return;                  // no channel in this warp
    float q0 = 0.f, q1 = 0.f, q2 = 0.f;
    if (cc < dim) {
      const float rr = row[cc], kk = row[dim + cc], rate = sigmoid_f(row[2 * dim + cc] + ab), w = expf(-a.decay * sigmoid_f(s_z[cc] + w0));
      s_ch[buf * dim + cc] = make_float4(w, rate * kk, kk, 0.f);
      s_kr[buf * dim + cc] = make_float2(kk, rr * w);
      q0 = kk * kk;
      q1 = rr * rate * kk;
      q2 = rr * kk;
    }
    q0 = warp_sum(q0);
    q1 = warp_sum(q1);
    q2 = warp_sum(q2);
    if (lane == 0) { red[buf][0][NT / 32 - 1 - warp] = q0; red[buf][1][NT / 32 - 1 - warp] = q1; red[buf][2][NT / 32 - 1 - warp] = q2; }
  };
  Item cur = first(blockIdx.y), nxt = next(cur), aft = next(nxt);
  fetch_state(cur, 0);
  fetch_row(cur, 0);
  fetch_row(nxt, 1);
  cp_async_commit();
  cp_async_wait_all();
  __syncthreads();
  low_rank(sm + l.row);
  __syncthreads();
  decay_logits();
  __syncthreads();
  channels(sm + l.row, 0);
  int sbuf = 0, rbuf = 0, step = 0;
  while (cur.b < n_seqs) {
    cp_async_wait_all();
    __syncthreads();                       // the state and the next token's projections have landed; this token's channels are ready
    const int r1 = rbuf == 2 ? 0 : rbuf + 1, r2 = r1 == 2 ? 0 : r1 + 1, kb = step & 1;
    if (nxt.i == 0) fetch_state(nxt, sbuf ^ 1);
    fetch_row(aft, r2);
    cp_async_commit();
    const Item later = next(aft);          // looked up ahead of its use
    const float* row = sm + l.row + rbuf * l.row_n;
    const float* row1 = sm + l.row + r1 * l.row_n;
    const float *s_v = row + rka, *s_g = s_v + W;
    float4* S = (float4*)(sm + l.state + sbuf * l.state_n) + grp * nv + col;
    const bool live = cur.n > 0, last = cur.i + 1 >= cur.n;
    low_rank(row1);
    if (active) {
      float4 rd = make_float4(0.f, 0.f, 0.f, 0.f), p = rd;
      const float2* kr_at = s_kr + kb * dim;
      rows([&](int d, int k) {
        const float2 kr = kr_at[d];
        const float4 x = S[k * ds];
        rd.x = fmaf(kr.x, x.x, rd.x); rd.y = fmaf(kr.x, x.y, rd.y); rd.z = fmaf(kr.x, x.z, rd.z); rd.w = fmaf(kr.x, x.w, rd.w);
        p.x = fmaf(kr.y, x.x, p.x); p.y = fmaf(kr.y, x.y, p.y); p.z = fmaf(kr.y, x.z, p.z); p.w = fmaf(kr.y, x.w, p.w);
      });
      *(float4*)(s_red + (size_t)(grp * 2) * W + 4 * col) = rd;
      *(float4*)(s_red + (size_t)(grp * 2 + 1) * W + 4 * col) = p;
    }
    __syncthreads();
    decay_logits();
    float o = 0.f;
    if (warp * 32 < W) {                   // one column per lane; W <= 256
      float q0 = 0.f, q1 = 0.f, q2 = 0.f;
      for (int j = 0; j * 32 < dim; j++) { q0 += red[kb][0][j]; q1 += red[kb][1][j]; q2 += red[kb][2][j]; }
      const float inv = 1.f / (q0 + kUnitEps);
      if (tid < W) {
        float rd = 0.f, p = 0.f;
#pragma unroll 8
        for (int g = 0; g < groups; g++) {
          rd += s_red[(size_t)(g * 2) * W + tid];
          p += s_red[(size_t)(g * 2 + 1) * W + tid];
        }
        rd *= inv;
        s_read[tid] = rd;
        o = p - q1 * rd + q2 * s_v[tid];   // padding columns are zero
      }
      const float ss = warp_sum(o * o);
      if (lane == 0) red1[warp] = ss;
    }
    __syncthreads();
    channels(row1, kb ^ 1);
    if (active) {
      const float4 v = *(const float4*)(s_v + 4 * col), rd = *(const float4*)(s_read + 4 * col);
      const float4* c_at = s_ch + kb * dim;
      auto updated = [&](int d, int k) {
        const float4 c = c_at[d], x = S[k * ds];
        return make_float4(fmaf(c.x, x.x, fmaf(c.z, v.x, -c.y * rd.x)), fmaf(c.x, x.y, fmaf(c.z, v.y, -c.y * rd.y)), fmaf(c.x, x.z, fmaf(c.z, v.z, -c.y * rd.z)),
                           fmaf(c.x, x.w, fmaf(c.z, v.w, -c.y * rd.w)));
      };
      float4* dst = state_of(cur.slot);
      if (!last) rows([&](int d, int k) { S[k * ds] = updated(d, k); });
      else if (live && cur.slot >= 0) rows([&](int d, int k) { dst[k * dg] = updated(d, k); });
    }
    float ss = 0.f;
    if (CL > 1 || warp * 32 < W)
      for (int j = 0; j * 32 < W; j++) ss += red1[j];
    if (CL > 1) {
      if (tid == 0) s_part[step & 1] = ss;
      cluster.sync();
      ss = 0.f;
      for (int p = 0; p < CL; p++) ss += *cluster.map_shared_rank(&s_part[step & 1], p);
    }
    if (tid < W && live) {
      if (e0 + tid < a.vdim) o *= wo * sigmoid_f(s_g[tid]) / sqrtf(ss / (float)a.vdim + a.eps);
      else o = 0.f;
      const size_t at = (size_t)(cur.t0 + cur.i) * a.ldo + (size_t)h * a.VP + e0 + tid;
      if (a.out_f32) a.out_f32[at] = o;
      if (a.out_bf16) a.out_bf16[at] = __float2bfloat16(o);
    }
    step++;
    rbuf = r1;
    if (nxt.i == 0) sbuf ^= 1;
    cur = nxt;
    nxt = aft;
    aft = later;
  }
  if (CL > 1) cluster.sync();              // peers may still be reading this CTA's sum
}

static int delta_fill(DeltaArgs& a, const float* in, int ld, const int* offs, int rank, const void* w2, int rank8, const float* w0, const float* ab,
                      const float* norm, float* state, const int* q_start, const int* q_len, const int* ctx_len, const int* slot, int n_seqs, int H, int dim,
                      int vdim, int VP, float decay, float eps, float* out_f32, void* out_bf16, int ldo) {
  if (n_seqs < 1 || H < 1 || dim < 1 || vdim < 1 || VP < vdim || VP % 8 || dim > kDeltaDim || VP > kDeltaDim || rank < 1 || rank8 < rank || rank8 % 8 ||
      rank8 > kDeltaRank || decay < 0.f || ldo < H * VP || ((uintptr_t)state % 16) || ((uintptr_t)w2 % 16) || !slot || (!out_f32 && !out_bf16))
    return B200_ERR_BAD_ARG;
  a.in = in; a.ld = ld; a.r_off = offs[0]; a.k_off = offs[1]; a.v_off = offs[2]; a.g_off = offs[3]; a.a_off = offs[4]; a.x_off = offs[5]; a.rank = rank;
  a.w2 = (const __nv_bfloat16*)w2; a.rank8 = rank8; a.w0 = w0; a.ab = ab; a.norm = norm; a.state = state; a.q_start = q_start; a.q_len = q_len;
  a.ctx_len = ctx_len; a.slot = slot; a.H = H; a.dim = dim; a.vdim = vdim; a.VP = VP; a.decay = decay; a.eps = eps; a.out_f32 = out_f32;
  a.out_bf16 = (__nv_bfloat16*)out_bf16; a.ldo = ldo;
  return 0;
}

// offs: columns of r, k, v, the output gate, the removal rate and the low-rank decay input in a row of `in`.
B200_API int b200_delta_recurrent(const float* in, int ld, const int* offs, int rank, const void* w2, int rank8, const float* w0, const float* ab,
                                  const float* norm, float* state, const int* q_start, const int* q_len, const int* ctx_len, const int* slot, int n_seqs,
                                  int H, int dim, int vdim, int VP, float decay, float eps, float* out_f32, void* out_bf16, int ldo, cudaStream_t st) {
  DeltaArgs a;
  int rc = delta_fill(a, in, ld, offs, rank, w2, rank8, w0, ab, norm, state, q_start, q_len, ctx_len, slot, n_seqs, H, dim, vdim, VP, decay, eps, out_f32,
                      out_bf16, ldo);
  if (rc) return rc;
  // CTAs per head: until a state share is 32 KB at most and the SMs are covered, eight (for the SMs' sake: sixteen) float4 columns each at least
  int CL = 1;
  while (CL < 8 && (VP / 4) % (2 * CL) == 0 && VP / 4 / (2 * CL) >= 8 && (dim * VP / CL > 8192 || (VP / CL > 64 && (long)H * n_seqs * CL < 148))) CL *= 2;
  const bool w64 = VP / CL == 64 && (dim == 64 || dim == 128);
  const int threads = w64 ? 128 : 256;
  const DeltaLayout l = delta_layout(dim, VP / CL, rank8, threads);
  const size_t smem = 4 * (size_t)l.total;
  if (smem > 200 * 1024) return B200_ERR_BAD_ARG;
  auto kern = !w64 ? delta_recurrent_kernel<0, 0, 256> : dim == 64 ? delta_recurrent_kernel<64, 16, 128> : delta_recurrent_kernel<128, 16, 128>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
  if (e != cudaSuccess) return (int)e;
  // shares of the sequences: no more CTAs than run at a time, all with about the same number of sequences
  const int fit = (int)(227 * 1024 / (smem + 1024)), most_fit = threads == 128 ? 3 : 2, resident = 148 * (fit < 1 ? 1 : fit > most_fit ? most_fit : fit);
  const int most = resident / (H * CL) > 1 ? resident / (H * CL) : 1, rounds = (n_seqs + most - 1) / most, shares = (n_seqs + rounds - 1) / rounds;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(H * CL, shares);
  cfg.blockDim = dim3(threads);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = CL;
  attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = b200_pdl_enabled() ? 2 : 1;
  return (int)cudaLaunchKernelEx(&cfg, kern, a, n_seqs, l);
}

// ------------------------------------------------------------------ prompts: 64-token chunks on the tensor cores
//
// With b_t the running sum of log w from the chunk's start, C its last token and y_t = u_t^T S_(t-1) what the removal of token t reads:
//   y_t = (u_t e^{b_(t-1)}) S + sum_{s<t} N[t][s] v_s - M[t][s] y_s      N[t][s] = sum_d u_td k_sd e^{b_(t-1)d - b_sd},  M with c for k
//   o_t = (r_t e^{b_t}) S + sum_{s<=t} A[t][s] v_s - B[t][s] y_s         A, B likewise with r e^{b_t}
//   S'  = diag(e^{b_C}) S + sum_s (k_s e^{b_C - b_s}) v_s^T - (c_s e^{b_C - b_s}) y_s^T
// y is linear in S: y = X S + P with (I + M) X = u e^{b_(t-1)} and (I + M) P = N V, so that
//   o = R S + Q      R = r e^b - B X,   Q = A V - B P
//   S' = G S + F     G = diag(e^{b_C}) - (c e^{b_C - b})^T X,   F = (k e^{b_C - b})^T V - (c e^{b_C - b})^T P
// delta_prepare_kernel solves for R, Q, G and F, all chunks and heads in parallel; delta_state_kernel walks a sequence's chunks with S in registers (one
// product each) and leaves every chunk's starting state behind; delta_output_kernel forms the outputs, norms and gates them, again in parallel.
//
// M is strictly lower triangular.  Its 16 x 16 diagonal blocks are inverted in fp32; the rest of the solve is products of blocks.  A warp of
// delta_prepare_kernel owns 16 columns of X or P (as rows of the MMA, so that its accumulators are operands of the next product as they lie) and needs no other.
//
// Operands enter the tensor cores as two bf16 numbers (value and remainder), products accumulate in fp32; only v, a plain projection, is rounded to bf16
// once.  The factors e^b and e^-b stay within e^(64 decay).

constexpr float kDeltaSpan = 60.f;       // most of GC * decay
constexpr int kBlk = 16 * 16;            // a 16 x 16 block of bf16; the halves of rows 4-7 and 12-15 change places (conflict-free for ldmatrix)
__device__ __forceinline__ int in_block(int t, int s) { return t * 16 + ((((s >> 3) ^ (t >> 2)) & 1) << 3) + (s & 7); }
constexpr int kRankSlice = 64;

struct DeltaWs {                         // per (chunk slot, head); fragments of 32 lanes
  uint4* r;                              // [DP / 16][4 token tiles of 16][2][lane]: R as the B operand of R S, values and remainders
  uint4* g;                              // [DP / 16][DP / 16][2][lane]: G likewise
  float4* q;                             // [value tiles][8 token tiles of 8][lane]: Q as accumulators
  float4* f;                             // [value tiles][DP / 8][lane]: F as accumulators
  uint4* s;                              // [value tiles][DP / 16][2][lane]: the state at the chunk's start as the A operand
  int nvt;                               // value tiles of 16
};

// Shared memory: scratch | k, c, r | u, whose place the matrices take once it is in registers | v.  Each operand in two parts (values, remainders).
template <int DP>
struct DeltaSmem {
  static constexpr int LQ = DP + 8, ROWS = GC * LQ, OP = 2 * ROWS * 2;      // OP: bytes of an operand
  static constexpr int LW = kRankSlice + 8, THREADS = DP >= 128 ? 512 : 256;
  static constexpr int kScratch = (4 * 16 * 17 + 2 * THREADS + GC + DP) * 4;         // fp32 diagonal blocks of M; column sums; unit-key factors; e^{b_C}
  static constexpr int kBlocks = 8 * 10 * kBlk * 2;                          // -M (diagonal: its inverse), N, A, -B
  static constexpr int kTail = OP > kBlocks ? OP : kBlocks;
  // only until the decays are known: tanh(x) in two parts and a slice of w2 over k, c, r; their product behind u
  static constexpr int kProduct = GC * (DP + 1) * 4;
  static_assert(2 * GC * LW * 2 + DP * LW * 2 <= 3 * OP, "the decay's operands fit the space of k, c and r");
  static int bytes(int nvt) {
    const int with_v = kTail + GC * (nvt * 16 + 8) * 2, with_product = OP + kProduct;
    return kScratch + 3 * OP + (with_v > with_product ? with_v : with_product);
  }
};

// Block (i, j <= i) of a lower triangular 64 x 64 matrix.
__device__ __forceinline__ int tri(int i, int j) { return i * (i + 1) / 2 + j; }

template <int DP>
__global__ void __launch_bounds__(DeltaSmem<DP>::THREADS, DP <= 64 ? 2 : 1) delta_prepare_kernel(const DeltaArgs a, const DeltaWs ws) {
  using L = DeltaSmem<DP>;
  constexpr int LQ = L::LQ, LW = L::LW, THREADS = L::THREADS, NW = THREADS / 32, NG = THREADS / (DP / 2), TPT = GC / NG, KD = DP / 16;
  extern __shared__ __align__(16) uint8_t smem[];
  float* sd = (float*)smem;                                      // [4][16][17]
  float* stot = sd + 4 * 16 * 17;                                // [NG][DP]
  float* sinv = stot + 2 * THREADS;                              // [GC]
  float* sdec = sinv + GC;                                       // [DP]
  __nv_bfloat16* sk = (__nv_bfloat16*)(smem + L::kScratch);      // values, then remainders, of each
  __nv_bfloat16 *sc = sk + 2 * L::ROWS, *sr = sc + 2 * L::ROWS, *su = sr + 2 * L::ROWS;
  __nv_bfloat16* sb = su;                                        // blocks: [4 matrices][value, remainder][10][kBlk]
  __nv_bfloat16* sv = su + L::kTail / 2;                         // [GC][LV]
  __nv_bfloat16* sx = sk;                                        // [2][GC][LW]   } only until the decays are known
  __nv_bfloat16* sw = sx + 2 * GC * LW;                          // [DP][LW]      }
  float* sz = (float*)(su + 2 * L::ROWS);                        // [GC][DP + 1]  }
  const int LV = ws.nvt * 16 + 8;
  const int c = blockIdx.x, h = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g4 = lane >> 2, t4 = lane & 3;
  pdl_wait();
  const int len = a.q_len[seq], qs = a.q_start[seq];
  if (c * GC >= len) {
    pdl_trigger();
    return;
  }
  const int n = min(GC, len - c * GC), t0 = qs + c * GC;
  const float* in = a.in + (size_t)t0 * a.ld;
  if (((a.vdim | a.dim | a.v_off | a.r_off | a.k_off | a.a_off | a.ld) & 3) == 0 && tid < 4 * GC && tid % GC < n) {      // rows read later, into L2 now
    const int what = tid / GC;
    const float* p = in + (size_t)(tid % GC) * a.ld + (what == 0 ? a.k_off + h * a.dim : what == 1 ? a.r_off + h * a.dim : what == 2 ? a.a_off + h * a.dim : a.v_off + h * a.vdim);
    prefetch_l2(p, (what == 3 ? a.vdim : a.dim) * 4);
  }
  // ---- z = W2 tanh(x): 64 tokens x DP channels, 64 ranks at a time; warp = 16 tokens x a share of the channels
  {
    constexpr int NT = DP / 2 / NW;                              // n8 tiles per warp
    float acc[NT][4] = {};
    const int m0 = (warp & 3) * 16, n0 = (warp >> 2) * NT * 8;
    for (int r0 = 0; r0 < a.rank; r0 += kRankSlice) {
      if (r0) __syncthreads();
      {
        constexpr int TS = THREADS / kRankSlice;                 // a thread: one rank of every TS-th token
        const int r = tid % kRankSlice, q = tid / kRankSlice;
        float x[GC / TS];
#pragma unroll
        for (int i = 0; i < GC / TS; i++) x[i] = q + TS * i < n && r0 + r < a.rank ? in[(size_t)(q + TS * i) * a.ld + a.x_off + r0 + r] : 0.f;
#pragma unroll
        for (int i = 0; i < GC / TS; i++) {
          const float e = __expf(-2.f * fabsf(x[i])), y = copysignf(__fdividef(1.f - e, 1.f + e), x[i]);      // tanh
          split_bf16(y, sx[(q + TS * i) * LW + r], sx[GC * LW + (q + TS * i) * LW + r]);
        }
      }
      for (int i = tid; i < DP * (kRankSlice / 8); i += THREADS) {
        const int d = i / (kRankSlice / 8), r = i % (kRankSlice / 8) * 8;
        *(uint4*)(sw + d * LW + r) = d < a.dim && r0 + r < a.rank8 ? *(const uint4*)(a.w2 + (size_t)(h * a.dim + d) * a.rank8 + r0 + r) : make_uint4(0u, 0u, 0u, 0u);
      }
      __syncthreads();
      const int ks = min(kRankSlice, a.rank - r0);
      for (int k0 = 0; k0 < ks; k0 += 16) {
        uint32_t ah[4], al[4];
        const int ra = (m0 + (lane & 15)) * LW + k0 + (lane >> 4) * 8;
        ldsm4(s32(sx + ra), ah);
        ldsm4(s32(sx + GC * LW + ra), al);
#pragma unroll
        for (int j = 0; j < NT; j += 2) {
          uint32_t w[4];
          ldsm4(s32(sw + (n0 + (j + (lane >> 4)) * 8 + (lane & 7)) * LW + k0 + ((lane >> 3) & 1) * 8), w);
          mma_bf16(acc[j], ah, w[0], w[1]);
          mma_bf16(acc[j + 1], ah, w[2], w[3]);
          mma_bf16(acc[j], al, w[0], w[1]);
          mma_bf16(acc[j + 1], al, w[2], w[3]);
        }
      }
    }
#pragma unroll
    for (int j = 0; j < NT; j++)
#pragma unroll
      for (int e = 0; e < 4; e++) sz[(m0 + g4 + 8 * (e >> 1)) * (DP + 1) + n0 + 8 * j + 2 * t4 + (e & 1)] = acc[j][e];
  }
  {                                                              // unit keys: a warp takes KT tokens
    constexpr int KT = GC / NW;
    float ss[KT] = {};
    for (int d = lane; d < a.dim; d += 32) {
      float x[KT];
#pragma unroll
      for (int i = 0; i < KT; i++) x[i] = warp * KT + i < n ? in[(size_t)(warp * KT + i) * a.ld + a.k_off + h * a.dim + d] : 0.f;
#pragma unroll
      for (int i = 0; i < KT; i++) ss[i] = fmaf(x[i], x[i], ss[i]);
    }
#pragma unroll
    for (int i = 0; i < KT; i++) {
      ss[i] = warp_sum(ss[i]);
      if (lane == i) sinv[warp * KT + i] = 1.f / sqrtf(ss[i] + kUnitEps);
    }
  }
  __syncthreads();
  // ---- running sums of the log decays, and the decayed operands: a thread owns two channels of TPT consecutive tokens
  {
    const int d = tid % (DP / 2) * 2, grp = tid / (DP / 2), c0 = h * a.dim + d;
    const bool l0 = d < a.dim, l1 = d + 1 < a.dim, even = ((a.dim | a.r_off | a.k_off | a.a_off | a.ld) & 1) == 0;
    const float2 w0 = make_float2(l0 ? a.w0[c0] : 0.f, l1 ? a.w0[c0 + 1] : 0.f), ab = make_float2(l0 ? a.ab[c0] : 0.f, l1 ? a.ab[c0 + 1] : 0.f);
    float2 b[TPT], sum = make_float2(0.f, 0.f);
#pragma unroll
    for (int i = 0; i < TPT; i++) {
      const int t = grp * TPT + i;
      if (t < n) {
        if (l0) sum.x -= a.decay * sigmoid_fast(sz[t * (DP + 1) + d] + w0.x);
        if (l1) sum.y -= a.decay * sigmoid_fast(sz[t * (DP + 1) + d + 1] + w0.y);
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
    if (grp == 0) *(float2*)(sdec + d) = make_float2(expf(total.x), expf(total.y));
    float2 eb = make_float2(__expf(before.x), __expf(before.y));      // e^{b_(t-1)}
    auto pair = [&](const float* p, bool row) -> float2 {
      if (!row || !l0) return make_float2(0.f, 0.f);
      if (even) return __ldg((const float2*)p);                  // an even head size: both channels exist
      return make_float2(__ldg(p), l1 ? __ldg(p + 1) : 0.f);
    };
    constexpr int LB = TPT < 4 ? TPT : 4;
#pragma unroll
    for (int i0 = 0; i0 < TPT; i0 += LB) {
      float2 r[LB], k[LB], x[LB];
#pragma unroll
      for (int i = 0; i < LB; i++) {
        const int t = grp * TPT + i0 + i;
        const float* row = in + (size_t)t * a.ld + c0;
        r[i] = pair(row + a.r_off, t < n);
        k[i] = pair(row + a.k_off, t < n);
        x[i] = pair(row + a.a_off, t < n);
      }
#pragma unroll
      for (int i = 0; i < LB; i++) {
        const int t = grp * TPT + i0 + i, at = t * LQ + d;
        const float ex = __expf(before.x + b[i0 + i].x), ey = __expf(before.y + b[i0 + i].y), inv = sinv[t];
        const float ix = __fdividef(1.f, ex), iy = __fdividef(1.f, ey), ux = k[i].x * inv, uy = k[i].y * inv;
        auto put = [&](__nv_bfloat16* p, float vx, float vy) {
          uint32_t hi, lo;
          split2(vx, vy, hi, lo);
          *(uint32_t*)(p + at) = hi;
          *(uint32_t*)(p + L::ROWS + at) = lo;
        };
        put(sr, r[i].x * ex, r[i].y * ey);
        put(su, ux * eb.x, uy * eb.y);
        put(sk, k[i].x * ix, k[i].y * iy);
        put(sc, -sigmoid_fast(x[i].x + ab.x) * ux * ix, -sigmoid_fast(x[i].y + ab.y) * uy * iy);      // negated: every product with it is taken off
        eb = make_float2(ex, ey);
      }
    }
  }
  __syncthreads();                                               // sz is no longer needed: blocks and v take its place
  if (((a.vdim | a.v_off | a.ld) & 3) == 0) {
    for (int i = tid; i < GC * ws.nvt * 4; i += THREADS) {
      const int t = i / (ws.nvt * 4), e = i % (ws.nvt * 4) * 4;
      float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
      if (t < n && e < a.vdim) x = __ldg((const float4*)(in + (size_t)t * a.ld + a.v_off + h * a.vdim + e));
      *(uint2*)(sv + t * LV + e) = make_uint2(pack_bf2(__float2bfloat16(x.x), __float2bfloat16(x.y)), pack_bf2(__float2bfloat16(x.z), __float2bfloat16(x.w)));
    }
  } else {
    for (int i = tid; i < GC * ws.nvt * 16; i += THREADS) {
      const int t = i / (ws.nvt * 16), e = i % (ws.nvt * 16);
      sv[t * LV + e] = __float2bfloat16(t < n && e < a.vdim ? in[(size_t)t * a.ld + a.v_off + h * a.vdim + e] : 0.f);
    }
  }
  // ---- the four triangular matrices, 40 blocks of 16 x 16, BPW per warp: (u, r) x (c, k)
  constexpr int BPW = (40 + NW - 1) / NW;
  float blocks[BPW][2][4];
#pragma unroll
  for (int q = 0; q < BPW; q++) {
    const int unit = min(warp * BPW + q, 39), mat = unit / 10, blk = unit % 10;        // mat 0: u c (-M), 1: u k (N), 2: r k (A), 3: r c (-B)
    const int i = blk >= 6 ? 3 : blk >= 3 ? 2 : blk >= 1 ? 1 : 0, j = blk - i * (i + 1) / 2;
    const __nv_bfloat16 *X = mat < 2 ? su : sr, *Y = (mat == 0 || mat == 3) ? sc : sk;
    float (&acc)[2][4] = blocks[q];
#pragma unroll
    for (int m = 0; m < 2; m++) acc[m][0] = acc[m][1] = acc[m][2] = acc[m][3] = 0.f;
#pragma unroll
    for (int k0 = 0; k0 < DP; k0 += 16) {
      uint32_t xh[4], xl[4], yh[4], yl[4];
      const int ra = (i * 16 + (lane & 15)) * LQ + k0 + (lane >> 4) * 8;
      const int rb = (j * 16 + (lane >> 4) * 8 + (lane & 7)) * LQ + k0 + ((lane >> 3) & 1) * 8;
      ldsm4(s32(X + ra), xh);
      ldsm4(s32(X + L::ROWS + ra), xl);
      ldsm4(s32(Y + rb), yh);
      ldsm4(s32(Y + L::ROWS + rb), yl);
      mma_bf16(acc[0], xh, yh[0], yh[1]);
      mma_bf16(acc[1], xh, yh[2], yh[3]);
      mma_bf16(acc[0], xh, yl[0], yl[1]);
      mma_bf16(acc[1], xh, yl[2], yl[3]);
      mma_bf16(acc[0], xl, yh[0], yh[1]);
      mma_bf16(acc[1], xl, yh[2], yh[3]);
    }
  }
  // rows d0..d0 + 16 (as MMA rows) of the tokens of tile i, from a [token][channel] operand kept in two parts
  auto columns = [&](const __nv_bfloat16* p, int d0, int i, float (&z)[2][4]) {
    uint32_t hi[4], lo[4];
    const int at = (i * 16 + (lane >> 4) * 8 + (lane & 7)) * LQ + d0 + ((lane >> 3) & 1) * 8;
    ldsm4t(s32(p + at), hi);
    ldsm4t(s32(p + L::ROWS + at), lo);
#pragma unroll
    for (int m = 0; m < 4; m++) {
      const float2 x = __bfloat1622float2(*(const __nv_bfloat162*)&hi[m]), y = __bfloat1622float2(*(const __nv_bfloat162*)&lo[m]);
      z[m >> 1][(m & 1) * 2] = x.x + y.x;
      z[m >> 1][(m & 1) * 2 + 1] = x.y + y.y;
    }
  };
  float u[4][2][4];                                              // this warp's columns of u: the matrices take its place
  if (warp < KD) {
#pragma unroll
    for (int i = 0; i < 4; i++) columns(su, warp * 16, i, u[i]);
  }
  __syncthreads();
#pragma unroll
  for (int q = 0; q < BPW; q++) {
    if (warp * BPW + q >= 40) break;
    const int unit = warp * BPW + q, mat = unit / 10, blk = unit % 10;
    const int i = blk >= 6 ? 3 : blk >= 3 ? 2 : blk >= 1 ? 1 : 0, j = blk - i * (i + 1) / 2;
    float (&acc)[2][4] = blocks[q];
    __nv_bfloat16* hi = sb + (mat * 2) * 10 * kBlk + blk * kBlk;
    __nv_bfloat16* lo = hi + 10 * kBlk;
#pragma unroll
    for (int m = 0; m < 2; m++)
#pragma unroll
      for (int hf = 0; hf < 2; hf++) {
        const int t = g4 + 8 * hf, s = 8 * m + 2 * t4;
        float x = acc[m][2 * hf], y = acc[m][2 * hf + 1];
        if (i == j) {
          const int last = mat < 2 ? t - 1 : t;                  // u meets earlier tokens only
          if (s > last) x = 0.f;
          if (s + 1 > last) y = 0.f;
        }
        if (mat == 0 && i == j) {
          sd[(i * 16 + t) * 17 + s] = x;
          sd[(i * 16 + t) * 17 + s + 1] = y;
        } else {
          uint32_t p, r;
          split2(x, y, p, r);
          *(uint32_t*)(hi + in_block(t, s)) = p;
          *(uint32_t*)(lo + in_block(t, s)) = r;
        }
      }
  }
  __syncthreads();
  if (warp < 2) {                                                // inverses of the diagonal blocks of I + M: a lane owns a column
    const int i = warp * 2 + (lane >> 4), s = lane & 15;
    const float* m = sd + i * 16 * 17;                           // -M
    float x[16];
#pragma unroll
    for (int t = 0; t < 16; t++) x[t] = t == s ? 1.f : 0.f;
#pragma unroll
    for (int k = 0; k < 16; k++)
#pragma unroll
      for (int t = k + 1; t < 16; t++) x[t] = fmaf(m[t * 17 + k], x[k], x[t]);
    __nv_bfloat16* hi = sb + tri(i, i) * kBlk;
#pragma unroll
    for (int t = 0; t < 16; t++) split_bf16(x[t], hi[in_block(t, s)], hi[10 * kBlk + in_block(t, s)]);
  }
  __syncthreads();

  // block (i, j) of matrix `mat` as the B operand (token columns, earlier tokens contracted)
  const int blk_at = in_block((lane >> 4) * 8 + (lane & 7), ((lane >> 3) & 1) * 8);
  auto block = [&](int mat, int i, int j, uint32_t (&hi)[4], uint32_t (&lo)[4]) {
    const __nv_bfloat16* p = sb + (mat * 2) * 10 * kBlk + tri(i, j) * kBlk + blk_at;
    ldsm4(s32(p), hi);
    ldsm4(s32(p + 10 * kBlk), lo);
  };
  auto mul = [&](float (&acc)[2][4], const uint32_t (&xh)[4], const uint32_t (&xl)[4], const uint32_t (&bh)[4], const uint32_t (&bl)[4]) {
    mma_bf16(acc[0], xh, bh[0], bh[1]);
    mma_bf16(acc[1], xh, bh[2], bh[3]);
    mma_bf16(acc[0], xh, bl[0], bl[1]);
    mma_bf16(acc[1], xh, bl[2], bl[3]);
    mma_bf16(acc[0], xl, bh[0], bh[1]);
    mma_bf16(acc[1], xl, bh[2], bh[3]);
  };
  auto mul_v = [&](float (&acc)[2][4], const uint32_t (&v)[4], const uint32_t (&bh)[4], const uint32_t (&bl)[4]) {
    mma_bf16(acc[0], v, bh[0], bh[1]);
    mma_bf16(acc[1], v, bh[2], bh[3]);
    mma_bf16(acc[0], v, bl[0], bl[1]);
    mma_bf16(acc[1], v, bl[2], bl[3]);
  };
  auto as_operand = [&](const float (&z)[2][4], uint32_t (&hi)[4], uint32_t (&lo)[4]) {
    split2(z[0][0], z[0][1], hi[0], lo[0]);
    split2(z[0][2], z[0][3], hi[1], lo[1]);
    split2(z[1][0], z[1][1], hi[2], lo[2]);
    split2(z[1][2], z[1][3], hi[3], lo[3]);
  };
  // (I + M) X = Z, tile by tile: z holds tile i of Z and of what the earlier tiles of X (xh, xl) take off it
  auto solve = [&](int i, float (&z)[2][4], uint32_t (&xh)[4][4], uint32_t (&xl)[4][4]) {
    uint32_t bh[4], bl[4], zh[4], zl[4];
#pragma unroll
    for (int j = 0; j < 3; j++) {
      if (j >= i) break;
      block(0, i, j, bh, bl);
      mul(z, xh[j], xl[j], bh, bl);
    }
    as_operand(z, zh, zl);
    float x[2][4] = {};
    block(0, i, i, bh, bl);
    mul(x, zh, zl, bh, bl);
    as_operand(x, xh[i], xl[i]);
  };
  const size_t slot = chunk_slot(qs, seq, c) * a.H + h;
  for (int cb = warp; cb < KD + ws.nvt; cb += NW) {
    uint32_t xh[4][4], xl[4][4], bh[4], bl[4];
    if (cb < KD) {                                               // 16 key channels: R and G
      const int d0 = cb * 16;
#pragma unroll
      for (int i = 0; i < 4; i++) {
        solve(i, u[i], xh, xl);
      }
      uint4* dst = ws.r + (slot * KD + cb) * 4 * 64 + lane;
#pragma unroll
      for (int i = 0; i < 4; i++) {
        float z[2][4];
        columns(sr, d0, i, z);
#pragma unroll
        for (int j = 0; j <= i; j++) {
          block(3, i, j, bh, bl);
          mul(z, xh[j], xl[j], bh, bl);
        }
        uint32_t hi[4], lo[4];
        as_operand(z, hi, lo);                                   // tiles (d 0-7, t 0-7), (d 8-15, t 0-7), (d 0-7, t 8-15), (d 8-15, t 8-15)
        dst[i * 64] = make_uint4(transpose_8x8(hi[0]), transpose_8x8(hi[1]), transpose_8x8(hi[2]), transpose_8x8(hi[3]));
        dst[i * 64 + 32] = make_uint4(transpose_8x8(lo[0]), transpose_8x8(lo[1]), transpose_8x8(lo[2]), transpose_8x8(lo[3]));
      }
      uint4* gd = ws.g + (slot * KD + cb) * KD * 64 + lane;
#pragma unroll
      for (int jn = 0; jn < KD; jn++) {
        float z[2][4] = {};
#pragma unroll
        for (int kt = 0; kt < 4; kt++) {
          const int at = (kt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LQ + jn * 16 + (lane >> 4) * 8;
          ldsm4t(s32(sc + at), bh);
          ldsm4t(s32(sc + L::ROWS + at), bl);
          mul(z, xh[kt], xl[kt], bh, bl);
        }
#pragma unroll
        for (int m = 0; m < 2; m++)
#pragma unroll
          for (int e = 0; e < 4; e++) {
            const int di = d0 + g4 + 8 * (e >> 1), dn = jn * 16 + 8 * m + 2 * t4 + (e & 1);
            z[m][e] = sdec[dn] * (z[m][e] + (di == dn ? 1.f : 0.f));
          }
        uint32_t hi[4], lo[4];
        as_operand(z, hi, lo);
        gd[jn * 64] = make_uint4(transpose_8x8(hi[0]), transpose_8x8(hi[1]), transpose_8x8(hi[2]), transpose_8x8(hi[3]));
        gd[jn * 64 + 32] = make_uint4(transpose_8x8(lo[0]), transpose_8x8(lo[1]), transpose_8x8(lo[2]), transpose_8x8(lo[3]));
      }
    } else {                                                     // 16 value columns: Q and F
      const int vb = cb - KD;
      uint32_t va[4][4];                                         // V^T: 16 value columns x 16 tokens each
#pragma unroll
      for (int j = 0; j < 4; j++) ldsm4t(s32(sv + (j * 16 + (lane >> 4) * 8 + (lane & 7)) * LV + vb * 16 + ((lane >> 3) & 1) * 8), va[j]);
#pragma unroll
      for (int i = 0; i < 4; i++) {
        float z[2][4] = {};
#pragma unroll
        for (int j = 0; j <= i; j++) {
          block(1, i, j, bh, bl);
          mul_v(z, va[j], bh, bl);
        }
        solve(i, z, xh, xl);
      }
      float4* q = ws.q + (slot * ws.nvt + vb) * 8 * 32 + lane;
#pragma unroll
      for (int i = 0; i < 4; i++) {
        float z[2][4] = {};
#pragma unroll
        for (int j = 0; j <= i; j++) {
          block(2, i, j, bh, bl);
          mul_v(z, va[j], bh, bl);
          block(3, i, j, bh, bl);
          mul(z, xh[j], xl[j], bh, bl);
        }
#pragma unroll
        for (int m = 0; m < 2; m++) q[(2 * i + m) * 32] = make_float4(z[m][0], z[m][1], z[m][2], z[m][3]);
      }
      float4* f = ws.f + (slot * ws.nvt + vb) * (DP / 8) * 32 + lane;
#pragma unroll
      for (int jn = 0; jn < KD; jn++) {
        float z[2][4] = {};
#pragma unroll
        for (int kt = 0; kt < 4; kt++) {
          const int at = (kt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LQ + jn * 16 + (lane >> 4) * 8;
          ldsm4t(s32(sk + at), bh);
          ldsm4t(s32(sk + L::ROWS + at), bl);
          mul_v(z, va[kt], bh, bl);
          ldsm4t(s32(sc + at), bh);
          ldsm4t(s32(sc + L::ROWS + at), bl);
          mul(z, xh[kt], xl[kt], bh, bl);
        }
#pragma unroll
        for (int m = 0; m < 2; m++) {
          const float2 e = *(const float2*)(sdec + jn * 16 + 8 * m + 2 * t4);
          f[(2 * jn + m) * 32] = make_float4(z[m][0] * e.x, z[m][1] * e.y, z[m][2] * e.x, z[m][3] * e.y);
        }
      }
    }
  }
  pdl_trigger();                                                 // late: the sequential kernel behind this one wants its CTAs spread over idle SMs
}

constexpr int state_stages(int dp) { return dp >= 128 ? 2 : 4; }
constexpr int state_bytes(int dp, int warps) { return state_stages(dp) * (dp * dp + warps * 16 * dp) * 4; }

// One CTA = some value tiles of one head of one sequence, a warp 16 value columns (as MMA rows) x all key channels: S'^T = S^T G^T + F^T.  The accumulators,
// split into values and remainders, are the A operand of the next chunk's product as they lie, and that is the form a chunk's starting state is stored in.
template <int DP>
__global__ void __launch_bounds__(128) delta_state_kernel(const DeltaArgs a, const DeltaWs ws) {
  constexpr int KD = DP / 16, GN = KD * KD * 64, ST = state_stages(DP);      // uint4 of G per chunk; stages of the ring
  extern __shared__ __align__(16) uint4 sg[];
  pdl_trigger();
  pdl_wait();
  const int h = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g4 = lane >> 2, t4 = lane & 3, NT = blockDim.x;
  const int vb0 = blockIdx.x * (NT >> 5), vb = vb0 + warp, vt = min(vb, ws.nvt - 1);
  const int FN = min(NT >> 5, ws.nvt - vb0) * (DP / 8) * 32, SN = GN + (NT >> 5) * (DP / 8) * 32;      // float4 of F; of a stage
  const bool mine = vb < ws.nvt;
  const int len = a.q_len[seq], qs = a.q_start[seq], slot = a.slot[seq];
  const bool fresh = a.ctx_len[seq] - len == 0 || slot < 0;
  const int nc = (len + GC - 1) / GC;
  float* S = a.state + ((size_t)max(slot, 0) * a.H + h) * a.dim * a.VP;
  const size_t base = chunk_slot(qs, seq, 0) * a.H + h;
  const uint4* gsrc = ws.g + base * GN;
  const size_t gstep = (size_t)a.H * GN;
  const float4* fsrc = ws.f + (base * ws.nvt + vb0) * (DP / 8) * 32;
  const size_t fstep = (size_t)a.H * ws.nvt * (DP / 8) * 32;
  auto load = [&](int c) {
    if (c < nc) {
      uint4* dst = sg + (c % ST) * SN;
#pragma unroll 4
      for (int i = tid; i < GN; i += NT) cp_async16(s32(dst + i), gsrc + c * gstep + i);
#pragma unroll 4
      for (int i = tid; i < FN; i += NT) cp_async16(s32(dst + GN + i), fsrc + c * fstep + i);
    }
    cp_async_commit();                  // empty past the end: keeps the count of groups in flight
  };
#pragma unroll
  for (int c = 0; c < ST - 1; c++) load(c);
  float acc[DP / 8][4];
#pragma unroll
  for (int j = 0; j < DP / 8; j++)
#pragma unroll
    for (int e = 0; e < 4; e++) {
      const int v = vt * 16 + g4 + 8 * (e >> 1), d = 8 * j + 2 * t4 + (e & 1);
      acc[j][e] = (!fresh && v < a.VP && d < a.dim) ? S[(size_t)d * a.VP + v] : 0.f;
    }
  for (int c = 0; c < nc; c++) {
    uint32_t sh[KD][4], sl[KD][4];
    uint4* frag = ws.s + ((base + (size_t)c * a.H) * ws.nvt + vt) * KD * 64 + lane;
#pragma unroll
    for (int kd = 0; kd < KD; kd++) {
      split2(acc[2 * kd][0], acc[2 * kd][1], sh[kd][0], sl[kd][0]);
      split2(acc[2 * kd][2], acc[2 * kd][3], sh[kd][1], sl[kd][1]);
      split2(acc[2 * kd + 1][0], acc[2 * kd + 1][1], sh[kd][2], sl[kd][2]);
      split2(acc[2 * kd + 1][2], acc[2 * kd + 1][3], sh[kd][3], sl[kd][3]);
      if (mine) {
        frag[kd * 64] = make_uint4(sh[kd][0], sh[kd][1], sh[kd][2], sh[kd][3]);
        frag[kd * 64 + 32] = make_uint4(sl[kd][0], sl[kd][1], sl[kd][2], sl[kd][3]);
      }
    }
    cp_async_wait<ST - 2>();
    __syncthreads();                    // chunk c has landed, and everyone is done with the stage that is refilled now
    load(c + ST - 1);
    const uint4* g = sg + (c % ST) * SN + lane;
    const float4* f = (const float4*)(sg + (c % ST) * SN + GN) + (vt - vb0) * (DP / 8) * 32 + lane;
#pragma unroll
    for (int j = 0; j < DP / 8; j++) {
      const float4 x = f[j * 32];
      acc[j][0] = x.x; acc[j][1] = x.y; acc[j][2] = x.z; acc[j][3] = x.w;
    }
#pragma unroll
    for (int kd = 0; kd < KD; kd++)
#pragma unroll
      for (int jn = 0; jn < KD; jn++) {
        const uint4 bh = g[(kd * KD + jn) * 64], bl = g[(kd * KD + jn) * 64 + 32];
        mma_bf16(acc[2 * jn], sh[kd], bh.x, bh.y);
        mma_bf16(acc[2 * jn + 1], sh[kd], bh.z, bh.w);
        mma_bf16(acc[2 * jn], sh[kd], bl.x, bl.y);
        mma_bf16(acc[2 * jn + 1], sh[kd], bl.z, bl.w);
        mma_bf16(acc[2 * jn], sl[kd], bh.x, bh.y);
        mma_bf16(acc[2 * jn + 1], sl[kd], bh.z, bh.w);
      }
  }
  cp_async_wait_all();
  if (slot >= 0 && mine) {
#pragma unroll
    for (int j = 0; j < DP / 8; j++)
#pragma unroll
      for (int e = 0; e < 4; e++) {
        const int v = vt * 16 + g4 + 8 * (e >> 1), d = 8 * j + 2 * t4 + (e & 1);
        if (v < a.VP && d < a.dim) S[(size_t)d * a.VP + v] = acc[j][e];
      }
  }
}

// Outputs of one chunk and head: O^T = S^T R^T + Q^T, then out = o / rms(o) * norm * sigmoid(g).  A warp takes half of the tokens of NV value tiles.
template <int DP, int NV>
__global__ void __launch_bounds__(256) delta_output_kernel(const DeltaArgs a, const DeltaWs ws) {
  constexpr int KD = DP / 16;
  extern __shared__ __align__(16) float so[];                  // [GC][nvt * 16 + 4]
  const int LO = ws.nvt * 16 + 4;
  __shared__ float s_ss[4][GC];
  pdl_trigger();
  pdl_wait();
  const int c = blockIdx.x, h = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x;
  const int warp = tid >> 5, lane = tid & 31, g4 = lane >> 2, t4 = lane & 3, vq = warp & 3, th = warp >> 2;
  const int len = a.q_len[seq], qs = a.q_start[seq];
  if (c * GC >= len) return;
  const int n = min(GC, len - c * GC), t0 = qs + c * GC;
  const bool with_state = c > 0 || !(a.ctx_len[seq] - len == 0 || a.slot[seq] < 0);
  const bool vec = ((a.vdim | a.g_off | a.ld | a.ldo) & 3) == 0 && ((uintptr_t)a.norm & 15) == 0;
  if (vec && tid < n) prefetch_l2(a.in + (size_t)(t0 + tid) * a.ld + a.g_off + h * a.vdim, a.vdim * 4);      // gates, read at the end
  const size_t slot = chunk_slot(qs, seq, c) * a.H + h;
  float acc[NV][4][4];                 // value tile vq + 4 i; token tile of 8 4 th + j
#pragma unroll
  for (int i = 0; i < NV; i++)
#pragma unroll
    for (int j = 0; j < 4; j++) {
      const float4 x = __ldg(ws.q + ((slot * ws.nvt + min(vq + 4 * i, ws.nvt - 1)) * 8 + 4 * th + j) * 32 + lane);
      acc[i][j][0] = x.x; acc[i][j][1] = x.y; acc[i][j][2] = x.z; acc[i][j][3] = x.w;
    }
  if (with_state) {
#pragma unroll
    for (int kd = 0; kd < KD; kd++) {
      uint4 rh[2], rl[2];
#pragma unroll
      for (int m = 0; m < 2; m++) {
        const uint4* p = ws.r + ((slot * KD + kd) * 4 + 2 * th + m) * 64 + lane;
        rh[m] = __ldg(p);
        rl[m] = __ldg(p + 32);
      }
#pragma unroll
      for (int i = 0; i < NV; i++) {
        const uint4* p = ws.s + ((slot * ws.nvt + min(vq + 4 * i, ws.nvt - 1)) * KD + kd) * 64 + lane;
        const uint4 xh = __ldg(p), xl = __ldg(p + 32);
        const uint32_t sh[4] = {xh.x, xh.y, xh.z, xh.w}, sl[4] = {xl.x, xl.y, xl.z, xl.w};
#pragma unroll
        for (int m = 0; m < 2; m++) {
          mma_bf16(acc[i][2 * m], sh, rh[m].x, rh[m].y);
          mma_bf16(acc[i][2 * m + 1], sh, rh[m].z, rh[m].w);
          mma_bf16(acc[i][2 * m], sh, rl[m].x, rl[m].y);
          mma_bf16(acc[i][2 * m + 1], sh, rl[m].z, rl[m].w);
          mma_bf16(acc[i][2 * m], sl, rh[m].x, rh[m].y);
          mma_bf16(acc[i][2 * m + 1], sl, rh[m].z, rh[m].w);
        }
      }
    }
  }
  // sums of squares per token (value columns past vdim hold zeros), and the tile through shared memory for whole-line stores
#pragma unroll
  for (int j = 0; j < 4; j++)
#pragma unroll
    for (int e = 0; e < 2; e++) {
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < NV; i++)
        if (vq + 4 * i < ws.nvt) ss += acc[i][j][e] * acc[i][j][e] + acc[i][j][e + 2] * acc[i][j][e + 2];
      ss += __shfl_xor_sync(0xffffffffu, ss, 4);
      ss += __shfl_xor_sync(0xffffffffu, ss, 8);
      ss += __shfl_xor_sync(0xffffffffu, ss, 16);
      if (g4 == 0) s_ss[vq][32 * th + 8 * j + 2 * t4 + e] = ss;
    }
#pragma unroll
  for (int i = 0; i < NV; i++)
    if (vq + 4 * i < ws.nvt) {
#pragma unroll
      for (int j = 0; j < 4; j++)
#pragma unroll
        for (int e = 0; e < 4; e++) so[(32 * th + 8 * j + 2 * t4 + (e & 1)) * LO + (vq + 4 * i) * 16 + g4 + 8 * (e >> 1)] = acc[i][j][e];
    }
  __syncthreads();
  if (tid < GC) s_ss[0][tid] = 1.f / sqrtf((s_ss[0][tid] + s_ss[1][tid] + s_ss[2][tid] + s_ss[3][tid]) / (float)a.vdim + a.eps);
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
      *(float4*)w = __ldg((const float4*)(a.norm + h * a.vdim + e));
    } else {
#pragma unroll
      for (int k = 0; k < 4; k++)
        if (e + k < a.vdim) {
          x[k] = __ldg(g + k);
          w[k] = __ldg(a.norm + h * a.vdim + e + k);
        }
    }
#pragma unroll
    for (int k = 0; k < 4; k++) y[k] *= r * w[k] * __fdividef(1.f, 1.f + __expf(-x[k]));      // the output gate: no part of the recurrence
    const size_t at = (size_t)(t0 + t) * a.ldo + (size_t)h * a.VP + e;
    if (a.out_f32) *(float4*)(a.out_f32 + at) = make_float4(y[0], y[1], y[2], y[3]);
    if (a.out_bf16)
      *(uint2*)(a.out_bf16 + at) = make_uint2(pack_bf2(__float2bfloat16(y[0]), __float2bfloat16(y[1])), pack_bf2(__float2bfloat16(y[2]), __float2bfloat16(y[3])));
  }
}

static int delta_dp(int dim) { return dim <= 32 ? 32 : dim <= 64 ? 64 : dim <= 128 ? 128 : 0; }

// Bytes of workspace for b200_delta_chunked; 0: sizes it does not take (the caller then uses b200_delta_recurrent).
B200_API size_t b200_delta_chunk_bytes(int T, int n_seqs, int H, int dim, int VP, float decay) {
  const int DP = delta_dp(dim), nvt = (VP + 15) / 16;
  if (!DP || VP > 128 || VP % 8 || decay * GC > kDeltaSpan) return 0;
  const size_t n = ((size_t)T / GC + n_seqs + 1) * H;
  return align256(n * DP * GC * 4) + align256(n * DP * DP * 4) + align256(n * nvt * 16 * GC * 4) + 2 * align256(n * nvt * 16 * DP * 4);
}

template <int DP>
static int launch_delta_chunked(const DeltaArgs& a, const DeltaWs& w, int n_seqs, int max_q, cudaStream_t st) {
  const int s1 = DeltaSmem<DP>::bytes(w.nvt), s3 = GC * (w.nvt * 16 + 4) * 4;
  static int configured = 0;
  if (s1 > configured) {
    cudaError_t e = cudaFuncSetAttribute(delta_prepare_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, s1);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(delta_state_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, state_bytes(DP, 4));
    if (e != cudaSuccess) return (int)e;
    configured = s1;
  }
  const int nc = (max_q + GC - 1) / GC;
  int rc = launch_pdl(delta_prepare_kernel<DP>, dim3(nc, a.H, n_seqs), dim3(DeltaSmem<DP>::THREADS), s1, st, a, w);
  if (rc) return rc;
  int warps = min(4, w.nvt);                 // fewer value tiles to a CTA until the SMs are covered
  while (warps > 1 && (long)a.H * n_seqs * ((w.nvt + warps / 2 - 1) / (warps / 2)) <= 148) warps >>= 1;
  rc = launch_pdl(delta_state_kernel<DP>, dim3((w.nvt + warps - 1) / warps, a.H, n_seqs), dim3(32 * warps), state_bytes(DP, warps), st, a, w);
  if (rc) return rc;
  auto out = w.nvt <= 4 ? delta_output_kernel<DP, 1> : delta_output_kernel<DP, 2>;
  return launch_pdl(out, dim3(nc, a.H, n_seqs), dim3(256), s3, st, a, w);
}

// As b200_delta_recurrent, for prompts: T rows in all, max_q = longest portion of a sequence; ws: b200_delta_chunk_bytes bytes, 256-byte aligned.
B200_API int b200_delta_chunked(const float* in, int ld, const int* offs, int rank, const void* w2, int rank8, const float* w0, const float* ab,
                                const float* norm, float* state, const int* q_start, const int* q_len, const int* ctx_len, const int* slot, int n_seqs,
                                int H, int dim, int vdim, int VP, float decay, float eps, float* out_f32, void* out_bf16, int ldo, int T, int max_q, void* ws,
                                size_t ws_bytes, cudaStream_t st) {
  DeltaArgs a;
  int rc = delta_fill(a, in, ld, offs, rank, w2, rank8, w0, ab, norm, state, q_start, q_len, ctx_len, slot, n_seqs, H, dim, vdim, VP, decay, eps, out_f32,
                      out_bf16, ldo);
  if (rc) return rc;
  const size_t need = b200_delta_chunk_bytes(T, n_seqs, H, dim, VP, decay);
  if (!need || ws_bytes < need || T < 1 || max_q < 1 || (ldo & 3) || ((uintptr_t)out_f32 % 16) || ((uintptr_t)out_bf16 % 8) || ((uintptr_t)ws % 256) ||
      ((uintptr_t)in % 16))
    return B200_ERR_BAD_ARG;
  const int DP = delta_dp(dim);
  const size_t m = ((size_t)T / GC + n_seqs + 1) * H;
  char* p = (char*)ws;
  auto take = [&](size_t bytes) { char* q = p; p += align256(bytes); return q; };
  DeltaWs w;
  w.nvt = (VP + 15) / 16;
  w.r = (uint4*)take(m * DP * GC * 4);
  w.g = (uint4*)take(m * DP * DP * 4);
  w.q = (float4*)take(m * w.nvt * 16 * GC * 4);
  w.f = (float4*)take(m * w.nvt * 16 * DP * 4);
  w.s = (uint4*)take(m * w.nvt * 16 * DP * 4);
  switch (DP) {
    case 32: return launch_delta_chunked<32>(a, w, n_seqs, max_q, st);
    case 64: return launch_delta_chunked<64>(a, w, n_seqs, max_q, st);
    case 128: return launch_delta_chunked<128>(a, w, n_seqs, max_q, st);
  }
  return B200_ERR_BAD_ARG;
}
