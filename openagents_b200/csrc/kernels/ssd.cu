// State-space duality (Mamba-2): a scalar decay per head and token.  With inner = H * P, N state dimensions and G groups of heads, a projection row holds
// [z: inner | x: inner | B: G N | C: G N | dt: H].  x, B and C pass a causal filter per channel and silu; then per head, with state S [N][P] (fp32, zero at
// a sequence's start), dt = softplus(dt' + dt_bias) and the head's group's B and C:
//   S_t = exp(-exp(A_log) dt) S_(t-1) + dt B_t x_t^T        y_t = S_t^T C_t + D x_t
// The gate silu(z) and the norm behind it are a kernel of their own (group_norm), because the norm's parts need not be heads.
// Every sequence owns a slot of the state and of the filter's inputs, a ring of `taps` rows indexed by position; a portion whose first token is at position
// 0 starts from zero without reading either.
//
// This file is compiled without fast math; step sizes, decays, their exponentials and the state are fp32.

#include "chunk_mma.cuh"
#include "warp_mma.cuh"

using namespace b200;

struct SsdArgs {
  const float* in;              // [T][ld] projections
  int ld, x_off, dt_off;        // x, B and C are the columns [x_off, x_off + CC)
  const float* cw;              // [CC][taps], the last one on the current token
  const float* cb;              // [CC]
  const float* dt_bias;         // [H]
  const float* A_log;           // [H]
  const float* D;               // [H]
  float* state;                 // [slots][H][N][PP]
  float* ring;                  // [slots][taps][CC]
  const int* q_start;
  const int* q_len;
  const int* ctx_len;           // tokens of the sequence after this portion
  const int* slot;              // < 0: start from zero, keep nothing
  int H, P, N, G, taps, PP, NP, CC;      // PP, NP: P and N padded to multiples of 8 and 16
  float* y;                     // [T][ldy], head h at column h * P
  int ldy;
};
constexpr int kSsdDim = 256;          // most state dimensions, and most value columns of a head

__device__ __forceinline__ float silu_f(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

// The filter's input of channel ch at position p < p0 (p0: the portion's first), from the ring.
__device__ __forceinline__ float ring_at(const SsdArgs& a, int slot, int p, int ch) {
  return p < 0 || slot < 0 ? 0.f : a.ring[((size_t)slot * a.taps + p % a.taps) * a.CC + ch];
}

// ------------------------------------------------------------------ the filter

// What the chunked and the token-by-token kernels of prompts read: x [T][H][PP], B and C [T][G][NP] (padding zero), dt and the log decay [T][H].
template <typename OT>
struct SsdConv {
  OT *x, *B, *C;
  float* dt;
  float* la;
};
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

// grid (token tiles, channel tiles, sequences); a thread owns one channel of the padded outputs, then one head's step size, over a tile of tokens.
constexpr int kConvTokens = 16;
template <typename OT, int TAPS>
__global__ void __launch_bounds__(256) ssd_conv_kernel(const SsdArgs a, const SsdConv<OT> o) {
  // triggers by ending: the sequential kernel behind this one wants its CTAs spread over idle SMs
  pdl_wait();
  const int seq = blockIdx.z, i0 = blockIdx.x * kConvTokens, len = a.q_len[seq];
  if (i0 >= len) return;
  const int m = min(kConvTokens, len - i0), qs = a.q_start[seq], slot = a.slot[seq], p0 = a.ctx_len[seq] - len;
  const int xn = a.H * a.PP, bn = a.G * a.NP, k = blockIdx.y * 256 + threadIdx.x;
  if (k >= xn + 2 * bn) {                                        // a head's step size
    const int h = k - xn - 2 * bn;
    if (h >= a.H) return;
    const float bias = a.dt_bias[h], A = -expf(a.A_log[h]);
    for (int i = 0; i < m; i++) {
      const size_t t = qs + i0 + i;
      const float dt = softplus_f(a.in[t * a.ld + a.dt_off + h] + bias);
      o.dt[t * a.H + h] = dt;
      o.la[t * a.H + h] = A * dt;
    }
    return;
  }
  int ch, width;
  OT* dst;
  if (k < xn) {
    const int h = k / a.PP, e = k % a.PP;
    ch = e < a.P ? h * a.P + e : -1;
    width = xn;
    dst = o.x + k;
  } else {
    const int q = k - xn, which = q / bn, j = q % bn, g = j / a.NP, e = j % a.NP;
    ch = e < a.N ? a.H * a.P + (which * a.G + g) * a.N + e : -1;
    width = bn;
    dst = (which ? o.C : o.B) + j;
  }
  dst += (size_t)(qs + i0) * width;
  if (ch < 0) {
    for (int i = 0; i < m; i++) put(dst + (size_t)i * width, 0.f);
    return;
  }
  const float* src = a.in + (size_t)(qs + i0) * a.ld + a.x_off + ch;
  auto input = [&](int i) {                                      // i relative to this tile, may be negative
    if (i0 + i >= 0) return src[(ptrdiff_t)i * a.ld];
    return ring_at(a, slot, p0 + i0 + i, ch);
  };
  const float bias = a.cb[ch];
  if constexpr (TAPS > 0) {
    float w[TAPS], v[kConvTokens + TAPS - 1];
#pragma unroll
    for (int j = 0; j < TAPS; j++) w[j] = a.cw[(size_t)ch * TAPS + j];
#pragma unroll
    for (int j = 0; j < TAPS - 1; j++) v[j] = input(j - TAPS + 1);
#pragma unroll
    for (int i = 0; i < kConvTokens; i++) v[TAPS - 1 + i] = i < m ? src[(size_t)i * a.ld] : 0.f;
#pragma unroll
    for (int i = 0; i < kConvTokens; i++) {
      float s = 0.f;
#pragma unroll
      for (int j = 0; j < TAPS; j++) s = fmaf(w[j], v[i + j], s);
      if (i < m) put(dst + (size_t)i * width, silu_f(s + bias));
    }
  } else {
    for (int i = 0; i < m; i++) {
      float s = 0.f;
      for (int j = 0; j < a.taps; j++) s = fmaf(a.cw[(size_t)ch * a.taps + j], input(i - a.taps + 1 + j), s);
      put(dst + (size_t)i * width, silu_f(s + bias));
    }
  }
}

// ------------------------------------------------------------------ token by token

// The CTAs of a head share its value columns and the sequences.  A CTA walks the tokens of its sequences one by one; while it works on one, the filtered inputs
// of the next, and with a new sequence its state, are on their way into the other half of a double buffer.  The state is updated in shared memory.
// FUSED (a few sequences with one token each): the filter is applied here, and its input written to the ring: the row of the current position, which no CTA
// reads.  Otherwise the filter has run (fp32), and the ring takes the portion's last inputs.
__device__ __forceinline__ void cp_async4(void* dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(s32(dst)), "l"(src) : "memory");
}
struct SsdLayout {                         // floats of shared memory: two states, two rows, the partial outputs
  int state_n, row_n, row, y, total;
};
static SsdLayout ssd_layout(int N, int W) {
  SsdLayout l;
  l.state_n = N * W;
  l.row_n = W + 2 * N + 4;                 // x | B | C | dt, log decay
  l.row_n = (l.row_n + 3) & ~3;
  l.row = 2 * l.state_n;
  l.y = l.row + 2 * l.row_n;
  l.total = l.y + 256 / (W / 4) * W;
  return l;
}
template <bool FUSED>
__global__ void __launch_bounds__(256, 4) ssd_recurrent_kernel(const SsdArgs a, const SsdConv<float> o, int n_seqs, const SsdLayout l) {
  extern __shared__ __align__(16) float sm[];
  const int CL = gridDim.x / a.H, part = blockIdx.x % CL, h = blockIdx.x / CL, tid = threadIdx.x;
  const int nv_all = a.PP >> 2, nv = nv_all / CL, W = nv * 4, e0 = part * W;     // this CTA's columns [e0, e0 + W)
  const int groups = 256 / nv, g = h / (a.H / a.G);
  float* s_y = sm + l.y;                   // [groups][W]
  pdl_trigger();
  const float A = -expf(a.A_log[h]), Dh = a.D[h], dtb = a.dt_bias[h];
  const int xc = a.H * a.P;
  // the filter's channels that this CTA needs: x columns, then B, then C of the group; `own`: those it keeps the ring of
  const int n_ch = W + 2 * a.N;
  auto channel = [&](int i) {
    if (i < W) return e0 + i < a.P ? h * a.P + e0 + i : -1;
    const int j = i - W, which = j / a.N;
    return xc + (which * a.G + g) * a.N + j - which * a.N;
  };
  const bool first_head = part == 0 && h % (a.H / a.G) == 0;
  auto own = [&](int i) { return i < W || first_head; };
  const int grp = tid / nv, col = tid % nv;
  const bool active = grp < groups;
  pdl_wait();
  struct Seq { int n, t0, slot, p0; bool fresh; };
  auto meta = [&](int b) {
    Seq q = {0, 0, -1, 0, true};
    if (b < n_seqs) {
      q.n = a.q_len[b];
      q.t0 = a.q_start[b];
      q.slot = a.slot[b];
      q.p0 = a.ctx_len[b] - q.n;
      q.fresh = q.p0 == 0 || q.slot < 0;
    }
    return q;
  };
  auto state_of = [&](int slot) { return (float4*)(a.state + ((size_t)max(slot, 0) * a.H + h) * a.N * a.PP) + part * nv; };
  auto fetch_state = [&](const Seq& q, int buf) {
    float4* dst = (float4*)(sm + buf * l.state_n);
    const float4* src = state_of(q.slot);
    if (!active) return;
    for (int d = grp; d < a.N; d += groups) {
      if (!q.fresh) cp_async16(s32(dst + d * nv + col), src + (size_t)d * nv_all + col);
      else dst[d * nv + col] = make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  auto fetch_row = [&](size_t t, int buf) {
    float* dst = sm + l.row + buf * l.row_n;
    for (int q = tid; q < n_ch + 2; q += 256) {
      const float* src;
      if (q < W) src = o.x + (t * a.H + h) * a.PP + e0 + q;
      else if (q < W + a.N) src = o.B + (t * a.G + g) * a.NP + q - W;
      else if (q < n_ch) src = o.C + (t * a.G + g) * a.NP + q - W - a.N;
      else src = (q == n_ch ? o.dt : o.la) + t * a.H + h;
      cp_async4(dst + q, src);
    }
  };
  auto filter_row = [&](const Seq& q, int buf) {          // FUSED
    float* dst = sm + l.row + buf * l.row_n;
    const float* row = a.in + (size_t)q.t0 * a.ld;
    for (int i = tid; i < n_ch; i += 256) {
      const int ch = channel(i);
      float s = 0.f;
      if (ch >= 0) {
        const float cur = row[a.x_off + ch], *w = a.cw + (size_t)ch * a.taps;
        if (!q.fresh)
          for (int j = 0; j < a.taps - 1; j++) s = fmaf(w[j], ring_at(a, q.slot, q.p0 - a.taps + 1 + j, ch), s);
        s = silu_f(fmaf(w[a.taps - 1], cur, s) + a.cb[ch]);
        if (q.slot >= 0 && own(i)) a.ring[((size_t)q.slot * a.taps + q.p0 % a.taps) * a.CC + ch] = cur;
      }
      dst[i] = s;
    }
    if (tid == 0) {
      dst[n_ch] = softplus_f(row[a.dt_off + h] + dtb);
      dst[n_ch + 1] = A * dst[n_ch];
    }
  };
  int b = blockIdx.y, i = 0, sbuf = 0, rbuf = 0;
  Seq cur = meta(b), nxt = meta(b + gridDim.y);
  while (b < n_seqs && cur.n < 1) {         // an entry without tokens
    b += gridDim.y;
    cur = nxt;
    nxt = meta(b + gridDim.y);
  }
  auto begin = [&]() {
    fetch_state(cur, sbuf);
    if (FUSED) filter_row(cur, rbuf);
    else fetch_row(cur.t0, rbuf);
    cp_async_commit();
  };
  if (b < n_seqs) begin();
  while (b < n_seqs) {
    cp_async_wait_all();
    __syncthreads();                       // this token's data has landed, and everyone is done with the other buffers
    const bool last = i + 1 == cur.n;
    if (!FUSED) {
      if (!last) {
        fetch_row(cur.t0 + i + 1, rbuf ^ 1);
      } else if (b + gridDim.y < n_seqs && nxt.n > 0) {
        fetch_state(nxt, sbuf ^ 1);
        fetch_row(nxt.t0, rbuf ^ 1);
      }
      cp_async_commit();
    }
    const float* row = sm + l.row + rbuf * l.row_n;
    const float *s_b = row + W, *s_c = s_b + a.N;
    const float dt = row[n_ch], al = expf(row[n_ch + 1]);
    if (active) {
      const bool keep = last && cur.slot >= 0;
      float4* S = (float4*)(sm + sbuf * l.state_n) + col;
      float4* dst = state_of(cur.slot) + col;
      float4 x = *(const float4*)(row + 4 * col);
      x.x *= dt; x.y *= dt; x.z *= dt; x.w *= dt;
      float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
      for (int d = grp; d < a.N; d += groups) {
        const float bb = s_b[d], cc = s_c[d];
        float4 v = S[d * nv];
        v.x = fmaf(al, v.x, bb * x.x);
        v.y = fmaf(al, v.y, bb * x.y);
        v.z = fmaf(al, v.z, bb * x.z);
        v.w = fmaf(al, v.w, bb * x.w);
        if (!last) S[d * nv] = v;
        else if (keep) dst[(size_t)d * nv_all] = v;
        y.x = fmaf(cc, v.x, y.x);
        y.y = fmaf(cc, v.y, y.y);
        y.z = fmaf(cc, v.z, y.z);
        y.w = fmaf(cc, v.w, y.w);
      }
      *(float4*)(s_y + grp * W + 4 * col) = y;
    }
    __syncthreads();
    if (tid < W && e0 + tid < a.P) {       // W <= 256
      float y = Dh * row[tid];
#pragma unroll 4
      for (int q = 0; q < groups; q++) y += s_y[q * W + tid];
      a.y[(size_t)(cur.t0 + i) * a.ldy + h * a.P + e0 + tid] = y;
    }
    rbuf ^= 1;
    i++;
    if (last) {
      if (!FUSED && cur.slot >= 0)
        for (int q = tid; q < n_ch; q += 256) {
          const int ch = channel(q);
          if (ch < 0 || !own(q)) continue;
          for (int j = max(0, cur.n - a.taps + 1); j < cur.n; j++)
            a.ring[((size_t)cur.slot * a.taps + (cur.p0 + j) % a.taps) * a.CC + ch] = a.in[(size_t)(cur.t0 + j) * a.ld + a.x_off + ch];
        }
      i = 0;
      sbuf ^= 1;
      bool skipped = false;
      do {                                 // past entries without tokens, whose successors were not fetched ahead
        b += gridDim.y;
        cur = nxt;
        nxt = meta(b + gridDim.y);
        if (b < n_seqs && cur.n < 1) skipped = true;
      } while (b < n_seqs && cur.n < 1);
      if ((FUSED || skipped) && b < n_seqs) {
        __syncthreads();
        begin();
      }
    }
  }
}

static int ssd_fill(SsdArgs& a, const float* in, int ld, int x_off, int dt_off, const float* cw, const float* cb, const float* dt_bias, const float* A_log,
                    const float* D, float* state, float* ring, const int* q_start, const int* q_len, const int* ctx_len, const int* slot, int n_seqs, int H,
                    int P, int N, int G, int taps, int PP, float* y, int ldy) {
  if (n_seqs < 1 || H < 1 || P < 1 || N < 1 || G < 1 || H % G || taps < 1 || PP < P || PP % 8 || PP > kSsdDim || N > kSsdDim || ldy < H * P ||
      ((uintptr_t)state % 16) || !ring || !slot || !y || ld < x_off + H * P + 2 * G * N)
    return B200_ERR_BAD_ARG;
  a.in = in; a.ld = ld; a.x_off = x_off; a.dt_off = dt_off; a.cw = cw; a.cb = cb; a.dt_bias = dt_bias; a.A_log = A_log; a.D = D; a.state = state;
  a.ring = ring; a.q_start = q_start; a.q_len = q_len; a.ctx_len = ctx_len; a.slot = slot; a.H = H; a.P = P; a.N = N; a.G = G; a.taps = taps; a.PP = PP;
  a.NP = (N + 15) / 16 * 16; a.CC = H * P + 2 * G * N; a.y = y; a.ldy = ldy;
  return 0;
}

template <bool FUSED>
static int launch_ssd_recurrent(const SsdArgs& a, const SsdConv<float>& o, int n_seqs, cudaStream_t st) {
  // CTAs per head: until a state share is 32 KB at most and the SMs are covered, eight float4 columns each at least
  int CL = 1;
  while (CL < 8 && (a.PP / 4) % (2 * CL) == 0 && a.PP / 4 / (2 * CL) >= 8 && (a.N * a.PP / CL > 8192 || (long)a.H * n_seqs * CL < 148)) CL *= 2;
  const SsdLayout l = ssd_layout(a.N, a.PP / CL);
  const size_t smem = 4 * (size_t)l.total;
  if (smem > 200 * 1024) return B200_ERR_BAD_ARG;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(ssd_recurrent_kernel<FUSED>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  // shares of the sequences: no more CTAs than run at a time, all with about the same number of sequences
  const int fit = (int)(227 * 1024 / (smem + 1024)), resident = 148 * (fit < 1 ? 1 : fit > 4 ? 4 : fit);
  const int most = resident / (a.H * CL) > 1 ? resident / (a.H * CL) : 1, rounds = (n_seqs + most - 1) / most;
  return launch_pdl(ssd_recurrent_kernel<FUSED>, dim3(a.H * CL, (n_seqs + rounds - 1) / rounds), dim3(256), smem, st, a, o, n_seqs, l);
}

template <typename OT>
static SsdConv<OT> ssd_conv_ws(const SsdArgs& a, char*& p, int T) {
  auto take = [&](size_t bytes) { char* q = p; p += align256(bytes); return q; };
  SsdConv<OT> o;
  o.x = (OT*)take((size_t)T * a.H * a.PP * sizeof(OT));
  o.B = (OT*)take((size_t)T * a.G * a.NP * sizeof(OT));
  o.C = (OT*)take((size_t)T * a.G * a.NP * sizeof(OT));
  o.dt = (float*)take((size_t)T * a.H * 4);
  o.la = (float*)take((size_t)T * a.H * 4);
  return o;
}
static size_t ssd_conv_bytes(int T, int H, int PP, int G, int NP, int size) {
  return align256((size_t)T * H * PP * size) + 2 * align256((size_t)T * G * NP * size) + 2 * align256((size_t)T * H * 4);
}
template <typename OT>
static int launch_ssd_conv(const SsdArgs& a, const SsdConv<OT>& o, int n_seqs, int max_q, cudaStream_t st) {
  const int channels = a.H * a.PP + 2 * a.G * a.NP + a.H;
  auto kern = a.taps == 4 ? ssd_conv_kernel<OT, 4> : ssd_conv_kernel<OT, 0>;
  return launch_pdl(kern, dim3((max_q + kConvTokens - 1) / kConvTokens, (channels + 255) / 256, n_seqs), dim3(256), 0, st, a, o);
}

#define SSD_PARAMS                                                                                                                                     \
  const float *in, int ld, int x_off, int dt_off, const float *cw, const float *cb, const float *dt_bias, const float *A_log, const float *D,         \
      float *state, float *ring, const int *q_start, const int *q_len, const int *ctx_len, const int *slot, int n_seqs, int H, int P, int N, int G,     \
      int taps, int PP, float *y, int ldy
#define SSD_FILL                                                                                                                                       \
  ssd_fill(a, in, ld, x_off, dt_off, cw, cb, dt_bias, A_log, D, state, ring, q_start, q_len, ctx_len, slot, n_seqs, H, P, N, G, taps, PP, y, ldy)

constexpr int kFusedSeqs = 4;           // decode steps of up to this many sequences apply the filter in the recurrence's kernel

// One token per sequence.  ws: b200_ssd_decode_bytes bytes, 256-byte aligned.
B200_API size_t b200_ssd_decode_bytes(int n_seqs, int H, int PP, int N, int G) {
  return n_seqs <= kFusedSeqs ? 0 : ssd_conv_bytes(n_seqs, H, PP, G, (N + 15) / 16 * 16, 4);
}
B200_API int b200_ssd_decode(SSD_PARAMS, void* ws, size_t ws_bytes, cudaStream_t st) {
  SsdArgs a;
  int rc = SSD_FILL;
  if (rc) return rc;
  if (n_seqs <= kFusedSeqs) return launch_ssd_recurrent<true>(a, SsdConv<float>{}, n_seqs, st);
  if (ws_bytes < b200_ssd_decode_bytes(n_seqs, H, PP, N, G) || ((uintptr_t)ws % 256)) return B200_ERR_BAD_ARG;
  char* p = (char*)ws;
  const SsdConv<float> o = ssd_conv_ws<float>(a, p, n_seqs);
  rc = launch_ssd_conv(a, o, n_seqs, 1, st);
  return rc ? rc : launch_ssd_recurrent<false>(a, o, n_seqs, st);
}

// ------------------------------------------------------------------ prompts: 64-token chunks on the tensor cores
//
// With b_t the running sum of log decays from the chunk's start and C its last token, per head:
//   y_t = e^{b_t} C_t S + sum_{s<=t} (C_t . B_s) e^{b_t - b_s} dt_s x_s + D x_t
//   S'  = e^{b_C} S + sum_s B_s (x_s dt_s e^{b_C - b_s})^T
// ssd_state_kernel walks a sequence's chunks with S in registers and leaves every chunk's starting state behind; ssd_output_kernel forms the outputs, all
// chunks and heads in parallel.  No exponent is ever positive.  x, B and C, which come out of a short filter, are bf16; what holds a step size, a decay
// or the state enters the tensor cores as two bf16 numbers (value and remainder), products accumulate in fp32.

struct SsdWs {
  SsdConv<__nv_bfloat16> c;
  uint4* s;                     // [chunk slots][H][P tiles of 16][NP / 16][2][lane]: the state at the chunk's start (value columns as rows)
  int npt, kn;                  // tiles of 16 value columns / state dimensions
};

// Steps and running log-decay sums of a chunk, in every warp: lane l holds tokens 2 l and 2 l + 1.
struct ChunkDecay {
  float2 dt, b;
  float total;
};
struct RawDecay {
  float2 dt, la;
};
__device__ __forceinline__ RawDecay load_decay(const SsdArgs& a, const SsdConv<__nv_bfloat16>& o, int t0, int n, int h, int lane) {
  const size_t at = (size_t)(t0 + 2 * lane) * a.H + h;
  const bool v0 = 2 * lane < n, v1 = 2 * lane + 1 < n;
  RawDecay r;
  r.dt = make_float2(v0 ? o.dt[at] : 0.f, v1 ? o.dt[at + a.H] : 0.f);
  r.la = make_float2(v0 ? o.la[at] : 0.f, v1 ? o.la[at + a.H] : 0.f);
  return r;
}
__device__ __forceinline__ ChunkDecay chunk_decay(const RawDecay& raw, int lane) {
  ChunkDecay r;
  r.dt = raw.dt;
  const float l0 = raw.la.x, l1 = raw.la.y;
  float s = l0 + l1;
#pragma unroll
  for (int d = 1; d < 32; d <<= 1) {
    const float x = __shfl_up_sync(0xffffffffu, s, d);
    if (lane >= d) s += x;
  }
  r.total = __shfl_sync(0xffffffffu, s, 31);
  float before = __shfl_up_sync(0xffffffffu, s, 1);
  if (lane == 0) before = 0.f;
  r.b = make_float2(before + l0, before + l0 + l1);
  return r;
}

constexpr int kSsdStages = 3;

// One CTA = 64 value columns x 2 DW state dimensions of one head of one sequence; a warp owns 16 value columns and half of the dimensions.  The state is kept
// transposed (value columns as the rows of the MMA), so that its accumulators, split in two, are operands of the output product as they lie.
template <int DW>
__global__ void __launch_bounds__(256) ssd_state_kernel(const SsdArgs a, const SsdWs ws) {
  constexpr int DS = 2 * DW, LN = DS + 8, LX = 72, STAGE = GC * (LN + LX), NJ = DW / 8;      // B slice | x
  extern __shared__ __align__(16) __nv_bfloat16 sb16[];
  pdl_trigger();
  pdl_wait();
  const int nslices = (a.NP + DS - 1) / DS;
  const int ps = blockIdx.x / nslices, n0 = blockIdx.x % nslices * DS, v0 = ps * 64, h = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x;
  const int warp = (tid >> 5) & 3, dw = (tid >> 7) * DW, lane = tid & 31, g4 = lane >> 2, t4 = lane & 3, g = h / (a.H / a.G);
  const int len = a.q_len[seq], qs = a.q_start[seq], slot = a.slot[seq], p0 = a.ctx_len[seq] - len;
  const bool fresh = p0 == 0 || slot < 0;
  const int nc = (len + GC - 1) / GC;
  float* S = a.state + ((size_t)max(slot, 0) * a.H + h) * a.N * a.PP;
  // this thread's 16-byte pieces of a chunk: two of x, and as many of B as its rows are long
  constexpr int BQ = DS / 8, BT = 256 / BQ;
  const int pt0 = tid / 8, px = (tid % 8) * 8, bt0 = tid / BQ, bx = (tid % BQ) * 8;
  const bool blive = n0 + bx < a.NP, xlive = v0 + px < a.PP;
  auto load = [&](int c) {
    if (c < nc) {
      __nv_bfloat16* st = sb16 + (c % kSsdStages) * STAGE;
#pragma unroll
      for (int m = 0; m < GC / BT; m++) {
        const int i = c * GC + bt0 + BT * m;
        __nv_bfloat16* db = st + (bt0 + BT * m) * LN + bx;
        if (blive && i < len) cp_async16(s32(db), ws.c.B + ((size_t)(qs + i) * a.G + g) * a.NP + n0 + bx);
        else *(uint4*)db = make_uint4(0u, 0u, 0u, 0u);
      }
#pragma unroll
      for (int m = 0; m < 2; m++) {
        const int i = c * GC + pt0 + 32 * m;
        __nv_bfloat16* dx = st + GC * LN + (pt0 + 32 * m) * LX + px;
        if (xlive && i < len) cp_async16(s32(dx), ws.c.x + ((size_t)(qs + i) * a.H + h) * a.PP + v0 + px);
        else *(uint4*)dx = make_uint4(0u, 0u, 0u, 0u);
      }
    }
    cp_async_commit();                  // empty past the end: keeps the count of groups in flight
  };
#pragma unroll
  for (int c = 0; c < kSsdStages - 1; c++) load(c);
  float acc[NJ][4];                      // rows v0 + 16 warp + g4 (+ 8), columns n0 + dw + 8 j + 2 t4 (+ 1)
#pragma unroll
  for (int j = 0; j < NJ; j++)
#pragma unroll
    for (int e = 0; e < 4; e++) {
      const int v = v0 + warp * 16 + g4 + 8 * (e >> 1), d = n0 + dw + 8 * j + 2 * t4 + (e & 1);
      acc[j][e] = (!fresh && v < a.PP && d < a.N) ? S[(size_t)d * a.PP + v] : 0.f;
    }
  const int pt = ps * 4 + warp;
  float f0, f1, dec;
  auto factors = [&](const RawDecay& raw) {
    const ChunkDecay dc = chunk_decay(raw, lane);
    f0 = dc.dt.x * expf(dc.total - dc.b.x);
    f1 = dc.dt.y * expf(dc.total - dc.b.y);
    dec = expf(dc.total);
  };
  factors(load_decay(a, ws.c, qs, min(GC, len), h, lane));
  for (int c = 0; c < nc; c++) {
    const RawDecay next = load_decay(a, ws.c, qs + (c + 1) * GC, len - (c + 1) * GC, h, lane);      // in flight until the products are done
    cp_async_wait<kSsdStages - 2>();
    __syncthreads();                    // chunk c has landed, and everyone is done with the stage that is refilled now
    load(c + kSsdStages - 1);
    const __nv_bfloat16 *sB = sb16 + (c % kSsdStages) * STAGE, *sX = sB + GC * LN;
    if (c > 0 || !fresh) {
#pragma unroll
      for (int kd = 0; kd < DW / 16; kd++) {
        const int kt = (n0 + dw) / 16 + kd;
        uint4 hi, lo;
        split2(acc[2 * kd][0], acc[2 * kd][1], hi.x, lo.x);
        split2(acc[2 * kd][2], acc[2 * kd][3], hi.y, lo.y);
        split2(acc[2 * kd + 1][0], acc[2 * kd + 1][1], hi.z, lo.z);
        split2(acc[2 * kd + 1][2], acc[2 * kd + 1][3], hi.w, lo.w);
        if (pt < ws.npt && kt < ws.kn) {
          uint4* frag = ws.s + (((chunk_slot(qs, seq, c) * a.H + h) * ws.npt + pt) * ws.kn + kt) * 64 + lane;
          frag[0] = hi;
          frag[32] = lo;
        }
      }
#pragma unroll
      for (int j = 0; j < NJ; j++)
#pragma unroll
        for (int e = 0; e < 4; e++) acc[j][e] *= dec;
    }
#pragma unroll
    for (int kt = 0; kt < GC / 16; kt++) {
      uint32_t xa[4], xh[4], xl[4];     // X^T: 16 value columns x 16 tokens, times the tokens' factors
      ldsm4t(s32(sX + (kt * 16 + (lane >> 4) * 8 + (lane & 7)) * LX + warp * 16 + ((lane >> 3) & 1) * 8), xa);
      const float fa = __shfl_sync(0xffffffffu, f0, kt * 8 + t4), fb = __shfl_sync(0xffffffffu, f1, kt * 8 + t4);
      const float fc = __shfl_sync(0xffffffffu, f0, kt * 8 + 4 + t4), fd = __shfl_sync(0xffffffffu, f1, kt * 8 + 4 + t4);
#pragma unroll
      for (int m = 0; m < 4; m++) {
        const float2 x = __bfloat1622float2(*(const __nv_bfloat162*)&xa[m]);
        split2(x.x * (m < 2 ? fa : fc), x.y * (m < 2 ? fb : fd), xh[m], xl[m]);
      }
      const int r = kt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8;
#pragma unroll
      for (int j = 0; j < NJ; j += 2) {
        uint32_t bb[4];
        ldsm4t(s32(sB + r * LN + dw + (j + (lane >> 4)) * 8), bb);
        mma_bf16(acc[j], xh, bb[0], bb[1]);
        mma_bf16(acc[j + 1], xh, bb[2], bb[3]);
        mma_bf16(acc[j], xl, bb[0], bb[1]);
        mma_bf16(acc[j + 1], xl, bb[2], bb[3]);
      }
    }
    factors(next);
  }
  cp_async_wait_all();
  if (slot < 0) return;
#pragma unroll
  for (int j = 0; j < NJ; j++)
#pragma unroll
    for (int e = 0; e < 4; e++) {
      const int v = v0 + warp * 16 + g4 + 8 * (e >> 1), d = n0 + dw + 8 * j + 2 * t4 + (e & 1);
      if (v < a.PP && d < a.N) S[(size_t)d * a.PP + v] = acc[j][e];
    }
  // the filter's last inputs: x channels by the head's first CTA of these columns, B and C by the group's first head
  if (n0 == 0)
    for (int q = tid; q < 64 * (a.taps - 1); q += 256) {
      const int e = v0 + q % 64, i = len - 1 - q / 64;
      if (e < a.P && i >= 0) a.ring[((size_t)slot * a.taps + (p0 + i) % a.taps) * a.CC + h * a.P + e] = a.in[(size_t)(qs + i) * a.ld + a.x_off + h * a.P + e];
    }
  if (ps == 0 && h % (a.H / a.G) == 0)
    for (int q = tid; q < 2 * DS * (a.taps - 1); q += 256) {
      const int d = n0 + q % DS, which = q / DS % 2, i = len - 1 - q / (2 * DS), ch = a.H * a.P + (which * a.G + g) * a.N + d;
      if (d < a.N && i >= 0) a.ring[((size_t)slot * a.taps + (p0 + i) % a.taps) * a.CC + ch] = a.in[(size_t)(qs + i) * a.ld + a.x_off + ch];
    }
}

// Outputs of one chunk and HB heads of a group over all their value columns: B and C, and the product C B^T, serve all of them.  A warp takes half of the
// tokens of NV value tiles.  While a head's outputs are formed, the next one's x is on its way.
template <int NV>
__global__ void __launch_bounds__(256, NV <= 2 ? 2 : 1) ssd_output_kernel(const SsdArgs a, const SsdWs ws, int HB) {
  constexpr int LA = GC + 8;
  extern __shared__ __align__(16) __nv_bfloat16 o16[];
  const int LN = a.NP + 8, LX = ws.npt * 16 + 8, LO = ws.npt * 16 + 4;
  __nv_bfloat16 *sC = o16, *sX0 = sC + GC * LN, *sAh = sX0 + 2 * GC * LX, *sAl = sAh + GC * LA, *sB = sAl + GC * LA;
  float* so = (float*)sB;                                      // [GC][LO], over B once it is used
  __shared__ float s_b[GC], s_dt[GC];
  pdl_trigger();
  pdl_wait();
  const int c = blockIdx.x, h0 = blockIdx.y * HB, seq = blockIdx.z, tid = threadIdx.x, g = h0 / (a.H / a.G);
  const int warp = tid >> 5, lane = tid & 31, g4 = lane >> 2, t4 = lane & 3;
  const int len = a.q_len[seq], qs = a.q_start[seq];
  if (c * GC >= len) return;
  const bool with_state = c > 0 || !(a.ctx_len[seq] - len == 0 || a.slot[seq] < 0);
  const int n = min(GC, len - c * GC), t0 = qs + c * GC;
  const int n8 = a.NP / 8, p8 = ws.npt * 2;
  for (GridWalk w(tid, 256, n8); w.r < 2 * GC; w.next()) {
    const int which = w.r >= GC, t = w.r - which * GC, x = w.c * 8;
    __nv_bfloat16* dst = (which ? sB : sC) + t * LN + x;
    if (t < n) cp_async16(s32(dst), (which ? ws.c.B : ws.c.C) + ((size_t)(t0 + t) * a.G + g) * a.NP + x);
    else *(uint4*)dst = make_uint4(0u, 0u, 0u, 0u);
  }
  auto load_x = [&](int k) {
    for (GridWalk w(tid, 256, p8); w.r < GC; w.next()) {
      const int t = w.r, x = w.c * 8;
      __nv_bfloat16* dst = sX0 + (k & 1) * GC * LX + t * LX + x;
      if (t < n && x < a.PP) cp_async16(s32(dst), ws.c.x + ((size_t)(t0 + t) * a.H + h0 + k) * a.PP + x);
      else *(uint4*)dst = make_uint4(0u, 0u, 0u, 0u);
    }
  };
  load_x(0);
  cp_async_commit();
  RawDecay raw = {};                                            // warp 0's
  if (warp == 0) raw = load_decay(a, ws.c, t0, n, h0, lane);
  cp_async_wait<0>();
  __syncthreads();
  // C B^T: warp = 16 tokens x 32 earlier ones
  const int m0 = (warp >> 1) * 16, n0 = (warp & 1) * 32;
  float cb[4][4] = {};
  if (n0 <= m0 + 15) {
    for (int k0 = 0; k0 < a.NP; k0 += 16) {
      uint32_t ca[4];
      ldsm4(s32(sC + (m0 + (lane & 15)) * LN + k0 + (lane >> 4) * 8), ca);
#pragma unroll
      for (int j = 0; j < 4; j += 2) {
        uint32_t bb[4];
        ldsm4(s32(sB + (n0 + (j + (lane >> 4)) * 8 + (lane & 7)) * LN + k0 + ((lane >> 3) & 1) * 8), bb);
        mma_bf16(cb[j], ca, bb[0], bb[1]);
        mma_bf16(cb[j + 1], ca, bb[2], bb[3]);
      }
    }
  }
  const int vq = warp & 3, th = warp >> 2;
  const bool vec = ((a.P | a.ldy) & 3) == 0 && ((uintptr_t)a.y & 15) == 0;
  for (int k = 0; k < HB; k++) {
    const int h = h0 + k;
    const __nv_bfloat16* sX = sX0 + (k & 1) * GC * LX;
    if (warp == 0) {
      const ChunkDecay dc = chunk_decay(raw, lane);
      *(float2*)(s_b + 2 * lane) = dc.b;
      *(float2*)(s_dt + 2 * lane) = dc.dt;
    }
    cp_async_wait<0>();
    __syncthreads();                                           // x and the decays of this head; the last one's outputs have been read
    if (k + 1 < HB) {
      load_x(k + 1);
      if (warp == 0) raw = load_decay(a, ws.c, t0, n, h + 1, lane);
    }
    cp_async_commit();
    const float bt[2] = {s_b[m0 + g4], s_b[m0 + g4 + 8]};
    // the decays on the hardware's exponential: these products become two bf16 numbers each.  Blocks above the diagonal stay as they are, zero.
#pragma unroll
    for (int j = 0; j < 4; j++)
#pragma unroll
      for (int hf = 0; hf < 2; hf++) {
        if (n0 > m0 + 15 && k) continue;
        const int t = m0 + g4 + 8 * hf, s = n0 + 8 * j + 2 * t4;
        const float2 bs = *(const float2*)(s_b + s), ds = *(const float2*)(s_dt + s);
        const float x = s <= t ? cb[j][2 * hf] * __expf(bt[hf] - bs.x) * ds.x : 0.f;
        const float y = s + 1 <= t ? cb[j][2 * hf + 1] * __expf(bt[hf] - bs.y) * ds.y : 0.f;
        uint32_t hi, lo;
        split2(x, y, hi, lo);
        *(uint32_t*)(sAh + t * LA + s) = hi;
        *(uint32_t*)(sAl + t * LA + s) = lo;
      }
    float acc[NV][4][4];                                       // value tile vq + 4 i; columns = tokens 32 th + 8 j + 2 t4 (+ 1)
#pragma unroll
    for (int i = 0; i < NV; i++)
#pragma unroll
      for (int j = 0; j < 4; j++) acc[i][j][0] = acc[i][j][1] = acc[i][j][2] = acc[i][j][3] = 0.f;
    if (with_state) {
      const uint4* frag = ws.s + (chunk_slot(qs, seq, c) * a.H + h) * ws.npt * ws.kn * 64 + lane;
#pragma unroll 4
      for (int kd = 0; kd < ws.kn; kd++) {
        uint32_t cc[2][4];
#pragma unroll
        for (int m = 0; m < 2; m++) ldsm4(s32(sC + (32 * th + 16 * m + (lane >> 4) * 8 + (lane & 7)) * LN + kd * 16 + ((lane >> 3) & 1) * 8), cc[m]);
#pragma unroll
        for (int i = 0; i < NV; i++) {
          const uint4* p = frag + ((size_t)min(vq + 4 * i, ws.npt - 1) * ws.kn + kd) * 64;
          const uint4 xh = __ldg(p), xl = __ldg(p + 32);
          const uint32_t sh[4] = {xh.x, xh.y, xh.z, xh.w}, sl[4] = {xl.x, xl.y, xl.z, xl.w};
#pragma unroll
          for (int m = 0; m < 2; m++) {
            mma_bf16(acc[i][2 * m], sh, cc[m][0], cc[m][1]);
            mma_bf16(acc[i][2 * m + 1], sh, cc[m][2], cc[m][3]);
            mma_bf16(acc[i][2 * m], sl, cc[m][0], cc[m][1]);
            mma_bf16(acc[i][2 * m + 1], sl, cc[m][2], cc[m][3]);
          }
        }
      }
#pragma unroll
      for (int j = 0; j < 4; j++) {
        const float2 b = *(const float2*)(s_b + 32 * th + 8 * j + 2 * t4);
        const float e0 = expf(b.x), e1 = expf(b.y);
#pragma unroll
        for (int i = 0; i < NV; i++) {
          acc[i][j][0] *= e0;
          acc[i][j][1] *= e1;
          acc[i][j][2] *= e0;
          acc[i][j][3] *= e1;
        }
      }
    }
    __syncthreads();                                           // the decayed products of all warps
#pragma unroll
    for (int kt = 0; kt < GC / 16; kt++) {
      if (kt * 16 >= 32 * th + 32) break;                      // later tokens than any of this warp's
      uint32_t xa[NV][4];
#pragma unroll
      for (int i = 0; i < NV; i++)
        ldsm4t(s32(sX + (kt * 16 + (lane >> 4) * 8 + (lane & 7)) * LX + min(vq + 4 * i, ws.npt - 1) * 16 + ((lane >> 3) & 1) * 8), xa[i]);
#pragma unroll
      for (int m = 0; m < 2; m++) {
        const int at = (32 * th + 16 * m + (lane >> 4) * 8 + (lane & 7)) * LA + kt * 16 + ((lane >> 3) & 1) * 8;
        uint32_t bh[4], bl[4];
        ldsm4(s32(sAh + at), bh);
        ldsm4(s32(sAl + at), bl);
#pragma unroll
        for (int i = 0; i < NV; i++) {
          mma_bf16(acc[i][2 * m], xa[i], bh[0], bh[1]);
          mma_bf16(acc[i][2 * m + 1], xa[i], bh[2], bh[3]);
          mma_bf16(acc[i][2 * m], xa[i], bl[0], bl[1]);
          mma_bf16(acc[i][2 * m + 1], xa[i], bl[2], bl[3]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < NV; i++)
      if (vq + 4 * i < ws.npt) {
#pragma unroll
        for (int j = 0; j < 4; j++)
#pragma unroll
          for (int e = 0; e < 4; e++) so[(32 * th + 8 * j + 2 * t4 + (e & 1)) * LO + (vq + 4 * i) * 16 + g4 + 8 * (e >> 1)] = acc[i][j][e];
      }
    __syncthreads();
    const float D = a.D[h];
    GridWalk w(tid, 256, vec ? a.P / 4 : a.P);
#pragma unroll 4
    for (; w.r < n; w.next()) {
      const int t = w.r;
      float* dst = a.y + (size_t)(t0 + t) * a.ldy + h * a.P;
      if (vec) {
        const int e = w.c * 4;
        float4 o = *(const float4*)(so + t * LO + e);
        const uint2 x = *(const uint2*)(sX + t * LX + e);
        const float2 x0 = __bfloat1622float2(*(const __nv_bfloat162*)&x.x), x1 = __bfloat1622float2(*(const __nv_bfloat162*)&x.y);
        o.x = fmaf(D, x0.x, o.x); o.y = fmaf(D, x0.y, o.y); o.z = fmaf(D, x1.x, o.z); o.w = fmaf(D, x1.y, o.w);
        *(float4*)(dst + e) = o;
      } else {
        dst[w.c] = fmaf(D, __bfloat162float(sX[t * LX + w.c]), so[t * LO + w.c]);
      }
    }
  }
}

// Bytes of workspace for b200_ssd_prefill.
B200_API size_t b200_ssd_prefill_bytes(int T, int n_seqs, int H, int PP, int N, int G, int exact) {
  const int NP = (N + 15) / 16 * 16;
  if (exact) return ssd_conv_bytes(T, H, PP, G, NP, 4);
  return ssd_conv_bytes(T, H, PP, G, NP, 2) + align256(((size_t)T / GC + n_seqs + 1) * H * ((PP + 15) / 16) * 16 * NP * 4);
}

template <int NV>
static int launch_ssd_output(const SsdArgs& a, const SsdWs& w, int n_seqs, int max_q, cudaStream_t st) {
  const size_t b = (size_t)GC * 2 * (a.NP + 8), tile = (size_t)GC * 4 * (w.npt * 16 + 4);
  const size_t smem = (size_t)GC * 2 * (a.NP + 8 + 2 * (w.npt * 16 + 8) + 2 * (GC + 8)) + (b > tile ? b : tile);
  if (smem > 225 * 1024) return B200_ERR_BAD_ARG;
  static size_t configured = 0;
  if (smem > configured) {
    cudaError_t e = cudaFuncSetAttribute(ssd_output_kernel<NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = smem;
  }
  const int chunks = (max_q + GC - 1) / GC, rep = a.H / a.G;
  int HB = 1;                                // heads to a CTA: more, as long as there are some CTAs to every SM
  while (HB < 8 && rep % (2 * HB) == 0 && (long)chunks * n_seqs * a.H / (2 * HB) >= 4 * 148) HB *= 2;
  return launch_pdl(ssd_output_kernel<NV>, dim3(chunks, a.H / HB, n_seqs), dim3(256), smem, st, a, w, HB);
}

// Prompts: T rows in all, max_q = longest portion of a sequence; ws: b200_ssd_prefill_bytes bytes, 256-byte aligned.  exact: token by token in fp32.
B200_API int b200_ssd_prefill(SSD_PARAMS, int T, int max_q, int exact, void* ws, size_t ws_bytes, cudaStream_t st) {
  SsdArgs a;
  int rc = SSD_FILL;
  if (rc) return rc;
  if (T < 1 || max_q < 1 || ws_bytes < b200_ssd_prefill_bytes(T, n_seqs, H, PP, N, G, exact) || ((uintptr_t)ws % 256)) return B200_ERR_BAD_ARG;
  char* p = (char*)ws;
  if (exact) {
    const SsdConv<float> o = ssd_conv_ws<float>(a, p, T);
    rc = launch_ssd_conv(a, o, n_seqs, max_q, st);
    return rc ? rc : launch_ssd_recurrent<false>(a, o, n_seqs, st);
  }
  SsdWs w;
  w.c = ssd_conv_ws<__nv_bfloat16>(a, p, T);
  w.s = (uint4*)p;
  w.npt = (PP + 15) / 16;
  w.kn = a.NP / 16;
  rc = launch_ssd_conv(a, w.c, n_seqs, max_q, st);
  if (rc) return rc;
  const int slices = a.NP <= 64 ? 1 : (a.NP + 127) / 128, s2 = kSsdStages * GC * ((a.NP <= 64 ? 64 : 128) + 8 + 72) * 2;
  auto walk = a.NP <= 64 ? ssd_state_kernel<32> : ssd_state_kernel<64>;
  cudaError_t e = cudaFuncSetAttribute(walk, cudaFuncAttributeMaxDynamicSharedMemorySize, s2);
  if (e != cudaSuccess) return (int)e;
  rc = launch_pdl(walk, dim3((w.npt + 3) / 4 * slices, H, n_seqs), dim3(256), (size_t)s2, st, a, w);
  if (rc) return rc;
  if (w.npt <= 4) return launch_ssd_output<1>(a, w, n_seqs, max_q, st);
  if (w.npt <= 8) return launch_ssd_output<2>(a, w, n_seqs, max_q, st);
  return launch_ssd_output<4>(a, w, n_seqs, max_q, st);
}
