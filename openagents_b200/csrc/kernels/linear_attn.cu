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
  const float* a2;         // [H * dim][rank]
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
      for (int r = 0; r < a.rank; r++) z = fmaf(a.a2[(size_t)c * a.rank + r], row[a.a_off + r], z);
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
