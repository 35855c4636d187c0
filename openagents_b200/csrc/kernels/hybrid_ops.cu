// Operators of hybrid decoders (attention and recurrent layers in one stack, norms around both ends of a sublayer): the
// residual step, Dynamic Tanh, the projection finish of an attention layer, attention in exact 32-bit arithmetic for any head size, the
// difference of two attention maps, the
// 32-bit matrix product, and the last step of the logits.
//
// This file is compiled without fast math: divisions, square roots, exponentials and hyperbolic tangents are the IEEE-accurate
// ones, because what runs here is what such models are required to compute in 32-bit.
#include "common.cuh"

using namespace b200;

// ------------------------------------------------------------------ residual step

// Per row:  x += y / rms(y) * gy   (when y is given; rms over D, eps inside the root)
//           h  = x / rms(x) * gh   (gh null: h = x) -> bf16 and/or fp32 (when either is given), columns D..ldh written as zeros
// i.e. the norm behind one sublayer, the residual sum and the norm ahead of the next in one pass over the row.
// zero_a / zero_b: buffers cleared on the side; y_clear: the row of y is left zeroed.  Both serve the K-split projections,
// which add into their outputs.
constexpr int kNormRegs = 8;
__global__ void __launch_bounds__(1024) norm_residual_kernel(float* __restrict__ y, int ldy, const float* __restrict__ gy,
                                                             float* __restrict__ x, int D, const float* __restrict__ gh,
                                                             float eps, __nv_bfloat16* __restrict__ hb,
                                                             float* __restrict__ hf, int ldh, int y_clear,
                                                             float4* __restrict__ zero_a, int na4, float4* __restrict__ zero_b,
                                                             int nb4) {
  __shared__ float red[32];
  const int t = blockIdx.x, nt = blockDim.x;
  float* xr = x + (size_t)t * D;
  float v[kNormRegs], w[kNormRegs];
  pdl_trigger();
  pdl_wait();
#pragma unroll
  for (int k = 0; k < kNormRegs; k++) {
    const int i = threadIdx.x + k * nt;
    v[k] = i < D ? xr[i] : 0.f;
    w[k] = (y && i < D) ? y[(size_t)t * ldy + i] : 0.f;
  }
  for (int i = blockIdx.x * nt + threadIdx.x; i < na4; i += gridDim.x * nt) zero_a[i] = make_float4(0.f, 0.f, 0.f, 0.f);
  for (int i = blockIdx.x * nt + threadIdx.x; i < nb4; i += gridDim.x * nt) zero_b[i] = make_float4(0.f, 0.f, 0.f, 0.f);
  if (y) {
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < kNormRegs; k++) ss += w[k] * w[k];
    for (int i = threadIdx.x + kNormRegs * nt; i < D; i += nt) {
      const float e = y[(size_t)t * ldy + i];
      ss += e * e;
    }
    const float r = 1.f / sqrtf(block_sum(ss, red) / (float)D + eps);
#pragma unroll
    for (int k = 0; k < kNormRegs; k++) {
      const int i = threadIdx.x + k * nt;
      if (i < D) {
        v[k] += w[k] * r * gy[i];
        xr[i] = v[k];
      }
    }
    for (int i = threadIdx.x + kNormRegs * nt; i < D; i += nt) xr[i] += y[(size_t)t * ldy + i] * r * gy[i];
    if (y_clear)
      for (int i = threadIdx.x; i < ldy; i += nt) y[(size_t)t * ldy + i] = 0.f;
  }
  if (!hb && !hf) return;
  float r = 1.f;
  if (gh) {
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < kNormRegs; k++) ss += v[k] * v[k];
    for (int i = threadIdx.x + kNormRegs * nt; i < D; i += nt) ss += xr[i] * xr[i];
    r = 1.f / sqrtf(block_sum(ss, red) / (float)D + eps);
  }
#pragma unroll
  for (int k = 0; k < kNormRegs; k++) {
    const int i = threadIdx.x + k * nt;
    if (i < ldh) {
      const float o = i < D ? (gh ? v[k] * r * gh[i] : v[k]) : 0.f;
      if (hb) hb[(size_t)t * ldh + i] = __float2bfloat16(o);
      if (hf) hf[(size_t)t * ldh + i] = o;
    }
  }
  for (int i = threadIdx.x + kNormRegs * nt; i < ldh; i += nt) {
    const float o = i < D ? (gh ? xr[i] * r * gh[i] : xr[i]) : 0.f;
    if (hb) hb[(size_t)t * ldh + i] = __float2bfloat16(o);
    if (hf) hf[(size_t)t * ldh + i] = o;
  }
}
// The same for rows of whole float4s that fit the registers of the block (every real model's width): 16-byte accesses, and blocks
// small enough for several rows per SM.
template <int R>
__global__ void __launch_bounds__(256) norm_residual_vec_kernel(float4* __restrict__ y, int ldy4, const float4* __restrict__ gy,
                                                                float4* __restrict__ x, int D4, const float4* __restrict__ gh,
                                                                float eps, __nv_bfloat16* __restrict__ hb,
                                                                float4* __restrict__ hf, int ldh4, int y_clear,
                                                                float4* __restrict__ zero_a, int na4, float4* __restrict__ zero_b,
                                                                int nb4) {
  __shared__ float red[32];
  const int t = blockIdx.x, tid = threadIdx.x, nt = blockDim.x;
  float4* xr = x + (size_t)t * D4;
  float4* yr = y + (size_t)t * ldy4;
  const float4 z = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 v[R], w[R];
  pdl_trigger();
  pdl_wait();
#pragma unroll
  for (int k = 0; k < R; k++) {
    const int i = tid + k * nt;
    v[k] = i < D4 ? xr[i] : z;
    w[k] = (y && i < D4) ? yr[i] : z;
  }
  for (int i = blockIdx.x * nt + tid; i < na4; i += gridDim.x * nt) zero_a[i] = z;
  for (int i = blockIdx.x * nt + tid; i < nb4; i += gridDim.x * nt) zero_b[i] = z;
  const float inv_d = 1.f / (float)(4 * D4);
  if (y) {
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < R; k++) ss += w[k].x * w[k].x + w[k].y * w[k].y + w[k].z * w[k].z + w[k].w * w[k].w;
    const float r = 1.f / sqrtf(block_sum(ss, red) * inv_d + eps);
#pragma unroll
    for (int k = 0; k < R; k++) {
      const int i = tid + k * nt;
      if (i >= D4) continue;
      const float4 g = gy[i];
      v[k].x += w[k].x * r * g.x;
      v[k].y += w[k].y * r * g.y;
      v[k].z += w[k].z * r * g.z;
      v[k].w += w[k].w * r * g.w;
      xr[i] = v[k];
      if (y_clear) yr[i] = z;
    }
  }
  if (!hb && !hf) return;
  float r = 1.f;
  if (gh) {
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < R; k++) ss += v[k].x * v[k].x + v[k].y * v[k].y + v[k].z * v[k].z + v[k].w * v[k].w;
    r = 1.f / sqrtf(block_sum(ss, red) * inv_d + eps);
  }
#pragma unroll
  for (int k = 0; k < R; k++) {
    const int i = tid + k * nt;
    if (i >= ldh4) continue;           // ldh4 > D4: padding columns are zeros
    float4 o = v[k];
    if (gh) {
      const float4 g = i < D4 ? gh[i] : z;
      o = make_float4(v[k].x * r * g.x, v[k].y * r * g.y, v[k].z * r * g.z, v[k].w * r * g.w);
    }
    if (hb) {
      const __nv_bfloat162 p0 = __floats2bfloat162_rn(o.x, o.y), p1 = __floats2bfloat162_rn(o.z, o.w);
      *(uint2*)(hb + ((size_t)t * ldh4 + i) * 4) = make_uint2(*(const uint32_t*)&p0, *(const uint32_t*)&p1);
    }
    if (hf) hf[(size_t)t * ldh4 + i] = o;
  }
}

// x fp32 [T][D]; y fp32 [T][ldy] or null; gains fp32 [D]; hb / hf [T][ldh].  zero_*_n: floats, multiples of 4.
B200_API int b200_norm_residual(float* y, int ldy, const float* gy, float* x, int T, int D, const float* gh, float eps, void* hb,
                                float* hf, int ldh, int y_clear, float* zero_a, long zero_a_n, float* zero_b, long zero_b_n,
                                cudaStream_t st) {
  if (T < 1 || D < 1 || !x || (y && (!gy || ldy < D)) || (gh && !hb && !hf) || ((hb || hf) && ldh < D)) return B200_ERR_BAD_ARG;
  if ((zero_a && (zero_a_n % 4 || (uintptr_t)zero_a % 16)) || (zero_b && (zero_b_n % 4 || (uintptr_t)zero_b % 16)))
    return B200_ERR_BAD_ARG;
  const uintptr_t align = (uintptr_t)x | (uintptr_t)y | (uintptr_t)gy | (uintptr_t)gh | (uintptr_t)hb | (uintptr_t)hf;
  if (align % 16 == 0 && ((D | ldy | ldh) & 3) == 0 && max(D, ldh) <= 256 * 4 * 8 && (!y || ldy == D || !y_clear)) {
    const int n4 = max(D, ldh) / 4, nt = n4 > 512 ? 256 : n4 > 128 ? 128 : 64, R = (n4 + nt - 1) / nt;
    auto kern = R <= 1 ? norm_residual_vec_kernel<1> : R <= 2 ? norm_residual_vec_kernel<2> : R <= 4 ? norm_residual_vec_kernel<4> : norm_residual_vec_kernel<8>;
    return launch_pdl(kern, dim3(T), dim3(nt), 0, st, (float4*)y, ldy / 4, (const float4*)gy, (float4*)x, D / 4, (const float4*)gh, eps,
                      (__nv_bfloat16*)hb, (float4*)hf, ldh / 4, y_clear, (float4*)zero_a, zero_a ? (int)(zero_a_n / 4) : 0, (float4*)zero_b,
                      zero_b ? (int)(zero_b_n / 4) : 0);
  }
  const int threads = D >= 4096 ? 1024 : D >= 2048 ? 512 : D >= 512 ? 256 : 128;
  return launch_pdl(norm_residual_kernel, dim3(T), dim3(threads), 0, st, y, ldy, gy, x, D, gh, eps, (__nv_bfloat16*)hb, hf, ldh,
                    y_clear, (float4*)zero_a, zero_a ? (int)(zero_a_n / 4) : 0, (float4*)zero_b, zero_b ? (int)(zero_b_n / 4) : 0);
}

// ------------------------------------------------------------------ Dynamic Tanh

// Per row:  x += emb[ids[t]]             (when emb is given: a looped stack's next pass takes the embedding in again)
//           h  = tanh(alpha x) * w + b   -> bf16 and/or fp32, columns D..ldh written as zeros
// No statistics, so rows are only a shape.  zero: a buffer cleared on the side for a K-split projection that adds into it.
struct DytArgs {
  float* x;                  // [T][D]
  int D, ldh;
  const int* ids;
  const __nv_bfloat16* emb;  // [vocab][D] or null
  int vocab;
  const float* alpha;        // one number
  const float* w;
  const float* b;
  __nv_bfloat16* hb;
  float* hf;
  float4* zero;
  int nz4;
};
__device__ __forceinline__ float dyt_one(float x, float alpha, float w, float b) { return fmaf(tanhf(alpha * x), w, b); }

__global__ void __launch_bounds__(256) norm_dyt_kernel(const DytArgs a) {
  const int t = blockIdx.x, nt = blockDim.x * gridDim.y, i0 = blockIdx.y * blockDim.x + threadIdx.x;
  const float alpha = *a.alpha;
  pdl_trigger();
  pdl_wait();
  for (int i = (blockIdx.x * gridDim.y + blockIdx.y) * blockDim.x + threadIdx.x; i < a.nz4; i += gridDim.x * nt)
    a.zero[i] = make_float4(0.f, 0.f, 0.f, 0.f);
  float* xr = a.x + (size_t)t * a.D;
  const int id = a.emb ? a.ids[t] : 0;
  const bool add = a.emb && id >= 0 && id < a.vocab;
  for (int i = i0; i < a.ldh; i += nt) {
    float o = 0.f;
    if (i < a.D) {
      float v = xr[i];
      if (add) {
        v += __bfloat162float(a.emb[(size_t)id * a.D + i]);
        xr[i] = v;
      }
      o = dyt_one(v, alpha, a.w[i], a.b[i]);
    }
    if (a.hb) a.hb[(size_t)t * a.ldh + i] = __float2bfloat16(o);
    if (a.hf) a.hf[(size_t)t * a.ldh + i] = o;
  }
}
// The same on 16-byte accesses (widths that are multiples of 4).
__global__ void __launch_bounds__(256) norm_dyt_vec_kernel(const DytArgs a) {
  const int t = blockIdx.x, nt = blockDim.x * gridDim.y, i0 = blockIdx.y * blockDim.x + threadIdx.x;
  const int D4 = a.D >> 2, l4 = a.ldh >> 2;
  const float alpha = *a.alpha;
  pdl_trigger();
  pdl_wait();
  for (int i = (blockIdx.x * gridDim.y + blockIdx.y) * blockDim.x + threadIdx.x; i < a.nz4; i += gridDim.x * nt)
    a.zero[i] = make_float4(0.f, 0.f, 0.f, 0.f);
  float4* xr = (float4*)(a.x + (size_t)t * a.D);
  const int id = a.emb ? a.ids[t] : 0;
  const bool add = a.emb && id >= 0 && id < a.vocab;
  for (int i = i0; i < l4; i += nt) {
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < D4) {
      float4 v = xr[i];
      const float4 w = ((const float4*)a.w)[i], b = ((const float4*)a.b)[i];
      if (add) {
        const uint2 e = ((const uint2*)(a.emb + (size_t)id * a.D))[i];
        const float2 e0 = __bfloat1622float2(*(const __nv_bfloat162*)&e.x), e1 = __bfloat1622float2(*(const __nv_bfloat162*)&e.y);
        v.x += e0.x; v.y += e0.y; v.z += e1.x; v.w += e1.y;
        xr[i] = v;
      }
      o = make_float4(dyt_one(v.x, alpha, w.x, b.x), dyt_one(v.y, alpha, w.y, b.y), dyt_one(v.z, alpha, w.z, b.z), dyt_one(v.w, alpha, w.w, b.w));
    }
    if (a.hb) {
      const __nv_bfloat162 p0 = __floats2bfloat162_rn(o.x, o.y), p1 = __floats2bfloat162_rn(o.z, o.w);
      *(uint2*)(a.hb + ((size_t)t * l4 + i) * 4) = make_uint2(*(const uint32_t*)&p0, *(const uint32_t*)&p1);
    }
    if (a.hf) ((float4*)a.hf)[(size_t)t * l4 + i] = o;
  }
}
B200_API int b200_norm_dyt(float* x, int T, int D, const int* ids, const void* emb, int vocab, const float* alpha, const float* w,
                           const float* b, void* hb, float* hf, int ldh, float* zero, long zero_n, cudaStream_t st) {
  if (T < 1 || D < 1 || ldh < D || !x || !alpha || !w || !b || (!hb && !hf) || (emb && !ids)) return B200_ERR_BAD_ARG;
  if (zero && (zero_n % 4 || (uintptr_t)zero % 16)) return B200_ERR_BAD_ARG;
  DytArgs a;
  a.x = x; a.D = D; a.ldh = ldh; a.ids = ids; a.emb = (const __nv_bfloat16*)emb; a.vocab = vocab; a.alpha = alpha; a.w = w; a.b = b;
  a.hb = (__nv_bfloat16*)hb; a.hf = hf; a.zero = (float4*)zero; a.nz4 = zero ? (int)(zero_n / 4) : 0;
  const uintptr_t align = (uintptr_t)x | (uintptr_t)w | (uintptr_t)b | (uintptr_t)hb | (uintptr_t)hf | (uintptr_t)emb;
  const bool vec = align % 16 == 0 && D % 4 == 0 && ldh % 4 == 0;
  const int per = vec ? ldh / 4 : ldh, threads = per > 128 ? 256 : 128;
  // a row has no reduction, so few rows are spread over several blocks each
  int gy = 1;
  while (gy * threads < per && (long)T * gy < 2 * 148) gy++;
  return launch_pdl(vec ? norm_dyt_vec_kernel : norm_dyt_kernel, dim3(T, gy), dim3(threads), 0, st, a);
}

// ------------------------------------------------------------------ depth average and the norms behind it

// Per row:  x = sum over j < n of w[j] * X_j   (X_j: row t of xs + j * stride; the embedding output and every layer's result so far)
//           out = x + add                     (the next layer adds its results to this row: `add` is a bias they carry, or null)
//           h1 = x / rms(x) * g1, h2 = x / rms(x) * g2   (two norms of the same x; each given or not; bf16 or fp32)
//           part_k = sum over j < n of pw[k][j] * X_j    (k < parts: what later layers will want of the same X_j, read once for all of them)
// base (or null): a row added to x as it is, such a partial sum from an earlier call.
// Rows are ld floats apart in xs, out and h, D of them live; the others are written as zeros.  zero: a buffer cleared on the side.
struct DepthArgs {
  const float* xs;
  size_t stride;
  const float* w;          // [n] or null (n = 1: x = X_0)
  int n, D, ld;
  float* out;              // or null
  const float* add;        // [D] or null
  const float* g1;         // [D] or null
  const float* g2;
  float eps;
  __nv_bfloat16* hb1;
  __nv_bfloat16* hb2;
  float* hf1;
  float* hf2;
  float4* zero;
  int nz4;
  const float* base;       // [T][ld] or null
  float* part;             // parts slabs of `stride` floats
  const float* pw;         // [parts][ldw]
  int parts, ldw;
};
constexpr int kDepthParts = 3;
__global__ void __launch_bounds__(256) depth_norm_kernel(const DepthArgs a) {
  extern __shared__ float depth_row[];               // [D]
  __shared__ float red[32];
  const int t = blockIdx.x, tid = threadIdx.x, nt = blockDim.x;
  pdl_trigger();
  pdl_wait();
  for (int i = blockIdx.x * nt + tid; i < a.nz4; i += gridDim.x * nt) a.zero[i] = make_float4(0.f, 0.f, 0.f, 0.f);
  const size_t at = (size_t)t * a.ld;
  float ss = 0.f;
  for (int i = tid; i < a.ld; i += nt) {
    float v = 0.f;
    float p[kDepthParts] = {};
    if (i < a.D) {
      const float* x = a.xs + at + i;
      if (a.base) v = a.base[at + i];
      if (!a.w) v += *x;
      else
        for (int j = 0; j < a.n; j++) {
          const float e = x[j * a.stride];
          v = fmaf(a.w[j], e, v);
#pragma unroll
          for (int k = 0; k < kDepthParts; k++)
            if (k < a.parts) p[k] = fmaf(a.pw[k * a.ldw + j], e, p[k]);
        }
      depth_row[i] = v;
      ss += v * v;
    }
#pragma unroll
    for (int k = 0; k < kDepthParts; k++)
      if (k < a.parts) a.part[k * a.stride + at + i] = p[k];
    if (a.out) a.out[at + i] = i < a.D && a.add ? v + a.add[i] : v;
  }
  if (!a.g1 && !a.g2) return;
  const float r = 1.f / sqrtf(block_sum(ss, red) / (float)a.D + a.eps);
  for (int i = tid; i < a.ld; i += nt) {               // every thread meets the elements it wrote
    const float v = i < a.D ? depth_row[i] * r : 0.f;
    if (a.g1) {
      const float o = i < a.D ? v * a.g1[i] : 0.f;
      if (a.hb1) a.hb1[at + i] = __float2bfloat16(o);
      if (a.hf1) a.hf1[at + i] = o;
    }
    if (a.g2) {
      const float o = i < a.D ? v * a.g2[i] : 0.f;
      if (a.hb2) a.hb2[at + i] = __float2bfloat16(o);
      if (a.hf2) a.hf2[at + i] = o;
    }
  }
}
// The same on 16-byte accesses with the row in registers (widths that are multiples of 4).  PARTS: whether there are partial sums to make.
__device__ __forceinline__ void fma4(float4& v, float w, const float4& e) {
  v.x = fmaf(w, e.x, v.x);
  v.y = fmaf(w, e.y, v.y);
  v.z = fmaf(w, e.z, v.z);
  v.w = fmaf(w, e.w, v.w);
}
template <int R, bool PARTS>
__global__ void __launch_bounds__(256) depth_norm_vec_kernel(const DepthArgs a) {
  __shared__ float red[32];
  const int t = blockIdx.x, tid = threadIdx.x, nt = blockDim.x, D4 = a.D >> 2, l4 = a.ld >> 2;
  const float4 z = make_float4(0.f, 0.f, 0.f, 0.f);
  pdl_trigger();
  pdl_wait();
  for (int i = blockIdx.x * nt + tid; i < a.nz4; i += gridDim.x * nt) a.zero[i] = z;
  const size_t at = (size_t)t * l4;
  float4 v[R], p[PARTS ? kDepthParts : 1][R];
#pragma unroll
  for (int k = 0; k < R; k++) v[k] = a.base && tid + k * nt < D4 ? ((const float4*)a.base)[at + tid + k * nt] : z;
  if constexpr (PARTS) {
#pragma unroll
    for (int m = 0; m < kDepthParts; m++)
#pragma unroll
      for (int k = 0; k < R; k++) p[m][k] = z;
  }
  const float4* x = (const float4*)a.xs + at;
  const size_t s4 = a.stride >> 2;
  if (!a.w) {
#pragma unroll
    for (int k = 0; k < R; k++)
      if (tid + k * nt < D4) fma4(v[k], 1.f, x[tid + k * nt]);
  } else {
    constexpr int U = R >= 8 ? 1 : R >= 4 ? 2 : 8 / R;            // layers in flight
    for (int j0 = 0; j0 < a.n; j0 += U) {
      float4 e[U][R];
      float w[U], pw[PARTS ? kDepthParts : 1][U];
#pragma unroll
      for (int u = 0; u < U; u++) {
        w[u] = j0 + u < a.n ? a.w[j0 + u] : 0.f;
        if constexpr (PARTS) {
#pragma unroll
          for (int m = 0; m < kDepthParts; m++) pw[m][u] = m < a.parts && j0 + u < a.n ? a.pw[m * a.ldw + j0 + u] : 0.f;
        }
#pragma unroll
        for (int k = 0; k < R; k++) e[u][k] = j0 + u < a.n && tid + k * nt < D4 ? x[(j0 + u) * s4 + tid + k * nt] : z;
      }
#pragma unroll
      for (int u = 0; u < U; u++)
#pragma unroll
        for (int k = 0; k < R; k++) {
          fma4(v[k], w[u], e[u][k]);
          if constexpr (PARTS) {
#pragma unroll
            for (int m = 0; m < kDepthParts; m++) fma4(p[m][k], pw[m][u], e[u][k]);
          }
        }
    }
  }
  if constexpr (PARTS) {
#pragma unroll
    for (int m = 0; m < kDepthParts; m++)
#pragma unroll
      for (int k = 0; k < R; k++)
        if (m < a.parts && tid + k * nt < l4) ((float4*)a.part)[m * s4 + at + tid + k * nt] = p[m][k];
  }
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < R; k++) {
    const int i = tid + k * nt;
    ss += v[k].x * v[k].x + v[k].y * v[k].y + v[k].z * v[k].z + v[k].w * v[k].w;
    if (a.out && i < l4) {
      const float4 b = a.add && i < D4 ? ((const float4*)a.add)[i] : z;
      ((float4*)a.out)[at + i] = make_float4(v[k].x + b.x, v[k].y + b.y, v[k].z + b.z, v[k].w + b.w);
    }
  }
  if (!a.g1 && !a.g2) return;
  const float r = 1.f / sqrtf(block_sum(ss, red) / (float)a.D + a.eps);
  auto put = [&](const float* g, __nv_bfloat16* hb, float* hf) {
#pragma unroll
    for (int k = 0; k < R; k++) {
      const int i = tid + k * nt;
      if (i >= l4) continue;
      const float4 w = i < D4 ? ((const float4*)g)[i] : z;
      const float4 o = make_float4(v[k].x * r * w.x, v[k].y * r * w.y, v[k].z * r * w.z, v[k].w * r * w.w);
      if (hb) {
        const __nv_bfloat162 p0 = __floats2bfloat162_rn(o.x, o.y), p1 = __floats2bfloat162_rn(o.z, o.w);
        *(uint2*)(hb + (at + i) * 4) = make_uint2(*(const uint32_t*)&p0, *(const uint32_t*)&p1);
      }
      if (hf) ((float4*)hf)[at + i] = o;
    }
  };
  if (a.g1) put(a.g1, a.hb1, a.hf1);
  if (a.g2) put(a.g2, a.hb2, a.hf2);
}
// xs fp32: n slabs `stride` floats apart, rows ld apart.  Outputs share ld; part: `parts` (at most 3) slabs as far apart.
B200_API int b200_depth_norm(const float* xs, size_t stride, const float* w, int n, int T, int D, int ld, float* out, const float* add,
                             const float* g1, const float* g2, float eps, void* hb1, void* hb2, float* hf1, float* hf2, float* zero,
                             long zero_n, const float* base, float* part, const float* pw, int parts, int ldw, cudaStream_t st) {
  if (parts < 0 || parts > kDepthParts || (parts && (!part || !pw || !w || ldw < n))) return B200_ERR_BAD_ARG;
  if (T < 1 || D < 1 || ld < D || n < 1 || !xs || (!w && n != 1) || (g1 && !hb1 && !hf1) || (g2 && !hb2 && !hf2)) return B200_ERR_BAD_ARG;
  if (zero && (zero_n % 4 || (uintptr_t)zero % 16)) return B200_ERR_BAD_ARG;
  DepthArgs a;
  a.xs = xs; a.stride = stride; a.w = w; a.n = n; a.D = D; a.ld = ld; a.out = out; a.add = add; a.g1 = g1; a.g2 = g2; a.eps = eps;
  a.hb1 = (__nv_bfloat16*)hb1; a.hb2 = (__nv_bfloat16*)hb2; a.hf1 = hf1; a.hf2 = hf2; a.zero = (float4*)zero; a.nz4 = zero ? (int)(zero_n / 4) : 0;
  a.base = base; a.part = part; a.pw = pw; a.parts = parts; a.ldw = ldw;
  const uintptr_t align = (uintptr_t)xs | (uintptr_t)out | (uintptr_t)add | (uintptr_t)g1 | (uintptr_t)g2 | (uintptr_t)hb1 | (uintptr_t)hb2 |
                          (uintptr_t)hf1 | (uintptr_t)hf2 | (uintptr_t)base | (uintptr_t)part;
  if (align % 16 == 0 && D % 4 == 0 && ld % 4 == 0 && stride % 4 == 0 && ld <= 256 * 4 * 8) {
    const int n4 = ld / 4, nt = n4 > 128 ? 256 : n4 > 64 ? 128 : 64, R = (n4 + nt - 1) / nt;
    auto kern = R <= 1 ? depth_norm_vec_kernel<1, false> : R <= 2 ? depth_norm_vec_kernel<2, false> : R <= 4 ? depth_norm_vec_kernel<4, false> : depth_norm_vec_kernel<8, false>;
    if (parts)
      kern = R <= 1 ? depth_norm_vec_kernel<1, true> : R <= 2 ? depth_norm_vec_kernel<2, true> : R <= 4 ? depth_norm_vec_kernel<4, true> : depth_norm_vec_kernel<8, true>;
    return launch_pdl(kern, dim3(T), dim3(nt), 0, st, a);
  }
  const size_t smem = (size_t)D * 4;
  if (smem > 200 * 1024) return B200_ERR_BAD_ARG;
  static size_t configured = 48 * 1024;
  if (smem > configured) {
    cudaError_t e = cudaFuncSetAttribute(depth_norm_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = smem;
  }
  return launch_pdl(depth_norm_kernel, dim3(T), dim3(256), smem, st, a);
}

// ------------------------------------------------------------------ PolyNorm

// Per row of F values z:  a N(z) + b N(z^2) + c N(z^3) + e, N dividing a row by its root mean square (powers element by element), with
// coef = (a, b, c, e).  in fp32 or bf16 [T][ldi]; out bf16 or fp32 [T][ldo], columns F..ldo zero.
constexpr int kPolyRegs = 8;
__device__ __forceinline__ float4 get4(const float* p, int i) { return ((const float4*)p)[i]; }
__device__ __forceinline__ float4 get4(const __nv_bfloat16* p, int i) {
  const uint2 v = ((const uint2*)p)[i];
  const float2 x = __bfloat1622float2(*(const __nv_bfloat162*)&v.x), y = __bfloat1622float2(*(const __nv_bfloat162*)&v.y);
  return make_float4(x.x, x.y, y.x, y.y);
}
__device__ __forceinline__ float get1(const float* p, int i) { return p[i]; }
__device__ __forceinline__ float get1(const __nv_bfloat16* p, int i) { return __bfloat162float(p[i]); }

template <typename IT>
__global__ void __launch_bounds__(512) poly_norm_kernel(const IT* __restrict__ in, int ldi, int F, const float* __restrict__ coef, float eps,
                                                        __nv_bfloat16* __restrict__ ob, float* __restrict__ of, int ldo, int vec) {
  __shared__ float red[3][32];
  const int t = blockIdx.x, tid = threadIdx.x, nt = blockDim.x;
  const float ca = coef[0], cb = coef[1], cc = coef[2], ce = coef[3];
  pdl_trigger();
  pdl_wait();
  const IT* zr = in + (size_t)t * ldi;
  const int F4 = F >> 2;
  float s2 = 0.f, s4 = 0.f, s6 = 0.f;
  auto stat = [&](float z) {
    const float z2 = z * z;
    s2 += z2;
    s4 = fmaf(z2, z2, s4);
    s6 = fmaf(z2 * z2, z2, s6);
  };
  float4 v[kPolyRegs];                                  // vec: the first part of the row stays in registers
  if (vec) {
#pragma unroll
    for (int k = 0; k < kPolyRegs; k++) {
      const int i = tid + k * nt;
      v[k] = i < F4 ? get4(zr, i) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int k = 0; k < kPolyRegs; k++) { stat(v[k].x); stat(v[k].y); stat(v[k].z); stat(v[k].w); }
    for (int i = tid + kPolyRegs * nt; i < F4; i += nt) {
      const float4 e = get4(zr, i);
      stat(e.x); stat(e.y); stat(e.z); stat(e.w);
    }
  } else {
    for (int i = tid; i < F; i += nt) stat(get1(zr, i));
  }
  const int lane = tid & 31, w = tid >> 5, nw = nt >> 5;
  s2 = warp_sum(s2); s4 = warp_sum(s4); s6 = warp_sum(s6);
  if (lane == 0) { red[0][w] = s2; red[1][w] = s4; red[2][w] = s6; }
  __syncthreads();
  s2 = warp_sum(lane < nw ? red[0][lane] : 0.f);
  s4 = warp_sum(lane < nw ? red[1][lane] : 0.f);
  s6 = warp_sum(lane < nw ? red[2][lane] : 0.f);
  const float a1 = ca / sqrtf(s2 / (float)F + eps), a2 = cb / sqrtf(s4 / (float)F + eps), a3 = cc / sqrtf(s6 / (float)F + eps);
  auto f = [&](float z) { return fmaf(z, fmaf(z, fmaf(z, a3, a2), a1), ce); };
  if (vec) {
    auto store = [&](int i, float4 z) {
      const float4 o = make_float4(f(z.x), f(z.y), f(z.z), f(z.w));
      if (ob) {
        const __nv_bfloat162 p0 = __floats2bfloat162_rn(o.x, o.y), p1 = __floats2bfloat162_rn(o.z, o.w);
        *(uint2*)(ob + (size_t)t * ldo + 4 * i) = make_uint2(*(const uint32_t*)&p0, *(const uint32_t*)&p1);
      }
      if (of) *(float4*)(of + (size_t)t * ldo + 4 * i) = o;
    };
#pragma unroll
    for (int k = 0; k < kPolyRegs; k++)
      if (tid + k * nt < F4) store(tid + k * nt, v[k]);
    for (int i = tid + kPolyRegs * nt; i < F4; i += nt) store(i, get4(zr, i));
  }
  for (int i = (vec ? F : 0) + tid; i < ldo; i += nt) {
    const float o = i < F ? f(get1(zr, i)) : 0.f;
    if (ob) ob[(size_t)t * ldo + i] = __float2bfloat16(o);
    if (of) of[(size_t)t * ldo + i] = o;
  }
}
B200_API int b200_poly_norm(const void* in, int in_bf16, int ldi, int T, int F, const float* coef, float eps, void* ob, float* of, int ldo,
                            cudaStream_t st) {
  if (T < 1 || F < 1 || ldi < F || ldo < F || !in || !coef || (!ob && !of) || of == in || ob == in) return B200_ERR_BAD_ARG;
  const int vec = F % 4 == 0 && ldi % 4 == 0 && ldo % 4 == 0 && (((uintptr_t)in | (uintptr_t)ob | (uintptr_t)of) & 15) == 0;
  const int threads = F >= 4096 ? 512 : F >= 1024 ? 256 : 128;
  if (in_bf16)
    return launch_pdl(poly_norm_kernel<__nv_bfloat16>, dim3(T), dim3(threads), 0, st, (const __nv_bfloat16*)in, ldi, F, coef, eps, (__nv_bfloat16*)ob, of, ldo, vec);
  return launch_pdl(poly_norm_kernel<float>, dim3(T), dim3(threads), 0, st, (const float*)in, ldi, F, coef, eps, (__nv_bfloat16*)ob, of, ldo, vec);
}

// ------------------------------------------------------------------ attention: finish of the projections

// One warp per (token, head) of a fused projection row: queries and keys are rotated on their first `rot` dimensions, then
// (qk_norm) divided by their root mean square over the head; queries are scaled, keys and values go to the paged cache.
//   style 0: dimension 2i turns with 2i + 1; style 1: i with i + rot / 2.
// Cache and query rows are padded to DK / DV columns; the padding is written as zeros.
// maps = 2 (differential attention): a key/value head has two key rows side by side ([map 1, map 2], DK columns each) and H counts
// the query rows of both maps, in the order (key/value head, map, query head of the group).  q_wide: a query row is as wide as
// both key rows and zero on the other map's half, so that one product with them gives its own map's scores.
struct QkvArgs {
  const float* in;         // [T][ld]
  int ld, q_off, k_off, v_off;     // k_off < 0: the layer has no keys and values of its own; v_off < 0: its values are its keys
  const int* pos;
  const int* slot;         // physical cache slot (page * page_size + offset); < 0: no cache write
  const float2* tab;       // [tab_len][rot / 2] (cos, sin)
  int tab_len;
  double base;
  int H, G, dim, vdim, DK, DV, rot, style, qk_norm, page_size;
  float eps, q_scale;
  float* q32;              // [T][H][DK or maps * DK] or null
  __half* q16;             // [T][H][DK] or null
  int maps, q_wide;
  const float* bias;       // added to the row's columns, or null
};
constexpr int kQkvPairs = 8;      // pairs per lane: head sizes up to 512

__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(__half* p, float v) { *p = __float2half(v); }

template <typename CT>
__global__ void __launch_bounds__(128) qkv_finish_kernel(const QkvArgs a, CT* __restrict__ kc, CT* __restrict__ vc) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, lane = threadIdx.x & 31;
  const int KR = a.G * a.maps;                            // key rows
  const int n_heads = a.H + (a.k_off >= 0 ? KR + (a.v_off >= 0 ? a.G : 0) : 0);
  const int hh = blockIdx.y * 4 + (threadIdx.x >> 5);
  if (hh >= n_heads) return;
  const int s = a.slot[t];
  const int page = s >= 0 ? s / a.page_size : 0, off = s >= 0 ? s % a.page_size : 0;
  const float* row = a.in + (size_t)t * a.ld;
  if (hh >= a.H + KR) {                                   // a value head
    if (s < 0) return;
    const int g = hh - a.H - KR;
    CT* dst = vc + (((size_t)page * a.G + g) * a.page_size + off) * a.DV;
    for (int e = lane; e < a.DV; e += 32) {
      const int c = a.v_off + g * a.vdim + e;
      put(dst + e, e < a.vdim ? row[c] + (a.bias ? a.bias[c] : 0.f) : 0.f);
    }
    return;
  }
  const bool is_q = hh < a.H;
  const int col = is_q ? a.q_off + hh * a.dim : a.k_off + (hh - a.H) * a.dim;
  const float* in = row + col;
  const float* bs = a.bias ? a.bias + col : nullptr;
  const int half = a.rot >> 1, n_pairs = (a.DK + 1) >> 1;
  const int p = a.pos[t];
  float u[kQkvPairs], w[kQkvPairs];
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < kQkvPairs; k++) {
    const int j = lane + 32 * k;
    u[k] = w[k] = 0.f;
    if (j < n_pairs) {
      const int i0 = (j < half && a.style == 1) ? j : 2 * j;
      const int i1 = (j < half && a.style == 1) ? j + half : 2 * j + 1;
      float x0 = i0 < a.dim ? in[i0] : 0.f, x1 = i1 < a.dim ? in[i1] : 0.f;
      if (bs) {
        if (i0 < a.dim) x0 += bs[i0];
        if (i1 < a.dim) x1 += bs[i1];
      }
      if (j < half) {
        float cs, sn;
        if (a.tab && p >= 0 && p < a.tab_len) {
          const float2 e = a.tab[(size_t)p * half + j];
          cs = e.x;
          sn = e.y;
        } else {
          double snd, csd;
          sincos((double)p * exp2(-2.0 * (double)j / (double)a.rot * log2(a.base)), &snd, &csd);
          cs = (float)csd;
          sn = (float)snd;
        }
        const float r0 = x0 * cs - x1 * sn, r1 = x1 * cs + x0 * sn;
        x0 = r0;
        x1 = r1;
      }
      u[k] = x0;
      w[k] = x1;
      ss += x0 * x0 + x1 * x1;
    }
  }
  float m = is_q ? a.q_scale : 1.f;
  if (a.qk_norm) m *= 1.f / sqrtf(warp_sum(ss) / (float)a.dim + a.eps);
  const int kr = hh - a.H, map = is_q ? hh / (a.H / KR) % a.maps : kr % a.maps;
  const int qw = a.q_wide ? a.maps * a.DK : a.DK;
  size_t q_at = ((size_t)t * a.H + hh) * qw;
  if (is_q && a.q_wide && a.q32)                          // the halves of the other maps
    for (int e = lane; e < qw; e += 32)
      if (e / a.DK != map) a.q32[q_at + e] = 0.f;
  if (a.q_wide) q_at += map * a.DK;
  CT* kd = is_q ? nullptr : kc + ((((size_t)page * a.G + kr / a.maps) * a.page_size + off) * a.maps + map) * a.DK;
  if (!is_q && s < 0) return;
#pragma unroll
  for (int k = 0; k < kQkvPairs; k++) {
    const int j = lane + 32 * k;
    if (j >= n_pairs) continue;
    const int i0 = (j < half && a.style == 1) ? j : 2 * j;
    const int i1 = (j < half && a.style == 1) ? j + half : 2 * j + 1;
    const float r0 = u[k] * m, r1 = w[k] * m;
    if (is_q) {
      if (a.q32) {
        a.q32[q_at + i0] = r0;
        if (i1 < a.DK) a.q32[q_at + i1] = r1;
      }
      if (a.q16) {
        a.q16[q_at + i0] = __float2half(r0);
        if (i1 < a.DK) a.q16[q_at + i1] = __float2half(r1);
      }
    } else {
      put(kd + i0, r0);
      if (i1 < a.DK) put(kd + i1, r1);
    }
  }
}
// The same where nothing rotates and nothing is normed: a thread takes four columns of one output row (head sizes and offsets that are multiples of 4).
__device__ __forceinline__ void put4(float* p, float4 v) { *(float4*)p = v; }
__device__ __forceinline__ void put4(__half* p, float4 v) {
  const __half2 a = __floats2half2_rn(v.x, v.y), b = __floats2half2_rn(v.z, v.w);
  *(uint2*)p = make_uint2(*(const uint32_t*)&a, *(const uint32_t*)&b);
}
template <typename CT>
__global__ void __launch_bounds__(256) qkv_copy_kernel(const QkvArgs a, CT* __restrict__ kc, CT* __restrict__ vc) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, i = blockIdx.y * 256 + threadIdx.x;
  const int KR = a.G * a.maps, qw = a.q_wide ? a.maps * a.DK : a.DK, q4 = qw >> 2, k4 = a.DK >> 2, v4 = a.DV >> 2;
  const int nq = a.H * q4, nk = a.k_off >= 0 ? KR * k4 : 0, nv = a.k_off >= 0 && a.v_off >= 0 ? a.G * v4 : 0;
  if (i >= nq + nk + nv) return;
  const float* row = a.in + (size_t)t * a.ld;
  int hh, c, col;
  bool in;                                                // within the head's own columns (else padding, or the other map's half)
  if (i < nq) {
    hh = i / q4;
    c = (i - hh * q4) << 2;
    const int cc = a.q_wide ? c - hh / (a.H / KR) % a.maps * a.DK : c;
    in = cc >= 0 && cc < a.dim;
    col = a.q_off + hh * a.dim + cc;
  } else if (i < nq + nk) {
    hh = (i - nq) / k4;
    c = (i - nq - hh * k4) << 2;
    in = c < a.dim;
    col = a.k_off + hh * a.dim + c;
  } else {
    hh = (i - nq - nk) / v4;
    c = (i - nq - nk - hh * v4) << 2;
    in = c < a.vdim;
    col = a.v_off + hh * a.vdim + c;
  }
  float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
  if (in) {
    v = *(const float4*)(row + col);
    if (a.bias) {
      const float4 b = *(const float4*)(a.bias + col);
      v.x += b.x; v.y += b.y; v.z += b.z; v.w += b.w;
    }
  }
  if (i < nq) {
    v.x *= a.q_scale; v.y *= a.q_scale; v.z *= a.q_scale; v.w *= a.q_scale;
    const size_t at = ((size_t)t * a.H + hh) * qw + c;
    if (a.q32) put4(a.q32 + at, v);
    if (a.q16) put4(a.q16 + at, v);
    return;
  }
  const int s = a.slot[t];
  if (s < 0) return;
  const int page = s / a.page_size, off = s % a.page_size;
  if (i < nq + nk) put4(kc + ((((size_t)page * a.G + hh / a.maps) * a.page_size + off) * a.maps + hh % a.maps) * a.DK + c, v);
  else put4(vc + (((size_t)page * a.G + hh) * a.page_size + off) * a.DV + c, v);
}
// cache_f32: kc / vc hold fp32 instead of fp16; layout [page][G][page_size][maps * DK or DV].
B200_API int b200_qkv_finish(const float* in, int ld, int T, int q_off, int k_off, int v_off, const int* pos, const int* slot,
                             const void* tab, int tab_len, double base, int H, int G, int dim, int vdim, int DK, int DV, int rot,
                             int style, int qk_norm, float eps, float q_scale, int page_size, float* q32, void* q16, void* kc,
                             void* vc, int cache_f32, int maps, int q_wide, const float* bias, cudaStream_t st) {
  if (T < 1 || H < 1 || G < 1 || dim < 1 || vdim < 1 || dim > DK || vdim > DV || DK > 64 * kQkvPairs || (rot & 1) || rot > dim || rot < 0)
    return B200_ERR_BAD_ARG;
  if ((k_off >= 0 && (!kc || (v_off >= 0 && !vc))) || (!q32 && !q16) || page_size < 1) return B200_ERR_BAD_ARG;
  if (maps < 1 || H % (G * maps) || (q_wide && q16)) return B200_ERR_BAD_ARG;
  QkvArgs a;
  a.in = in; a.ld = ld; a.q_off = q_off; a.k_off = k_off; a.v_off = v_off; a.pos = pos; a.slot = slot; a.tab = (const float2*)tab;
  a.tab_len = tab ? tab_len : 0; a.base = base; a.H = H; a.G = G; a.dim = dim; a.vdim = vdim; a.DK = DK; a.DV = DV; a.rot = rot;
  a.style = style; a.qk_norm = qk_norm; a.page_size = page_size; a.eps = eps; a.q_scale = q_scale; a.q32 = q32; a.q16 = (__half*)q16;
  a.maps = maps; a.q_wide = q_wide; a.bias = bias;
  if (rot == 0 && !qk_norm && ((ld | q_off | dim | vdim | DK | DV) & 3) == 0 && (k_off < 0 || ((k_off | max(v_off, 0)) & 3) == 0) &&
      (((uintptr_t)in | (uintptr_t)bias | (uintptr_t)q32 | (uintptr_t)q16 | (uintptr_t)kc | (uintptr_t)vc) & 15) == 0) {
    const int quads = (H * (q_wide ? maps : 1) * DK + (k_off >= 0 ? G * (maps * DK + (v_off >= 0 ? DV : 0)) : 0)) / 4;
    const dim3 g(T, (quads + 255) / 256);
    if (cache_f32) return launch_pdl(qkv_copy_kernel<float>, g, dim3(256), 0, st, a, (float*)kc, (float*)vc);
    return launch_pdl(qkv_copy_kernel<__half>, g, dim3(256), 0, st, a, (__half*)kc, (__half*)vc);
  }
  const int n_heads = H + (k_off >= 0 ? (maps + (v_off >= 0)) * G : 0);
  const dim3 grid(T, (n_heads + 3) / 4);
  if (cache_f32) return launch_pdl(qkv_finish_kernel<float>, grid, dim3(128), 0, st, a, (float*)kc, (float*)vc);
  return launch_pdl(qkv_finish_kernel<__half>, grid, dim3(128), 0, st, a, (__half*)kc, (__half*)vc);
}

// ------------------------------------------------------------------ attention: finish of projections that are normed as whole rows

// One CTA per token: q and k are each divided by the root mean square of the WHOLE projection row (all heads together) and multiplied by a weight per column
// (q_w / k_w; null: left alone), then rotated on the first `rot` dimensions of every head with the (cos, sin) table (style as in qkv_finish); queries
// are scaled.  Values (v_norm) are divided by their root mean square per head, then (lam) mixed with the first mixing layer's values of the same token:
// v <- (1 - lam) v + lam v_first; without lam but with v_first they are written there.  Keys and values go to the paged cache, padding zero.
struct RowQkvArgs {
  const float* in;         // [T][ld]
  int ld, q_off, k_off, v_off;
  const float* q_w;        // [H * dim] or null
  const float* k_w;        // [G * dim] or null
  const int* pos;
  const int* slot;
  const float2* tab;       // [tab_len][rot / 2]
  int tab_len;
  int H, G, dim, vdim, DK, DV, rot, style, page_size, v_norm;
  float eps, q_scale;
  const float* lam;        // one number or null
  float* v_first;          // [T][G * vdim] or null
  float* q32;              // [T][H][DK] or null
  __half* q16;             // [T][H][DK] or null
};
template <typename CT, bool VEC>
__global__ void __launch_bounds__(512) row_qkv_finish_kernel(const RowQkvArgs a, CT* __restrict__ kc, CT* __restrict__ vc) {
  extern __shared__ __align__(16) float row_s[];           // q row | k row
  __shared__ float red[2][16];
  pdl_trigger();
  if (VEC && blockIdx.x < 8 && threadIdx.x < 2) {          // the weights, needed behind the sums, into L2 now
    const float* w = threadIdx.x ? a.k_w : a.q_w;
    if (w) prefetch_l2(w, (threadIdx.x ? a.G : a.H) * a.dim * 4);
  }
  pdl_wait();
  const int t = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nt = blockDim.x, nw = nt >> 5;
  const float* row = a.in + (size_t)t * a.ld;
  const int nq = a.H * a.dim, nk = a.G * a.dim, s = a.slot[t], p = a.pos[t];
  const int page = s >= 0 ? s / a.page_size : 0, off = s >= 0 ? s % a.page_size : 0;
  float sq = 0.f, sk = 0.f;
  if constexpr (VEC) {
    auto sum = [](float4 v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; };
#pragma unroll 4
    for (int i = tid; i < nq / 4; i += nt) {
      const float4 v = *(const float4*)(row + a.q_off + 4 * i);
      *(float4*)(row_s + 4 * i) = v;
      sq += sum(v);
    }
    for (int i = tid; i < nk / 4; i += nt) {
      const float4 v = *(const float4*)(row + a.k_off + 4 * i);
      *(float4*)(row_s + nq + 4 * i) = v;
      sk += sum(v);
    }
  } else {
    for (int i = tid; i < nq; i += nt) {
      const float v = row[a.q_off + i];
      row_s[i] = v;
      sq += v * v;
    }
    for (int i = tid; i < nk; i += nt) {
      const float v = row[a.k_off + i];
      row_s[nq + i] = v;
      sk += v * v;
    }
  }
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if (lane == 0) { red[0][warp] = sq; red[1][warp] = sk; }
  const float lam = a.lam ? *a.lam : 0.f;
  for (int g = warp; g < a.G; g += nw) {                    // a warp per value head
    const float* v = row + a.v_off + g * a.vdim;
    float ss = 0.f;
    if (a.v_norm)
      for (int e = lane; e < a.vdim; e += 32) ss += v[e] * v[e];
    const float r = a.v_norm ? 1.f / sqrtf(warp_sum(ss) / (float)a.vdim + a.eps) : 1.f;
    float* first = a.v_first ? a.v_first + ((size_t)t * a.G + g) * a.vdim : nullptr;
    CT* dst = vc + (((size_t)page * a.G + g) * a.page_size + off) * a.DV;
    for (int e = lane; e < a.DV; e += 32) {
      float x = 0.f;
      if (e < a.vdim) {
        x = v[e] * r;
        if (a.lam) x = (1.f - lam) * x + lam * first[e];
        else if (first) first[e] = x;
      }
      if (s >= 0) put(dst + e, x);
    }
  }
  __syncthreads();
  sq = sk = 0.f;
  for (int i = 0; i < nw; i++) { sq += red[0][i]; sk += red[1][i]; }
  const float rq = a.q_w ? 1.f / sqrtf(sq / (float)nq + a.eps) : 1.f, rk = a.k_w ? 1.f / sqrtf(sk / (float)nk + a.eps) : 1.f;
  const int half = a.rot >> 1;
  const float2* cs = a.tab + (size_t)min(max(p, 0), a.tab_len - 1) * half;
  if constexpr (VEC) {                                     // four columns of a head, and the four they turn with
    const int skip = a.style == 1 ? half : 0, units = (a.DK - skip) >> 2;
    for (int i = tid; i < (a.H + a.G) * units; i += nt) {
      const int hh = i / units, u = i - hh * units;
      const bool is_q = hh < a.H;
      if (!is_q && s < 0) continue;
      const int c = 4 * u < half || a.style == 0 ? 4 * u : 4 * u + skip;
      const float* src = row_s + hh * a.dim;               // the k row follows the q row
      const float* w = is_q ? a.q_w ? a.q_w + hh * a.dim : nullptr : a.k_w ? a.k_w + (hh - a.H) * a.dim : nullptr;
      const float r = is_q ? rq : rk, m = is_q ? a.q_scale : 1.f;
      auto get = [&](int at) {
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (at < a.dim) {
          v = *(const float4*)(src + at);
          if (w) {
            const float4 g = __ldg((const float4*)(w + at));
            v = make_float4(v.x * r * g.x, v.y * r * g.y, v.z * r * g.z, v.w * r * g.w);
          }
        }
        return v;
      };
      auto store = [&](int at, float4 v) {
        v.x *= m; v.y *= m; v.z *= m; v.w *= m;
        if (is_q) {
          const size_t o = ((size_t)t * a.H + hh) * a.DK + at;
          if (a.q32) put4(a.q32 + o, v);
          if (a.q16) put4(a.q16 + o, v);
        } else {
          put4(kc + (((size_t)page * a.G + hh - a.H) * a.page_size + off) * a.DK + at, v);
        }
      };
      float4 x = get(c);
      if (a.style == 1 && c < half) {
        float4 y = get(c + half);
        const float4 e0 = __ldg((const float4*)(cs + c)), e1 = __ldg((const float4*)(cs + c + 2));
        const float4 x1 = make_float4(x.x * e0.x - y.x * e0.y, x.y * e0.z - y.y * e0.w, x.z * e1.x - y.z * e1.y, x.w * e1.z - y.w * e1.w);
        y = make_float4(y.x * e0.x + x.x * e0.y, y.y * e0.z + x.y * e0.w, y.z * e1.x + x.z * e1.y, y.w * e1.z + x.w * e1.w);
        store(c, x1);
        store(c + half, y);
        continue;
      }
      if (a.style == 0 && c < a.rot) {
        const float4 e = __ldg((const float4*)(cs + c / 2));
        x = make_float4(x.x * e.x - x.y * e.y, x.y * e.x + x.x * e.y, x.z * e.z - x.w * e.w, x.w * e.z + x.z * e.w);
      }
      store(c, x);
    }
  } else {
    const int pairs = (a.DK + 1) >> 1;
    for (int i = tid; i < (a.H + a.G) * pairs; i += nt) {
      const int hh = i / pairs, j = i - hh * pairs;
      const bool is_q = hh < a.H;
      if (!is_q && s < 0) continue;
      const int i0 = j < half && a.style == 1 ? j : 2 * j, i1 = j < half && a.style == 1 ? j + half : 2 * j + 1;
      const float* src = row_s + hh * a.dim;
      const float* w = is_q ? a.q_w ? a.q_w + hh * a.dim : nullptr : a.k_w ? a.k_w + (hh - a.H) * a.dim : nullptr;
      const float r = is_q ? rq : rk, m = is_q ? a.q_scale : 1.f;
      float x = i0 < a.dim ? (w ? src[i0] * r * w[i0] : src[i0]) : 0.f, y = i1 < a.dim ? (w ? src[i1] * r * w[i1] : src[i1]) : 0.f;
      if (j < half) {
        const float2 e = cs[j];
        const float x1 = x * e.x - y * e.y;
        y = y * e.x + x * e.y;
        x = x1;
      }
      if (is_q) {
        const size_t o = ((size_t)t * a.H + hh) * a.DK;
        if (a.q32) { a.q32[o + i0] = x * m; if (i1 < a.DK) a.q32[o + i1] = y * m; }
        if (a.q16) { a.q16[o + i0] = __float2half(x * m); if (i1 < a.DK) a.q16[o + i1] = __float2half(y * m); }
      } else {
        CT* kd = kc + (((size_t)page * a.G + hh - a.H) * a.page_size + off) * a.DK;
        put(kd + i0, x);
        if (i1 < a.DK) put(kd + i1, y);
      }
    }
  }
}
// cache_f32: kc / vc hold fp32 instead of fp16; layout [page][G][page_size][DK or DV].
B200_API int b200_row_qkv_finish(const float* in, int ld, int T, int q_off, int k_off, int v_off, const float* q_w, const float* k_w, const int* pos,
                                 const int* slot, const void* tab, int tab_len, int H, int G, int dim, int vdim, int DK, int DV, int rot, int style,
                                 int v_norm, float eps, float q_scale, int page_size, const float* lam, float* v_first, float* q32, void* q16, void* kc,
                                 void* vc, int cache_f32, cudaStream_t st) {
  if (T < 1 || H < 1 || G < 1 || H % G || dim < 1 || vdim < 1 || dim > DK || vdim > DV || (rot & 1) || rot > dim || rot < 0 || page_size < 1 || !kc || !vc ||
      (!q32 && !q16) || (rot && (!tab || tab_len < 1)) || (lam && !v_first))
    return B200_ERR_BAD_ARG;
  const size_t smem = (size_t)(H + G) * dim * 4;
  if (smem > 200 * 1024) return B200_ERR_BAD_ARG;
  RowQkvArgs a;
  a.in = in; a.ld = ld; a.q_off = q_off; a.k_off = k_off; a.v_off = v_off; a.q_w = q_w; a.k_w = k_w; a.pos = pos; a.slot = slot; a.tab = (const float2*)tab;
  a.tab_len = tab_len; a.H = H; a.G = G; a.dim = dim; a.vdim = vdim; a.DK = DK; a.DV = DV; a.rot = rot; a.style = style; a.page_size = page_size;
  a.v_norm = v_norm; a.eps = eps; a.q_scale = q_scale; a.lam = lam; a.v_first = v_first; a.q32 = q32; a.q16 = (__half*)q16;
  const bool vec = ((ld | q_off | k_off | dim | DK) & 3) == 0 && rot % 8 == 0 &&
                   (((uintptr_t)in | (uintptr_t)q_w | (uintptr_t)k_w | (uintptr_t)tab | (uintptr_t)q32 | (uintptr_t)q16 | (uintptr_t)kc) & 15) == 0;
  auto run = [&](auto kern, auto* k, auto* v) {
    if (smem > 48 * 1024) {
      cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
      if (e != cudaSuccess) return (int)e;
    }
    return launch_pdl(kern, dim3(T), dim3(T <= 2 * 148 && (H + G) * dim >= 2048 ? 512 : 256), smem, st, a, k, v);
  };
  if (cache_f32)
    return vec ? run(row_qkv_finish_kernel<float, true>, (float*)kc, (float*)vc) : run(row_qkv_finish_kernel<float, false>, (float*)kc, (float*)vc);
  return vec ? run(row_qkv_finish_kernel<__half, true>, (__half*)kc, (__half*)vc) : run(row_qkv_finish_kernel<__half, false>, (__half*)kc, (__half*)vc);
}

// ------------------------------------------------------------------ gated norm in equal parts

// Per row of D values y:  v = y * silu(z)   (z null: v = y), each of NG equal parts of v divided by its own root mean square, times w [D].
// y fp32 [T][ldy], z fp32 [T][ldz]; out bf16 and/or fp32 [T][ldo], columns D..ldo zero.  One CTA per (row, part).
__global__ void __launch_bounds__(256) group_norm_kernel(const float* __restrict__ y, int ldy, const float* __restrict__ z, int ldz, int D, int NG,
                                                         const float* __restrict__ w, float eps, __nv_bfloat16* __restrict__ ob, float* __restrict__ of,
                                                         int ldo, int vec) {
  extern __shared__ __align__(16) float part_s[];          // [D / NG]
  __shared__ float red[32];
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, g = blockIdx.y, n = D / NG, tid = threadIdx.x, nt = blockDim.x;
  const float* yr = y + (size_t)t * ldy + g * n;
  const float* zr = z ? z + (size_t)t * ldz + g * n : nullptr;
  const size_t at = (size_t)t * ldo + g * n;
  auto gate = [](float a, float b) { return a * (b / (1.f + expf(-b))); };
  float ss = 0.f;
  if (vec) {
#pragma unroll 4
    for (int i = tid; i < n / 4; i += nt) {
      float4 v = *(const float4*)(yr + 4 * i);
      if (zr) {
        const float4 q = *(const float4*)(zr + 4 * i);
        v = make_float4(gate(v.x, q.x), gate(v.y, q.y), gate(v.z, q.z), gate(v.w, q.w));
      }
      *(float4*)(part_s + 4 * i) = v;
      ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
  } else {
    for (int i = tid; i < n; i += nt) {
      const float v = zr ? gate(yr[i], zr[i]) : yr[i];
      part_s[i] = v;
      ss += v * v;
    }
  }
  const float r = 1.f / sqrtf(block_sum(ss, red) / (float)n + eps);
  if (vec) {
    for (int i = tid; i < n / 4; i += nt) {                // every thread meets the elements it wrote
      const float4 v = *(const float4*)(part_s + 4 * i), q = *(const float4*)(w + g * n + 4 * i);
      const float4 o = make_float4(v.x * r * q.x, v.y * r * q.y, v.z * r * q.z, v.w * r * q.w);
      if (ob) {
        const __nv_bfloat162 p0 = __floats2bfloat162_rn(o.x, o.y), p1 = __floats2bfloat162_rn(o.z, o.w);
        *(uint2*)(ob + at + 4 * i) = make_uint2(*(const uint32_t*)&p0, *(const uint32_t*)&p1);
      }
      if (of) *(float4*)(of + at + 4 * i) = o;
    }
  } else {
    for (int i = tid; i < n; i += nt) {
      const float o = part_s[i] * r * w[g * n + i];
      if (ob) ob[at + i] = __float2bfloat16(o);
      if (of) of[at + i] = o;
    }
  }
  if (g == NG - 1)
    for (int i = D + tid; i < ldo; i += nt) {
      if (ob) ob[(size_t)t * ldo + i] = __float2bfloat16(0.f);
      if (of) of[(size_t)t * ldo + i] = 0.f;
    }
}
B200_API int b200_group_norm(const float* y, int ldy, const float* z, int ldz, int T, int D, int NG, const float* w, float eps, void* ob, float* of, int ldo,
                             cudaStream_t st) {
  if (T < 1 || D < 1 || NG < 1 || D % NG || ldy < D || (z && ldz < D) || ldo < D || !y || !w || (!ob && !of)) return B200_ERR_BAD_ARG;
  const int n = D / NG;
  const size_t smem = (size_t)n * 4;
  if (smem > 200 * 1024) return B200_ERR_BAD_ARG;
  const int vec = ((n | ldy | ldz | ldo) & 3) == 0 && (((uintptr_t)y | (uintptr_t)z | (uintptr_t)w | (uintptr_t)ob | (uintptr_t)of) & 15) == 0;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(group_norm_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e != cudaSuccess) return (int)e;
  }
  const int threads = n >= 1024 ? 256 : n >= 256 ? 128 : 64;
  return launch_pdl(group_norm_kernel, dim3(T, NG), dim3(threads), smem, st, y, ldy, z, z ? ldz : 0, D, NG, w, eps, (__nv_bfloat16*)ob, of, ldo, vec);
}

// ------------------------------------------------------------------ attention in 32-bit arithmetic, any head size

// Causal grouped-query attention over the paged cache, prompts and decoding alike: one warp per query row, eight rows per CTA
// sharing key tiles of 32.  Lane j scores key j of a tile; the weights are then broadcast lane by lane while the lanes hold
// the output columns.  Everything is fp32 whatever the cache holds.  gate [T][ldg] (or null): the output of head h is
// multiplied by sigmoid(gate[t][h]).  chunk > 0: a query sees its own chunk of that many positions only.  sinks [H] (or null): one more
// term of the denominator per head.  maps: see qkv_finish (query rows are DK wide).  KS: columns of a key row in the cache.  vc null: the
// values are the first DV columns of the key row (latent attention).  window > 0: a query sees that many positions, itself the last.
// slopes [H] (or null): slopes[h] times the distance is taken off a score.  slices > 1 (mixed heads, values are keys): a key row is that many
// heads' keys of DK columns side by side, a query row is as wide and meets all of them, and the values are the slice of the head's own group.
struct AttnExactArgs {
  const float* q;          // [T][H][DK], scaled
  const int* page_table;
  const int* q_start;
  const int* q_len;
  const int* ctx_len;
  const float* gate;
  const float* sinks;
  const float* slopes;
  int ldg, max_pages, H, G, DK, DV, KS, maps, chunk, shared_kv, window, slices;
  float* out_f32;          // [T][ldo], head h at column h * DV
  __nv_bfloat16* out_bf16;
  int ldo;
};
constexpr int kExactRows = 8, kExactKeys = 32;

__device__ __forceinline__ float get(const float* p) { return *p; }
__device__ __forceinline__ float get(const __half* p) { return __half2float(*p); }

// kExactCols: output columns per lane (value sizes up to 32 times that)
template <typename CT, int kExactCols>
__global__ void __launch_bounds__(32 * kExactRows) attn_exact_kernel(const AttnExactArgs a, const CT* __restrict__ kc,
                                                                     const CT* __restrict__ vc) {
  extern __shared__ __align__(16) float sm[];
  float* sQ = sm;                                   // [rows][QW]
  const int QW = a.DK * a.slices;                   // columns of a query row
  float* sK = sQ + kExactRows * QW;                 // [keys][DK + 1]
  const int ldv = a.shared_kv ? a.DK + 1 : a.DV;
  float* sV = a.shared_kv ? sK : sK + kExactKeys * (a.DK + 1);         // [keys][ldv]
  pdl_trigger();
  pdl_wait();
  const int seq = blockIdx.z, h = blockIdx.y, q0 = blockIdx.x * kExactRows;
  const int qlen = a.q_len[seq];
  if (q0 >= qlen) return;
  const int ctx = a.ctx_len[seq], qs = a.q_start[seq], row_k = h / (a.H / (a.G * a.maps));
  const int kh = row_k / a.maps, own = h / (a.H / a.slices);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int* pt = a.page_table + (size_t)seq * a.max_pages;
  const int rows = min(kExactRows, qlen - q0), pos0 = ctx - qlen + q0, qpos = pos0 + warp;
  for (int i = tid; i < rows * QW; i += blockDim.x) {
    const int r = i / QW, c = i % QW;
    sQ[i] = a.q[((size_t)(qs + q0 + r) * a.H + h) * QW + c];
  }
  float acc[kExactCols];
#pragma unroll
  for (int i = 0; i < kExactCols; i++) acc[i] = 0.f;
  float m = -INFINITY, l = 0.f;
  const float slope = a.slopes ? a.slopes[h] : 0.f;
  const int k_end = pos0 + rows;                    // keys [k_begin, k_end) matter to some row
  const int k_begin = a.chunk > 0 ? pos0 / a.chunk * a.chunk : a.window > 0 ? max(0, pos0 - a.window + 1) : 0;
  const int q_first = a.chunk > 0 ? qpos / a.chunk * a.chunk : a.window > 0 ? qpos - a.window + 1 : 0;
  for (int k0 = k_begin; k0 < k_end; k0 += kExactKeys) {
    const int nk = min(kExactKeys, k_end - k0);
    const bool seen = warp < rows && lane < nk && k0 + lane <= qpos && k0 + lane >= q_first;
    float s = seen ? -slope * (float)(qpos - k0 - lane) : -INFINITY;
    for (int u = 1; u <= a.slices; u++) {           // the own slice comes last: its keys are then the values
      const int sl = (own + u) % a.slices, k_col = (a.slices > 1 ? sl : row_k % a.maps) * a.DK;
      __syncthreads();
      for (int i = tid; i < nk * a.DK; i += blockDim.x) {
        const int r = i / a.DK, c = i % a.DK, key = k0 + r;
        sK[r * (a.DK + 1) + c] = get(kc + (((size_t)pt[key >> 4] * a.G + kh) * 16 + (key & 15)) * a.KS + k_col + c);
      }
      for (int i = tid; i < nk * a.DV && !a.shared_kv; i += blockDim.x) {
        const int r = i / a.DV, c = i % a.DV, key = k0 + r;
        sV[r * a.DV + c] = get(vc + (((size_t)pt[key >> 4] * a.G + kh) * 16 + (key & 15)) * a.DV + c);
      }
      __syncthreads();
      if (seen) {
        const float* kr = sK + lane * (a.DK + 1);
        const float* qr = sQ + warp * QW + (a.slices > 1 ? sl * a.DK : 0);
        float dot = 0.f;
        for (int c = 0; c < a.DK; c++) dot = fmaf(qr[c], kr[c], dot);
        s += dot;
      }
    }
    if (warp >= rows) continue;
    const float mn = fmaxf(m, warp_max(s));
    if (mn == -INFINITY) continue;
    const float corr = m == -INFINITY ? 0.f : expf(m - mn);
    const float p = s == -INFINITY ? 0.f : expf(s - mn);
    l = l * corr + warp_sum(p);
    m = mn;
#pragma unroll
    for (int i = 0; i < kExactCols; i++) acc[i] *= corr;
    for (int j = 0; j < nk; j++) {
      const float pj = __shfl_sync(0xffffffffu, p, j);
      const float* vr = sV + j * ldv;
#pragma unroll
      for (int i = 0; i < kExactCols; i++) {
        const int e = lane + 32 * i;
        if (e < a.DV) acc[i] = fmaf(pj, vr[e], acc[i]);
      }
    }
  }
  if (warp >= rows) return;
  const size_t t = (size_t)(qs + q0 + warp);
  float inv = l > 0.f ? 1.f / l : 0.f;
  if (a.sinks) {
    const float sk = a.sinks[h], mn = fmaxf(m, sk), c = m == -INFINITY ? 0.f : expf(m - mn);
    inv = c / (l * c + expf(sk - mn));
  }
  if (a.gate) inv *= 1.f / (1.f + expf(-a.gate[t * a.ldg + h]));
#pragma unroll
  for (int i = 0; i < kExactCols; i++) {
    const int e = lane + 32 * i;
    if (e >= a.DV) continue;
    const size_t at = t * a.ldo + (size_t)h * a.DV + e;
    if (a.out_f32) a.out_f32[at] = acc[i] * inv;
    if (a.out_bf16) a.out_bf16[at] = __float2bfloat16(acc[i] * inv);
  }
}
template <typename CT, int NC>
static int launch_exact_nc(dim3 grid, size_t smem, const AttnExactArgs& a, const CT* kc, const CT* vc, cudaStream_t st) {
  auto kern = attn_exact_kernel<CT, NC>;
  static size_t configured = 48 * 1024;
  if (smem > configured) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = smem;
  }
  return launch_pdl(kern, grid, dim3(32 * kExactRows), smem, st, a, kc, vc);
}
template <typename CT>
static int launch_exact(int DV, dim3 grid, size_t smem, const AttnExactArgs& a, const CT* kc, const CT* vc, cudaStream_t st) {
  if (DV <= 128) return launch_exact_nc<CT, 4>(grid, smem, a, kc, vc, st);
  if (DV <= 512) return launch_exact_nc<CT, 16>(grid, smem, a, kc, vc, st);
  return launch_exact_nc<CT, 32>(grid, smem, a, kc, vc, st);
}
B200_API int b200_attn_exact(const float* q, const void* kc, const void* vc, int cache_f32, const int* page_table, int max_pages,
                             const int* q_start, const int* q_len, const int* ctx_len, int n_seqs, int max_q, int H, int G, int DK,
                             int DV, const float* gate, int ldg, float* out_f32, void* out_bf16, int ldo, int KS, int maps, int chunk,
                             const float* sinks, int window, const float* slopes, int slices, cudaStream_t st) {
  if (G < 1 || maps < 1 || H % (G * maps) || n_seqs < 1 || max_q < 1 || DK < 1 || DV < 1 || DV > 1024 || ldo < H * DV || KS < maps * DK || chunk < 0)
    return B200_ERR_BAD_ARG;
  if (!vc && (DV > DK || maps != 1)) return B200_ERR_BAD_ARG;
  if (window < 0 || (window && chunk) || slices < 1 || (slices > 1 && (vc || G != 1 || maps != 1 || H % slices || KS < slices * DK))) return B200_ERR_BAD_ARG;
  AttnExactArgs a;
  a.q = q; a.page_table = page_table; a.q_start = q_start; a.q_len = q_len; a.ctx_len = ctx_len; a.gate = gate; a.ldg = ldg;
  a.max_pages = max_pages; a.H = H; a.G = G; a.DK = DK; a.DV = DV; a.out_f32 = out_f32; a.out_bf16 = (__nv_bfloat16*)out_bf16; a.ldo = ldo;
  a.KS = KS; a.maps = maps; a.chunk = chunk; a.sinks = sinks; a.shared_kv = vc ? 0 : 1; a.window = window; a.slopes = slopes; a.slices = slices;
  const size_t smem = 4 * ((size_t)kExactRows * DK * slices + (size_t)kExactKeys * (DK + 1) + (vc ? (size_t)kExactKeys * DV : 0));
  if (smem > 200 * 1024) return B200_ERR_BAD_ARG;
  const dim3 grid((max_q + kExactRows - 1) / kExactRows, H, n_seqs);
  if (cache_f32) return launch_exact<float>(DV, grid, smem, a, (const float*)kc, (const float*)vc, st);
  return launch_exact<__half>(DV, grid, smem, a, (const __half*)kc, (const __half*)vc, st);
}

// ------------------------------------------------------------------ differential attention: the difference of two maps

// One warp per (token, head): o = a1 - lambda a2 over the two maps' outputs, divided by its root mean square over the head's values, times
// `mult`.  in [T][2 H][DV] in qkv_finish's order; out [T][ldo] with head h at column h * DV, padding columns zero.
__global__ void __launch_bounds__(128) diff_combine_kernel(const float* __restrict__ in, const float* __restrict__ lambda, int H, int G, int vdim, int DV,
                                                           float eps, float mult, float* __restrict__ out_f32, __nv_bfloat16* __restrict__ out_bf16,
                                                           int ldo) {
  const float lam = *lambda;
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, h = blockIdx.y * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (h >= H) return;
  const int rep = H / G, g = h / rep, r = h % rep;
  const float* a1 = in + ((size_t)t * 2 * H + (g * 2) * rep + r) * DV;
  const float* a2 = a1 + (size_t)rep * DV;
  float ss = 0.f;
  for (int e = lane; e < vdim; e += 32) {
    const float o = a1[e] - lam * a2[e];
    ss += o * o;
  }
  const float m = mult / sqrtf(warp_sum(ss) / (float)vdim + eps);
  for (int e = lane; e < DV; e += 32) {
    const float o = e < vdim ? (a1[e] - lam * a2[e]) * m : 0.f;
    const size_t at = (size_t)t * ldo + (size_t)h * DV + e;
    if (out_f32) out_f32[at] = o;
    if (out_bf16) out_bf16[at] = __float2bfloat16(o);
  }
}
B200_API int b200_diff_combine(const float* in, const float* lambda, int T, int H, int G, int vdim, int DV, float eps, float mult,
                               float* out_f32, void* out_bf16, int ldo, cudaStream_t st) {
  if (T < 1 || G < 1 || H % G || vdim < 1 || vdim > DV || ldo < H * DV || (!out_f32 && !out_bf16)) return B200_ERR_BAD_ARG;
  return launch_pdl(diff_combine_kernel, dim3(T, (H + 3) / 4), dim3(128), 0, st, in, lambda, H, G, vdim, DV, eps, mult, out_f32,
                    (__nv_bfloat16*)out_bf16, ldo);
}

// ------------------------------------------------------------------ matrix product in 32-bit

// C[M][N] = act(alpha A[M][K] W[N][K]^T), times sigmoid(gate[M][N]) where given, added into C (accumulate) or stored: fp32 activations, bf16-stored weights (their expansion is exact), fp32 multiply-adds on the
// CUDA cores.  The 32-bit mode's projection; 64 x 64 tiles, 16 K columns staged at a time, 4 x 4 outputs per thread.
// col_scale [N] (or null) multiplies what is stored or added.  heads > 1: head z multiplies columns z * head_k of A with rows z * N of W into columns z * head_ldc of C.
__global__ void __launch_bounds__(256) gemm_f32_kernel(const float* __restrict__ A, int lda, const __nv_bfloat16* __restrict__ W,
                                                       int ldb, float* __restrict__ C, int ldc, int M, int N, int K, int act, float alpha,
                                                       int accumulate, const float* __restrict__ gate, int ldg, int head_k, int head_ldc,
                                                       const float* __restrict__ col_scale) {
  __shared__ float sA[16][68], sB[16][68];
  pdl_trigger();
  pdl_wait();
  A += (size_t)blockIdx.z * head_k;
  W += (size_t)blockIdx.z * N * ldb;
  C += (size_t)blockIdx.z * head_ldc;
  if (gate) gate += (size_t)blockIdx.z * head_ldc;
  const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64, tid = threadIdx.x;
  const int tx = tid & 15, ty = tid >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += 16) {
    for (int i = tid; i < 1024; i += 256) {
      const int r = i >> 4, c = i & 15, k = k0 + c;
      sA[c][r] = (m0 + r < M && k < K) ? A[(size_t)(m0 + r) * lda + k] : 0.f;
      sB[c][r] = (n0 + r < N && k < K) ? __bfloat162float(W[(size_t)(n0 + r) * ldb + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; k++) {
      const float4 x = *(const float4*)&sA[k][ty * 4], w = *(const float4*)&sB[k][tx * 4];
      const float xa[4] = {x.x, x.y, x.z, x.w}, wa[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
      for (int i = 0; i < 4; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) acc[i][j] = fmaf(xa[i], wa[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; i++)
#pragma unroll
    for (int j = 0; j < 4; j++) {
      const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (m >= M || n >= N) continue;
      float v = acc[i][j] * alpha;
      if (act == 1) v = v > 0.f ? v * v : 0.f;
      else if (act == 2) v = gelu_erf(v);
      if (gate) v *= 1.f / (1.f + expf(-gate[(size_t)m * ldg + n]));
      if (col_scale) v *= col_scale[n];
      float* c = C + (size_t)m * ldc + n;
      *c = accumulate ? *c + v : v;
    }
}
// act: 0 none, 1 the square of relu, 2 the erf gelu.
B200_API int b200_gemm_f32(const float* A, int lda, const void* W, int ldb, float* C, int ldc, int M, int N, int K, int act,
                           float alpha, int accumulate, const float* gate, int ldg, int heads, int head_k, int head_ldc, const float* col_scale,
                           cudaStream_t st) {
  if (M < 1 || N < 1 || K < 1 || heads < 1 || (col_scale && heads > 1) || lda < (heads - 1) * head_k + K || ldb < K || ldc < (heads - 1) * head_ldc + N || act < 0 || act > 2)
    return B200_ERR_BAD_ARG;
  return launch_pdl(gemm_f32_kernel, dim3((N + 63) / 64, (M + 63) / 64, heads), dim3(256), 0, st, A, lda, (const __nv_bfloat16*)W, ldb, C,
                    ldc, M, N, K, act, alpha, accumulate, gate, ldg, head_k, head_ldc, col_scale);
}

// ------------------------------------------------------------------ one small mat-vec per head

// out[t][z * head_ldc + n] = alpha * sum_k A[t][z * head_k + k] W[z * N + n][k], times sigmoid(gate[t][z * head_ldc + n]) where given: gemm_f32's
// per-head product for 1..8 rows.  LPR lanes share a weight row (LPR * 8 columns per pass); a group of them holds four rows in flight.
template <int T, int LPR>
__global__ void __launch_bounds__(256) head_matvec_kernel(const float* __restrict__ A, int lda, const __nv_bfloat16* __restrict__ W, int ldb,
                                                          float* __restrict__ out, int ldc, int rows, int N, int K, float alpha,
                                                          const float* __restrict__ gate, int ldg, int head_k, int head_ldc) {
  extern __shared__ __align__(16) float xs[];          // [T][K]
  const int z = blockIdx.y, grp = threadIdx.x / LPR, gl = threadIdx.x % LPR, n0 = (blockIdx.x * (256 / LPR) + grp) * 4;
  const __nv_bfloat16* w = W + (size_t)z * N * ldb;
  uint4 q[4];
  auto fetch = [&](int k) {
#pragma unroll
    for (int r = 0; r < 4; r++) q[r] = ldg_stream(w + (size_t)min(n0 + r, N - 1) * ldb + k);
  };
  const bool live = n0 < N;
  if (live && gl * 8 < K) fetch(gl * 8);               // weights do not wait for the kernel before this one
  pdl_trigger();
  pdl_wait();
  for (int i = threadIdx.x; i < T * K; i += 256) {
    const int t = i / K, k = i - t * K;
    xs[i] = t < rows ? A[(size_t)t * lda + (size_t)z * head_k + k] : 0.f;
  }
  __syncthreads();
  float acc[4][T];
#pragma unroll
  for (int r = 0; r < 4; r++)
#pragma unroll
    for (int t = 0; t < T; t++) acc[r][t] = 0.f;
  for (int k = gl * 8; k < K && live; k += LPR * 8) {
    if (k != gl * 8) fetch(k);
#pragma unroll
    for (int t = 0; t < T; t++) {
      const float4 x0 = *(const float4*)(xs + t * K + k), x1 = *(const float4*)(xs + t * K + k + 4);
#pragma unroll
      for (int r = 0; r < 4; r++) {
        const __nv_bfloat162* p = (const __nv_bfloat162*)&q[r];
        float2 f;
        f = __bfloat1622float2(p[0]); acc[r][t] += f.x * x0.x + f.y * x0.y;
        f = __bfloat1622float2(p[1]); acc[r][t] += f.x * x0.z + f.y * x0.w;
        f = __bfloat1622float2(p[2]); acc[r][t] += f.x * x1.x + f.y * x1.y;
        f = __bfloat1622float2(p[3]); acc[r][t] += f.x * x1.z + f.y * x1.w;
      }
    }
  }
#pragma unroll
  for (int r = 0; r < 4; r++)
#pragma unroll
    for (int t = 0; t < T; t++) {
#pragma unroll
      for (int o = LPR / 2; o > 0; o >>= 1) acc[r][t] += __shfl_xor_sync(0xffffffffu, acc[r][t], o);
    }
  if (gl != 0 || !live) return;
#pragma unroll
  for (int r = 0; r < 4; r++)
#pragma unroll
    for (int t = 0; t < T; t++) {
      if (n0 + r >= N || t >= rows) continue;
      const int c = z * head_ldc + n0 + r;
      float v = acc[r][t] * alpha;
      if (gate) v *= 1.f / (1.f + expf(-gate[(size_t)t * ldg + c]));
      out[(size_t)t * ldc + c] = v;
    }
}
template <int T>
static int launch_head_matvec(const float* A, int lda, const __nv_bfloat16* W, int ldb, float* out, int ldc, int rows, int heads, int N, int K, float alpha,
                              const float* gate, int ldg, int head_k, int head_ldc, cudaStream_t st) {
  const size_t smem = (size_t)T * K * 4;
  const int lpr = K <= 64 ? 8 : K <= 128 ? 16 : 32;
  const dim3 grid((N + 1024 / lpr - 1) / (1024 / lpr), heads);
  auto kern = lpr == 8 ? head_matvec_kernel<T, 8> : lpr == 16 ? head_matvec_kernel<T, 16> : head_matvec_kernel<T, 32>;
  return launch_pdl(kern, grid, dim3(256), smem, st, A, lda, W, ldb, out, ldc, rows, N, K, alpha, gate, ldg, head_k, head_ldc);
}
// A fp32 [rows][lda], W bf16 [heads * N][ldb]; rows <= 8, K a multiple of 8 (48 KB of activations at most).
B200_API int b200_head_matvec(const float* A, int lda, const void* W, int ldb, float* out, int ldc, int rows, int heads, int N, int K, float alpha,
                              const float* gate, int ldg, int head_k, int head_ldc, cudaStream_t st) {
  if (rows < 1 || rows > 8 || heads < 1 || N < 1 || K < 8 || K % 8 || ldb % 8 || ((uintptr_t)W & 15) || K > head_k || N > head_ldc) return B200_ERR_BAD_ARG;
  const int T = rows <= 1 ? 1 : rows <= 2 ? 2 : rows <= 4 ? 4 : 8;
  if ((size_t)T * K * 4 > 48 * 1024) return B200_ERR_BAD_ARG;
  const __nv_bfloat16* w = (const __nv_bfloat16*)W;
  switch (T) {
    case 1: return launch_head_matvec<1>(A, lda, w, ldb, out, ldc, rows, heads, N, K, alpha, gate, ldg, head_k, head_ldc, st);
    case 2: return launch_head_matvec<2>(A, lda, w, ldb, out, ldc, rows, heads, N, K, alpha, gate, ldg, head_k, head_ldc, st);
    case 4: return launch_head_matvec<4>(A, lda, w, ldb, out, ldc, rows, heads, N, K, alpha, gate, ldg, head_k, head_ldc, st);
  }
  return launch_head_matvec<8>(A, lda, w, ldb, out, ldc, rows, heads, N, K, alpha, gate, ldg, head_k, head_ldc, st);
}

// ------------------------------------------------------------------ last step of the logits

// l <- l * scale, then (cap > 0) l <- cap * tanh(l / cap), in place.
__global__ void __launch_bounds__(256) logits_finish_kernel(float* __restrict__ l, size_t n, float scale, float cap) {
  pdl_trigger();
  pdl_wait();
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
    float v = l[i] * scale;
    if (cap > 0.f) v = cap * tanhf(v / cap);
    l[i] = v;
  }
}
B200_API int b200_logits_finish(float* logits, size_t n, float scale, float cap, cudaStream_t st) {
  if (n < 1) return B200_ERR_BAD_ARG;
  const size_t blocks = (n + 1023) / 1024;
  return launch_pdl(logits_finish_kernel, dim3((unsigned)(blocks < 2368 ? blocks : 2368)), dim3(256), 0, st, logits, n, scale, cap);
}
