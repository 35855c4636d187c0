// Operators of hybrid decoders (attention and recurrent layers in one stack, norms around both ends of a sublayer): the
// residual step, the projection finish of an attention layer, attention in exact 32-bit arithmetic for any head size, the
// 32-bit matrix product, and the last step of the logits.
//
// This file is compiled without fast math: divisions, square roots, exponentials and hyperbolic tangents are the IEEE-accurate
// ones, because what runs here is what such models are required to compute in 32-bit.
#include "common.cuh"

using namespace b200;

// ------------------------------------------------------------------ residual step

// Per row:  x += y / rms(y) * gy   (when y is given; rms over D, eps inside the root)
//           h  = x / rms(x) * gh   (when gh is given) -> bf16 and/or fp32, columns D..ldh written as zeros
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
  if (!gh) return;
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < kNormRegs; k++) ss += v[k] * v[k];
  for (int i = threadIdx.x + kNormRegs * nt; i < D; i += nt) ss += xr[i] * xr[i];
  const float r = 1.f / sqrtf(block_sum(ss, red) / (float)D + eps);
#pragma unroll
  for (int k = 0; k < kNormRegs; k++) {
    const int i = threadIdx.x + k * nt;
    if (i < ldh) {
      const float o = i < D ? v[k] * r * gh[i] : 0.f;
      if (hb) hb[(size_t)t * ldh + i] = __float2bfloat16(o);
      if (hf) hf[(size_t)t * ldh + i] = o;
    }
  }
  for (int i = threadIdx.x + kNormRegs * nt; i < ldh; i += nt) {
    const float o = i < D ? xr[i] * r * gh[i] : 0.f;
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
  if (!gh) return;
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < R; k++) ss += v[k].x * v[k].x + v[k].y * v[k].y + v[k].z * v[k].z + v[k].w * v[k].w;
  const float r = 1.f / sqrtf(block_sum(ss, red) * inv_d + eps);
#pragma unroll
  for (int k = 0; k < R; k++) {
    const int i = tid + k * nt;
    if (i >= ldh4) continue;           // ldh4 > D4: padding columns are zeros
    const float4 g = i < D4 ? gh[i] : z;
    const float4 o = make_float4(v[k].x * r * g.x, v[k].y * r * g.y, v[k].z * r * g.z, v[k].w * r * g.w);
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
  if (T < 1 || D < 1 || !x || (y && (!gy || ldy < D)) || (gh && (ldh < D || (!hb && !hf)))) return B200_ERR_BAD_ARG;
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

// ------------------------------------------------------------------ attention: finish of the projections

// One warp per (token, head) of a fused projection row: queries and keys are rotated on their first `rot` dimensions, then
// (qk_norm) divided by their root mean square over the head; queries are scaled, keys and values go to the paged cache.
//   style 0: dimension 2i turns with 2i + 1; style 1: i with i + rot / 2.
// Cache and query rows are padded to DK / DV columns; the padding is written as zeros.
struct QkvArgs {
  const float* in;         // [T][ld]
  int ld, q_off, k_off, v_off;     // k_off < 0: the layer has no keys and values of its own
  const int* pos;
  const int* slot;         // physical cache slot (page * page_size + offset); < 0: no cache write
  const float2* tab;       // [tab_len][rot / 2] (cos, sin)
  int tab_len;
  double base;
  int H, G, dim, vdim, DK, DV, rot, style, qk_norm, page_size;
  float eps, q_scale;
  float* q32;              // [T][H][DK] or null
  __half* q16;             // [T][H][DK] or null
};
constexpr int kQkvPairs = 8;      // pairs per lane: head sizes up to 512

__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(__half* p, float v) { *p = __float2half(v); }

template <typename CT>
__global__ void __launch_bounds__(128) qkv_finish_kernel(const QkvArgs a, CT* __restrict__ kc, CT* __restrict__ vc) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, lane = threadIdx.x & 31;
  const int n_heads = a.H + (a.k_off >= 0 ? 2 * a.G : 0);
  const int hh = blockIdx.y * 4 + (threadIdx.x >> 5);
  if (hh >= n_heads) return;
  const int s = a.slot[t];
  const int page = s >= 0 ? s / a.page_size : 0, off = s >= 0 ? s % a.page_size : 0;
  const float* row = a.in + (size_t)t * a.ld;
  if (hh >= a.H + a.G) {                                  // a value head
    if (s < 0) return;
    const int g = hh - a.H - a.G;
    CT* dst = vc + (((size_t)page * a.G + g) * a.page_size + off) * a.DV;
    for (int e = lane; e < a.DV; e += 32) put(dst + e, e < a.vdim ? row[a.v_off + g * a.vdim + e] : 0.f);
    return;
  }
  const bool is_q = hh < a.H;
  const float* in = row + (is_q ? a.q_off + hh * a.dim : a.k_off + (hh - a.H) * a.dim);
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
  const size_t q_at = ((size_t)t * a.H + hh) * a.DK;
  CT* kd = is_q ? nullptr : kc + (((size_t)page * a.G + (hh - a.H)) * a.page_size + off) * a.DK;
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
// cache_f32: kc / vc hold fp32 instead of fp16; layout [page][G][page_size][DK or DV].
B200_API int b200_qkv_finish(const float* in, int ld, int T, int q_off, int k_off, int v_off, const int* pos, const int* slot,
                             const void* tab, int tab_len, double base, int H, int G, int dim, int vdim, int DK, int DV, int rot,
                             int style, int qk_norm, float eps, float q_scale, int page_size, float* q32, void* q16, void* kc,
                             void* vc, int cache_f32, cudaStream_t st) {
  if (T < 1 || H < 1 || G < 1 || dim < 1 || vdim < 1 || dim > DK || vdim > DV || DK > 64 * kQkvPairs || (rot & 1) || rot > dim || rot < 0)
    return B200_ERR_BAD_ARG;
  if ((k_off >= 0 && (!kc || !vc)) || (!q32 && !q16) || page_size < 1) return B200_ERR_BAD_ARG;
  QkvArgs a;
  a.in = in; a.ld = ld; a.q_off = q_off; a.k_off = k_off; a.v_off = v_off; a.pos = pos; a.slot = slot; a.tab = (const float2*)tab;
  a.tab_len = tab ? tab_len : 0; a.base = base; a.H = H; a.G = G; a.dim = dim; a.vdim = vdim; a.DK = DK; a.DV = DV; a.rot = rot;
  a.style = style; a.qk_norm = qk_norm; a.page_size = page_size; a.eps = eps; a.q_scale = q_scale; a.q32 = q32; a.q16 = (__half*)q16;
  const int n_heads = H + (k_off >= 0 ? 2 * G : 0);
  const dim3 grid(T, (n_heads + 3) / 4);
  if (cache_f32) return launch_pdl(qkv_finish_kernel<float>, grid, dim3(128), 0, st, a, (float*)kc, (float*)vc);
  return launch_pdl(qkv_finish_kernel<__half>, grid, dim3(128), 0, st, a, (__half*)kc, (__half*)vc);
}

// ------------------------------------------------------------------ attention in 32-bit arithmetic, any head size

// Causal grouped-query attention over the paged cache, prompts and decoding alike: one warp per query row, eight rows per CTA
// sharing key tiles of 32.  Lane j scores key j of a tile; the weights are then broadcast lane by lane while the lanes hold
// the output columns.  Everything is fp32 whatever the cache holds.  gate [T][ldg] (or null): the output of head h is
// multiplied by sigmoid(gate[t][h]).
struct AttnExactArgs {
  const float* q;          // [T][H][DK], scaled
  const int* page_table;
  const int* q_start;
  const int* q_len;
  const int* ctx_len;
  const float* gate;
  int ldg, max_pages, H, G, DK, DV;
  float* out_f32;          // [T][ldo], head h at column h * DV
  __nv_bfloat16* out_bf16;
  int ldo;
};
constexpr int kExactRows = 8, kExactKeys = 32, kExactCols = 16;     // columns per lane: value sizes up to 512

__device__ __forceinline__ float get(const float* p) { return *p; }
__device__ __forceinline__ float get(const __half* p) { return __half2float(*p); }

template <typename CT>
__global__ void __launch_bounds__(32 * kExactRows) attn_exact_kernel(const AttnExactArgs a, const CT* __restrict__ kc,
                                                                     const CT* __restrict__ vc) {
  extern __shared__ __align__(16) float sm[];
  float* sQ = sm;                                   // [rows][DK]
  float* sK = sQ + kExactRows * a.DK;               // [keys][DK + 1]
  float* sV = sK + kExactKeys * (a.DK + 1);         // [keys][DV]
  pdl_trigger();
  pdl_wait();
  const int seq = blockIdx.z, h = blockIdx.y, q0 = blockIdx.x * kExactRows;
  const int qlen = a.q_len[seq];
  if (q0 >= qlen) return;
  const int ctx = a.ctx_len[seq], qs = a.q_start[seq], kh = h / (a.H / a.G);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int* pt = a.page_table + (size_t)seq * a.max_pages;
  const int rows = min(kExactRows, qlen - q0), pos0 = ctx - qlen + q0, qpos = pos0 + warp;
  for (int i = tid; i < rows * a.DK; i += blockDim.x) {
    const int r = i / a.DK, c = i % a.DK;
    sQ[i] = a.q[((size_t)(qs + q0 + r) * a.H + h) * a.DK + c];
  }
  float acc[kExactCols];
#pragma unroll
  for (int i = 0; i < kExactCols; i++) acc[i] = 0.f;
  float m = -INFINITY, l = 0.f;
  const int k_end = pos0 + rows;                    // keys [0, k_end) matter to some row
  for (int k0 = 0; k0 < k_end; k0 += kExactKeys) {
    __syncthreads();
    const int nk = min(kExactKeys, k_end - k0);
    for (int i = tid; i < nk * a.DK; i += blockDim.x) {
      const int r = i / a.DK, c = i % a.DK, key = k0 + r;
      sK[r * (a.DK + 1) + c] = get(kc + (((size_t)pt[key >> 4] * a.G + kh) * 16 + (key & 15)) * a.DK + c);
    }
    for (int i = tid; i < nk * a.DV; i += blockDim.x) {
      const int r = i / a.DV, c = i % a.DV, key = k0 + r;
      sV[r * a.DV + c] = get(vc + (((size_t)pt[key >> 4] * a.G + kh) * 16 + (key & 15)) * a.DV + c);
    }
    __syncthreads();
    if (warp >= rows) continue;
    float s = -INFINITY;
    if (lane < nk && k0 + lane <= qpos) {
      const float* kr = sK + lane * (a.DK + 1);
      const float* qr = sQ + warp * a.DK;
      s = 0.f;
      for (int c = 0; c < a.DK; c++) s = fmaf(qr[c], kr[c], s);
    }
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
      const float* vr = sV + j * a.DV;
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
B200_API int b200_attn_exact(const float* q, const void* kc, const void* vc, int cache_f32, const int* page_table, int max_pages,
                             const int* q_start, const int* q_len, const int* ctx_len, int n_seqs, int max_q, int H, int G, int DK,
                             int DV, const float* gate, int ldg, float* out_f32, void* out_bf16, int ldo, cudaStream_t st) {
  if (G < 1 || H % G || n_seqs < 1 || max_q < 1 || DK < 1 || DV < 1 || DV > 32 * kExactCols || ldo < H * DV) return B200_ERR_BAD_ARG;
  AttnExactArgs a;
  a.q = q; a.page_table = page_table; a.q_start = q_start; a.q_len = q_len; a.ctx_len = ctx_len; a.gate = gate; a.ldg = ldg;
  a.max_pages = max_pages; a.H = H; a.G = G; a.DK = DK; a.DV = DV; a.out_f32 = out_f32; a.out_bf16 = (__nv_bfloat16*)out_bf16; a.ldo = ldo;
  const size_t smem = 4 * ((size_t)kExactRows * DK + (size_t)kExactKeys * (DK + 1) + (size_t)kExactKeys * DV);
  if (smem > 200 * 1024) return B200_ERR_BAD_ARG;
  const dim3 grid((max_q + kExactRows - 1) / kExactRows, H, n_seqs), block(32 * kExactRows);
  static size_t configured = 48 * 1024;
  if (smem > configured) {
    cudaError_t e = cudaFuncSetAttribute(attn_exact_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(attn_exact_kernel<__half>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = smem;
  }
  if (cache_f32) return launch_pdl(attn_exact_kernel<float>, grid, block, smem, st, a, (const float*)kc, (const float*)vc);
  return launch_pdl(attn_exact_kernel<__half>, grid, block, smem, st, a, (const __half*)kc, (const __half*)vc);
}

// ------------------------------------------------------------------ matrix product in 32-bit

// C[M][N] = act(A[M][K] W[N][K]^T): fp32 activations, bf16-stored weights (their expansion is exact), fp32 multiply-adds on the
// CUDA cores.  The 32-bit mode's projection; 64 x 64 tiles, 16 K columns staged at a time, 4 x 4 outputs per thread.
__global__ void __launch_bounds__(256) gemm_f32_kernel(const float* __restrict__ A, int lda, const __nv_bfloat16* __restrict__ W,
                                                       int ldb, float* __restrict__ C, int ldc, int M, int N, int K, int act) {
  __shared__ float sA[16][68], sB[16][68];
  pdl_trigger();
  pdl_wait();
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
      float v = acc[i][j];
      if (act == 1) v = v > 0.f ? v * v : 0.f;
      C[(size_t)m * ldc + n] = v;
    }
}
// act: 0 none, 1 the square of relu.
B200_API int b200_gemm_f32(const float* A, int lda, const void* W, int ldb, float* C, int ldc, int M, int N, int K, int act,
                           cudaStream_t st) {
  if (M < 1 || N < 1 || K < 1 || lda < K || ldb < K || ldc < N || act < 0 || act > 1) return B200_ERR_BAD_ARG;
  return launch_pdl(gemm_f32_kernel, dim3((N + 63) / 64, (M + 63) / 64), dim3(256), 0, st, A, lda, (const __nv_bfloat16*)W, ldb, C,
                    ldc, M, N, K, act);
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
