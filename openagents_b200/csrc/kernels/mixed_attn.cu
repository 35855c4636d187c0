// Attention whose heads' scores are mixed ahead of the softmax: score_h <- sum_g T[h][g] score_g, with keys that are the values too, a bias
// that grows with the distance, a sliding window and a term of one in the softmax's denominator.
//
// The mixture is linear in the queries, so it can be taken either on them or on the scores:
//   sum_g T[h][g] (q_g . k_c(g)) = Q'_h . K,   K = [k_0 | k_1 | ...] (all key heads of a token side by side),
//                                              Q'_h = [sum over g of group 0 of T[h][g] q_g | the same of group 1 | ...]
// Prompts take the first form: every head then attends on its own, with wide queries on a key row that all heads share, whose slice of the
// head's group is the value.  Distances: the biases of the mixture add up to one slope per head.
// A cache row is K: [page][16][G * DK], fp16 (or fp32 in the 32-bit mode).
//
// This file is compiled without fast math.
#include "common.cuh"

using namespace b200;

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
// walks the heads: REP multiply-adds per result, results leave as whole rows.
template <int REP, typename CT>
__global__ void __launch_bounds__(256) mixed_finish_kernel(const MixedArgs a, CT* __restrict__ kc) {
  extern __shared__ __align__(16) float sT[];       // [H][H]
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, tid = threadIdx.x, rep = REP ? REP : a.H / a.G;
  for (int i = tid; i < a.H * a.H; i += 256) sT[i] = a.mix[i];
  __syncthreads();
  const float* row = a.in + (size_t)t * a.ld;
  const int n8 = a.G * a.DK >> 3, d8 = a.DK >> 3;   // pieces of eight columns of a cache row, of one head
  const int shares = max(1, 256 / n8), per = (a.H + shares - 1) / shares;
  auto fetch = [&](int col, int d, float (&v)[8]) {
#pragma unroll
    for (int i = 0; i < 8; i++) v[i] = d + i < a.dim ? row[col + d + i] + (a.bias ? a.bias[col + d + i] : 0.f) : 0.f;
  };
  for (int it = tid; it < n8 * shares; it += 256) {
    const int p = it % n8, c = p / d8, d = (p % d8) << 3, h0 = it / n8 * per, h1 = min(a.H, h0 + per);
    float q[REP ? REP : 1][8];
    if constexpr (REP > 0) {
#pragma unroll
      for (int r = 0; r < REP; r++) {
        fetch((c * REP + r) * a.dim, d, q[r]);
#pragma unroll
        for (int i = 0; i < 8; i++) q[r][i] *= a.q_scale;
      }
    }
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
  const int s = a.slot[t];
  if (s < 0) return;
  for (int p = tid; p < n8; p += 256) {
    float v[8];
    fetch(a.k_off + p / d8 * a.dim, (p % d8) << 3, v);
    put8(kc + ((size_t)(s / a.page_size) * a.page_size + s % a.page_size) * n8 * 8 + p * 8, v);
  }
}
template <typename CT>
static int launch_mixed_finish(int T, const MixedArgs& a, CT* kc, cudaStream_t st) {
  const size_t smem = (size_t)a.H * a.H * 4;
  auto kern = mixed_finish_kernel<0, CT>;
  switch (a.H / a.G) {
    case 1: kern = mixed_finish_kernel<1, CT>; break;
    case 2: kern = mixed_finish_kernel<2, CT>; break;
    case 4: kern = mixed_finish_kernel<4, CT>; break;
    case 8: kern = mixed_finish_kernel<8, CT>; break;
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
  return cache_f32 ? launch_mixed_finish(T, a, (float*)kc, st) : launch_mixed_finish(T, a, (__half*)kc, st);
}
