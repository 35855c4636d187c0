// What the chunked forms of recurrent layers share: 64-token chunks and their slots in a workspace, fp32 values as two bf16 numbers (value and
// remainder, about 16 bits of mantissa) for the tensor cores, and the warp-level instructions on them.
#pragma once
#include "common.cuh"

namespace b200 {

constexpr int GC = 64;                 // tokens per chunk

// Walks (row, column) of a row-major grid in steps of a block, without a division per step.
struct GridWalk {
  int r, c, dr, dc, cols;
  __device__ __forceinline__ GridWalk(int start, int step, int n_cols) : r(start / n_cols), c(start % n_cols), dr(step / n_cols), dc(step % n_cols), cols(n_cols) {}
  __device__ __forceinline__ void next() {
    r += dr;
    c += dc;
    if (c >= cols) {
      c -= cols;
      r++;
    }
  }
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

static inline size_t align256(size_t n) { return (n + 255) & ~(size_t)255; }

}  // namespace b200
