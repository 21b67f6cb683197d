// Pieces of the mma.sync kernels of composed models.
#pragma once
#include "gemm_mma.cuh"

__device__ __forceinline__ void ldmatrix_x4_t(unsigned& r0, unsigned& r1, unsigned& r2, unsigned& r3, const void* p) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(s));
}
__device__ __forceinline__ unsigned pack_bf16(float lo, float hi) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<const unsigned*>(&v);
}
// fp32 operands of a bf16 product: the sum of this many bf16 pieces
constexpr int PIECES = 3;

// two fp32 values -> PIECES packed pairs of bf16 that sum up to them
__device__ __forceinline__ void split2(float x, float y, unsigned (&p)[PIECES]) {
#pragma unroll
  for (int i = 0; i < PIECES; ++i) {
    p[i] = pack_bf16(x, y);
    const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&p[i]));
    x -= f.x;
    y -= f.y;
  }
}
