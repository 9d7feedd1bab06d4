// Products of 32-bit numbers on the tensor cores in three TF32 terms (mma.sync m16n8k8): x = hi + lo with hi cut off to TF32's 11
// bits, and hi hi' + hi lo' + lo hi' keeps about 21 bits of a product.
#pragma once
#include <stdint.h>

struct Split {
  uint32_t hi, lo;
};
__device__ __forceinline__ Split split(float x) {
  Split s;
  s.hi = __float_as_uint(x) & 0xffffe000u;
  s.lo = __float_as_uint(x - __uint_as_float(s.hi));
  return s;
}
__device__ __forceinline__ void mma_tf32(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0,
                                         uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
struct FragA {
  Split v[4];
};
__device__ __forceinline__ FragA frag_a(float a0, float a1, float a2, float a3) {
  return FragA{{split(a0), split(a1), split(a2), split(a3)}};
}
__device__ __forceinline__ void mma3(float (&c)[4], const FragA& a, const float2& b) {
  const Split x = split(b.x), y = split(b.y);
  mma_tf32(c, a.v[0].lo, a.v[1].lo, a.v[2].lo, a.v[3].lo, x.hi, y.hi);
  mma_tf32(c, a.v[0].hi, a.v[1].hi, a.v[2].hi, a.v[3].hi, x.lo, y.lo);
  mma_tf32(c, a.v[0].hi, a.v[1].hi, a.v[2].hi, a.v[3].hi, x.hi, y.hi);
}
