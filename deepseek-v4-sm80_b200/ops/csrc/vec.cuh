// Element access shared by the kernels that exist for bf16 and for fp32 activations.
#pragma once
#include "common.cuh"

__device__ __forceinline__ float ld_f(const float* p) { return *p; }
__device__ __forceinline__ float ld_f(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st_f(float* p, float v) { *p = v; }
__device__ __forceinline__ void st_f(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ float4 ld_f4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 ld_f4(const __nv_bfloat16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void st_f4(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void st_f4(__nv_bfloat16* p, const float4& v) {
  __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 u;
  u.x = *reinterpret_cast<uint32_t*>(&a);
  u.y = *reinterpret_cast<uint32_t*>(&b);
  *reinterpret_cast<uint2*>(p) = u;
}
// W consecutive values, W = 1 or 4 (then aligned to four elements)
template <int W>
__device__ __forceinline__ void ld_w(const float* p, float (&v)[W]) {
  if constexpr (W == 4) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    v[0] = f.x, v[1] = f.y, v[2] = f.z, v[3] = f.w;
  } else {
    v[0] = *p;
  }
}
template <int W, typename T>
__device__ __forceinline__ void st_w(T* p, const float (&v)[W]) {
  if constexpr (W == 4)
    st_f4(p, make_float4(v[0], v[1], v[2], v[3]));
  else
    st_f(p, v[0]);
}
// sum over the CTA (blockDim.x a multiple of 32, at most 1024); sh: 32 floats
__device__ __forceinline__ float cta_sum(float v, float* sh) {
  v = warp_sum(v);
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31, nw = blockDim.x >> 5;
  __syncthreads();
  if (l == 0) sh[w] = v;
  __syncthreads();
  return warp_sum(l < nw ? sh[l] : 0.f);
}

// Epilogue activations of the projections (the numbers are part of the host interface).
// The gates pair columns: the weight rows come in blocks of 16 gate and 16 up rows, and the result is half as wide.
enum GemmAct : int { kActNone = 0, kActRelu2 = 1, kActTanh = 2, kActGeluGate = 3, kActSiluGate = 4, kActClampGate = 5 };
constexpr int kGateBlock = 16;
__host__ __device__ __forceinline__ bool gated_act(int act) { return act >= kActGeluGate && act <= kActClampGate; }
__device__ __forceinline__ float gemm_act(float v, int act) {
  if (act == kActRelu2) {
    v = fmaxf(v, 0.f);
    return v * v;
  }
  return act == kActTanh ? tanhf(v) : v;
}

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
// the same for results that are rounded to T: 1e-6 relative is enough for bf16
template <typename T>
__device__ __forceinline__ float sigmoid_for(float z) {
  return sizeof(T) == 2 ? __fdividef(1.f, 1.f + __expf(-z)) : sigmoid_f(z);
}
// gate(z) * up.  silu: z sigmoid(z);  gelu: 0.5 z (1 + tanh(w)) = z sigmoid(2 w),  w = sqrt(2 / pi) (z + 0.044715 z^3);
// clamp: g sigmoid(1.702 g) (u + 1) for g = min(z, limit), u = min(max(up, -limit), limit)
__device__ __forceinline__ float gate_mul(float z, float up, int act, float limit) {
  if (act == kActClampGate) {
    z = fminf(z, limit);
    return z * sigmoid_f(1.702f * z) * (fminf(fmaxf(up, -limit), limit) + 1.f);
  }
  const float w = act == kActSiluGate ? z : 1.5957691216057308f * fmaf(0.044715f * z * z, z, z);
  return z * sigmoid_f(w) * up;
}
// v: a row's 32 consecutive columns (16 gate, 16 up) -> its 16 gated values in v[0..15]
__device__ __forceinline__ void gate_block(float* v, int act, float limit) {
#pragma unroll
  for (int j = 0; j < kGateBlock; ++j) v[j] = gate_mul(v[j], v[j + kGateBlock], act, limit);
}
// 16 consecutive values, dst 16-byte aligned
__device__ __forceinline__ void st_f16x(__nv_bfloat16* dst, const float* v) {
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    uint4 u;
    __nv_bfloat162* p = reinterpret_cast<__nv_bfloat162*>(&u);
#pragma unroll
    for (int e = 0; e < 4; ++e) p[e] = __floats2bfloat162_rn(v[8 * i + 2 * e], v[8 * i + 2 * e + 1]);
    reinterpret_cast<uint4*>(dst)[i] = u;
  }
}
__device__ __forceinline__ void st_f16x(float* dst, const float* v) {
#pragma unroll
  for (int i = 0; i < 4; ++i) st_f4(dst + 4 * i, make_float4(v[4 * i], v[4 * i + 1], v[4 * i + 2], v[4 * i + 3]));
}

// First and last row of a request's rows in the batch: rows of a request stand together at consecutive positions.
__device__ __forceinline__ bool seg_first(const int* slots, const int* pos, int t) {
  return t == 0 || slots[t - 1] != slots[t] || pos[t - 1] + 1 != pos[t];
}
__device__ __forceinline__ bool seg_last(const int* slots, const int* pos, int t, int rows) {
  return t + 1 >= rows || slots[t + 1] != slots[t] || pos[t + 1] != pos[t] + 1;
}
