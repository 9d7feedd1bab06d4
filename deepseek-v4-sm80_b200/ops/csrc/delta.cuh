// Shared pieces of the gated delta rule kernels (delta.cu, delta_chunk.cu).
#pragma once
#include "vec.cuh"

__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
// logarithm of the decay of a key channel; ea = exp(A_log) of the head
__device__ __forceinline__ float log_decay(float rate, float dt_bias, float ea) { return -ea * softplus_f(rate + dt_bias); }
// The same in two special-function instructions.  The absolute error stays at a rounding of the sum of logarithms it goes into.
__device__ __forceinline__ float log_decay_fast(float rate, float dt_bias, float ea) {
  const float x = rate + dt_bias;
  return -ea * (fmaxf(x, 0.f) + __logf(1.f + __expf(-fabsf(x))));
}

// Where the parts of the merged projection stand, and the inputs the short convolutions keep.
struct ConvCols {
  int ld;                 // row stride of p
  int at_k, at_v;         // first columns of k and v (q: 0)
  int nqk, nv;            // channels of q (and of k), and of v
  int taps;
  __device__ __forceinline__ int col(int c) const {      // column of channel c of q | k | v
    return c < nqk ? c : c < 2 * nqk ? at_k + c - nqk : at_v + c - 2 * nqk;
  }
};

// before[j] <- input number n - (taps - 1) + j of a portion of n tokens whose rows start at t0 (older ones from `before`
// itself, zeros ahead of position 0).  A thread owns whole channels c0, c0 + step, ...
template <typename T>
__device__ __forceinline__ void keep_conv_inputs(const T* __restrict__ p, T* before, const ConvCols& a, int t0, int n,
                                                 bool fresh, int c0, int step) {
  const int C = 2 * a.nqk + a.nv;
  for (int c = c0; c < C; c += step) {
    const int col = a.col(c);
    for (int j = 0; j < a.taps - 1; ++j) {
      const int i = n - (a.taps - 1) + j;
      T v;
      if (i >= 0)
        v = p[(size_t)(t0 + i) * a.ld + col];
      else
        st_f(&v, fresh ? 0.f : ld_f(before + (size_t)(j + n) * C + c));   // j + n > j: not overwritten yet
      before[(size_t)j * C + c] = v;
    }
  }
}
