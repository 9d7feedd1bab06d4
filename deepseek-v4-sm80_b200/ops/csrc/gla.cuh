// Gated linear attention: what the kernels of gla.cu (token by token) and gla_chunk.cu (chunks) share.
//
//   S_t = diag(g_t) S_{t-1} + k_t v_t^T,   o_t = S_t^T q_t                (S is [key channel, value], fp32)
//
// Where g and k come from (Gates):
//   kGiven    log g per head and a factor of k per head, prepared by mlstm_gates; the values have a column of ones behind them, so
//             the state carries the sum of the weighted keys as one more column
//   kStep     a step size per head: dt = softplus(raw + bias), log g = -exp(A_log) dt, k dt; groups of heads share q and k
//   kForget   per key channel: g = low + (1 - low) sigmoid(raw + bias), k = 1 - g; q goes through silu
#pragma once
#include "vec.cuh"

enum Gates : int { kGiven = 0, kStep = 1, kForget = 2 };

struct GlaArgs {
  int ldq, ldk, ldv;      // row strides; query / key head h / group
  const float* raw;       // kGiven: log g [rows][heads]; kStep, kForget: the projection [rows][heads] / [rows][heads * d]
  const float* fac;       // kGiven: factor of k [rows][heads]
  const float* bias;      // kStep: [heads]; kForget: [heads * d]
  const float* par;       // kStep: A_log [heads]; kForget: low [heads * d]
  float q_mul;
  int heads, group, d, e; // e values per head
  int ew;                 // columns of the state: e, plus the column of ones for kGiven, rounded up to 4
  float* state;           // [slots + 1][heads][d][ew]
  float* out;             // [rows][heads][ew]
  const int* slots;
  const int* pos;
};

__device__ __forceinline__ float softplus_of(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

// A head's gate of a row (kGiven, kStep): log g and the factor of k.
struct HeadGate {
  float log_g, fac;
};
template <int MODE>
__device__ __forceinline__ HeadGate head_gate(const GlaArgs& a, size_t row, int head) {
  const float raw = a.raw[row * a.heads + head];
  if constexpr (MODE == kGiven) return {raw, a.fac[row * a.heads + head]};
  const float dt = softplus_of(raw + a.bias[head]);
  return {-expf(a.par[head]) * dt, dt};
}
// A key channel's forget gate: what is written (1 - g) and what is kept.
struct ChannelGate {
  float write, keep;
  // log g without the cancellation near g = 1
  __device__ __forceinline__ float log_keep() const { return write < 0.5f ? log1pf(-write) : logf(keep); }
};
__device__ __forceinline__ ChannelGate channel_gate(float z, float low) {
  const float e = expf(-fabsf(z)), big = 1.f / (1.f + e), small = e * big;     // sigmoid(|z|) and sigmoid(-|z|)
  const float up = z >= 0.f ? big : small, down = z >= 0.f ? small : big;
  return {(1.f - low) * down, fmaf(1.f - low, up, low)};
}
