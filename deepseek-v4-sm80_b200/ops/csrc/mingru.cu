// Element-wise gated recurrence whose gates read only the current token (minGRU), with an output gate:
//
//   z = sigmoid(p_z + b_z),   u = p_u + b_u,   c = u + 1/2 for u >= 0, sigmoid(u) below
//   S_t = (1 - z) S_{t-1} + z c,               y = S_t * silu(p_g)
//
// p [tokens][z | u | g] fp32 comes from one projection, S [width] fp32 belongs to the request's slot.  The steps are maps
// S -> a S + b, which compose to (a1 a2, a2 b1 + b2): products of the decays themselves, so portions of any length run in parallel
// without logarithms.
//   mingru_step   one thread per request and W elements, token by token: decode and short portions
//   mingru_scan   a CTA takes `CT` neighbouring elements of one request and all its tokens: 256 threads hold 8 tokens each, the
//                 maps are combined over lanes and warps, the state is carried from tile to tile.  The next tile's inputs are
//                 fetched before the current tile is combined.
#include "vec.cuh"

namespace {

struct MinGruArgs {
  const float* p;
  int ld, at_u, at_g;      // row stride, first columns of u and of g
  const float *bz, *bu;    // [width]
  float* state;            // [slots + 1][width]
  const int *slots, *pos, *seg_off, *num_valid;
  int width;
};

// z and u with their biases -> the step's map (a, b).  1 - sigmoid(z) = e^-z sigmoid(z), without cancellation.  Where bf16 comes out,
// both reciprocals are one: 1 / p = q / (p q).
template <typename T>
__device__ __forceinline__ void gru_map(float z, float u, float& a, float& b) {
  if constexpr (sizeof(T) == 2) {
    const float ez = __expf(fminf(-z, 40.f)), eu = __expf(fminf(-u, 40.f));
    const float p = 1.f + ez, q = 1.f + eu, r = __fdividef(1.f, p * q);
    const float s = q * r;
    a = ez * s;
    b = s * (u >= 0.f ? u + 0.5f : p * r);
  } else {
    const float ez = expf(fminf(-z, 80.f)), s = 1.f / (1.f + ez);
    a = ez * s;
    b = s * (u >= 0.f ? u + 0.5f : sigmoid_f(u));
  }
}

template <typename T, int W>
__global__ void __launch_bounds__(128) mingru_step_kernel(T* __restrict__ y, const MinGruArgs a) {
  pdl_entry();
  const int seg = blockIdx.y, c = (blockIdx.x * 128 + threadIdx.x) * W;
  if (c >= a.width || (a.num_valid && seg >= *a.num_valid)) return;
  const int t0 = a.seg_off ? a.seg_off[seg] : seg, t1 = a.seg_off ? a.seg_off[seg + 1] : seg + 1;
  if (t1 <= t0) return;
  float* st = a.state + (size_t)a.slots[t0] * a.width + c;
  float s[W], bz[W], bu[W];
  ld_w<W>(a.bz + c, bz);
  ld_w<W>(a.bu + c, bu);
#pragma unroll
  for (int i = 0; i < W; ++i) s[i] = 0.f;
  if (a.pos[t0] != 0) ld_w<W>(st, s);
  for (int t = t0; t < t1; ++t) {
    const float* row = a.p + (size_t)t * a.ld + c;
    float z[W], u[W], g[W], o[W];
    ld_w<W>(row, z);
    ld_w<W>(row + a.at_u, u);
    ld_w<W>(row + a.at_g, g);
#pragma unroll
    for (int i = 0; i < W; ++i) {
      float ka, kb;
      gru_map<T>(z[i] + bz[i], u[i] + bu[i], ka, kb);
      s[i] = fmaf(ka, s[i], kb);
      o[i] = s[i] * g[i] * sigmoid_for<T>(g[i]);
    }
    st_w<W>(y + (size_t)t * a.width + c, o);
  }
  st_w<W>(st, s);
}

constexpr int kGruThreads = 256, kGruTokens = 8, kGruWarps = kGruThreads / 32;

template <typename T, int CT>
__global__ void __launch_bounds__(kGruThreads, 2) mingru_scan_kernel(T* __restrict__ y, const MinGruArgs a) {
  pdl_entry();
  constexpr int L = kGruTokens, SUB = 32 / CT, TT = kGruThreads / CT * L;   // token groups per warp, tokens per tile
  __shared__ float2 maps[2][kGruWarps][CT];
  const int seg = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int ch = lane % CT, sub = lane / CT, c = blockIdx.x * CT + ch;
  const bool in = c < a.width;
  const int t0 = a.seg_off ? a.seg_off[seg] : seg, t1 = a.seg_off ? a.seg_off[seg + 1] : seg + 1;
  if (t1 <= t0) return;
  float* st = a.state + (size_t)a.slots[t0] * a.width + c;
  const float bz = in ? a.bz[c] : 0.f, bu = in ? a.bu[c] : 0.f;
  float s_in = in && a.pos[t0] != 0 ? *st : 0.f;
  const int mine = (warp * SUB + sub) * L;                                  // first token of this thread within a tile
  float z[L], u[L], g[L];
  auto fetch = [&](int tile) {
    const float* row = a.p + (size_t)(tile + mine) * a.ld + c;
#pragma unroll
    for (int j = 0; j < L; ++j) {
      const bool ok = in && tile + mine + j < t1;
      z[j] = ok ? row[(size_t)j * a.ld] : 0.f;
      u[j] = ok ? row[(size_t)j * a.ld + a.at_u] : 0.f;
      g[j] = ok ? row[(size_t)j * a.ld + a.at_g] : 0.f;
    }
  };
  fetch(t0);
  int buf = 0;
  for (int tile = t0; tile < t1; tile += TT, buf ^= 1) {
    float ka[L], kb[L], gate[L];
    float A = 1.f, B = 0.f;
#pragma unroll
    for (int j = 0; j < L; ++j) {
      gru_map<T>(z[j] + bz, u[j] + bu, ka[j], kb[j]);
      if (tile + mine + j >= t1) ka[j] = 1.f, kb[j] = 0.f;
      gate[j] = g[j];
      B = fmaf(ka[j], B, kb[j]);
      A *= ka[j];
    }
    if (tile + TT < t1) fetch(tile + TT);
    // inclusive over the token groups of the warp
#pragma unroll
    for (int off = CT; off < 32; off <<= 1) {
      const float pa = __shfl_up_sync(0xffffffffu, A, off), pb = __shfl_up_sync(0xffffffffu, B, off);
      if (lane >= off) B = fmaf(A, pb, B), A *= pa;
    }
    if (sub == SUB - 1) maps[buf][warp][ch] = make_float2(A, B);
    float ea = 1.f, eb = 0.f;                                               // of the groups ahead of this one in the warp
    if constexpr (SUB > 1) {
      const float pa = __shfl_up_sync(0xffffffffu, A, CT), pb = __shfl_up_sync(0xffffffffu, B, CT);
      if (sub > 0) ea = pa, eb = pb;
    }
    __syncthreads();      // one per tile: a warp can be at most one tile ahead, in the other buffer
    float s = s_in;
#pragma unroll
    for (int w = 0; w < kGruWarps; ++w) {
      const float2 m = maps[buf][w][ch];
      if (w == warp) s = s_in;
      s_in = fmaf(m.x, s_in, m.y);
    }
    s = fmaf(ea, s, eb);
#pragma unroll
    for (int j = 0; j < L; ++j) {
      s = fmaf(ka[j], s, kb[j]);
      if (in && tile + mine + j < t1)
        st_f(y + (size_t)(tile + mine + j) * a.width + c, s * gate[j] * sigmoid_for<T>(gate[j]));
    }
  }
  if (in && threadIdx.x < CT) *st = s_in;
}

template <typename T>
int launch_gru(void* y, const MinGruArgs& a, int segs, int longest, int ct, cudaStream_t st) {
  auto go = [&](auto kern, int per, int threads) {
    dsv4_launch(kern, dim3((a.width + per - 1) / per, segs), threads, 0, st, (T*)y, a);
  };
  if (longest <= 16) {
    const bool wide = a.width % 4 == 0 && a.ld % 4 == 0 && a.at_u % 4 == 0 && a.at_g % 4 == 0 && ((uintptr_t)a.p & 15) == 0;
    if (wide)
      go(mingru_step_kernel<T, 4>, 512, 128);
    else
      go(mingru_step_kernel<T, 1>, 128, 128);
  } else if (ct == 32) {
    go(mingru_scan_kernel<T, 32>, 32, kGruThreads);
  } else if (ct == 16) {
    go(mingru_scan_kernel<T, 16>, 16, kGruThreads);
  } else if (ct == 8) {
    go(mingru_scan_kernel<T, 8>, 8, kGruThreads);
  } else {
    return 801;
  }
  return (int)cudaGetLastError();
}

}  // namespace

// p fp32 [rows, ld], z at column 0, u and g at at_u and at_g; y [rows, width] (fp32: its type, 0 = bf16); state fp32 [slots + 1,
// width].  segs requests, their rows as in seg_off [segs + 1], or null: a row each.  longest: rows of the longest request; ct:
// elements per CTA of longer portions (8, 16 or 32).
DSV4_API int dsv4_mingru(const float* p, int ld, int at_u, int at_g, const float* bz, const float* bu, float* state, void* y,
                         const int* slots, const int* pos, const int* seg_off, int segs, const int* num_valid, int longest,
                         int ct, int width, int fp32, cudaStream_t st) {
  if (segs <= 0) return 0;
  if (segs > 65535 || width < 1 || (longest > 1 && !seg_off) || (seg_off && num_valid)) return 800;
  const MinGruArgs a{p, ld, at_u, at_g, bz, bu, state, slots, pos, seg_off, num_valid, width};
  return fp32 ? launch_gru<float>(y, a, segs, longest, ct, st) : launch_gru<__nv_bfloat16>(y, a, segs, longest, ct, st);
}
