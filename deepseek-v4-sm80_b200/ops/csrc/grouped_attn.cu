// Causal attention with several query heads to a key head over paged keys and values (bf16 or fp32 caches): what happens
// between the q | k | v projection and the output projection.
//
//   s_ij = cap tanh(q_i . k_j scale / cap) + rel[h, min(i - j, last)] - slope_h (i - j)
//   w_ij = e^{s_ij} / (e^{sink_h} + sum_j' e^{s_ij'})       or, without any normalisation,  w_ij = sigmoid(s_ij + b_h)
//
// cap, rel, slope and sink are optional.  With a chunk size, position i only sees keys from i / chunk * chunk on; with a window, the
// last `window` positions up to itself.  Where the values were turned by their positions ahead of the cache, a head's result is
// turned back by the query's; and it may be multiplied by a gate per token and head.  Kernels:
//   rotate_store     bias, norms, rotation, query temperature; keys and values to their cache rows
//   head_store       the same with a norm per head, either layout of the rotated pairs, and values that turn
//   grouped_attn     tensor cores (mma.sync): the (token, query head) rows of a key head are consecutive, and all of them see
//                    a prefix of the same keys, so a CTA takes 16 .. 64 rows of one request and key head and streams the keys
//                    and values once for all of them.  grid.y splits the keys when the row tiles alone leave SMs idle;
//                    grouped_merge adds the partial results in split order, turns them back and gates them.  Decode, and short
//                    portions of prompts.
//   grouped_row      one warp per row on the CUDA cores, fp32 throughout: models served in 32-bit floats, other sizes
//   kv_gather        a request's keys and (transposed) values side by side, for the prompt kernel in flash_attn.cu
#include "mma16.cuh"

namespace {

// ------------------------------------------------------------------ behind the projection
struct RotateArgs {
  int ld;                    // row stride of qkv
  const float* bias;         // [(H + G) dim + G vdim] or null
  const float* freq;         // [pairs] or null
  int pairs;
  float coef;                // query temperature 1 + coef ln((pos + 1) / every + 1); every 0: none
  int every;
  const float* gain;         // [(H + G) dim]: q and k are divided by the root mean square of all their rows, times this; or null
  int unit_v;                // every head's values are divided by their root mean square
  float eps, v_mul;          // and the values multiplied by v_mul
  const int* pos;
  const int* out_loc;
  int heads, kv_heads, dim, vdim;
};

// One CTA per token; cos and sin of its angles and the norms' sums in shared memory.  W consecutive values per thread and chunk
// (even, or 1); NC > 0: all chunks of the row in registers, which the norms want.
template <typename T, int W, int NC>
__global__ void __launch_bounds__(256) rotate_store_kernel(const T* __restrict__ qkv, T* __restrict__ q,
                                                           T* __restrict__ keys, T* __restrict__ values,
                                                           const RotateArgs a) {
  pdl_entry();
  extern __shared__ float2 cs[];
  __shared__ float sums[2][8];
  float* part = reinterpret_cast<float*>(cs + a.pairs);   // NC > 0: sums of squares of the chunks of v; else of the heads
  const int t = blockIdx.x, pos = a.pos[t], loc = a.out_loc[t], warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int nq = a.heads * a.dim, nk = a.kv_heads * a.dim, nv = a.kv_heads * a.vdim;
  const T* src = qkv + (size_t)t * a.ld;
  auto at = [&](int i) { return ld_f(src + i) + (a.bias ? a.bias[i] : 0.f); };
  auto load = [&](int i, float (&v)[W]) {
    if constexpr (W == 1) {
      v[0] = at(i);
    } else {
#pragma unroll
      for (int j = 0; j < W; j += 4) {
        float4 x = ld_f4(src + i + j);
        if (a.bias) {
          const float4 b = ld_f4(a.bias + i + j);
          x.x += b.x, x.y += b.y, x.z += b.z, x.w += b.w;
        }
        v[j] = x.x, v[j + 1] = x.y, v[j + 2] = x.z, v[j + 3] = x.w;
      }
    }
  };
  float row[NC > 0 ? NC : 1][W];
  float sq = 0.f, sk = 0.f;
  if constexpr (NC > 0) {
#pragma unroll
    for (int n = 0; n < NC; ++n) {
      const int i = (n * 256 + (int)threadIdx.x) * W;
      if (i < nq + nk + nv) load(i, row[n]);
    }
#pragma unroll
    for (int n = 0; n < NC; ++n) {
      const int i = (n * 256 + (int)threadIdx.x) * W;
      if (i >= nq + nk + nv) continue;
      float s = 0.f;
#pragma unroll
      for (int j = 0; j < W; ++j) s = fmaf(row[n][j], row[n][j], s);
      if (i < nq) sq += s;
      else if (i < nq + nk) sk += s;
      else if (a.unit_v) part[(i - nq - nk) / W] = s;
    }
  } else {
    for (int i = threadIdx.x; a.gain && i < nq + nk; i += 256) {
      const float x = at(i);
      if (i < nq) sq += x * x; else sk += x * x;
    }
    for (int g = warp; a.unit_v && g < a.kv_heads; g += 8) {
      float s = 0.f;
      for (int i = lane; i < a.vdim; i += 32) {
        const float x = at(nq + nk + g * a.vdim + i);
        s += x * x;
      }
      s = warp_sum(s);
      if (lane == 0) part[g] = s;
    }
  }
  if (a.gain) {
    sq = warp_sum(sq), sk = warp_sum(sk);
    if (lane == 0) sums[0][warp] = sq, sums[1][warp] = sk;
  }
  for (int i = threadIdx.x; i < a.pairs; i += 256) {
    float s, c;
    sincosf((float)pos * a.freq[i], &s, &c);
    cs[i] = make_float2(c, s);
  }
  const float temp = a.every ? 1.f + a.coef * logf((float)((pos + 1) / a.every + 1)) : 1.f;
  __syncthreads();
  float inv[2] = {1.f, 1.f};       // of q and of k
  if (a.gain) {
#pragma unroll
    for (int p = 0; p < 2; ++p) {
      float s = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) s += sums[p][w];
      inv[p] = 1.f / sqrtf(s / (p ? nk : nq) + a.eps);
    }
  }
  auto place = [&](int i, float (&v)[W]) {
    if (i < nq + nk) {
      const float sc = i < nq ? inv[0] : inv[1];
      if (a.gain) {
        float gn[W];
        if constexpr (W == 1) {
          gn[0] = a.gain[i];
        } else {
#pragma unroll
          for (int j = 0; j < W; j += 4) {
            const float4 f = ld_f4(a.gain + i + j);
            gn[j] = f.x, gn[j + 1] = f.y, gn[j + 2] = f.z, gn[j + 3] = f.w;
          }
        }
#pragma unroll
        for (int j = 0; j < W; ++j) v[j] *= sc * gn[j];
      }
      const int e = i % a.dim;
      if constexpr (W == 1) {
        if (e < 2 * a.pairs) {
          const int o = e & 1 ? i - 1 : i + 1;
          const float2 r = cs[e >> 1];
          const float other = at(o) * (a.gain ? sc * a.gain[o] : 1.f);
          v[0] = e & 1 ? v[0] * r.x + other * r.y : v[0] * r.x - other * r.y;
        }
      } else {
#pragma unroll
        for (int j = 0; j < W; j += 2)
          if (e + j < 2 * a.pairs) {
            const float2 r = cs[(e + j) >> 1];
            const float x = v[j], y = v[j + 1];
            v[j] = x * r.x - y * r.y, v[j + 1] = y * r.x + x * r.y;
          }
      }
    } else {
      float sc = a.v_mul;
      if (a.unit_v) {
        const int head = (i - nq - nk) / a.vdim;
        float s = 0.f;
        if constexpr (NC > 0) {
          for (int p = 0; p < a.vdim / W; ++p) s += part[head * (a.vdim / W) + p];
        } else {
          s = part[head];
        }
        sc /= sqrtf(s / a.vdim + a.eps);
      }
#pragma unroll
      for (int j = 0; j < W; ++j) v[j] *= sc;
    }
    T* dst;
    if (i < nq) {
#pragma unroll
      for (int j = 0; j < W; ++j) v[j] *= temp;
      dst = q + (size_t)t * nq + i;
    } else {
      if (loc < 0) return;
      dst = i < nq + nk ? keys + (size_t)loc * nk + (i - nq) : values + (size_t)loc * nv + (i - nq - nk);
    }
    if constexpr (W == 1) {
      st_f(dst, v[0]);
    } else {
#pragma unroll
      for (int j = 0; j < W; j += 4) st_f4(dst + j, make_float4(v[j], v[j + 1], v[j + 2], v[j + 3]));
    }
  };
  if constexpr (NC > 0) {
#pragma unroll
    for (int n = 0; n < NC; ++n) {
      const int i = (n * 256 + (int)threadIdx.x) * W;
      if (i < nq + nk + nv) place(i, row[n]);
    }
  } else {
    for (int i = threadIdx.x * W; i < nq + nk + nv; i += 256 * W) {
      load(i, row[0]);
      place(i, row[0]);
    }
  }
}

// ------------------------------------------------------------------ norms per head, values that turn
struct HeadStoreArgs {
  int ld;                    // row stride of qkv
  const float* bias;         // [(H + G) dim + G vdim] or null
  const float* gain;         // [2][dim]: every q and k head is divided by its root mean square, times its row; or null
  float eps;
  const float* freq;         // [pairs]: the first 2 * pairs dimensions of q and k heads turn; or null
  int pairs, halves;         // partners: dimensions i and i + pairs (halves), or 2 i and 2 i + 1
  float mul;                 // factor of their cos and sin
  const float* vfreq;        // [vdim / 2]: whole value heads turn, in the same layout; or null
  float2* turn;              // [rows][vdim / 2]: cos and sin of the values' angles, for what turns the results back
  const int *pos, *out_loc;
  int heads, kv_heads, dim, vdim;
};

// One CTA per token, the row in registers: a thread's unit is eight values of a head, two groups of four that hold each other's
// partners.  Heads of q and k are a power of two of units wide, so that the lanes of a head sum up its squares.  Few tokens take a
// thread per unit (NU = 1), many take CTAs of kUnitThreads.
constexpr int kUnitThreads = 128;
template <typename T, int NU>
__global__ void __launch_bounds__(NU == 1 ? 1024 : kUnitThreads) head_store_units_kernel(const T* __restrict__ qkv, T* __restrict__ q,
                                                                        T* __restrict__ keys, T* __restrict__ values,
                                                                        const HeadStoreArgs a) {
  pdl_entry();
  extern __shared__ __align__(16) float hs_row[];
  const int t = blockIdx.x, pos = a.pos[t], loc = a.out_loc[t], tid = threadIdx.x, nt = blockDim.x;
  const int nq = a.heads * a.dim, nk = a.kv_heads * a.dim, nv = a.kv_heads * a.vdim, n = nq + nk + nv, vhalf = a.vdim / 2;
  float2* cs = reinterpret_cast<float2*>(hs_row);
  float2* vcs = cs + a.pairs;
  const T* src = qkv + (size_t)t * a.ld;
  // first columns (in the row) of the two groups of unit u; m: turned pairs of its head, k: the unit's first pair (< m) or none
  auto place = [&](int u, int& c0, int& c1, int& m, int& k) {
    const bool is_v = u * 8 >= nq + nk;
    const int w = is_v ? a.vdim : a.dim, base = is_v ? nq + nk : 0;
    const int h = (u * 8 - base) / w, e = u - (base + h * w) / 8;      // unit of its head
    m = is_v ? (a.vfreq ? vhalf : 0) : a.pairs;
    k = e * 4;
    c0 = base + h * w;
    if (a.halves && k < m)
      c1 = c0 + m + k, c0 += k;
    else
      c0 += e * 8, c1 = c0 + 4;
  };
  float4 x[NU][2];
#pragma unroll
  for (int i = 0; i < NU; ++i) {
    const int u = i * nt + tid;
    if (u * 8 >= n) continue;
    int c0, c1, m, k;
    place(u, c0, c1, m, k);
    x[i][0] = ld_f4(src + c0), x[i][1] = ld_f4(src + c1);
  }
  for (int i = tid; i < a.pairs; i += nt) {
    float s, c;
    sincosf((float)pos * a.freq[i], &s, &c);
    cs[i] = make_float2(c * a.mul, s * a.mul);
  }
  for (int i = tid; a.vfreq && i < vhalf; i += nt) {
    float s, c;
    sincosf((float)pos * a.vfreq[i], &s, &c);
    vcs[i] = make_float2(c, s);
    a.turn[(size_t)t * vhalf + i] = make_float2(c, s);
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < NU; ++i) {
    const int u = i * nt + tid;
    const bool in = u * 8 < n;
    int c0 = 0, c1 = 4, m = 0, k = 0;
    float v[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = 0.f;
    if (in) {
      place(u, c0, c1, m, k);
      float4 b0 = make_float4(0.f, 0.f, 0.f, 0.f), b1 = b0;
      if (a.bias) b0 = ld_f4(a.bias + c0), b1 = ld_f4(a.bias + c1);
      v[0] = x[i][0].x + b0.x, v[1] = x[i][0].y + b0.y, v[2] = x[i][0].z + b0.z, v[3] = x[i][0].w + b0.w;
      v[4] = x[i][1].x + b1.x, v[5] = x[i][1].y + b1.y, v[6] = x[i][1].z + b1.z, v[7] = x[i][1].w + b1.w;
    }
    if (a.gain) {
      float s = 0.f;
#pragma unroll
      for (int j = 0; j < 8; ++j) s = fmaf(v[j], v[j], s);
      for (int off = a.dim / 16; off > 0; off >>= 1) s += __shfl_xor_sync(0xffffffffu, s, off);
      if (in && c0 < nq + nk) {
        const float sc = 1.f / sqrtf(s / a.dim + a.eps);
        const float* g = a.gain + (c0 < nq ? 0 : a.dim);
        const float4 g0 = ld_f4(g + c0 % a.dim), g1 = ld_f4(g + c1 % a.dim);
        v[0] *= sc * g0.x, v[1] *= sc * g0.y, v[2] *= sc * g0.z, v[3] *= sc * g0.w;
        v[4] *= sc * g1.x, v[5] *= sc * g1.y, v[6] *= sc * g1.z, v[7] *= sc * g1.w;
      }
    }
    if (!in) continue;
    if (k < m) {
      const float4* tab = reinterpret_cast<const float4*>((c0 < nq + nk ? cs : vcs) + k);      // two pairs each
      const float4 r0 = tab[0], r1 = tab[1];
      const float co[4] = {r0.x, r0.z, r1.x, r1.z}, si[4] = {r0.y, r0.w, r1.y, r1.w};
      if (a.halves) {
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float y = v[j] * co[j] - v[4 + j] * si[j];
          v[4 + j] = v[4 + j] * co[j] + v[j] * si[j], v[j] = y;
        }
      } else {
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float y = v[2 * j] * co[j] - v[2 * j + 1] * si[j];
          v[2 * j + 1] = v[2 * j + 1] * co[j] + v[2 * j] * si[j], v[2 * j] = y;
        }
      }
    }
    T *d0 = q + (size_t)t * nq + c0, *d1 = q + (size_t)t * nq + c1;
    if (c0 >= nq) {
      if (loc < 0) continue;
      T* base = c0 < nq + nk ? keys + (size_t)loc * nk - nq : values + (size_t)loc * nv - (nq + nk);
      d0 = base + c0, d1 = base + c1;
    }
    st_f4(d0, make_float4(v[0], v[1], v[2], v[3]));
    st_f4(d1, make_float4(v[4], v[5], v[6], v[7]));
  }
}

// Other sizes: the row with its bias passes through shared memory, where a warp norms a head in place and partners meet.  W
// consecutive values per thread and access.
template <typename T, int W>
__global__ void __launch_bounds__(256) head_store_kernel(const T* __restrict__ qkv, T* __restrict__ q, T* __restrict__ keys,
                                                         T* __restrict__ values, const HeadStoreArgs a) {
  pdl_entry();
  extern __shared__ __align__(16) float hs_row[];
  const int t = blockIdx.x, pos = a.pos[t], loc = a.out_loc[t], warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int nq = a.heads * a.dim, nk = a.kv_heads * a.dim, nv = a.kv_heads * a.vdim, n = nq + nk + nv, vhalf = a.vdim / 2;
  float* row = hs_row;
  float2* cs = reinterpret_cast<float2*>(hs_row + (n + 3) / 4 * 4);
  float2* vcs = cs + a.pairs;
  const T* src = qkv + (size_t)t * a.ld;
  for (int i = threadIdx.x * W; i < n; i += 256 * W) {
    if constexpr (W == 1) {
      row[i] = ld_f(src + i) + (a.bias ? a.bias[i] : 0.f);
    } else {
#pragma unroll
      for (int j = 0; j < W; j += 4) {
        float4 x = ld_f4(src + i + j);
        if (a.bias) {
          const float4 b = ld_f4(a.bias + i + j);
          x.x += b.x, x.y += b.y, x.z += b.z, x.w += b.w;
        }
        *reinterpret_cast<float4*>(row + i + j) = x;
      }
    }
  }
  for (int i = threadIdx.x; i < a.pairs; i += 256) {
    float s, c;
    sincosf((float)pos * a.freq[i], &s, &c);
    cs[i] = make_float2(c * a.mul, s * a.mul);
  }
  for (int i = threadIdx.x; a.vfreq && i < vhalf; i += 256) {
    float s, c;
    sincosf((float)pos * a.vfreq[i], &s, &c);
    vcs[i] = make_float2(c, s);
    a.turn[(size_t)t * vhalf + i] = make_float2(c, s);
  }
  __syncthreads();
  if (a.gain) {
    for (int h = warp; h < a.heads + a.kv_heads; h += 8) {
      float* x = row + h * a.dim;
      const float* g = a.gain + (h < a.heads ? 0 : a.dim);
      float s = 0.f;
      for (int i = lane; i < a.dim; i += 32) s = fmaf(x[i], x[i], s);
      const float sc = 1.f / sqrtf(warp_sum(s) / a.dim + a.eps);
      for (int i = lane; i < a.dim; i += 32) x[i] *= sc * g[i];
    }
    __syncthreads();
  }
  for (int i = threadIdx.x * W; i < n; i += 256 * W) {
    const bool is_v = i >= nq + nk;
    const int e = is_v ? (i - nq - nk) % a.vdim : i % a.dim;
    const int m = is_v ? (a.vfreq ? vhalf : 0) : a.pairs;
    const float2* tab = is_v ? vcs : cs;
    float v[W];
#pragma unroll
    for (int j = 0; j < W; ++j) {
      const int k = e + j;
      v[j] = row[i + j];
      if (k >= 2 * m) continue;
      const bool second = a.halves ? k >= m : k & 1;
      const int pair = a.halves ? (second ? k - m : k) : k >> 1, away = a.halves ? m : 1;
      const float other = row[second ? i + j - away : i + j + away];
      const float2 r = tab[pair];
      v[j] = second ? v[j] * r.x + other * r.y : v[j] * r.x - other * r.y;
    }
    T* dst;
    if (i < nq) {
      dst = q + (size_t)t * nq + i;
    } else {
      if (loc < 0) continue;
      dst = is_v ? values + (size_t)loc * nv + (i - nq - nk) : keys + (size_t)loc * nk + (i - nq);
    }
    if constexpr (W == 1) {
      st_f(dst, v[0]);
    } else {
#pragma unroll
      for (int j = 0; j < W; j += 4) st_f4(dst + j, make_float4(v[j], v[j + 1], v[j + 2], v[j + 3]));
    }
  }
}

// ------------------------------------------------------------------ few rows: tensor cores
struct AttnArgs {
  const int* slots;
  const int* pos;
  const int* page_table;
  int ld_pt;
  const int* tiles;      // [tiles][2]: row range of a tile (rows of a key head: token * group + query head), or null: tiles
                         // of every token's own rows
  int n_tiles;
  const int* num_valid;  // tokens >= *num_valid are padding, or null
  int rows;              // tokens
  int kv_heads, group, dim, vdim;
  float scale, cap;      // cap 0: scores are not capped
  const float* sink;     // [H] or null
  const float* rel;      // [H][n_rel] or null
  int n_rel;
  const float* slope;    // [H]: taken off per position of distance; or null
  int chunk;             // > 0: keys are seen from the start of the query's chunk of this many positions on; the tokens of a
                         // tile then lie in one chunk
  int window;            // > 0: position i sees the keys i - window + 1 .. i
  const float* wbias;    // [H]: a key's weight is sigmoid(score + wbias), not normalised; or null: softmax
  const float2* turn;    // [rows][vdim / 2] cos and sin: results are turned back by these angles (partners half of vdim apart); or
                         // null
  const void* gate;      // [rows] activations of stride ld_gate, one per head: results are multiplied by its sigmoid; or null
  int ld_gate;
  int nsplit;
  int partial;           // results go to part_acc and part_ml, for grouped_merge
  float* part_acc;       // [T * H][nsplit][vdim]
  float* part_ml;        // [T * H][nsplit][2]
};
__device__ __forceinline__ int first_key(const AttnArgs& a, int pos) {
  return a.chunk ? pos / a.chunk * a.chunk : a.window ? max(0, pos - a.window + 1) : 0;
}
// column c of a result whose pair (c mod half, + half) holds u and v, turned back
__device__ __forceinline__ float turned_back(float u, float v, const float2& cs, bool second) {
  return second ? v * cs.x - u * cs.y : u * cs.x + v * cs.y;
}

constexpr int kKT = 64;       // keys per tile
constexpr int kSP = kKT + 4;  // floats per score row

template <int P, int MT>      // head sizes padded to P, MT x 16 rows
struct AttnCfg {
  static constexpr int M = MT * 16;
  static constexpr int RG = MT == 4 ? 2 : 1;       // warp row groups of the S phase
  static constexpr int WM = MT / RG;               // m16 tiles per warp
  static constexpr int KG = 8 / RG;                // key groups
  static constexpr int WN = kKT / KG / 8;          // n8 tiles per warp
  static constexpr int DW = P / 8;                 // output columns per warp
  static constexpr int NT = DW / 8;
  static constexpr int SMEM = M * P * 2 + 4 * kKT * P * 2 + M * kSP * 4 + M * kKT * 2 + 5 * M * 4;
};

template <int P, int MT>
__global__ void __launch_bounds__(256) grouped_attn_kernel(const __nv_bfloat16* __restrict__ q,
                                                           const __nv_bfloat16* __restrict__ keys,
                                                           const __nv_bfloat16* __restrict__ values,
                                                           __nv_bfloat16* __restrict__ o, const AttnArgs a) {
  pdl_entry();
  using C = AttnCfg<P, MT>;
  constexpr int M = C::M, WM = C::WM, WN = C::WN, NT = C::NT;
  extern __shared__ __align__(128) uint8_t attn_smem[];
  __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(attn_smem);  // [M][P] swizzled
  __nv_bfloat16* ksm = qs + M * P;                                  // [2][kKT][P] swizzled
  __nv_bfloat16* vsm = ksm + 2 * kKT * P;                           // [2][kKT][P] swizzled
  float* ss = reinterpret_cast<float*>(vsm + 2 * kKT * P);          // [M][kSP]
  __nv_bfloat16* pb = reinterpret_cast<__nv_bfloat16*>(ss + M * kSP);  // [M][kKT] swizzled
  float* ms = reinterpret_cast<float*>(pb + M * kKT);
  float* ls = ms + M;
  float* alpha = ls + M;
  int* see = reinterpret_cast<int*>(alpha + M);                     // end of the keys the row sees
  int* from = see + M;                                              // and their beginning

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = blockIdx.z, split = blockIdx.y, R = a.group, dch = a.dim / 8, vch = a.vdim / 8;
  const int ldq = a.kv_heads * R * a.dim, ldk = a.kv_heads * a.dim, ldv = a.kv_heads * a.vdim;
  int row0, row1;
  if (a.tiles) {
    row0 = a.tiles[blockIdx.x * 2], row1 = a.tiles[blockIdx.x * 2 + 1];
  } else {
    const int tpt = (R + M - 1) / M, t = blockIdx.x / tpt;
    row0 = t * R + blockIdx.x % tpt * M;
    row1 = min(row0 + M, (t + 1) * R);
  }
  if (a.num_valid && row0 / R >= *a.num_valid) return;
  const int t_last = (row1 - 1) / R;
  const int key0 = first_key(a, a.pos[row0 / R]);                     // first key; keys are counted from there
  const int nkeys = a.pos[t_last] + 1 - key0;   // of the tile's last token, the one that sees most
  const int* pt = a.page_table + (size_t)a.slots[t_last] * a.ld_pt + key0;
  // place of row r of the tile in q (elements) and in the lists of (token, head) rows
  auto head_row = [&](int r) { return (size_t)((row0 + r) / R) * (a.kv_heads * R) + g * R + (row0 + r) % R; };

  const int ktiles = (nkeys + kKT - 1) / kKT;
  const int per = (ktiles + a.nsplit - 1) / a.nsplit;
  const int kt0 = split * per, kt1 = min(kt0 + per, ktiles);
  if (kt0 >= kt1) {  // nothing for this split: an empty partial
    if (a.partial)
      for (int r = tid; r < row1 - row0; r += 256) {
        float* ml = a.part_ml + (head_row(r) * a.nsplit + split) * 2;
        ml[0] = -1e30f, ml[1] = 0.f;
      }
    return;
  }

  for (int i = tid; i < M * (P / 8); i += 256) {
    const int r = i / (P / 8), c = i % (P / 8);
    uint4 v = make_uint4(0, 0, 0, 0);
    if (row0 + r < row1 && c < dch)
      v = reinterpret_cast<const uint4*>(q + (size_t)((row0 + r) / R) * ldq + (g * R + (row0 + r) % R) * a.dim)[c];
    reinterpret_cast<uint4*>(qs + r * P)[swz(r, c)] = v;
  }
  if (tid < M) {
    ms[tid] = -1e30f, ls[tid] = 0.f;
    see[tid] = row0 + tid < row1 ? a.pos[(row0 + tid) / R] + 1 - key0 : 0;
    from[tid] = a.window ? max(0, see[tid] - a.window) : 0;
  }

  // four threads fetch the key and the value of one row
  const int fk = tid >> 2, fp = tid & 3;
  auto key_loc = [&](int kt) {
    const int key = kt * kKT + fk;
    return (kt < kt1 && key < nkeys) ? pt[key] : -1;
  };
  auto issue = [&](int loc, int buf) {
    __nv_bfloat16 *kd = ksm + ((size_t)buf * kKT + fk) * P, *vd = vsm + ((size_t)buf * kKT + fk) * P;
    const __nv_bfloat16 *kp = keys + (size_t)max(loc, 0) * ldk + g * a.dim, *vp = values + (size_t)max(loc, 0) * ldv + g * a.vdim;
#pragma unroll
    for (int c = fp; c < P / 8; c += 4) {
      const bool in_k = loc >= 0 && c < dch, in_v = loc >= 0 && c < vch;
      cpa16_zfill(kd + swz(fk, c) * 8, in_k ? kp + c * 8 : keys, in_k);
      cpa16_zfill(vd + swz(fk, c) * 8, in_v ? vp + c * 8 : values, in_v);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };

  float acc[MT][NT][4];
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < NT; ++j) acc[i][j][0] = acc[i][j][1] = acc[i][j][2] = acc[i][j][3] = 0.f;

  issue(key_loc(kt0), kt0 & 1);
  int loc_next = key_loc(kt0 + 1);
  const float sc2 = a.scale * kLog2e, cap2 = a.cap * kLog2e;   // scores in powers of two
  const float ce = a.cap > 0.f ? 2.f * kLog2e / cap2 : 0.f;
  const int rg = warp / C::KG, kg = warp % C::KG;
  const int kend = (a.dim + 31) / 32 * 2;                      // 16-wide steps of the score product, two at a time
  for (int kt = kt0; kt < kt1; ++kt) {
    const int buf = kt & 1;
    if (kt + 1 < kt1) {
      issue(loc_next, buf ^ 1);
      loc_next = key_loc(kt + 2);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const __nv_bfloat16 *kb = ksm + (size_t)buf * kKT * P, *vb = vsm + (size_t)buf * kKT * P;
    // ---- scores: rows [rg * WM * 16, +WM * 16) x keys [kg * WN * 8, +WN * 8)
    {
      float s[2][WM][WN][4] = {};
#pragma unroll 2
      for (int ks = 0; ks < kend; ks += 2) {
        uint32_t bf[WN][4];
#pragma unroll
        for (int j = 0; j < WN; ++j) {
          const int br = (kg * WN + j) * 8 + (lane & 7);
          ldsm4(bf[j], kb + br * P + swz(br, ks * 2 + (lane >> 3)) * 8);
        }
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
          for (int i = 0; i < WM; ++i) {
            const int ar = (rg * WM + i) * 16 + (lane & 15);
            uint32_t af[4];
            ldsm4(af, qs + ar * P + swz(ar, (ks + h) * 2 + (lane >> 4)) * 8);
#pragma unroll
            for (int j = 0; j < WN; ++j) mma16816(s[h][i][j], af, bf[j][2 * h], bf[j][2 * h + 1]);
          }
      }
#pragma unroll
      for (int i = 0; i < WM; ++i)
#pragma unroll
        for (int j = 0; j < WN; ++j) {
          const int r = (rg * WM + i) * 16 + (lane >> 2), c = (kg * WN + j) * 8 + (lane & 3) * 2;
          *reinterpret_cast<float2*>(ss + r * kSP + c) =
              make_float2((s[0][i][j][0] + s[1][i][j][0]) * sc2, (s[0][i][j][1] + s[1][i][j][1]) * sc2);
          *reinterpret_cast<float2*>(ss + (r + 8) * kSP + c) =
              make_float2((s[0][i][j][2] + s[1][i][j][2]) * sc2, (s[0][i][j][3] + s[1][i][j][3]) * sc2);
        }
    }
    __syncthreads();
    // ---- cap, bias, online softmax
    {
      constexpr int TPR = 256 / M, PER = kKT / TPR;  // threads per row, keys per thread (4, 8 or 16)
      const int r = tid / TPR, seg = tid % TPR;
      const int lim = see[r] - kt * kKT - seg * PER, low = from[r] - kt * kKT - seg * PER;
      float v[PER];
      float mx = -1e30f;
#pragma unroll
      for (int i = 0; i < PER; i += 4) {
        const float4 f = *reinterpret_cast<const float4*>(ss + r * kSP + seg * PER + i);
        v[i] = f.x, v[i + 1] = f.y, v[i + 2] = f.z, v[i + 3] = f.w;
      }
      if (a.cap > 0.f) {
#pragma unroll
        for (int i = 0; i < PER; ++i) v[i] = softcap_ex2(v[i], ce, cap2);
      }
      if (a.rel && lim > 0) {       // distance of key i: lim - 1 - i
        const float* rel = a.rel + (size_t)(g * R + (row0 + r) % R) * a.n_rel;
#pragma unroll
        for (int i = 0; i < PER; ++i) v[i] = fmaf(rel[max(min(lim - 1 - i, a.n_rel - 1), 0)], kLog2e, v[i]);
      }
      if (a.slope) {
        const float slope = row0 + r < row1 ? a.slope[g * R + (row0 + r) % R] * kLog2e : 0.f;
#pragma unroll
        for (int i = 0; i < PER; ++i) v[i] = fmaf(-slope, (float)(lim - 1 - i), v[i]);
      }
#pragma unroll
      for (int i = 0; i < PER; ++i) {
        v[i] = i < lim && i >= low ? v[i] : -INFINITY;
        mx = fmaxf(mx, v[i]);
      }
#pragma unroll
      for (int off = TPR / 2; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
      const float m_old = ms[r], m_new = a.wbias ? 0.f : fmaxf(m_old, mx);
      float sum = 0.f;
      __align__(16) __nv_bfloat16 e[PER];
      if (a.wbias) {
        const float wb = row0 + r < row1 ? a.wbias[g * R + (row0 + r) % R] * kLog2e : 0.f;
#pragma unroll
        for (int i = 0; i < PER; ++i) e[i] = f2bf(sigmoid_ex2(v[i] + wb));
      } else {
#pragma unroll
        for (int i = 0; i < PER; ++i) {
          e[i] = f2bf(exp2f(v[i] - m_new));
          sum += bf2f(e[i]);   // the weights as they enter the product add up to what they are divided by
        }
      }
#pragma unroll
      for (int off = TPR / 2; off > 0; off >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
      if constexpr (PER >= 8) {
#pragma unroll
        for (int i = 0; i < PER; i += 8)
          reinterpret_cast<uint4*>(pb + r * kKT)[swz(r, (seg * PER + i) / 8)] = *reinterpret_cast<uint4*>(e + i);
      } else {
        *reinterpret_cast<uint2*>(pb + r * kKT + swz(r, seg / 2) * 8 + (seg & 1) * 4) = *reinterpret_cast<uint2*>(e);
      }
      __syncwarp();
      if (seg == 0) {
        const float al = a.wbias ? 1.f : exp2f(m_old - m_new);
        alpha[r] = al;
        ms[r] = m_new;
        ls[r] = a.wbias ? 1.f : ls[r] * al + sum;
      }
    }
    __syncthreads();
    // ---- o += P V: all rows, output columns [warp * DW, +DW)
    if (warp * C::DW < a.vdim) {
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        const float a0 = alpha[i * 16 + (lane >> 2)], a1 = alpha[i * 16 + (lane >> 2) + 8];
#pragma unroll
        for (int j = 0; j < NT; ++j) acc[i][j][0] *= a0, acc[i][j][1] *= a0, acc[i][j][2] *= a1, acc[i][j][3] *= a1;
      }
#pragma unroll
      for (int kk = 0; kk < kKT / 16; ++kk) {
        uint32_t pf[MT][4];
#pragma unroll
        for (int i = 0; i < MT; ++i) {
          const int pr = i * 16 + (lane & 15);
          ldsm4(pf[i], pb + pr * kKT + swz(pr, kk * 2 + (lane >> 4)) * 8);
        }
        const int vr = kk * 16 + (lane & 15);
        if constexpr (NT == 1) {
          uint32_t v0, v1;
          ldsm2_t(v0, v1, vb + vr * P + swz(vr, warp) * 8);
#pragma unroll
          for (int i = 0; i < MT; ++i) mma16816(acc[i][0], pf[i], v0, v1);
        } else {
#pragma unroll
          for (int j = 0; j < NT; j += 2) {
            uint32_t vf[4];
            ldsm4_t(vf, vb + vr * P + swz(vr, warp * (C::DW / 8) + j + (lane >> 4)) * 8);
#pragma unroll
            for (int i = 0; i < MT; ++i) {
              mma16816(acc[i][j], pf[i], vf[0], vf[1]);
              mma16816(acc[i][j + 1], pf[i], vf[2], vf[3]);
            }
          }
        }
      }
    }
    __syncthreads();
  }
  // ---- result or partial
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = i * 16 + (lane >> 2) + half * 8;
      if (row0 + r >= row1) continue;
      const size_t row = head_row(r);
      float inv = 1.f;
      if (!a.partial && !a.wbias) {
        float l = ls[r], f = 1.f;
        if (a.sink) {   // one more term of the sum, without a key or a value
          const float s2 = a.sink[g * R + (row0 + r) % R] * kLog2e, mm = fmaxf(ms[r], s2);
          f = exp2f(ms[r] - mm);
          l = l * f + exp2f(s2 - mm);
        }
        inv = f / l;
      }
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        const int c = warp * C::DW + j * 8 + (lane & 3) * 2;
        if (c >= a.vdim) continue;
        const float x = acc[i][j][half * 2], y = acc[i][j][half * 2 + 1];
        if (a.partial)
          *reinterpret_cast<float2*>(a.part_acc + (row * a.nsplit + split) * a.vdim + c) = make_float2(x, y);
        else
          *reinterpret_cast<__nv_bfloat162*>(o + row * a.vdim + c) = __floats2bfloat162_rn(x * inv, y * inv);
      }
    }
  if (a.partial && tid < M && row0 + tid < row1) {
    float* ml = a.part_ml + (head_row(tid) * a.nsplit + split) * 2;
    ml[0] = ms[tid], ml[1] = ls[tid];
  }
}

// o[row] = sum_s acc_s 2^(m_s - M) / (2^(sink - M) + sum_s l_s 2^(m_s - M)) for the rows of the tiles of M rows that
// grouped_attn_kernel worked on (the plain sum where weights are not normalised), turned back and gated; one warp per row.
__global__ void __launch_bounds__(128) grouped_merge_kernel(__nv_bfloat16* __restrict__ o, const AttnArgs a, int M) {
  pdl_entry();
  const int R = a.group, n = a.nsplit, g = blockIdx.y, lane = threadIdx.x & 31;
  int row0, row1;
  if (a.tiles) {
    row0 = a.tiles[blockIdx.x * 2], row1 = a.tiles[blockIdx.x * 2 + 1];
  } else {
    const int tpt = (R + M - 1) / M, t = blockIdx.x / tpt;
    row0 = t * R + blockIdx.x % tpt * M;
    row1 = min(row0 + M, (t + 1) * R);
  }
  if (a.num_valid && row0 / R >= *a.num_valid) return;
  for (int r = row0 + (threadIdx.x >> 5); r < row1; r += 4) {
    const int h = g * R + r % R;
    const size_t row = (size_t)(r / R) * (a.kv_heads * R) + h;
    const float* ml = a.part_ml + row * n * 2;
    const float s2 = a.sink ? a.sink[h] * kLog2e : -1e30f;
    // lane s holds split s (at most 32)
    const float ms = lane < n ? ml[lane * 2] : -1e30f, ls = lane < n ? ml[lane * 2 + 1] : 0.f;
    const float mx = fmaxf(warp_max(ms), s2);
    const float f = ls > 0.f ? a.wbias ? 1.f : exp2f(ms - mx) : 0.f;
    const float sum = warp_sum(ls * f) + (a.sink ? exp2f(s2 - mx) : 0.f);
    float mul = a.wbias ? 1.f : 1.f / sum;
    if (a.gate) mul *= sigmoid_f(bf2f(static_cast<const __nv_bfloat16*>(a.gate)[(size_t)(r / R) * a.ld_gate + h]));
    const float* acc = a.part_acc + row * n * a.vdim;
    if (a.turn) {
      const int half = a.vdim / 2;
      const float2* turn = a.turn + (size_t)(r / R) * half;
      for (int c0 = 0; c0 < half; c0 += 32) {
        const int c = c0 + lane;
        float u = 0.f, v = 0.f;
        for (int s = 0; s < n; ++s) {
          const float fs = __shfl_sync(0xffffffffu, f, s);
          if (fs > 0.f && c < half) u = fmaf(acc[s * a.vdim + c], fs, u), v = fmaf(acc[s * a.vdim + c + half], fs, v);
        }
        if (c < half) {
          const float2 cs = turn[c];
          o[row * a.vdim + c] = f2bf(turned_back(u, v, cs, false) * mul);
          o[row * a.vdim + c + half] = f2bf(turned_back(u, v, cs, true) * mul);
        }
      }
      continue;
    }
    for (int c0 = 0; c0 < a.vdim; c0 += 32) {
      const int c = c0 + lane;
      float v = 0.f;
      for (int s = 0; s < n; ++s) {
        const float fs = __shfl_sync(0xffffffffu, f, s);
        if (fs > 0.f && c < a.vdim) v = fmaf(acc[s * a.vdim + c], fs, v);
      }
      if (c < a.vdim) o[row * a.vdim + c] = f2bf(v * mul);
    }
  }
}

// ------------------------------------------------------------------ one warp per row, fp32 arithmetic
template <typename T, int NI>
__global__ void __launch_bounds__(128) grouped_row_kernel(const T* __restrict__ q, const T* __restrict__ keys,
                                                          const T* __restrict__ values, T* __restrict__ o,
                                                          const AttnArgs a) {
  pdl_entry();
  constexpr int KB = 4;     // keys at a time
  const int row = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const int H = a.kv_heads * a.group;
  if (row >= a.rows * H) return;
  const int t = row / H, h = row % H, g = h / a.group;
  if (a.num_valid && t >= *a.num_valid) return;
  const int key0 = first_key(a, a.pos[t]), nkeys = a.pos[t] + 1 - key0;
  const int* pt = a.page_table + (size_t)a.slots[t] * a.ld_pt + key0;
  const float slope = a.slope ? a.slope[h] : 0.f, wb = a.wbias ? a.wbias[h] : 0.f;
  const T *kb = keys + g * a.dim, *vb = values + g * a.vdim;
  const size_t ldk = (size_t)a.kv_heads * a.dim, ldv = (size_t)a.kv_heads * a.vdim;
  const float* rel = a.rel ? a.rel + (size_t)h * a.n_rel : nullptr;
  float qv[NI], acc[NI];
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int c = i * 32 + lane;
    qv[i] = c < a.dim ? ld_f(q + (size_t)row * a.dim + c) : 0.f;
    acc[i] = 0.f;
  }
  float m = -1e30f, l = 0.f;
  if (a.sink) m = a.sink[h], l = 1.f;
  for (int k0 = 0; k0 < nkeys; k0 += 32) {
    const int mine = pt[min(k0 + lane, nkeys - 1)];
    const int n = min(32, nkeys - k0);
    for (int k = 0; k < n; k += KB) {
      size_t loc[KB];
      float s[KB];
#pragma unroll
      for (int j = 0; j < KB; ++j) {
        loc[j] = (size_t)__shfl_sync(0xffffffffu, mine, k + j);    // places past the last key repeat it
        const T* kp = kb + loc[j] * ldk;
        s[j] = 0.f;
#pragma unroll
        for (int i = 0; i < NI; ++i)
          if (i * 32 + lane < a.dim) s[j] = fmaf(qv[i], ld_f(kp + i * 32 + lane), s[j]);
      }
      float mn = m;
#pragma unroll
      for (int j = 0; j < KB; ++j) {
        s[j] = warp_sum(s[j]) * a.scale;
        if (a.cap > 0.f) s[j] = a.cap * tanhf(s[j] / a.cap);
        if (rel) s[j] += rel[min(max(nkeys - 1 - (k0 + k + j), 0), a.n_rel - 1)];
        s[j] = fmaf(-slope, (float)(nkeys - 1 - (k0 + k + j)), s[j]);
        if (k + j >= n) s[j] = -INFINITY;
        mn = fmaxf(mn, s[j]);
      }
      if (!a.wbias) {
        const float al = expf(m - mn);
        m = mn;
        l *= al;
#pragma unroll
        for (int i = 0; i < NI; ++i) acc[i] *= al;
      }
#pragma unroll
      for (int j = 0; j < KB; ++j) {
        const float p = a.wbias ? sigmoid_f(s[j] + wb) : expf(s[j] - mn);
        const T* vp = vb + loc[j] * ldv;
        l += p;
#pragma unroll
        for (int i = 0; i < NI; ++i)
          if (i * 32 + lane < a.vdim) acc[i] = fmaf(p, ld_f(vp + i * 32 + lane), acc[i]);
      }
    }
  }
  float mul = a.wbias ? 1.f : 1.f / l;
  if (a.gate) mul *= sigmoid_f(ld_f(static_cast<const T*>(a.gate) + (size_t)t * a.ld_gate + h));
  if (a.turn) {
    __shared__ float whole[4][NI * 32];
    float* w = whole[threadIdx.x >> 5];
#pragma unroll
    for (int i = 0; i < NI; ++i) w[i * 32 + lane] = acc[i];
    __syncwarp();
    const int half = a.vdim / 2;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int c = i * 32 + lane;
      if (c >= a.vdim) continue;
      const int u = c < half ? c : c - half;
      acc[i] = turned_back(w[u], w[u + half], a.turn[(size_t)t * half + u], c >= half);
    }
  }
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int c = i * 32 + lane;
    if (c < a.vdim) st_f(o + (size_t)row * a.vdim + c, acc[i] * mul);
  }
}

// ------------------------------------------------------------------ keys and values of long portions, side by side
// ctx_k[dst + j] = keys of key j of every listed request; ctx_vt[:, dst + j] = its values; zeros in the padding behind them.
// list: [segs][4] = slot, keys, first row of the copy (a multiple of 64), first key.  One CTA: 64 keys x 64 columns of k or v.
__global__ void __launch_bounds__(256) kv_gather_kernel(const __nv_bfloat16* __restrict__ keys,
                                                        const __nv_bfloat16* __restrict__ values,
                                                        __nv_bfloat16* __restrict__ ctx_k, __nv_bfloat16* __restrict__ ctx_vt,
                                                        const int* __restrict__ list, int segs, int total,
                                                        const int* __restrict__ page_table, int ld_pt, int kw, int vw) {
  pdl_entry();
  __shared__ __nv_bfloat16 tile[64][66];
  const int row0 = blockIdx.x * 64, kblocks = (kw + 63) / 64, tid = threadIdx.x;
  int lo = 0, hi = segs - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (list[mid * 4 + 2] <= row0) lo = mid; else hi = mid - 1;
  }
  const int j0 = row0 - list[lo * 4 + 2], n = list[lo * 4 + 1];
  const int* pt = page_table + (size_t)list[lo * 4] * ld_pt + list[lo * 4 + 3];
  const bool is_k = (int)blockIdx.y < kblocks;
  const int c0 = (is_k ? blockIdx.y : blockIdx.y - kblocks) * 64, w = is_k ? kw : vw;
  const __nv_bfloat16* src = is_k ? keys : values;
  for (int i = tid; i < 64 * 8; i += 256) {
    const int r = i >> 3, c = (i & 7) * 8;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (j0 + r < n && c0 + c < w) v = *reinterpret_cast<const uint4*>(src + (size_t)pt[j0 + r] * w + c0 + c);
    if (is_k) {
      if (row0 + r < total && c0 + c < w) *reinterpret_cast<uint4*>(ctx_k + (size_t)(row0 + r) * w + c0 + c) = v;
    } else {
      uint32_t* d = reinterpret_cast<uint32_t*>(&tile[r][c]);
      d[0] = v.x, d[1] = v.y, d[2] = v.z, d[3] = v.w;
    }
  }
  if (is_k) return;
  __syncthreads();
  for (int i = tid; i < 64 * 8; i += 256) {
    const int c = i >> 3, r = (i & 7) * 8;
    if (c0 + c >= w) continue;
    __align__(16) __nv_bfloat16 v[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] = tile[r + e][c];
    *reinterpret_cast<uint4*>(ctx_vt + (size_t)(c0 + c) * total + row0 + r) = *reinterpret_cast<uint4*>(v);
  }
}

template <int P, int MT>
int launch_attn(const void* q, const void* k, const void* v, void* o, const AttnArgs& a, cudaStream_t st) {
  using C = AttnCfg<P, MT>;
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(grouped_attn_kernel<P, MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM) !=
        cudaSuccess)
      return 671;
    set = true;
  }
  dsv4_launch(grouped_attn_kernel<P, MT>, dim3(a.n_tiles, a.nsplit, a.kv_heads), 256, C::SMEM, st, (const __nv_bfloat16*)q,
              (const __nv_bfloat16*)k, (const __nv_bfloat16*)v, (__nv_bfloat16*)o, a);
  if (a.partial)
    dsv4_launch(grouped_merge_kernel, dim3(a.n_tiles, a.kv_heads), 128, 0, st, (__nv_bfloat16*)o, a, C::M);
  return (int)cudaGetLastError();
}
template <int P>
int dispatch_attn(int m, const void* q, const void* k, const void* v, void* o, const AttnArgs& a, cudaStream_t st) {
  switch (m) {
    case 16: return launch_attn<P, 1>(q, k, v, o, a, st);
    case 32: return launch_attn<P, 2>(q, k, v, o, a, st);
    case 64: return launch_attn<P, 4>(q, k, v, o, a, st);
    default: return 672;
  }
}
template <typename T>
int launch_row(const void* q, const void* k, const void* v, void* o, const AttnArgs& a, cudaStream_t st) {
  const int grid = (a.rows * a.kv_heads * a.group + 3) / 4, w = a.dim > a.vdim ? a.dim : a.vdim;
  const T *tq = (const T*)q, *tk = (const T*)k, *tv = (const T*)v;
  if (w <= 64)
    dsv4_launch(grouped_row_kernel<T, 2>, grid, 128, 0, st, tq, tk, tv, (T*)o, a);
  else if (w <= 128)
    dsv4_launch(grouped_row_kernel<T, 4>, grid, 128, 0, st, tq, tk, tv, (T*)o, a);
  else if (w <= 256)
    dsv4_launch(grouped_row_kernel<T, 8>, grid, 128, 0, st, tq, tk, tv, (T*)o, a);
  else if (w <= 512)
    dsv4_launch(grouped_row_kernel<T, 16>, grid, 128, 0, st, tq, tk, tv, (T*)o, a);
  else
    return 673;
  return (int)cudaGetLastError();
}

template <typename T, int W>
void launch_rotate(const void* qkv, void* q, void* keys, void* values, const RotateArgs& a, int rows, cudaStream_t st) {
  const int nv = a.kv_heads * a.vdim, chunks = ((a.heads + a.kv_heads) * a.dim + nv + 256 * W - 1) / (256 * W);
  const bool norms = a.gain || a.unit_v, in_regs = norms && W > 1 && chunks <= 4;
  const size_t smem = a.pairs * sizeof(float2) + (a.unit_v ? (in_regs ? nv / W : a.kv_heads) * sizeof(float) : 0);
  auto go = [&](auto kern) {
    dsv4_launch(kern, rows, 256, smem, st, (const T*)qkv, (T*)q, (T*)keys, (T*)values, a);
  };
  if constexpr (W > 1) {
    if (in_regs && chunks <= 1) return go(rotate_store_kernel<T, W, 1>);
    if (in_regs && chunks <= 2) return go(rotate_store_kernel<T, W, 2>);
    if (in_regs) return go(rotate_store_kernel<T, W, 4>);
  }
  go(rotate_store_kernel<T, W, 0>);
}

}  // namespace

// qkv [rows, ld]: q (heads x dim) | k (kv_heads x dim) | v (kv_heads x vdim); q_out [rows, heads * dim]; caches
// [locations, kv_heads * dim] and [locations, kv_heads * vdim].  pairs: rotated pairs per head; every 0: no temperature; gain,
// unit_v: norms as in RotateArgs.
DSV4_API int dsv4_rotate_store(const void* qkv, int ld, const float* bias, const float* freq, int pairs, float coef, int every,
                               const float* gain, int unit_v, float eps, float v_mul, const int* pos, const int* out_loc, void* q_out, void* keys, void* values, int rows,
                               int heads, int kv_heads, int dim, int vdim, int fp32, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (pairs < 0 || 2 * pairs > dim || pairs > 4096 || (pairs && !freq) || every < 0 || kv_heads > 1024) return 674;
  const RotateArgs a{ld, bias, freq, pairs, coef, every, gain, unit_v, eps, v_mul, pos, out_loc, heads, kv_heads, dim, vdim};
  const bool wide = dim % 8 == 0 && vdim % 8 == 0 && ld % 8 == 0 && ((uintptr_t)qkv & 15) == 0;
  if (fp32)
    wide ? launch_rotate<float, 4>(qkv, q_out, keys, values, a, rows, st)
         : launch_rotate<float, 1>(qkv, q_out, keys, values, a, rows, st);
  else
    wide ? launch_rotate<__nv_bfloat16, 8>(qkv, q_out, keys, values, a, rows, st)
         : launch_rotate<__nv_bfloat16, 1>(qkv, q_out, keys, values, a, rows, st);
  return (int)cudaGetLastError();
}

// Norms per head and rotation in either layout, values included (see HeadStoreArgs).  qkv, q_out and the caches as above; turn [rows,
// vdim / 2, 2] receives the values' cos and sin if vfreq is given.
DSV4_API int dsv4_head_store(const void* qkv, int ld, const float* bias, const float* gain, float eps, const float* freq,
                             int pairs, int halves, float mul, const float* vfreq, float* turn, const int* pos,
                             const int* out_loc, void* q_out, void* keys, void* values, int rows, int heads, int kv_heads,
                             int dim, int vdim, int fp32, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (pairs < 0 || 2 * pairs > dim || (pairs && !freq) || (vfreq && (vdim % 2 || !turn))) return 680;
  const HeadStoreArgs a{ld, bias, gain, eps, freq, pairs, halves, mul, vfreq, reinterpret_cast<float2*>(turn), pos, out_loc,
                        heads, kv_heads, dim, vdim};
  const int n = (heads + kv_heads) * dim + kv_heads * vdim;
  const size_t smem = (size_t)(n + 3) / 4 * 16 + (pairs + (vfreq ? vdim / 2 : 0)) * sizeof(float2);
  if (smem > 200 * 1024) return 681;
  const bool wide = dim % 8 == 0 && vdim % 8 == 0 && ld % 8 == 0 && ((uintptr_t)qkv & 15) == 0;
  const int units = (n / 8 + kUnitThreads - 1) / kUnitThreads, lanes = dim / 8;
  if (wide && pairs % 4 == 0 && lanes <= 32 && (lanes & (lanes - 1)) == 0 && units <= 8) {
    const int threads = rows <= 512 && n <= 8192 ? (n / 8 + 31) / 32 * 32 : kUnitThreads;
    const size_t small = (pairs + (vfreq ? vdim / 2 : 0)) * sizeof(float2);
    auto go = [&](auto kern, auto type) {
      using T = decltype(type);
      dsv4_launch(kern, rows, threads, small, st, (const T*)qkv, (T*)q_out, (T*)keys, (T*)values, a);
    };
    auto pick = [&](auto type) {
      using T = decltype(type);
      if (units <= 1 || threads != kUnitThreads) go(head_store_units_kernel<T, 1>, type);
      else if (units <= 3) go(head_store_units_kernel<T, 3>, type);
      else if (units <= 5) go(head_store_units_kernel<T, 5>, type);
      else go(head_store_units_kernel<T, 8>, type);
    };
    if (fp32) pick(float());
    else pick(__nv_bfloat16());
    return (int)cudaGetLastError();
  }
  auto go = [&](auto kern, auto type) {
    using T = decltype(type);
    if (smem > 48 * 1024 && cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess)
      return 682;
    dsv4_launch(kern, rows, 256, smem, st, (const T*)qkv, (T*)q_out, (T*)keys, (T*)values, a);
    return (int)cudaGetLastError();
  };
  if (fp32) return wide ? go(head_store_kernel<float, 4>, float()) : go(head_store_kernel<float, 1>, float());
  return wide ? go(head_store_kernel<__nv_bfloat16, 8>, __nv_bfloat16()) : go(head_store_kernel<__nv_bfloat16, 1>, __nv_bfloat16());
}

// q [rows, heads * dim], o [rows, heads * vdim].  m: rows per CTA (16, 32 or 64; 0 = the one-warp-per-row kernel, which takes
// every token).  tiles: [n_tiles][2] row ranges (see AttnArgs), or null: n_tiles covers every token's own rows.  nsplit > 1
// (at most 32) needs part_acc [rows * heads, nsplit, vdim] and part_ml [rows * heads, nsplit, 2], and so do turn and gate unless
// m is 0.
DSV4_API int dsv4_grouped_attention(const void* q, const void* keys, const void* values, void* o, const int* slots,
                                    const int* pos, const int* page_table, int ld_pt, const int* tiles, int n_tiles,
                                    const int* num_valid, int rows, int kv_heads, int group, int dim, int vdim, float scale,
                                    float cap, const float* sink, const float* rel, int n_rel, const float* slope,
                                    int chunk, int window, const float* wbias, const float* turn, const void* gate, int ld_gate,
                                    int m, int nsplit, float* part_acc, float* part_ml, int fp32, cudaStream_t st) {
  if (rows <= 0) return 0;
  const int partial = nsplit > 1 || (m && (turn || gate));
  if (nsplit < 1 || nsplit > 32 || (partial && (!part_acc || !part_ml)) || (rel && n_rel < 1)) return 675;
  if (kv_heads < 1 || kv_heads > 65535 || group < 1 || chunk < 0 || window < 0 || (chunk && window)) return 676;
  if ((wbias && sink) || (turn && vdim % 2)) return 683;
  const AttnArgs a{slots, pos, page_table, ld_pt, tiles, n_tiles, num_valid, rows, kv_heads, group, dim, vdim, scale, cap,
                   sink, rel, n_rel, slope, chunk, window, wbias, reinterpret_cast<const float2*>(turn), gate, ld_gate, nsplit,
                   partial, part_acc, part_ml};
  if (m == 0)
    return fp32 ? launch_row<float>(q, keys, values, o, a, st) : launch_row<__nv_bfloat16>(q, keys, values, o, a, st);
  if (fp32 || dim % 8 || vdim % 8) return 677;
  if (n_tiles <= 0) return 0;
  const int w = dim > vdim ? dim : vdim;
  if (w <= 64) return dispatch_attn<64>(m, q, keys, values, o, a, st);
  if (w <= 128) return dispatch_attn<128>(m, q, keys, values, o, a, st);
  if (w <= 256) return dispatch_attn<256>(m, q, keys, values, o, a, st);
  return 678;
}

// ctx_k [total, kw], ctx_vt [vw, total]; total and the first rows of list are multiples of 64.
DSV4_API int dsv4_kv_gather(const void* keys, const void* values, void* ctx_k, void* ctx_vt, const int* list, int segs,
                            int total, const int* page_table, int ld_pt, int kw, int vw, cudaStream_t st) {
  if (total <= 0) return 0;
  if (kw % 8 || vw % 8 || total % 64 || segs < 1) return 679;
  dsv4_launch(kv_gather_kernel, dim3(total / 64, (kw + 63) / 64 + (vw + 63) / 64), 256, 0, st, (const __nv_bfloat16*)keys,
              (const __nv_bfloat16*)values, (__nv_bfloat16*)ctx_k, (__nv_bfloat16*)ctx_vt, list, segs, total, page_table,
              ld_pt, kw, vw);
  return (int)cudaGetLastError();
}
