// Gated linear attention (gla.cuh) token by token (decode, short portions, models served in 32-bit floats), and what stands
// around it:
//   mlstm_gates      exponential input and sigmoid forget gates with a running maximum -> log g, factor of k, floor
//   causal_conv      short causal convolution per channel with bias and silu, and the inputs it keeps
//   gla_scan         the recurrence over a portion, state in registers
//   gla_step         one token per request: the state streams through once
//   gla_norm_*       normaliser, skip, gate and norms behind the recurrence
#include "gla.cuh"

namespace {

// ------------------------------------------------------------------ gates with a running maximum
struct MlstmArgs {
  const float* z;          // [rows][2 heads]: input gates, then forget gates
  const float* bias;       // [2 heads]
  float cap;
  float* top;              // [slots + 1][heads]: the running maximum m
  float *log_g, *fac, *floor;   // [rows][heads]
  const int *slots, *pos, *seg_off, *num_valid;
  int heads;
};

// i = cap tanh(z_i / cap), f = log sigmoid(cap tanh(z_f / cap));  m_t = max(f_t + m_{t-1}, i_t), m_{-1} = 0;
// log g = f_t + m_{t-1} - m_t, factor e^{i_t - m_t}, floor e^{-m_t}.  m is a prefix of the maps m -> max(F + m, M), which compose
// to (F1 + F2, max(M1 + F2, M2)).  One CTA per (segment, head).
__global__ void __launch_bounds__(1024) mlstm_gates_kernel(const MlstmArgs a) {
  pdl_entry();
  __shared__ float fs[32], ms[32];
  const int seg = blockIdx.x, head = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  if (a.num_valid && seg >= *a.num_valid) return;
  const int t0 = a.seg_off ? a.seg_off[seg] : seg, t1 = a.seg_off ? a.seg_off[seg + 1] : seg + 1;
  if (t1 <= t0) return;
  float* top = a.top + (size_t)a.slots[t0] * a.heads + head;
  float m_in = a.pos[t0] == 0 ? 0.f : *top;
  const float bi = a.bias[head], bf = a.bias[a.heads + head];
  for (int c0 = t0; c0 < t1; c0 += blockDim.x) {
    const int t = c0 + threadIdx.x;
    float i = -INFINITY, f = 0.f;
    if (t < t1) {
      i = a.cap * tanhf((a.z[(size_t)t * 2 * a.heads + head] + bi) / a.cap);
      f = -softplus_of(-a.cap * tanhf((a.z[(size_t)t * 2 * a.heads + a.heads + head] + bf) / a.cap));
    }
    float F = f, M = i;
#pragma unroll
    for (int off = 1; off < 32; off <<= 1) {
      const float fp = __shfl_up_sync(0xffffffffu, F, off), mp = __shfl_up_sync(0xffffffffu, M, off);
      if (lane >= off) M = fmaxf(mp + F, M), F += fp;
    }
    __syncthreads();
    if (lane == 31) fs[warp] = F, ms[warp] = M;
    __syncthreads();
    float m = m_in;                     // ahead of this warp, then of this token
    for (int w = 0; w < warp; ++w) m = fmaxf(fs[w] + m, ms[w]);
    const float mine = fmaxf(F + m, M);
    const float up = __shfl_up_sync(0xffffffffu, mine, 1);
    const float before = lane ? up : m;
    if (t < t1) {
      const size_t at = (size_t)t * a.heads + head;
      a.log_g[at] = fminf(f + before - mine, 0.f);
      a.fac[at] = expf(fminf(i - mine, 0.f));
      a.floor[at] = expf(-mine);
    }
    for (int w = 0; w < nw; ++w) m_in = fmaxf(fs[w] + m_in, ms[w]);
  }
  if (threadIdx.x == 0) *top = m_in;
}

// ------------------------------------------------------------------ short convolution
struct CausalConvArgs {
  int ld, C;               // row stride of p, channels
  const float* taps;       // [n][C], the last row is the current token's
  const float* bias;       // [C]
  const int *slots, *pos, *seg_off, *num_valid;
  const int* tiles;        // [n_tiles][2]: segment, token within it; or null: a segment of one token per row
  int n, span;             // taps, tokens per tile
};

// One thread: W channels over a tile of tokens of one segment, the last N - 1 inputs in registers.  The tile that begins the
// segment alone reads `before` (span >= N - 1) and afterwards leaves the segment's last inputs there.
template <typename T, int N, int W>
__global__ void __launch_bounds__(128) causal_conv_kernel(const T* __restrict__ p, T* before, T* __restrict__ out,
                                                          const CausalConvArgs a) {
  pdl_entry();
  const int c = (blockIdx.x * 128 + threadIdx.x) * W;
  if (c >= a.C) return;
  const int seg = a.tiles ? a.tiles[blockIdx.y * 2] : blockIdx.y, o0 = a.tiles ? a.tiles[blockIdx.y * 2 + 1] : 0;
  if (a.num_valid && seg >= *a.num_valid) return;
  const int t0 = a.seg_off ? a.seg_off[seg] : seg, len = a.seg_off ? a.seg_off[seg + 1] - t0 : 1;
  const int m = min(a.span, len - o0);
  const bool fresh = a.pos[t0] == 0;
  T* kept = before + (size_t)a.slots[t0] * (N - 1) * a.C + c;
  const T* src = p + (size_t)t0 * a.ld + c;
  // input o of the segment, o < 0: from the slot
  auto input = [&](int o, float (&x)[W]) {
    if (o < 0 && fresh) {
#pragma unroll
      for (int j = 0; j < W; ++j) x[j] = 0.f;
      return;
    }
    const T* s = o >= 0 ? src + (size_t)o * a.ld : kept + (size_t)(N - 1 + o) * a.C;
    if constexpr (W == 4) {
      const float4 f = ld_f4(s);
      x[0] = f.x, x[1] = f.y, x[2] = f.z, x[3] = f.w;
    } else {
      x[0] = ld_f(s);
    }
  };
  float w[N][W], b[W], x[N][W];          // x[j]: j tokens back
#pragma unroll
  for (int j = 0; j < N; ++j) ld_w<W>(a.taps + (size_t)(N - 1 - j) * a.C + c, w[j]);
  ld_w<W>(a.bias + c, b);
#pragma unroll
  for (int j = 1; j < N; ++j) input(o0 - j, x[j - 1]);
#pragma unroll 4
  for (int o = o0; o < o0 + m; ++o) {
#pragma unroll
    for (int j = N - 1; j > 0; --j)
#pragma unroll
      for (int i = 0; i < W; ++i) x[j][i] = x[j - 1][i];
    input(o, x[0]);
    float y[W];
#pragma unroll
    for (int i = 0; i < W; ++i) {
      y[i] = b[i];
#pragma unroll
      for (int j = 0; j < N; ++j) y[i] = fmaf(x[j][i], w[j][i], y[i]);
      y[i] *= sigmoid_for<T>(y[i]);
    }
    st_w<W>(out + (size_t)(t0 + o) * a.C + c, y);
  }
  if (o0 == 0) {
    float keep[N > 1 ? N - 1 : 1][W];
#pragma unroll
    for (int j = 0; j < N - 1; ++j) input(len - (N - 1) + j, keep[j]);
#pragma unroll
    for (int j = 0; j < N - 1; ++j) st_w<W>(kept + (size_t)j * a.C, keep[j]);
  }
}

// ------------------------------------------------------------------ recurrence
constexpr int kTC = 8;        // tokens staged at a time
constexpr int kKK = 16;       // keys per thread
constexpr int kGS = kKK + 4;  // floats between two key groups in shared memory (keeps 16-byte reads conflict-free)

// One CTA per (segment, head, vb columns).  A thread owns kKK keys x 4 columns of the state; sums over keys are shuffles over the
// G neighbouring threads of a column group.
template <typename T, int DP, int MODE>
__global__ void __launch_bounds__(512) gla_scan_kernel(const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v,
                                                       const int* __restrict__ seg_off, const int* __restrict__ num_valid,
                                                       int vb, const GlaArgs a) {
  pdl_entry();
  constexpr int G = DP / kKK, LD = G * kGS;
  __shared__ __align__(16) float qs[kTC][LD], ks[kTC][LD], gs[MODE == kForget ? kTC : 1][MODE == kForget ? LD : 1];
  __shared__ HeadGate gate[kTC];     // keep (g itself), factor of k (applied to the values)
  extern __shared__ __align__(16) float vs[];          // [kTC][vb]
  const int seg = blockIdx.x, head = blockIdx.y, v0 = blockIdx.z * vb, tid = threadIdx.x, NT = blockDim.x;
  if (num_valid && seg >= *num_valid) return;
  const int t0 = seg_off ? seg_off[seg] : seg, t1 = seg_off ? seg_off[seg + 1] : seg + 1;
  const int n = t1 - t0, d = a.d, ew = a.ew;
  if (n <= 0) return;
  const bool fresh = a.pos[t0] == 0;
  const int g = tid % G, col = v0 + tid / G * 4, at_k = head / a.group * d;
  const bool active = tid / G * 4 < vb && col < ew;

  float s[kKK][4];
  float* st = a.state + ((size_t)a.slots[t0] * a.heads + head) * d * ew;
#pragma unroll
  for (int i = 0; i < kKK; ++i) {
    const int key = g * kKK + i;
    s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
    if (!fresh && key < d && active) ld_w<4>(st + (size_t)key * ew + col, s[i]);
  }
  for (int c0 = 0; c0 < n; c0 += kTC) {
    const int m = min(kTC, n - c0);
    __syncthreads();
    if constexpr (MODE != kForget) {
      for (int tok = tid; tok < m; tok += NT) {
        const HeadGate f = head_gate<MODE>(a, t0 + c0 + tok, head);
        gate[tok] = {expf(f.log_g), f.fac};
      }
    }
    for (int i = tid; i < m * DP; i += NT) {
      const int tok = i / DP, c = i % DP, at = c / kKK * kGS + c % kKK;
      const bool in = c < d;                     // keys past d are zero: they never touch the state
      const size_t row = t0 + c0 + tok;
      float qv = 0.f, kv = 0.f;
      if (in) qv = ld_f(q + row * a.ldq + at_k + c);
      if constexpr (MODE == kForget) {
        const int ch = head * d + c;
        ChannelGate f{0.f, 0.f};
        if (in) f = channel_gate(a.raw[row * a.heads * d + ch] + a.bias[ch], a.par[ch]);
        kv = f.write, gs[tok][at] = f.keep;
        qv *= sigmoid_f(qv);
      } else if (in) {
        kv = ld_f(k + row * a.ldk + at_k + c);
      }
      qs[tok][at] = qv * a.q_mul, ks[tok][at] = kv;
    }
    for (int i = tid; i < m * vb; i += NT) {
      const int c = v0 + i % vb;
      vs[i] = c < a.e ? ld_f(v + (size_t)(t0 + c0 + i / vb) * a.ldv + head * a.e + c) : MODE == kGiven && c == a.e ? 1.f : 0.f;
    }
    __syncthreads();
    for (int tok = 0; tok < m; ++tok) {
      const float *qp = qs[tok] + g * kGS, *kp = ks[tok] + g * kGS;
      float vv[4] = {}, pq[4] = {};
      if (active) ld_w<4>(vs + tok * vb + tid / G * 4, vv);
      const float all = MODE == kForget ? 0.f : gate[tok].log_g;
      if constexpr (MODE != kForget) {
#pragma unroll
        for (int j = 0; j < 4; ++j) vv[j] *= gate[tok].fac;
      }
#pragma unroll
      for (int i = 0; i < kKK; i += 4) {
        float gg[4] = {all, all, all, all}, kk[4], qq[4];
        if constexpr (MODE == kForget) ld_w<4>(gs[tok] + g * kGS + i, gg);
        ld_w<4>(kp + i, kk);
        ld_w<4>(qp + i, qq);
#pragma unroll
        for (int h = 0; h < 4; ++h)
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            s[i + h][j] = fmaf(gg[h], s[i + h][j], kk[h] * vv[j]);
            pq[j] = fmaf(qq[h], s[i + h][j], pq[j]);
          }
      }
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int off = 1; off < G; off <<= 1) pq[j] += __shfl_xor_sync(0xffffffffu, pq[j], off);
      if (g == 0 && active) st_w<4>(a.out + ((size_t)(t0 + c0 + tok) * a.heads + head) * ew + col, pq);
    }
  }
#pragma unroll
  for (int i = 0; i < kKK; ++i) {
    const int key = g * kKK + i;
    if (key < d && active) st_w<4>(st + (size_t)key * ew + col, s[i]);
  }
}

// One CTA per (row, head), one token: a thread takes four columns of every KG-th key, so a row of the state is one contiguous
// access; the KG partial sums of a column meet in shared memory.
template <typename T, int MODE>
__global__ void __launch_bounds__(256, 3) gla_step_kernel(const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v,
                                                       const int* __restrict__ num_valid, const GlaArgs a) {
  pdl_entry();
  constexpr int B = 8;             // keys in flight
  __shared__ float qs[256], ks[256], gs[MODE == kForget ? 256 : 1];
  __shared__ float4 part[256];
  const int row = blockIdx.x, head = blockIdx.y, tid = threadIdx.x, d = a.d, ew = a.ew;
  if (num_valid && row >= *num_valid) return;
  const int nq = ew / 4, KG = 256 / nq, kg = tid / nq, col = tid % nq * 4, at_k = head / a.group * d;
  const bool fresh = a.pos[row] == 0, active = kg < KG;
  float4* st = reinterpret_cast<float4*>(a.state + ((size_t)a.slots[row] * a.heads + head) * d * ew + col);
  float4 s[B];
  auto fetch = [&](int k0) {
#pragma unroll
    for (int i = 0; i < B; ++i) {
      const int key = k0 + i * KG + kg;
      s[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (active && !fresh && key < d) s[i] = st[(size_t)key * nq];
    }
  };
  fetch(0);
  float keep = 0.f, fac = 1.f;
  if constexpr (MODE != kForget) {
    const HeadGate f = head_gate<MODE>(a, row, head);
    keep = expf(f.log_g), fac = f.fac;
  }
  for (int c = tid; c < d; c += 256) {
    float qv = ld_f(q + (size_t)row * a.ldq + at_k + c);
    if constexpr (MODE == kForget) {
      const int ch = head * d + c;
      const ChannelGate f = channel_gate(a.raw[(size_t)row * a.heads * d + ch] + a.bias[ch], a.par[ch]);
      ks[c] = f.write, gs[c] = f.keep;
      qv *= sigmoid_f(qv);
    } else {
      ks[c] = ld_f(k + (size_t)row * a.ldk + at_k + c);
    }
    qs[c] = qv * a.q_mul;
  }
  float vv[4] = {};
  if (active)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int c = col + j;
      if (c < a.e) vv[j] = fac * ld_f(v + (size_t)row * a.ldv + head * a.e + c);
      else if (MODE == kGiven && c == a.e) vv[j] = fac;
    }
  __syncthreads();
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
  for (int k0 = 0; k0 < d; k0 += B * KG) {
    if (k0 > 0) fetch(k0);
#pragma unroll
    for (int i = 0; i < B; ++i) {
      const int key = k0 + i * KG + kg;
      if (!active || key >= d) continue;
      const float g = MODE == kForget ? gs[MODE == kForget ? key : 0] : keep, kk = ks[key], qq = qs[key];
      float4 x = s[i];
      x.x = fmaf(g, x.x, kk * vv[0]), x.y = fmaf(g, x.y, kk * vv[1]), x.z = fmaf(g, x.z, kk * vv[2]), x.w = fmaf(g, x.w, kk * vv[3]);
      o.x = fmaf(qq, x.x, o.x), o.y = fmaf(qq, x.y, o.y), o.z = fmaf(qq, x.z, o.z), o.w = fmaf(qq, x.w, o.w);
      st[(size_t)key * nq] = x;
    }
  }
  part[tid] = o;
  __syncthreads();
  if (tid < nq) {
    for (int i = 1; i < KG; ++i) {
      const float4 x = part[i * nq + tid];
      o.x += x.x, o.y += x.y, o.z += x.z, o.w += x.w;
    }
    reinterpret_cast<float4*>(a.out + ((size_t)row * a.heads + head) * ew)[tid] = o;
  }
}

// ------------------------------------------------------------------ behind the recurrence
struct HeadNormArgs {
  const float* o;          // [rows][heads][ew]
  const float* floor;      // [rows][heads]: o is divided by max(|o[e]|, floor) + 1e-6 first; or null
  const float* gain;       // [e], or [heads * e] (per_head)
  int per_head, ldg, ldy;  // row strides of gate and y
  float eps, mul;
  int heads, e, ew, total;
};
// y = o / rms(o) * gain * mul (* sigmoid(gate)), one warp per R consecutive (row, head)s of up to NI x 128 values, e and the strides
// multiples of 4
template <typename T, int NI, int R>
__global__ void __launch_bounds__(256) gla_norm_heads_kernel(const T* __restrict__ gate, T* __restrict__ y, const HeadNormArgs a) {
  pdl_entry();
  const int r0 = (blockIdx.x * 8 + (threadIdx.x >> 5)) * R;
  const int lane = threadIdx.x & 31;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 o[R][NI], g[R][NI];
  float den[R], ss[R];
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int at = min(r0 + i, a.total - 1), head = at % a.heads;
    const size_t r = at, row = at / a.heads;
#pragma unroll
    for (int n = 0; n < NI; ++n) {
      const int c = (n * 32 + lane) * 4;
      o[i][n] = c < a.e ? ld_f4(a.o + r * a.ew + c) : zero;
      g[i][n] = gate && c < a.e ? ld_f4(gate + row * a.ldg + head * a.e + c) : zero;
    }
    den[i] = a.floor ? fmaxf(fabsf(a.o[r * a.ew + a.e]), a.floor[r]) + 1e-6f : 1.f;
  }
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const float f = 1.f / den[i];
    ss[i] = 0.f;
#pragma unroll
    for (int n = 0; n < NI; ++n) {
      float4& x = o[i][n];
      x.x *= f, x.y *= f, x.z *= f, x.w *= f;
      ss[i] += (x.x * x.x + x.y * x.y) + (x.z * x.z + x.w * x.w);
    }
  }
#pragma unroll
  for (int off = 16; off > 0; off >>= 1)
#pragma unroll
    for (int i = 0; i < R; ++i) ss[i] += __shfl_xor_sync(0xffffffffu, ss[i], off);
#pragma unroll
  for (int i = 0; i < R; ++i) {
    if (r0 + i >= a.total) break;
    const size_t row = (r0 + i) / a.heads;
    const int head = (r0 + i) % a.heads;
    const float inv = a.mul / sqrtf(ss[i] / a.e + a.eps);
#pragma unroll
    for (int n = 0; n < NI; ++n) {
      const int c = (n * 32 + lane) * 4;
      if (c >= a.e) continue;
      const float4 gn = ld_f4(a.gain + (a.per_head ? head * a.e : 0) + c), x = o[i][n], z = g[i][n];
      float4 w = make_float4(x.x * inv * gn.x, x.y * inv * gn.y, x.z * inv * gn.z, x.w * inv * gn.w);
      if (gate) w.x *= sigmoid_for<T>(z.x), w.y *= sigmoid_for<T>(z.y), w.z *= sigmoid_for<T>(z.z), w.w *= sigmoid_for<T>(z.w);
      st_f4(y + row * a.ldy + head * a.e + c, w);
    }
  }
}
// any sizes, one warp per (row, head)
template <typename T>
__global__ void __launch_bounds__(256) gla_norm_heads_any_kernel(const T* __restrict__ gate, T* __restrict__ y,
                                                                 const HeadNormArgs a) {
  pdl_entry();
  const int r = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (r >= a.total) return;
  const size_t row = r / a.heads;
  const int head = r % a.heads;
  const float* o = a.o + (size_t)r * a.ew;
  const float f = 1.f / (a.floor ? fmaxf(fabsf(o[a.e]), a.floor[r]) + 1e-6f : 1.f);
  const float* gain = a.gain + (a.per_head ? head * a.e : 0);
  float ss = 0.f;
  for (int c = lane; c < a.e; c += 32) ss += o[c] * f * (o[c] * f);
  const float inv = a.mul / sqrtf(warp_sum(ss) / a.e + a.eps);
  for (int c = lane; c < a.e; c += 32) {
    float x = o[c] * f * inv * gain[c];
    if (gate) x *= sigmoid_for<T>(ld_f(gate + row * a.ldg + head * a.e + c));
    st_f(y + row * a.ldy + head * a.e + c, x);
  }
}

struct GroupNormArgs {
  const float* o;          // [rows][heads][ew]
  const float* skip;       // [heads]
  const float* gain;       // [heads * e]
  int ldx, ldz, groups, heads, e, ew;
  float eps;
};
// v = (o + skip x) silu(z);  y = v / rms of its group * gain.  One CTA per (row, group of consecutive values).
template <typename T, int NV>
__global__ void __launch_bounds__(128) gla_norm_groups_kernel(const T* __restrict__ x, const T* __restrict__ z, T* __restrict__ y,
                                                              const GroupNormArgs a) {
  pdl_entry();
  __shared__ float sh[32];
  const size_t row = blockIdx.x;
  const int inner = a.heads * a.e, w = inner / a.groups, c0 = blockIdx.y * w;
  const float* o = a.o + row * a.heads * a.ew;
  auto value = [&](int c) {
    const int h = c / a.e;
    const float zz = ld_f(z + row * a.ldz + c);
    return fmaf(a.skip[h], ld_f(x + row * a.ldx + c), o[h * a.ew + c - h * a.e]) * zz * sigmoid_for<T>(zz);
  };
  float ss = 0.f;
  if constexpr (NV > 0) {       // w, c0, e and the strides are multiples of 4
    float4 keep[NV];
#pragma unroll
    for (int n = 0; n < NV; ++n) {
      const int i = (n * 128 + (int)threadIdx.x) * 4, c = c0 + i;
      keep[n] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (i >= w) continue;
      const int h = c / a.e;
      const float sk = a.skip[h];
      const float4 oo = ld_f4(o + h * a.ew + c - h * a.e), xx = ld_f4(x + row * a.ldx + c), zz = ld_f4(z + row * a.ldz + c);
      keep[n] = make_float4(fmaf(sk, xx.x, oo.x) * zz.x * sigmoid_for<T>(zz.x), fmaf(sk, xx.y, oo.y) * zz.y * sigmoid_for<T>(zz.y),
                            fmaf(sk, xx.z, oo.z) * zz.z * sigmoid_for<T>(zz.z), fmaf(sk, xx.w, oo.w) * zz.w * sigmoid_for<T>(zz.w));
      ss += (keep[n].x * keep[n].x + keep[n].y * keep[n].y) + (keep[n].z * keep[n].z + keep[n].w * keep[n].w);
    }
    const float inv = 1.f / sqrtf(cta_sum(ss, sh) / w + a.eps);
#pragma unroll
    for (int n = 0; n < NV; ++n) {
      const int i = (n * 128 + (int)threadIdx.x) * 4;
      if (i >= w) continue;
      const float4 gn = ld_f4(a.gain + c0 + i);
      st_f4(y + row * inner + c0 + i, make_float4(keep[n].x * inv * gn.x, keep[n].y * inv * gn.y, keep[n].z * inv * gn.z,
                                                  keep[n].w * inv * gn.w));
    }
  } else {
    for (int i = threadIdx.x; i < w; i += 128) {
      const float v = value(c0 + i);
      ss += v * v;
    }
    const float inv = 1.f / sqrtf(cta_sum(ss, sh) / w + a.eps);
    for (int i = threadIdx.x; i < w; i += 128) st_f(y + row * inner + c0 + i, value(c0 + i) * inv * a.gain[c0 + i]);
  }
}

// ------------------------------------------------------------------ launchers
template <typename T, int DP, int MODE>
int launch_gla(const void* q, const void* k, const void* v, const GlaArgs& a, const int* seg_off, int segs,
               const int* num_valid, cudaStream_t st) {
  constexpr int G = DP / kKK, MAXC = 512 / G * 4;
  const int parts = (a.ew + MAXC - 1) / MAXC, vb = ((a.ew + parts - 1) / parts + 3) / 4 * 4;
  const int threads = (G * vb / 4 + 31) / 32 * 32;
  dsv4_launch(gla_scan_kernel<T, DP, MODE>, dim3(segs, a.heads, (a.ew + vb - 1) / vb), threads, kTC * vb * sizeof(float), st,
              (const T*)q, (const T*)k, (const T*)v, seg_off, num_valid, vb, a);
  return (int)cudaGetLastError();
}
template <typename T, int MODE>
int dispatch_gla(const void* q, const void* k, const void* v, const GlaArgs& a, const int* seg_off, int segs,
                 const int* num_valid, cudaStream_t st) {
  if (a.d <= 32) return launch_gla<T, 32, MODE>(q, k, v, a, seg_off, segs, num_valid, st);
  if (a.d <= 64) return launch_gla<T, 64, MODE>(q, k, v, a, seg_off, segs, num_valid, st);
  if (a.d <= 128) return launch_gla<T, 128, MODE>(q, k, v, a, seg_off, segs, num_valid, st);
  return launch_gla<T, 256, MODE>(q, k, v, a, seg_off, segs, num_valid, st);
}
template <typename T, int MODE>
int launch_step(const void* q, const void* k, const void* v, const GlaArgs& a, int rows, const int* num_valid, cudaStream_t st) {
  dsv4_launch(gla_step_kernel<T, MODE>, dim3(rows, a.heads), 256, 0, st, (const T*)q, (const T*)k, (const T*)v, num_valid, a);
  return (int)cudaGetLastError();
}
template <typename T>
int dispatch_gla_mode(int mode, const void* q, const void* k, const void* v, const GlaArgs& a, const int* seg_off, int segs,
                      const int* num_valid, cudaStream_t st) {
  if (!seg_off && a.ew <= 1024) {
    if (mode == kGiven) return launch_step<T, kGiven>(q, k, v, a, segs, num_valid, st);
    if (mode == kStep) return launch_step<T, kStep>(q, k, v, a, segs, num_valid, st);
    return launch_step<T, kForget>(q, k, v, a, segs, num_valid, st);
  }
  if (mode == kGiven) return dispatch_gla<T, kGiven>(q, k, v, a, seg_off, segs, num_valid, st);
  if (mode == kStep) return dispatch_gla<T, kStep>(q, k, v, a, seg_off, segs, num_valid, st);
  return dispatch_gla<T, kForget>(q, k, v, a, seg_off, segs, num_valid, st);
}
template <typename T, int N>
void launch_causal(const void* p, void* before, void* out, const CausalConvArgs& a, int tiles, bool wide, cudaStream_t st) {
  if (wide)
    dsv4_launch(causal_conv_kernel<T, N, 4>, dim3((a.C / 4 + 127) / 128, tiles), 128, 0, st, (const T*)p, (T*)before, (T*)out, a);
  else
    dsv4_launch(causal_conv_kernel<T, N, 1>, dim3((a.C + 127) / 128, tiles), 128, 0, st, (const T*)p, (T*)before, (T*)out, a);
}
template <typename T>
int dispatch_causal(const void* p, void* before, void* out, const CausalConvArgs& a, int tiles, cudaStream_t st) {
  const bool wide = a.C % 4 == 0 && a.ld % 4 == 0 && ((uintptr_t)p & (4 * sizeof(T) - 1)) == 0;
  switch (a.n) {
    case 1: launch_causal<T, 1>(p, before, out, a, tiles, wide, st); break;
    case 2: launch_causal<T, 2>(p, before, out, a, tiles, wide, st); break;
    case 3: launch_causal<T, 3>(p, before, out, a, tiles, wide, st); break;
    case 4: launch_causal<T, 4>(p, before, out, a, tiles, wide, st); break;
    case 5: launch_causal<T, 5>(p, before, out, a, tiles, wide, st); break;
    case 6: launch_causal<T, 6>(p, before, out, a, tiles, wide, st); break;
    case 7: launch_causal<T, 7>(p, before, out, a, tiles, wide, st); break;
    case 8: launch_causal<T, 8>(p, before, out, a, tiles, wide, st); break;
    default: return 702;
  }
  return (int)cudaGetLastError();
}
template <typename T>
int launch_norm_heads(const void* gate, void* y, const HeadNormArgs& a, cudaStream_t st) {
  auto go = [&](auto kern, int r) {
    dsv4_launch(kern, (unsigned)((a.total + 8 * r - 1) / (8 * r)), 256, 0, st, (const T*)gate, (T*)y, a);
  };
  const bool wide = a.e % 4 == 0 && a.ldy % 4 == 0 && a.ldg % 4 == 0 && ((uintptr_t)gate & (4 * sizeof(T) - 1)) == 0;
  if (!wide || a.e > 256)
    go(gla_norm_heads_any_kernel<T>, 1);
  else if (a.e > 128)
    go(gla_norm_heads_kernel<T, 2, 2>, 2);
  else
    go(gla_norm_heads_kernel<T, 1, 4>, 4);
  return (int)cudaGetLastError();
}
template <typename T>
int launch_norm_groups(const void* x, const void* z, void* y, const GroupNormArgs& a, int rows, cudaStream_t st) {
  const int w = a.heads * a.e / a.groups;
  const dim3 grid(rows, a.groups);
  auto go = [&](auto kern) { dsv4_launch(kern, grid, 128, 0, st, (const T*)x, (const T*)z, (T*)y, a); };
  const uintptr_t align = 4 * sizeof(T) - 1;
  const bool wide = w % 4 == 0 && a.e % 4 == 0 && a.ldx % 4 == 0 && a.ldz % 4 == 0 && (((uintptr_t)x | (uintptr_t)z) & align) == 0;
  if (!wide || w > 8192)
    go(gla_norm_groups_kernel<T, 0>);
  else if (w <= 512)
    go(gla_norm_groups_kernel<T, 1>);
  else if (w <= 1024)
    go(gla_norm_groups_kernel<T, 2>);
  else if (w <= 2048)
    go(gla_norm_groups_kernel<T, 4>);
  else if (w <= 4096)
    go(gla_norm_groups_kernel<T, 8>);
  else
    go(gla_norm_groups_kernel<T, 16>);
  return (int)cudaGetLastError();
}

}  // namespace

// z [rows, 2 heads] fp32; log_g, fac, floor [rows, heads]; top [slots + 1, heads] is advanced.  longest: tokens of the longest
// segment.  segs: segments (seg_off given) or rows; from *num_valid on they are padding.
DSV4_API int dsv4_mlstm_gates(const float* z, const float* bias, float cap, float* top, float* log_g, float* fac, float* floor,
                              const int* slots, const int* pos, const int* seg_off, int segs, const int* num_valid, int heads,
                              int longest, cudaStream_t st) {
  if (segs <= 0) return 0;
  if (heads < 1 || heads > 65535 || cap <= 0.f) return 700;
  const MlstmArgs a{z, bias, cap, top, log_g, fac, floor, slots, pos, seg_off, num_valid, heads};
  const int threads = longest >= 1024 ? 1024 : longest > 256 ? 512 : longest > 32 ? 256 : 32;
  dsv4_launch(mlstm_gates_kernel, dim3(segs, heads), threads, 0, st, a);
  return (int)cudaGetLastError();
}

// out[t] = silu(bias + sum_j taps[j] p[t - (n - 1) + j]) per channel; p: C columns with row stride ld; before [slots + 1, n - 1, C]
// holds the inputs ahead of a segment and is moved on.  tiles [n_tiles][2] = segment, first token within it, every `span` tokens
// (span >= n - 1); or null: n_tiles rows, a segment each.  At most 8 taps.
DSV4_API int dsv4_causal_conv(const void* p, int ld, const float* taps, int n, const float* bias, void* before, void* out, int C,
                              const int* slots, const int* pos, const int* seg_off, const int* tiles, int n_tiles, int span,
                              const int* num_valid, int fp32, cudaStream_t st) {
  if (n_tiles <= 0) return 0;
  if (C < 1 || n < 1 || n_tiles > 65535 || (tiles && (!seg_off || span < n - 1))) return 701;
  const CausalConvArgs a{ld, C, taps, bias, slots, pos, tiles ? seg_off : nullptr, num_valid, tiles, n, tiles ? span : 1};
  return fp32 ? dispatch_causal<float>(p, before, out, a, n_tiles, st)
              : dispatch_causal<__nv_bfloat16>(p, before, out, a, n_tiles, st);
}

// See GlaArgs.  out [rows, heads, ew].  segs: segments (seg_off given), or rows of one token each.
DSV4_API int dsv4_gla_scan(int mode, const void* q, int ldq, const void* k, int ldk, const void* v, int ldv, const float* raw,
                           const float* fac, const float* bias, const float* par, float q_mul, float* state, float* out,
                           const int* slots, const int* pos, const int* seg_off, int segs, const int* num_valid, int heads,
                           int group, int d, int e, int ew, int fp32, cudaStream_t st) {
  if (segs <= 0) return 0;
  if (mode < 0 || mode > 2 || heads < 1 || heads > 65535 || group < 1 || d < 1 || d > 256 || e < 1 || ew % 4 ||
      ew < e + (mode == kGiven))
    return 703;
  const GlaArgs a{ldq, ldk, ldv, raw, fac, bias, par, q_mul, heads, group, d, e, ew, state, out, slots, pos};
  return fp32 ? dispatch_gla_mode<float>(mode, q, k, v, a, seg_off, segs, num_valid, st)
              : dispatch_gla_mode<__nv_bfloat16>(mode, q, k, v, a, seg_off, segs, num_valid, st);
}

// See HeadNormArgs; gate (row stride ldg) may be null; y [rows, ldy].
DSV4_API int dsv4_gla_norm_heads(const float* o, const float* floor, const void* gate, int ldg, const float* gain, int per_head,
                                 float eps, float mul, void* y, int ldy, int rows, int heads, int e, int ew, int fp32,
                                 cudaStream_t st) {
  if (rows <= 0) return 0;
  if ((long long)rows * heads > 1 << 30) return 705;
  const HeadNormArgs a{o, floor, gain, per_head, ldg, ldy, eps, mul, heads, e, ew, rows * heads};
  return fp32 ? launch_norm_heads<float>(gate, y, a, st) : launch_norm_heads<__nv_bfloat16>(gate, y, a, st);
}

// See GroupNormArgs; x, z: row strides ldx, ldz; y [rows, heads * e].
DSV4_API int dsv4_gla_norm_groups(const float* o, const float* skip, const void* x, int ldx, const void* z, int ldz,
                                  const float* gain, int groups, float eps, void* y, int rows, int heads, int e, int ew,
                                  int fp32, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (groups < 1 || groups > 65535 || heads * e % groups) return 704;
  const GroupNormArgs a{o, skip, gain, ldx, ldz, groups, heads, e, ew, eps};
  return fp32 ? launch_norm_groups<float>(x, z, y, a, rows, st) : launch_norm_groups<__nv_bfloat16>(x, z, y, a, rows, st);
}
