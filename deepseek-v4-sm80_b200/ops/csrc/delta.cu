// Gated delta rule with a decay per head and key channel: the short convolutions in front of it, the recurrence token by
// token (decode, short portions, models served in 32-bit floats), and the per-head norm with its gate behind it.
//
//   S <- diag(g_t) S,   u_t = beta_t (v_t - S^T k_t),   S <- S + k_t u_t^T,   o_t = S^T q_t        (S is [key, value])
//   g_t = exp(-exp(A_log) softplus(rate_t + dt_bias)),  beta_t = sigmoid(b_t),  y_t = o_t / rms(o_t) * gain * sigmoid(gate_t)
//
// With S' = diag(g) S:  o = S'^T q + (k . q) u, so one pass over the state gives both S'^T k and S'^T q.
// State per request slot: S [heads][d][e] in fp32 and the last taps - 1 inputs of the convolutions.  A request at position 0
// starts from zeros whatever its slot held before.
#include "delta.cuh"

namespace {

// ------------------------------------------------------------------ short convolutions, silu, unit vectors
struct ConvArgs {
  ConvCols cols;
  const float* taps;      // [n][channels]
  const int* slots;
  const int* pos;
  int rows, d, e, kv_heads, heads;
};

// A head of q, k or v.
struct ConvUnit {
  int part, head, width, ch0, col0;
  __device__ __forceinline__ ConvUnit(const ConvArgs& a, int unit) {
    part = unit < a.kv_heads ? 0 : unit < 2 * a.kv_heads ? 1 : 2;
    head = unit - part * a.kv_heads, width = part == 2 ? a.e : a.d;
    ch0 = part * a.cols.nqk + head * width;
    col0 = a.cols.col(ch0);
  }
};

// One warp per head and TB tokens, N taps: every input is read once, the taps and the last N - 1 inputs stay in registers.
// NI x 4 x 32 channels at most, sizes multiples of 4.
template <typename T, int NI, int N, int TB>
__global__ void __launch_bounds__(256) conv_unit_tile_kernel(const T* __restrict__ p, const T* __restrict__ before,
                                                             float* __restrict__ q, float* __restrict__ k,
                                                             T* __restrict__ v, const ConvArgs a) {
  pdl_entry();
  const int t0 = (blockIdx.y * 8 + (threadIdx.x >> 5)) * TB, lane = threadIdx.x & 31;
  if (t0 >= a.rows) return;
  const ConvUnit un(a, blockIdx.x);
  const int C = 2 * a.cols.nqk + a.cols.nv;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  int slot[TB], pos[TB];
  float4 x[TB][NI], w[N][NI], old[N > 1 ? N - 1 : 1][NI];    // old[b]: b + 1 tokens back
#pragma unroll
  for (int i = 0; i < TB; ++i) {
    const int t = min(t0 + i, a.rows - 1);
    slot[i] = a.slots[t], pos[i] = a.pos[t];
#pragma unroll
    for (int n = 0; n < NI; ++n) {
      const int c = (n * 32 + lane) * 4;
      x[i][n] = c < un.width ? ld_f4(p + (size_t)t * a.cols.ld + un.col0 + c) : zero;
    }
  }
#pragma unroll
  for (int b = 0; b < N; ++b)
#pragma unroll
    for (int n = 0; n < NI; ++n) {
      const int c = (n * 32 + lane) * 4;
      w[b][n] = c < un.width ? ld_f4(a.taps + (size_t)(N - 1 - b) * C + un.ch0 + c) : zero;   // b tokens back
    }
#pragma unroll
  for (int i = 0; i < TB; ++i) {
    const int t = t0 + i;
    if (t >= a.rows) return;
    if (i == 0 || slot[i] != slot[i > 0 ? i - 1 : 0] || pos[i] != pos[i > 0 ? i - 1 : 0] + 1) {
      int have = 1;               // rows of this portion that the convolution reads; older inputs come from the slot
#pragma unroll
      for (int b = 1; b < N; ++b)
        if (have == b && t - b >= 0 && a.slots[t - b] == slot[i] && a.pos[t - b] == pos[i] - b) ++have;
#pragma unroll
      for (int b = 1; b < N; ++b)
#pragma unroll
        for (int n = 0; n < NI; ++n) {
          const int c = (n * 32 + lane) * 4;
          float4 o = zero;
          if (c < un.width && pos[i] - b >= 0) {
            if (b < have) {
              o = ld_f4(p + (size_t)(t - b) * a.cols.ld + un.col0 + c);
            } else {
              const T* src = before + ((size_t)slot[i] * (N - 1) + N - 2 - (b - have)) * C + un.ch0 + c;
              o = make_float4(ld_f(src), ld_f(src + 1), ld_f(src + 2), ld_f(src + 3));
            }
          }
          old[b - 1][n] = o;
        }
    }
    float4 y[NI];
    float ss = 0.f;
#pragma unroll
    for (int n = 0; n < NI; ++n) {
      float4 s = make_float4(x[i][n].x * w[0][n].x, x[i][n].y * w[0][n].y, x[i][n].z * w[0][n].z, x[i][n].w * w[0][n].w);
#pragma unroll
      for (int b = 1; b < N; ++b) {
        const float4 o = old[b - 1][n], f = w[b][n];
        s.x = fmaf(o.x, f.x, s.x), s.y = fmaf(o.y, f.y, s.y), s.z = fmaf(o.z, f.z, s.z), s.w = fmaf(o.w, f.w, s.w);
      }
      s.x *= sigmoid_for<T>(s.x), s.y *= sigmoid_for<T>(s.y), s.z *= sigmoid_for<T>(s.z), s.w *= sigmoid_for<T>(s.w);
      ss += (s.x * s.x + s.y * s.y) + (s.z * s.z + s.w * s.w);
      y[n] = s;
#pragma unroll
      for (int b = N - 2; b > 0; --b) old[b][n] = old[b - 1][n];
      if (N > 1) old[0][n] = x[i][n];
    }
    float sc = 1.f;
    if (un.part < 2) {
      sc = 1.f / sqrtf(warp_sum(ss) + 1e-6f);
      if (un.part == 0) sc *= 1.f / sqrtf((float)a.d);
    }
#pragma unroll
    for (int n = 0; n < NI; ++n) {
      const int c = (n * 32 + lane) * 4;
      if (c >= un.width) continue;
      const float4 s = make_float4(y[n].x * sc, y[n].y * sc, y[n].z * sc, y[n].w * sc);
      if (un.part == 2)
        st_f4(v + (size_t)t * a.cols.nv + un.head * un.width + c, s);
      else
        st_f4((un.part ? k : q) + (size_t)t * a.cols.nqk + un.head * un.width + c, s);
    }
  }
}

// Any number of taps, any sizes: one warp per (token, head of q, k or v).
template <typename T, int W>     // W consecutive channels per lane and step (4, or 1 for sizes that are no multiple of 4)
__global__ void __launch_bounds__(256) conv_unit_kernel(const T* __restrict__ p, const T* __restrict__ before,
                                                        float* __restrict__ q, float* __restrict__ k, T* __restrict__ v,
                                                        const ConvArgs a) {
  pdl_entry();
  const int t = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (t >= a.rows) return;
  const int n = a.cols.taps, C = 2 * a.cols.nqk + a.cols.nv;
  const ConvUnit un(a, blockIdx.x);
  const int part = un.part, head = un.head, width = un.width, ch0 = un.ch0, col0 = un.col0;
  const int slot = a.slots[t], pos = a.pos[t];
  int have = 1;                   // rows of this portion up to and including this one that the convolution reads
  while (have < n && t - have >= 0 && a.slots[t - have] == slot && a.pos[t - have] == pos - have) ++have;
  constexpr int NI = W == 4 ? 2 : 8;   // up to 256 channels
  float y[NI][W];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int c = (i * 32 + lane) * W;
#pragma unroll
    for (int j = 0; j < W; ++j) y[i][j] = 0.f;
    if (c >= width) continue;
    for (int b = 0; b < n; ++b) {            // b tokens back
      float x[W], w[W];
      if (b < have) {
        const T* src = p + (size_t)(t - b) * a.cols.ld + col0 + c;
        if constexpr (W == 4) {
          const float4 f = ld_f4(src);
          x[0] = f.x, x[1] = f.y, x[2] = f.z, x[3] = f.w;
        } else {
          x[0] = ld_f(src);
        }
      } else {
        // `have` rows of the portion were used up: b - have tokens ahead of it
        if (pos - b < 0) break;
        const T* src = before + ((size_t)slot * (n - 1) + (n - 1) - 1 - (b - have)) * C + ch0 + c;
#pragma unroll
        for (int j = 0; j < W; ++j) x[j] = ld_f(src + j);
      }
      ld_w<W>(a.taps + (size_t)(n - 1 - b) * C + ch0 + c, w);
#pragma unroll
      for (int j = 0; j < W; ++j) y[i][j] = fmaf(x[j], w[j], y[i][j]);
    }
#pragma unroll
    for (int j = 0; j < W; ++j) {
      y[i][j] *= sigmoid_f(y[i][j]);
      ss += y[i][j] * y[i][j];
    }
  }
  float sc = 1.f;
  if (part < 2) {
    sc = 1.f / sqrtf(warp_sum(ss) + 1e-6f);
    if (part == 0) sc *= 1.f / sqrtf((float)a.d);
  }
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int c = (i * 32 + lane) * W;
    if (c >= width) continue;
#pragma unroll
    for (int j = 0; j < W; ++j) y[i][j] *= sc;
    if (part == 2)
      st_w<W>(v + (size_t)t * a.cols.nv + head * width + c, y[i]);
    else
      st_w<W>((part ? k : q) + (size_t)t * a.cols.nqk + head * width + c, y[i]);
  }
}

// ------------------------------------------------------------------ recurrence
struct ScanArgs {
  const float* q;         // [rows][kv_heads][d]
  const float* k;
  const float* rate;      // [rows][heads][d]
  const float* dt_bias;   // [heads][d]
  const float* a_log;     // [heads]
  int at_b;               // column of p with the step sizes' logits
  const float* gain;      // [e]
  float eps;
  float* state;           // [slots + 1][heads][d][e]
  float* raw;             // [rows][heads][e]: outputs ahead of the norm, when a head's columns are split over CTAs
  const int* slots;
  const int* pos;
  const int* seg_off;     // [segments + 1] or null: segment s is row s
  const int* num_valid;   // segments (rows) from here on are padding, or null
  int heads, group, d, e;
  ConvCols cols;
};

constexpr int kTC = 8;        // tokens staged at a time
constexpr int kKK = 16;       // keys per thread
constexpr int kVV = 4;        // value columns per thread
constexpr int kGS = kKK + 4;  // floats between two key groups in shared memory (keeps 16-byte reads conflict-free)

template <int DP, int VB>
struct ScanCfg {
  static constexpr int G = DP / kKK;                 // threads that share four value columns
  static constexpr int THREADS = G * (VB / kVV);
};

// One CTA per (segment, head, VB value columns).  The state sits in registers: a thread owns kKK keys x kVV columns; sums over
// keys are shuffles over the G neighbouring threads of a column group.
template <typename T, int DP, int VB>
__global__ void __launch_bounds__(ScanCfg<DP, VB>::THREADS) delta_scan_kernel(const T* __restrict__ p,
                                                                              const T* __restrict__ v,
                                                                              const T* __restrict__ gate, T* before,
                                                                              T* __restrict__ y, const ScanArgs a) {
  pdl_entry();
  using C = ScanCfg<DP, VB>;
  constexpr int G = C::G, NT = C::THREADS, LD = G * kGS;
  __shared__ __align__(16) float qs[kTC][LD], ks[kTC][LD], gs[kTC][LD], vs[kTC][VB], os[kTC][VB];
  __shared__ float beta[kTC], kq[kTC];
  const int seg = blockIdx.x, head = blockIdx.y, v0 = blockIdx.z * VB;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  if (a.num_valid && seg >= *a.num_valid) return;
  const int t0 = a.seg_off ? a.seg_off[seg] : seg, t1 = a.seg_off ? a.seg_off[seg + 1] : seg + 1;
  const int n = t1 - t0, d = a.d, e = a.e;
  if (n <= 0) return;
  const int slot = a.slots[t0], kvh = head / a.group;
  const bool fresh = a.pos[t0] == 0;
  const int g = tid % G, col = v0 + tid / G * kVV;
  const float ea = expf(a.a_log[head]);
  const bool vec = e % 4 == 0;

  float s[kKK][kVV];
  float* st = a.state + ((size_t)slot * a.heads + head) * d * e;
#pragma unroll
  for (int i = 0; i < kKK; ++i) {
    const int key = g * kKK + i;
    s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
    if (fresh || key >= d || col >= e) continue;
    if (vec) {
      ld_w<4>(st + (size_t)key * e + col, s[i]);
    } else {
#pragma unroll
      for (int j = 0; j < kVV; ++j)
        if (col + j < e) s[i][j] = st[(size_t)key * e + col + j];
    }
  }
  for (int c0 = 0; c0 < n; c0 += kTC) {
    const int m = min(kTC, n - c0);
    __syncthreads();
    for (int i = tid; i < m * DP; i += NT) {
      const int tok = i / DP, c = i % DP, at = c / kKK * kGS + c % kKK;
      const bool in = c < d;                     // keys past d are zero: they never touch the state
      const size_t row = t0 + c0 + tok;
      qs[tok][at] = in ? a.q[row * a.cols.nqk + kvh * d + c] : 0.f;
      ks[tok][at] = in ? a.k[row * a.cols.nqk + kvh * d + c] : 0.f;
      gs[tok][at] = in ? expf(log_decay(a.rate[row * a.heads * d + head * d + c], a.dt_bias[head * d + c], ea)) : 0.f;
    }
    for (int i = tid; i < m * VB; i += NT) {
      const int tok = i / VB, c = v0 + i % VB;
      vs[tok][i % VB] = c < e ? ld_f(v + (size_t)(t0 + c0 + tok) * a.cols.nv + head * e + c) : 0.f;
    }
    for (int tok = tid; tok < m; tok += NT) beta[tok] = sigmoid_f(ld_f(p + (size_t)(t0 + c0 + tok) * a.cols.ld + a.at_b + head));
    __syncthreads();
    for (int tok = warp; tok < m; tok += NT / 32) {
      float x = 0.f;
      for (int c = lane; c < DP; c += 32) x += qs[tok][c / kKK * kGS + c % kKK] * ks[tok][c / kKK * kGS + c % kKK];
      x = warp_sum(x);
      if (lane == 0) kq[tok] = x;
    }
    __syncthreads();
    for (int tok = 0; tok < m; ++tok) {
      const float *qp = qs[tok] + g * kGS, *kp = ks[tok] + g * kGS, *gp = gs[tok] + g * kGS;
      float pk[kVV] = {}, pq[kVV] = {};
#pragma unroll
      for (int i = 0; i < kKK; i += 4) {
        float gg[4], kk[4], qq[4];
        ld_w<4>(gp + i, gg);
        ld_w<4>(kp + i, kk);
        ld_w<4>(qp + i, qq);
#pragma unroll
        for (int h = 0; h < 4; ++h)
#pragma unroll
          for (int j = 0; j < kVV; ++j) {
            s[i + h][j] *= gg[h];
            pk[j] = fmaf(kk[h], s[i + h][j], pk[j]);
            pq[j] = fmaf(qq[h], s[i + h][j], pq[j]);
          }
      }
#pragma unroll
      for (int j = 0; j < kVV; ++j)
#pragma unroll
        for (int off = 1; off < G; off <<= 1) {
          pk[j] += __shfl_xor_sync(0xffffffffu, pk[j], off);
          pq[j] += __shfl_xor_sync(0xffffffffu, pq[j], off);
        }
      float vv[kVV], u[kVV];
      ld_w<4>(vs[tok] + tid / G * kVV, vv);
      const float bt = beta[tok], dot = kq[tok];
#pragma unroll
      for (int j = 0; j < kVV; ++j) u[j] = bt * (vv[j] - pk[j]);
#pragma unroll
      for (int i = 0; i < kKK; i += 4) {
        float kk[4];
        ld_w<4>(kp + i, kk);
#pragma unroll
        for (int h = 0; h < 4; ++h)
#pragma unroll
          for (int j = 0; j < kVV; ++j) s[i + h][j] = fmaf(kk[h], u[j], s[i + h][j]);
      }
      if (g == 0) {
#pragma unroll
        for (int j = 0; j < kVV; ++j) pq[j] = fmaf(dot, u[j], pq[j]);
        st_w<4>(os[tok] + tid / G * kVV, pq);
      }
    }
    __syncthreads();
    for (int tok = warp; tok < m; tok += NT / 32) {
      const size_t row = ((size_t)(t0 + c0 + tok) * a.heads + head) * e;
      if (gridDim.z > 1) {
        for (int c = lane; c < VB && v0 + c < e; c += 32) a.raw[row + v0 + c] = os[tok][c];
        continue;
      }
      float x = 0.f;
      for (int c = lane; c < e; c += 32) x += os[tok][c] * os[tok][c];
      const float inv = 1.f / sqrtf(warp_sum(x) / e + a.eps);
      for (int c = lane; c < e; c += 32) st_f(y + row + c, os[tok][c] * inv * a.gain[c] * sigmoid_f(ld_f(gate + row + c)));
    }
  }
#pragma unroll
  for (int i = 0; i < kKK; ++i) {
    const int key = g * kKK + i;
    if (key >= d || col >= e) continue;
    if (vec) {
      st_w<4>(st + (size_t)key * e + col, s[i]);
    } else {
#pragma unroll
      for (int j = 0; j < kVV; ++j)
        if (col + j < e) st[(size_t)key * e + col + j] = s[i][j];
    }
  }
  if (blockIdx.z == 0)     // the heads of a segment share the channels
    keep_conv_inputs(p, before + (size_t)slot * (a.cols.taps - 1) * (2 * a.cols.nqk + a.cols.nv), a.cols, t0, n, fresh,
                     head * NT + tid, a.heads * NT);
}

// y = o / rms(o) * gain * sigmoid(gate), one warp per (token, head)
template <typename T>
__global__ void __launch_bounds__(256) head_norm_gate_kernel(const float* __restrict__ raw, const T* __restrict__ gate,
                                                             const float* __restrict__ gain, float eps,
                                                             T* __restrict__ y, long long total, int e) {
  pdl_entry();
  const long long r = blockIdx.x * 8ll + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (r >= total) return;
  const float* o = raw + r * e;
  float x = 0.f;
  if (e % 4 == 0 && e <= 256) {
    float4 keep[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int c = (i * 32 + lane) * 4;
      keep[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < e) keep[i] = ld_f4(o + c);
      x += keep[i].x * keep[i].x + keep[i].y * keep[i].y + keep[i].z * keep[i].z + keep[i].w * keep[i].w;
    }
    const float inv = 1.f / sqrtf(warp_sum(x) / e + eps);
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int c = (i * 32 + lane) * 4;
      if (c >= e) continue;
      const float4 gt = ld_f4(gate + r * e + c), gn = ld_f4(gain + c);
      st_f4(y + r * e + c, make_float4(keep[i].x * inv * gn.x * sigmoid_for<T>(gt.x), keep[i].y * inv * gn.y * sigmoid_for<T>(gt.y),
                                       keep[i].z * inv * gn.z * sigmoid_for<T>(gt.z), keep[i].w * inv * gn.w * sigmoid_for<T>(gt.w)));
    }
    return;
  }
  for (int c = lane; c < e; c += 32) x += o[c] * o[c];
  const float inv = 1.f / sqrtf(warp_sum(x) / e + eps);
  for (int c = lane; c < e; c += 32) st_f(y + r * e + c, o[c] * inv * gain[c] * sigmoid_for<T>(ld_f(gate + r * e + c)));
}

template <typename T, int DP, int VB>
int launch_scan(const void* p, const void* v, const void* gate, void* before, void* y, const ScanArgs& a, int segs,
                cudaStream_t st) {
  dsv4_launch(delta_scan_kernel<T, DP, VB>, dim3(segs, a.heads, (a.e + VB - 1) / VB), ScanCfg<DP, VB>::THREADS, 0, st,
              (const T*)p, (const T*)v, (const T*)gate, (T*)before, (T*)y, a);
  return (int)cudaGetLastError();
}
template <typename T>
int dispatch_scan(const void* p, const void* v, const void* gate, void* before, void* y, const ScanArgs& a, int vb,
                  int segs, cudaStream_t st) {
  if (a.d <= 32) return vb == 64 ? launch_scan<T, 32, 64>(p, v, gate, before, y, a, segs, st)
                                 : launch_scan<T, 32, 128>(p, v, gate, before, y, a, segs, st);
  if (a.d <= 64) return vb == 64 ? launch_scan<T, 64, 64>(p, v, gate, before, y, a, segs, st)
                                 : launch_scan<T, 64, 128>(p, v, gate, before, y, a, segs, st);
  if (a.d <= 128) return vb == 64 ? launch_scan<T, 128, 64>(p, v, gate, before, y, a, segs, st)
                                  : launch_scan<T, 128, 128>(p, v, gate, before, y, a, segs, st);
  if (a.d <= 256 && vb == 64) return launch_scan<T, 256, 64>(p, v, gate, before, y, a, segs, st);
  return 680;
}
template <typename T, int NI, int N>
void launch_conv_tile(const void* p, const void* before, float* q, float* k, void* v, const ConvArgs& a, cudaStream_t st) {
  const int units = 2 * a.kv_heads + a.heads;
  if (a.rows <= 1024)
    dsv4_launch(conv_unit_tile_kernel<T, NI, N, 1>, dim3(units, (a.rows + 7) / 8), 256, 0, st, (const T*)p, (const T*)before,
                q, k, (T*)v, a);
  else
    dsv4_launch(conv_unit_tile_kernel<T, NI, N, 4>, dim3(units, (a.rows + 31) / 32), 256, 0, st, (const T*)p,
                (const T*)before, q, k, (T*)v, a);
}
template <typename T, int NI>
bool dispatch_conv_tile(const void* p, const void* before, float* q, float* k, void* v, const ConvArgs& a, cudaStream_t st) {
  switch (a.cols.taps) {
    case 2: launch_conv_tile<T, NI, 2>(p, before, q, k, v, a, st); return true;
    case 3: launch_conv_tile<T, NI, 3>(p, before, q, k, v, a, st); return true;
    case 4: launch_conv_tile<T, NI, 4>(p, before, q, k, v, a, st); return true;
    default: return false;
  }
}
template <typename T>
void launch_conv(const void* p, const void* before, float* q, float* k, void* v, const ConvArgs& a, bool wide,
                 cudaStream_t st) {
  const dim3 grid(2 * a.kv_heads + a.heads, (a.rows + 7) / 8);
  if (wide && (a.d > 128 || a.e > 128 ? dispatch_conv_tile<T, 2>(p, before, q, k, v, a, st)
                                      : dispatch_conv_tile<T, 1>(p, before, q, k, v, a, st)))
    return;
  if (wide)
    dsv4_launch(conv_unit_kernel<T, 4>, grid, 256, 0, st, (const T*)p, (const T*)before, q, k, (T*)v, a);
  else
    dsv4_launch(conv_unit_kernel<T, 1>, grid, 256, 0, st, (const T*)p, (const T*)before, q, k, (T*)v, a);
}

}  // namespace

// p [rows, ld]: columns q from 0, k from at_k, v from at_v; taps [n_taps, channels] over q | k | v, the last row is the current
// token's; before [slots + 1, n_taps - 1, channels].  q, k: fp32 [rows, kv_heads * d], v: [rows, heads * e].
DSV4_API int dsv4_conv_unit(const void* p, int ld, int at_k, int at_v, const float* taps, int n_taps, const void* before,
                            const int* slots, const int* pos, float* q, float* k, void* v, int rows, int heads, int kv_heads,
                            int d, int e, int fp32, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (d < 1 || e < 1 || d > 256 || e > 256 || n_taps < 1 || rows > 8 * 65535) return 681;
  const ConvArgs a{{ld, at_k, at_v, kv_heads * d, heads * e, n_taps}, taps, slots, pos, rows, d, e, kv_heads, heads};
  const bool wide = d % 4 == 0 && e % 4 == 0 && ld % 4 == 0 && at_k % 4 == 0 && at_v % 4 == 0;
  if (fp32)
    launch_conv<float>(p, before, q, k, v, a, wide, st);
  else
    launch_conv<__nv_bfloat16>(p, before, q, k, v, a, wide, st);
  return (int)cudaGetLastError();
}

// segs: segments (seg_off given) or rows.  vb: value columns per CTA (64 or 128; 64 for d > 128); raw [rows, heads * e] is
// needed when a head has more columns, and dsv4_head_norm_gate has to follow then.
DSV4_API int dsv4_delta_scan(const void* p, int ld, int at_k, int at_v, int at_b, int n_taps, const float* q, const float* k,
                             const void* v, const float* rate, const float* dt_bias, const float* a_log, const void* gate,
                             const float* gain, float eps, float* state, void* before, float* raw, const int* slots,
                             const int* pos, const int* seg_off, int segs, const int* num_valid, int heads, int kv_heads,
                             int d, int e, int vb, void* y, int fp32, cudaStream_t st) {
  if (segs <= 0) return 0;
  if (heads < 1 || heads > 65535 || kv_heads < 1 || heads % kv_heads || d < 1 || e < 1 || (vb != 64 && vb != 128)) return 682;
  if (e > vb && !raw) return 683;
  const ScanArgs s{q, k, rate, dt_bias, a_log, at_b, gain, eps, state, raw, slots, pos, seg_off, num_valid, heads,
                   heads / kv_heads, d, e, {ld, at_k, at_v, kv_heads * d, heads * e, n_taps}};
  return fp32 ? dispatch_scan<float>(p, v, gate, before, y, s, vb, segs, st)
              : dispatch_scan<__nv_bfloat16>(p, v, gate, before, y, s, vb, segs, st);
}

DSV4_API int dsv4_head_norm_gate(const float* raw, const void* gate, const float* gain, float eps, void* y, int rows,
                                 int heads, int e, int fp32, cudaStream_t st) {
  if (rows <= 0) return 0;
  const long long total = (long long)rows * heads;
  const unsigned grid = (unsigned)((total + 7) / 8);
  if (fp32)
    dsv4_launch(head_norm_gate_kernel<float>, grid, 256, 0, st, raw, (const float*)gate, gain, eps, (float*)y, total, e);
  else
    dsv4_launch(head_norm_gate_kernel<__nv_bfloat16>, grid, 256, 0, st, raw, (const __nv_bfloat16*)gate, gain, eps,
                (__nv_bfloat16*)y, total, e);
  return (int)cudaGetLastError();
}
