// Gated linear attention (gla.cuh) of long prompt portions in chunks of 64 tokens, bf16 activations.  With L_t = sum_{j <= t} log
// g_j inside a chunk and S the state before it,
//
//   o_t    = (q_t e^{L_t})^T S + sum_{s <= t} A_ts v_s,        A_ts = q_t . (k_s e^{L_t - L_s})
//   S_next = diag(e^{L_63}) S + sum_s (k_s e^{L_63 - L_s}) v_s^T
//
// so that only the carry S -> S_next runs in sequence:
//   gla_chunk_state_kernel   every (chunk, head, 128 value columns): its own contribution U and e^{L_63}
//   gla_chunk_carry_kernel   per state element: walks a request's chunks, leaves the state before each chunk in U's place
//   gla_chunk_out_kernel     every (chunk, head, 128 value columns): the outputs
//
// Products run on the tensor cores in TF32.  bf16 operands are exact in TF32; fp32 ones are split, x = hi + lo with hi cut off to
// TF32's 11 bits, and hi hi' + hi lo' + lo hi' keeps about 21 bits of a product.  Sums are fp32.
//
// Decays per head: A is q . k times e^{L_t - L_s} (never positive).  Decays per channel: A is the product of q e^{L_t - L_ref} and
// k e^{L_ref - L_s} with a reference inside each block of 16 tokens; across blocks the references' difference goes onto k, where it
// cannot grow.  Inside a block exponents may be positive, which is safe up to e^60; a chunk with decays beyond that takes its
// exponentials pair by pair on the CUDA cores.  log g per channel is clamped at -40 (g below 1e-17).
//
// Fragments of m16n8k8 (lane = 4 g + t): A rows g, g + 8, B column g, C rows g, g + 8 and columns 2t, 2t + 1.  The order of the
// contraction index is free as long as A and B agree: places t, t + 4 stand for 2t, 2t + 1 where that makes them neighbours.
#include "gla.cuh"
#include "tf32.cuh"

namespace {

constexpr int kC = 64;            // tokens of a chunk
constexpr int kCols = 128;        // value columns per CTA
constexpr float kMinLog = -40.f;
constexpr float kSafe = 60.f;
constexpr int kThreads = 256;
constexpr int kVL = kCols + 8;    // row stride of the values (8 mod 32: conflict-free)
constexpr int kAL = kC + 4;       // row stride of A (4 mod 32: conflict-free as an A operand)

struct ChunkArgs {
  GlaArgs g;
  const int* chunks;      // [chunks][2]: first row, tokens
  float* us;              // [chunks][heads][d][ew] contributions, then states
  float* decay;           // [chunks][heads] or, per channel, [chunks][heads][d]: e^{L_63}
};

using bf16 = __nv_bfloat16;

__device__ __forceinline__ float2 ld_f2(const float* p) { return *reinterpret_cast<const float2*>(p); }
// exact TF32 (bf16 values): no low part
__device__ __forceinline__ uint32_t bits(float x) { return __float_as_uint(x); }

// Running sums of log g per head over the chunk (64 tokens, two per lane of warp 0) and the factors of k.
template <int MODE>
__device__ __forceinline__ void head_logs(const GlaArgs& a, int t0, int m, int head, float* ls, float* fac) {
  if (threadIdx.x >= 32) return;
  const int lane = threadIdx.x;
  float l[2], f[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    l[i] = f[i] = 0.f;
    if (2 * lane + i < m) {
      const HeadGate h = head_gate<MODE>(a, t0 + 2 * lane + i, head);
      l[i] = h.log_g, f[i] = h.fac;
    }
  }
  float sum = l[0] + l[1];
#pragma unroll
  for (int off = 1; off < 32; off <<= 1) {
    const float up = __shfl_up_sync(0xffffffffu, sum, off);
    if (lane >= off) sum += up;
  }
  const float prev = __shfl_up_sync(0xffffffffu, sum, 1), base = lane ? prev : 0.f;
  ls[2 * lane] = base + l[0], ls[2 * lane + 1] = base + l[0] + l[1];
  fac[2 * lane] = f[0], fac[2 * lane + 1] = f[1];
}

// [kC][LD] <- columns [c0, c0 + d) of the chunk's rows, zeros past d and past the last token; d, c0 multiples of 8.
template <int DP, int LD>
__device__ __forceinline__ void load_rows(const bf16* p, int ld, int t0, int m, int c0, int d, float* dst) {
  constexpr int N = kC * DP / 8 / kThreads;
  uint4 u[N];
#pragma unroll
  for (int n = 0; n < N; ++n) {
    const int i = threadIdx.x + n * kThreads, t = i / (DP / 8), c = i % (DP / 8) * 8;
    u[n] = make_uint4(0, 0, 0, 0);
    if (t < m && c < d) u[n] = *reinterpret_cast<const uint4*>(p + (size_t)(t0 + t) * ld + c0 + c);
  }
#pragma unroll
  for (int n = 0; n < N; ++n) {
    const int i = threadIdx.x + n * kThreads, t = i / (DP / 8), c = i % (DP / 8) * 8;
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u[n]);
    const float2 x = __bfloat1622float2(h[0]), y = __bfloat1622float2(h[1]), z = __bfloat1622float2(h[2]),
                 w = __bfloat1622float2(h[3]);
    st_f4(dst + t * LD + c, make_float4(x.x, x.y, y.x, y.y));
    st_f4(dst + t * LD + c + 4, make_float4(z.x, z.y, w.x, w.y));
  }
}

// Per channel: ks <- k = 1 - g, ls <- running sums of log g (first per half of the chunk, then joined).
template <int DP, int LD>
__device__ __forceinline__ void channel_logs(const GlaArgs& a, int t0, int m, int head, float* ks, float* ls) {
#pragma unroll 4
  for (int i = threadIdx.x; i < kC * DP / 4; i += kThreads) {
    const int t = i / (DP / 4), x = i % (DP / 4) * 4;
    float4 k = make_float4(0.f, 0.f, 0.f, 0.f), l = k;
    if (t < m && x < a.d) {
      const int ch = head * a.d + x;
      const float4 z = ld_f4(a.raw + (size_t)(t0 + t) * a.heads * a.d + ch), b = ld_f4(a.bias + ch), low = ld_f4(a.par + ch);
      const ChannelGate f0 = channel_gate(z.x + b.x, low.x), f1 = channel_gate(z.y + b.y, low.y),
                        f2 = channel_gate(z.z + b.z, low.z), f3 = channel_gate(z.w + b.w, low.w);
      k = make_float4(f0.write, f1.write, f2.write, f3.write);
      l = make_float4(fmaxf(f0.log_keep(), kMinLog), fmaxf(f1.log_keep(), kMinLog), fmaxf(f2.log_keep(), kMinLog),
                      fmaxf(f3.log_keep(), kMinLog));
    }
    st_f4(ks + t * LD + x, k);
    st_f4(ls + t * LD + x, l);
  }
  __syncthreads();
  const int half = threadIdx.x / DP, c = threadIdx.x % DP;
  if (half < 2) {
    float v[kC / 2];
#pragma unroll
    for (int t = 0; t < kC / 2; ++t) v[t] = ls[(half * kC / 2 + t) * LD + c];
#pragma unroll
    for (int t = 1; t < kC / 2; ++t) v[t] += v[t - 1];
#pragma unroll
    for (int t = 0; t < kC / 2; ++t) ls[(half * kC / 2 + t) * LD + c] = v[t];
  }
  __syncthreads();
  for (int i = threadIdx.x; i < kC / 2 * DP; i += kThreads) ls[(kC / 2 + i / DP) * LD + i % DP] += ls[(kC / 2 - 1) * LD + i % DP];
  __syncthreads();
}

// ------------------------------------------------------------------ contributions
template <int DP, int MODE>
struct StateCfg {
  static constexpr int LD = DP + 8;
  static constexpr int MW = DP / 16 < 4 ? DP / 16 : 4, NW = 8 / MW;      // warps along the keys and along the columns
  static constexpr int MT = DP / 16 / MW, NT = kCols / 8 / NW;           // tiles of a warp
  static constexpr int SMEM = (kC * LD * (MODE == kForget ? 2 : 1) + kC * kVL + 2 * kC) * 4;
};

template <int DP, int MODE>
__global__ void __launch_bounds__(kThreads) gla_chunk_state_kernel(const bf16* __restrict__ k, const bf16* __restrict__ v,
                                                                   const ChunkArgs a) {
  pdl_entry();
  using C = StateCfg<DP, MODE>;
  constexpr int LD = C::LD;
  extern __shared__ __align__(16) float sm[];
  float* ks = sm;                                           // [kC][LD] k e^{L_63 - L}
  float* vs = ks + kC * LD;                                 // [kC][kVL]
  float* ls = vs + kC * kVL;                                // [kC] or [kC][LD]
  float* fac = ls + (MODE == kForget ? kC * LD : kC);       // [kC]
  const int c = blockIdx.x, head = blockIdx.y, v0 = blockIdx.z * kCols, d = a.g.d, e = a.g.e, ew = a.g.ew, tid = threadIdx.x;
  const int t0 = a.chunks[c * 2], m = a.chunks[c * 2 + 1];
  const size_t ch = (size_t)c * a.g.heads + head;
  load_rows<kCols, kVL>(v, a.g.ldv, t0, m, head * e + v0, e - v0, vs);
  if constexpr (MODE == kForget) {
    channel_logs<DP, LD>(a.g, t0, m, head, ks, ls);
    for (int i = tid; i < kC * DP; i += kThreads) {
      const int t = i / DP, x = i % DP;
      ks[t * LD + x] *= __expf(ls[(kC - 1) * LD + x] - ls[t * LD + x]);
    }
    if (v0 == 0 && tid < d) a.decay[ch * d + tid] = expf(ls[(kC - 1) * LD + tid]);
  } else {
    load_rows<DP, LD>(k, a.g.ldk, t0, m, head / a.g.group * d, d, ks);
    head_logs<MODE>(a.g, t0, m, head, ls, fac);
    __syncthreads();
    for (int i = tid; i < kC * DP; i += kThreads) {
      const int t = i / DP, x = i % DP;
      ks[t * LD + x] *= __expf(ls[kC - 1] - ls[t]) * fac[t];
    }
    if (v0 == 0 && tid == 0) a.decay[ch] = expf(ls[kC - 1]);
  }
  __syncthreads();
  float* u = a.us + ch * d * ew;
  const int warp = tid >> 5, lane = tid & 31, g = lane >> 2, tt = lane & 3;
  const int m0 = warp % C::MW * C::MT * 16, n0 = warp / C::MW * C::NT * 8;
  float acc[C::MT][C::NT][4] = {};
#pragma unroll 1
  for (int s = 0; s < kC; s += 8) {
    FragA f[C::MT];
#pragma unroll
    for (int i = 0; i < C::MT; ++i) {
      const float *p0 = ks + (s + tt) * LD + m0 + i * 16 + g, *p1 = p0 + 4 * LD;
      f[i] = frag_a(p0[0], p0[8], p1[0], p1[8]);
    }
#pragma unroll
    for (int j = 0; j < C::NT; ++j) {
      const uint32_t b0 = bits(vs[(s + tt) * kVL + n0 + j * 8 + g]), b1 = bits(vs[(s + tt + 4) * kVL + n0 + j * 8 + g]);
#pragma unroll
      for (int i = 0; i < C::MT; ++i) {
        mma_tf32(acc[i][j], f[i].v[0].lo, f[i].v[1].lo, f[i].v[2].lo, f[i].v[3].lo, b0, b1);
        mma_tf32(acc[i][j], f[i].v[0].hi, f[i].v[1].hi, f[i].v[2].hi, f[i].v[3].hi, b0, b1);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < C::MT; ++i)
#pragma unroll
    for (int j = 0; j < C::NT; ++j)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int key = m0 + i * 16 + g + h * 8, x = v0 + n0 + j * 8 + 2 * tt;
        if (key < d && x < e) *reinterpret_cast<float2*>(u + (size_t)key * ew + x) = make_float2(acc[i][j][2 * h], acc[i][j][2 * h + 1]);
      }
  if (MODE == kGiven && v0 == 0 && tid < d) {       // the column of ones, and the padding behind it
    float s = 0.f;
#pragma unroll 8
    for (int t = 0; t < kC; ++t) s += ks[t * LD + tid];
    for (int x = e; x < ew; ++x) u[(size_t)tid * ew + x] = x == e ? s : 0.f;
  }
}

// ------------------------------------------------------------------ carry
// One thread per 4 consecutive state elements of one key.  segs: [n][4] = slot, first chunk, chunks, first row.
template <bool CHANNEL>
__global__ void __launch_bounds__(128) gla_chunk_carry_kernel(const ChunkArgs a, const int* __restrict__ segs) {
  pdl_entry();
  const int seg = blockIdx.x, head = blockIdx.y, d = a.g.d, ew = a.g.ew, heads = a.g.heads;
  const int i = (blockIdx.z * 128 + threadIdx.x) * 4;
  if (i >= d * ew) return;
  const int slot = segs[seg * 4], c0 = segs[seg * 4 + 1], n = segs[seg * 4 + 2], row = segs[seg * 4 + 3];
  const size_t per = (size_t)d * ew, step = heads * per, dstep = CHANNEL ? (size_t)heads * d : heads;
  float* st = a.g.state + ((size_t)slot * heads + head) * per + i;
  float s[4] = {};
  if (a.g.pos[row] != 0) ld_w<4>(st, s);
  float* u = a.us + ((size_t)c0 * heads + head) * per + i;
  const float* w = a.decay + (CHANNEL ? ((size_t)c0 * heads + head) * d + i / ew : (size_t)c0 * heads + head);
  constexpr int B = 8;
  for (int c = 0; c < n; c += B) {
    float uv[B][4], wv[B];
#pragma unroll
    for (int j = 0; j < B; ++j)
      if (c + j < n) ld_w<4>(u + (c + j) * step, uv[j]), wv[j] = w[(c + j) * dstep];
#pragma unroll
    for (int j = 0; j < B; ++j)
      if (c + j < n) {
        st_w<4>(u + (c + j) * step, s);
#pragma unroll
        for (int x = 0; x < 4; ++x) s[x] = fmaf(wv[j], s[x], uv[j][x]);
      }
  }
  st_w<4>(st, s);
}

// ------------------------------------------------------------------ outputs
template <int DP, int MODE>
struct OutCfg {
  static constexpr int LD = DP + 8;
  static constexpr int KV = LD > kVL ? LD : kVL;               // k, later the values
  static constexpr int EXTRA = MODE == kForget ? kC * LD + 4 * DP : 2 * kC + DP;
  static constexpr int SMEM = (kC * LD + kC * KV + kC * kAL + EXTRA) * 4;
};

template <int DP, int MODE>
__global__ void __launch_bounds__(kThreads) gla_chunk_out_kernel(const bf16* __restrict__ q, const bf16* __restrict__ k,
                                                                 const bf16* __restrict__ v, const ChunkArgs a) {
  pdl_entry();
  using C = OutCfg<DP, MODE>;
  constexpr int LD = C::LD;
  extern __shared__ __align__(16) float sm[];
  float* qs = sm;                       // [kC][LD]
  float* ks = qs + kC * LD;             // [kC][LD], then values [kC][kVL]
  float* am = ks + kC * C::KV;          // [kC][kAL] A, zero above the diagonal
  float* ls = am + kC * kAL;            // [kC] or [kC][LD] running logs
  float* fac = ls + (MODE == kForget ? kC * LD : kC);   // per head: [kC] factors of k; per channel: [4][DP] L of the references
  float* ns = fac + kC;                 // kGiven: [DP] the column of ones of the state
  const int c = blockIdx.x, head = blockIdx.y, v0 = blockIdx.z * kCols, d = a.g.d, e = a.g.e, ew = a.g.ew, tid = threadIdx.x;
  const int t0 = a.chunks[c * 2], m = a.chunks[c * 2 + 1], at_k = head / a.g.group * d;
  const int warp = tid >> 5, lane = tid & 31, g = lane >> 2, tt = lane & 3;
  const float* u = a.us + ((size_t)c * a.g.heads + head) * d * ew;
  load_rows<DP, LD>(q, a.g.ldq, t0, m, at_k, d, qs);
  for (int i = tid; i < kC * kAL; i += kThreads) am[i] = 0.f;
  bool wild = false;
  if constexpr (MODE == kForget) {
    channel_logs<DP, LD>(a.g, t0, m, head, ks, ls);
    for (int i = tid; i < 4 * DP; i += kThreads) {
      const int b = i / DP, x = i % DP;
      const float* l = ls + b * 16 * LD + x;
      fac[i] = l[7 * LD];
      wild |= fmaxf(l[0] - l[7 * LD], l[7 * LD] - l[15 * LD]) > kSafe;
    }
    wild = __syncthreads_or(wild);
    for (int i = tid; i < kC * DP / 4; i += kThreads) {
      const int t = i / (DP / 4), x = i % (DP / 4) * 4;
      float4 y = ld_f4(qs + t * LD + x);
      y.x *= a.g.q_mul * sigmoid_f(y.x), y.y *= a.g.q_mul * sigmoid_f(y.y);
      y.z *= a.g.q_mul * sigmoid_f(y.z), y.w *= a.g.q_mul * sigmoid_f(y.w);
      if (!wild) {
        const float4 l = ld_f4(ls + t * LD + x), r = ld_f4(fac + t / 16 * DP + x);
        float4 z = ld_f4(ks + t * LD + x);
        y.x *= __expf(l.x - r.x), y.y *= __expf(l.y - r.y), y.z *= __expf(l.z - r.z), y.w *= __expf(l.w - r.w);
        z.x *= __expf(r.x - l.x), z.y *= __expf(r.y - l.y), z.z *= __expf(r.z - l.z), z.w *= __expf(r.w - l.w);
        st_f4(ks + t * LD + x, z);
      }
      st_f4(qs + t * LD + x, y);
    }
  } else {
    load_rows<DP, LD>(k, a.g.ldk, t0, m, at_k, d, ks);
    head_logs<MODE>(a.g, t0, m, head, ls, fac);
    if (MODE == kGiven && tid < DP) ns[tid] = tid < d ? u[(size_t)tid * ew + e] : 0.f;
  }
  __syncthreads();
  // ---- A: sources [8 warp, +8) against the row tiles at or below them
  if (MODE == kForget && wild) {
    for (int i = tid; i < kC * (kC + 1) / 2; i += kThreads) {
      int t = (int)((sqrtf(8.f * i + 1.f) - 1.f) * 0.5f);        // i = t (t + 1) / 2 + s, s <= t
      while (t * (t + 1) / 2 > i) --t;
      while ((t + 1) * (t + 2) / 2 <= i) ++t;
      const int s = i - t * (t + 1) / 2;
      float x = 0.f;
      for (int j = 0; j < d; ++j) x = fmaf(qs[t * LD + j] * ks[s * LD + j], __expf(ls[t * LD + j] - ls[s * LD + j]), x);
      am[t * kAL + s] = x;
    }
  } else {
    const int i0 = warp / 2;
    float acc[4][4] = {};
#pragma unroll 2
    for (int x = 2 * tt; x < DP; x += 8) {
      const float2 y = ld_f2(ks + (warp * 8 + g) * LD + x);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        if (i < i0) continue;
        const float2 r0 = ld_f2(qs + (i * 16 + g) * LD + x), r1 = ld_f2(qs + (i * 16 + 8 + g) * LD + x);
        if constexpr (MODE == kForget) {
          float2 z = y;
          if (i > i0) {
            const float2 hi = ld_f2(fac + i * DP + x), lo = ld_f2(fac + i0 * DP + x);
            z.x *= __expf(hi.x - lo.x), z.y *= __expf(hi.y - lo.y);
          }
          mma3(acc[i], frag_a(r0.x, r1.x, r0.y, r1.y), z);
        } else {
          mma_tf32(acc[i], bits(r0.x), bits(r1.x), bits(r0.y), bits(r1.y), bits(y.x), bits(y.y));
        }
      }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int t = i * 16 + g + (j >> 1) * 8, s = warp * 8 + 2 * tt + (j & 1);
        if (i < i0 || s > t) continue;
        float x = acc[i][j];
        if constexpr (MODE != kForget) x *= a.g.q_mul * __expf(ls[t] - ls[s]) * fac[s];
        am[t * kAL + s] = x;
      }
  }
  __syncthreads();
  load_rows<kCols, kVL>(v, a.g.ldv, t0, m, head * e + v0, e - v0, ks);
  if constexpr (MODE == kForget) {     // q e^L
    for (int i = tid; i < kC * DP; i += kThreads) {
      const int t = i / DP, x = i % DP;
      qs[t * LD + x] *= __expf(wild ? ls[t * LD + x] : fac[t / 16 * DP + x]);
    }
    __syncthreads();
  }
  // ---- outputs: all 64 tokens x columns [16 warp, +16)
  const int n0 = warp * 16;
  float acc[4][2][4] = {};
  if (v0 + n0 < e) {
#pragma unroll 2
    for (int x = 2 * tt; x < DP; x += 8) {
      float2 b[2];
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int col = v0 + n0 + j * 8 + g;
        const float* p = u + (size_t)x * ew + col;
        b[j] = make_float2(x < d && col < e ? p[0] : 0.f, x + 1 < d && col < e ? p[ew] : 0.f);
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float2 r0 = ld_f2(qs + (i * 16 + g) * LD + x), r1 = ld_f2(qs + (i * 16 + 8 + g) * LD + x);
        if constexpr (MODE == kForget) {
          const FragA f = frag_a(r0.x, r1.x, r0.y, r1.y);
#pragma unroll
          for (int j = 0; j < 2; ++j) mma3(acc[i][j], f, b[j]);
        } else {
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            const Split y0 = split(b[j].x), y1 = split(b[j].y);
            mma_tf32(acc[i][j], bits(r0.x), bits(r1.x), bits(r0.y), bits(r1.y), y0.lo, y1.lo);
            mma_tf32(acc[i][j], bits(r0.x), bits(r1.x), bits(r0.y), bits(r1.y), y0.hi, y1.hi);
          }
        }
      }
    }
    if constexpr (MODE != kForget) {
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float f0 = a.g.q_mul * __expf(ls[i * 16 + g]), f1 = a.g.q_mul * __expf(ls[i * 16 + 8 + g]);
#pragma unroll
        for (int j = 0; j < 2; ++j) acc[i][j][0] *= f0, acc[i][j][1] *= f0, acc[i][j][2] *= f1, acc[i][j][3] *= f1;
      }
    }
  }
  __syncthreads();                        // the values are in place
  if (v0 + n0 < e) {
#pragma unroll
    for (int s = 0; s < kC; s += 8) {
      uint32_t b[2][2];
#pragma unroll
      for (int j = 0; j < 2; ++j)
        b[j][0] = bits(ks[(s + tt) * kVL + n0 + j * 8 + g]), b[j][1] = bits(ks[(s + tt + 4) * kVL + n0 + j * 8 + g]);
#pragma unroll
      for (int i = s / 16; i < 4; ++i) {
        const float *p0 = am + (i * 16 + g) * kAL + s + tt, *p1 = p0 + 8 * kAL;
        const FragA f = frag_a(p0[0], p1[0], p0[4], p1[4]);
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          mma_tf32(acc[i][j], f.v[0].lo, f.v[1].lo, f.v[2].lo, f.v[3].lo, b[j][0], b[j][1]);
          mma_tf32(acc[i][j], f.v[0].hi, f.v[1].hi, f.v[2].hi, f.v[3].hi, b[j][0], b[j][1]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int t = i * 16 + g + h * 8;
        if (t >= m) continue;
        float* o = a.g.out + ((size_t)(t0 + t) * a.g.heads + head) * ew + v0 + n0 + 2 * tt;
#pragma unroll
        for (int j = 0; j < 2; ++j)
          if (v0 + n0 + j * 8 + 2 * tt < e) *reinterpret_cast<float2*>(o + j * 8) = make_float2(acc[i][j][2 * h], acc[i][j][2 * h + 1]);
      }
  }
  if (MODE == kGiven && v0 == 0) {        // the column of ones
    for (int t = warp; t < m; t += kThreads / 32) {
      float x = 0.f, y = 0.f;
      for (int j = lane; j < DP; j += 32) x = fmaf(qs[t * LD + j], ns[j], x);
      for (int s = lane; s <= t; s += 32) y += am[t * kAL + s];
      x = warp_sum(fmaf(a.g.q_mul * __expf(ls[t]), x, y));
      if (lane == 0) a.g.out[((size_t)(t0 + t) * a.g.heads + head) * ew + e] = x;
    }
  }
}

template <int DP, int MODE>
int launch_chunks(const bf16* q, const bf16* k, const bf16* v, const ChunkArgs& a, int n_chunks, const int* segs, int n_segs,
                  cudaStream_t st) {
  using S = StateCfg<DP, MODE>;
  using O = OutCfg<DP, MODE>;
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(gla_chunk_state_kernel<DP, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, S::SMEM) !=
            cudaSuccess ||
        cudaFuncSetAttribute(gla_chunk_out_kernel<DP, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, O::SMEM) != cudaSuccess)
      return 711;
    set = true;
  }
  const dim3 grid(n_chunks, a.g.heads, (a.g.e + kCols - 1) / kCols);
  dsv4_launch(gla_chunk_state_kernel<DP, MODE>, grid, kThreads, S::SMEM, st, k, v, a);
  dsv4_launch(gla_chunk_carry_kernel<MODE == kForget>, dim3(n_segs, a.g.heads, (a.g.d * a.g.ew / 4 + 127) / 128), 128, 0, st, a, segs);
  dsv4_launch(gla_chunk_out_kernel<DP, MODE>, grid, kThreads, O::SMEM, st, q, k, v, a);
  return (int)cudaGetLastError();
}
template <int MODE>
int dispatch_chunks(const bf16* q, const bf16* k, const bf16* v, const ChunkArgs& a, int n_chunks, const int* segs, int n_segs,
                    cudaStream_t st) {
  if (a.g.d <= 32) return launch_chunks<32, MODE>(q, k, v, a, n_chunks, segs, n_segs, st);
  if (a.g.d <= 64) return launch_chunks<64, MODE>(q, k, v, a, n_chunks, segs, n_segs, st);
  return launch_chunks<128, MODE>(q, k, v, a, n_chunks, segs, n_segs, st);
}

}  // namespace

// Arguments as in dsv4_gla_scan, q, k and v bf16 with rows and first columns on 16 bytes; d, e multiples of 8, d <= 128.  chunks
// [n_chunks][2] = first row, tokens (at most 64; a request's chunks stand together), segs [n_segs][4] = slot, first chunk, chunks,
// first row; us [n_chunks, heads, d, ew] and decay [n_chunks, heads (, d for mode 2)] scratch.
DSV4_API int dsv4_gla_chunked(int mode, const void* q, int ldq, const void* k, int ldk, const void* v, int ldv, const float* raw,
                              const float* fac, const float* bias, const float* par, float q_mul, float* state, float* out,
                              const int* pos, const int* chunks, int n_chunks, const int* segs, int n_segs, float* us,
                              float* decay, int heads, int group, int d, int e, int ew, cudaStream_t st) {
  if (n_chunks <= 0 || n_segs <= 0) return 0;
  if (mode < 0 || mode > 2 || heads < 1 || heads > 65535 || group < 1 || d < 8 || d % 8 || e < 8 || e % 8 || d > 128 || ew % 4 ||
      ew < e + (mode == kGiven))
    return 712;
  if (ldq % 8 || ldk % 8 || ldv % 8 || (((uintptr_t)q | (uintptr_t)k | (uintptr_t)v) & 15)) return 713;
  const ChunkArgs a{{ldq, ldk, ldv, raw, fac, bias, par, q_mul, heads, group, d, e, ew, state, out, nullptr, pos}, chunks, us, decay};
  const bf16 *bq = (const bf16*)q, *bk = (const bf16*)k, *bv = (const bf16*)v;
  if (mode == kGiven) return dispatch_chunks<kGiven>(bq, bk, bv, a, n_chunks, segs, n_segs, st);
  if (mode == kStep) return dispatch_chunks<kStep>(bq, bk, bv, a, n_chunks, segs, n_segs, st);
  return dispatch_chunks<kForget>(bq, bk, bv, a, n_chunks, segs, n_segs, st);
}
