// Gated linear attention (gla.cuh) of long prompt portions in chunks of 64 tokens, bf16 activations.  With L_t = sum_{j <= t} log
// g_j inside a chunk and S the state before it,
//
//   o_t    = (q_t e^{L_t})^T S + sum_{s <= t} A_ts v_s,        A_ts = q_t . (k_s e^{L_t - L_s})
//   S_next = diag(e^{L_63}) S + sum_s (k_s e^{L_63 - L_s}) v_s^T
//
// so that only the carry S -> S_next runs in sequence:
//   gla_chunk_state_kernel   every (chunk, head, 64 or 128 value columns): its own contribution U and e^{L_63}
//   gla_chunk_carry_kernel   per state element: walks a request's chunks, leaves the state before each chunk in U's place
//   gla_chunk_out_kernel     every (chunk, head, 64 or 128 value columns): the outputs
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
// contraction index is free as long as A and B agree: places t, t + 4 stand for 2t, 2t + 1, which are neighbours in memory and in the
// registers that ldmatrix fills from bf16 tiles.
#include "gla.cuh"
#include "mma16.cuh"
#include "tf32.cuh"

namespace {

constexpr int kC = 64;            // tokens of a chunk
constexpr float kMinLog = -40.f;
constexpr float kSafe = 60.f;
constexpr int kThreads = 256;
constexpr int kAL = kC + 8;       // row stride of A (8 mod 32: conflict-free 8-byte reads)

struct ChunkArgs {
  GlaArgs g;
  const int* chunks;      // [chunks][2]: first row, tokens
  float* us;              // [chunks][heads][d][ew] contributions, then states
  float* decay;           // [chunks][heads] or, per channel, [chunks][heads][d]: e^{L_63}
};

using bf16 = __nv_bfloat16;

__device__ __forceinline__ float2 ld_f2(const float* p) { return *reinterpret_cast<const float2*>(p); }
// The two bf16 values of a register as 32-bit floats, which TF32 holds exactly.
__device__ __forceinline__ uint32_t lo16(uint32_t r) { return r << 16; }
__device__ __forceinline__ uint32_t hi16(uint32_t r) { return r & 0xffff0000u; }

// Columns [c0, c0 + n) of the chunk's rows in 16-byte pieces, zeros past n and past the last token; n, c0 multiples of 8.
template <int P>
struct Rows {
  static constexpr int N = kC * P / 8 / kThreads;
  uint4 u[N];
  __device__ __forceinline__ void load(const bf16* p, int ld, int t0, int m, int c0, int n) {
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int x = threadIdx.x + i * kThreads, t = x / (P / 8), c = x % (P / 8) * 8;
      u[i] = make_uint4(0, 0, 0, 0);
      if (t < m && c < n) u[i] = *reinterpret_cast<const uint4*>(p + (size_t)(t0 + t) * ld + c0 + c);
    }
  }
  // as bf16 [kC][P + 8]: the padding keeps ldmatrix free of bank conflicts
  __device__ __forceinline__ void store(bf16* dst) const {
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int x = threadIdx.x + i * kThreads;
      *reinterpret_cast<uint4*>(dst + x / (P / 8) * (P + 8) + x % (P / 8) * 8) = u[i];
    }
  }
  // as floats [kC][P + 8]
  __device__ __forceinline__ void store(float* dst) const {
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int x = threadIdx.x + i * kThreads;
      float* d = dst + x / (P / 8) * (P + 8) + x % (P / 8) * 8;
      const uint32_t r[4] = {u[i].x, u[i].y, u[i].z, u[i].w};
#pragma unroll
      for (int j = 0; j < 4; j += 2)
        st_f4(d + 2 * j, make_float4(__uint_as_float(lo16(r[j])), __uint_as_float(hi16(r[j])), __uint_as_float(lo16(r[j + 1])),
                                     __uint_as_float(hi16(r[j + 1]))));
    }
  }
};
template <int P>
__device__ __forceinline__ const bf16* tile16(const bf16* base, int row, int col) {     // ldmatrix address of a 16 x 16 tile
  const int lane = threadIdx.x & 31;
  return base + (row + (lane & 15)) * (P + 8) + col + (lane >> 4) * 8;
}

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
template <int DP, int CW, int MODE>
struct StateCfg {
  static constexpr int LD = DP + 8;
  static constexpr int MW = DP / 16 < 4 ? DP / 16 : 4, NW = 8 / MW;      // warps along the keys and along the columns
  static constexpr int MT = DP / 16 / MW, NT = CW / 8 / NW;              // tiles of a warp
  static constexpr int KS = MODE == kForget ? 2 * kC * LD * 4 : kC * LD * 2 + 2 * kC * 4;
  static constexpr int SMEM = KS + kC * (CW + 8) * 2;
};

template <int DP, int CW, int MODE>
__global__ void __launch_bounds__(kThreads, 2) gla_chunk_state_kernel(const bf16* __restrict__ k, const bf16* __restrict__ v,
                                                                      const ChunkArgs a) {
  pdl_entry();
  using C = StateCfg<DP, CW, MODE>;
  constexpr int LD = C::LD;
  extern __shared__ __align__(16) float sm[];
  // per channel: k e^{L_63 - L} and L as floats [kC][LD]; per head: e^{L_63 - L} fac and L [kC], k as bf16 [kC][LD]
  float *w = sm, *ls = sm + (MODE == kForget ? kC * LD : kC);
  bf16* ks = reinterpret_cast<bf16*>(ls + kC);
  bf16* vs = reinterpret_cast<bf16*>(reinterpret_cast<uint8_t*>(sm) + C::KS);      // [kC][CW + 8]
  const int c = blockIdx.x, head = blockIdx.y, v0 = blockIdx.z * CW, d = a.g.d, e = a.g.e, ew = a.g.ew, tid = threadIdx.x;
  const int t0 = a.chunks[c * 2], m = a.chunks[c * 2 + 1];
  const size_t ch = (size_t)c * a.g.heads + head;
  Rows<CW> rv;
  rv.load(v, a.g.ldv, t0, m, head * e + v0, e - v0);
  if constexpr (MODE == kForget) {
    channel_logs<DP, LD>(a.g, t0, m, head, w, ls);
    for (int i = tid; i < kC * DP; i += kThreads) {
      const int t = i / DP, x = i % DP;
      w[t * LD + x] *= __expf(ls[(kC - 1) * LD + x] - ls[t * LD + x]);
    }
    if (v0 == 0 && tid < d) a.decay[ch * d + tid] = expf(ls[(kC - 1) * LD + tid]);
  } else {
    Rows<DP> rk;
    rk.load(k, a.g.ldk, t0, m, head / a.g.group * d, d);
    head_logs<MODE>(a.g, t0, m, head, ls, w);
    rk.store(ks);
    __syncthreads();
    if (tid < kC) w[tid] *= __expf(ls[kC - 1] - ls[tid]);
    if (v0 == 0 && tid == 0) a.decay[ch] = expf(ls[kC - 1]);
  }
  rv.store(vs);
  __syncthreads();
  float* u = a.us + ch * d * ew;
  const int warp = tid >> 5, lane = tid & 31, g = lane >> 2, tt = lane & 3;
  const int m0 = warp % C::MW * C::MT * 16, n0 = warp / C::MW * C::NT * 8;
  float acc[C::MT][C::NT][4] = {};
#pragma unroll
  for (int s = 0; s < kC; s += 16) {
    uint32_t b[C::NT][2];                       // [columns][8 tokens each]
#pragma unroll
    for (int j = 0; j < C::NT; j += 2) {
      uint32_t r[4];
      ldsm4_t(r, tile16<CW>(vs, s, n0 + j * 8));
      b[j][0] = r[0], b[j][1] = r[1], b[j + 1][0] = r[2], b[j + 1][1] = r[3];
    }
#pragma unroll
    for (int i = 0; i < C::MT; ++i) {
      FragA f[2];
      if constexpr (MODE == kForget) {
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const float *p0 = w + (s + h * 8 + 2 * tt) * LD + m0 + i * 16 + g, *p1 = p0 + LD;
          f[h] = frag_a(p0[0], p0[8], p1[0], p1[8]);
        }
      } else {
        uint32_t r[4];                          // keys m0 + i 16 .. +8 (r0, r1), +8 .. +16 (r2, r3)
        ldsm4_t(r, tile16<DP>(ks, s, m0 + i * 16));
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const float2 x = ld_f2(w + s + h * 8 + 2 * tt);
          f[h] = frag_a(__uint_as_float(lo16(r[h])) * x.x, __uint_as_float(lo16(r[2 + h])) * x.x,
                        __uint_as_float(hi16(r[h])) * x.y, __uint_as_float(hi16(r[2 + h])) * x.y);
        }
      }
#pragma unroll
      for (int h = 0; h < 2; ++h)
#pragma unroll
        for (int j = 0; j < C::NT; ++j) {
          mma_tf32(acc[i][j], f[h].v[0].lo, f[h].v[1].lo, f[h].v[2].lo, f[h].v[3].lo, lo16(b[j][h]), hi16(b[j][h]));
          mma_tf32(acc[i][j], f[h].v[0].hi, f[h].v[1].hi, f[h].v[2].hi, f[h].v[3].hi, lo16(b[j][h]), hi16(b[j][h]));
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
    for (int t = 0; t < kC; ++t) s = fmaf(bf2f(ks[t * LD + tid]), w[t], s);
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
template <int DP, int CW, int MODE>
struct OutCfg {
  static constexpr int LD = DP + 8, VL = CW + 8;
  static constexpr int NW = CW / 16, MW = 8 / NW, MT = 4 / MW;      // warps along the columns and along the tokens; row tiles
  // per channel: q and k as floats, their logs (later A), the references' logs; the values take k's place
  static constexpr int LS = kC * LD > kC * kAL ? kC * LD : kC * kAL;
  static constexpr int KV = kC * LD * 4 > kC * VL * 2 ? kC * LD * 4 : kC * VL * 2;
  // per head: q and k as bf16, values, A, logs, factors, the state's column of ones
  static constexpr int SMEM = MODE == kForget ? kC * LD * 4 + KV + LS * 4 + 4 * DP * 4
                                              : 2 * kC * LD * 2 + kC * VL * 2 + (kC * kAL + 2 * kC + DP) * 4;
};

template <int DP, int CW, int MODE>
__global__ void __launch_bounds__(kThreads, 2) gla_chunk_out_kernel(const bf16* __restrict__ q, const bf16* __restrict__ k,
                                                                    const bf16* __restrict__ v, const ChunkArgs a) {
  pdl_entry();
  using C = OutCfg<DP, CW, MODE>;
  constexpr int LD = C::LD, VL = C::VL, MT = C::MT;
  extern __shared__ __align__(16) uint8_t raw[];
  // per channel
  float* qf = reinterpret_cast<float*>(raw);                      // [kC][LD]
  float* kf = qf + kC * LD;                                       // [kC][LD]
  float* lf = reinterpret_cast<float*>(raw + kC * LD * 4 + C::KV);       // [kC][LD], then A
  float* ref = lf + C::LS;                                        // [4][DP]
  // per head
  bf16 *qs = reinterpret_cast<bf16*>(raw), *ks = qs + kC * LD;    // [kC][LD]
  bf16* vs = MODE == kForget ? reinterpret_cast<bf16*>(kf) : ks + kC * LD;       // [kC][VL]
  float* am = MODE == kForget ? lf : reinterpret_cast<float*>(vs + kC * VL);     // [kC][kAL] A, zero above the diagonal
  float *ls = am + kC * kAL, *fac = ls + kC, *ns = fac + kC;      // [kC], [kC], [DP]
  const int c = blockIdx.x, head = blockIdx.y, v0 = blockIdx.z * CW, d = a.g.d, e = a.g.e, ew = a.g.ew, tid = threadIdx.x;
  const int t0 = a.chunks[c * 2], m = a.chunks[c * 2 + 1], at_k = head / a.g.group * d;
  const int warp = tid >> 5, lane = tid & 31, g = lane >> 2, tt = lane & 3;
  const float* u = a.us + ((size_t)c * a.g.heads + head) * d * ew;
  Rows<CW> rv;
  {
    Rows<DP> rq;
    rq.load(q, a.g.ldq, t0, m, at_k, d);
    rv.load(v, a.g.ldv, t0, m, head * e + v0, e - v0);
    if constexpr (MODE == kForget) {
      rq.store(qf);
    } else {
      Rows<DP> rk;
      rk.load(k, a.g.ldk, t0, m, at_k, d);
      rq.store(qs);
      rk.store(ks);
      rv.store(vs);
    }
  }
  bool wild = false;
  if constexpr (MODE == kForget) {
    channel_logs<DP, LD>(a.g, t0, m, head, kf, lf);
    for (int i = tid; i < 4 * DP; i += kThreads) {
      const float* l = lf + i / DP * 16 * LD + i % DP;
      ref[i] = l[7 * LD];
      wild |= fmaxf(l[0] - l[7 * LD], l[7 * LD] - l[15 * LD]) > kSafe;
    }
    wild = __syncthreads_or(wild);
    for (int i = tid; i < kC * DP / 4; i += kThreads) {
      const int t = i / (DP / 4), x = i % (DP / 4) * 4;
      float4 y = ld_f4(qf + t * LD + x);
      y.x *= a.g.q_mul * sigmoid_f(y.x), y.y *= a.g.q_mul * sigmoid_f(y.y);
      y.z *= a.g.q_mul * sigmoid_f(y.z), y.w *= a.g.q_mul * sigmoid_f(y.w);
      if (!wild) {
        const float4 l = ld_f4(lf + t * LD + x), r = ld_f4(ref + t / 16 * DP + x);
        float4 z = ld_f4(kf + t * LD + x);
        y.x *= __expf(l.x - r.x), y.y *= __expf(l.y - r.y), y.z *= __expf(l.z - r.z), y.w *= __expf(l.w - r.w);
        z.x *= __expf(r.x - l.x), z.y *= __expf(r.y - l.y), z.z *= __expf(r.z - l.z), z.w *= __expf(r.w - l.w);
        st_f4(kf + t * LD + x, z);
      }
      st_f4(qf + t * LD + x, y);
    }
  } else {
    head_logs<MODE>(a.g, t0, m, head, ls, fac);
    if (MODE == kGiven && tid < DP) ns[tid] = tid < d ? u[(size_t)tid * ew + e] : 0.f;
    for (int i = tid; i < kC * kAL; i += kThreads) am[i] = 0.f;
  }
  __syncthreads();
  // ---- A.  The 20 tiles (16 tokens x 8 sources) at or below the diagonal: warps 0-3 take three of the sources [8 warp, +8),
  // warps 4-7 two of what is left.
  constexpr int kPairs = (kC * (kC + 1) / 2 + kThreads - 1) / kThreads;
  int ti[3], si[3];
#pragma unroll
  for (int j = 0; j < 3; ++j) {
    const int p = warp - 4;
    ti[j] = warp < 4 ? j + 1 : j == 0 ? (p < 2 ? 0 : 2) : 3;
    si[j] = warp < 4 ? warp : j == 0 ? (p < 2 ? p : 7 - p) : 7 - p;
  }
  const int nt = warp < 4 ? 3 : 2;
  float acc3[3][4] = {};
  float pair[MODE == kForget ? kPairs : 1];
  if constexpr (MODE == kForget) {
    if (wild) {
#pragma unroll 1
      for (int n = 0; n < kPairs; ++n) {
        const int i = n * kThreads + tid;
        float x = 0.f;
        if (i < kC * (kC + 1) / 2) {
          int t = (int)((sqrtf(8.f * i + 1.f) - 1.f) * 0.5f);        // i = t (t + 1) / 2 + s, s <= t
          while (t * (t + 1) / 2 > i) --t;
          while ((t + 1) * (t + 2) / 2 <= i) ++t;
          const int s = i - t * (t + 1) / 2;
          for (int j = 0; j < d; ++j) x = fmaf(qf[t * LD + j] * kf[s * LD + j], __expf(lf[t * LD + j] - lf[s * LD + j]), x);
        }
#pragma unroll
        for (int j = 0; j < kPairs; ++j)
          if (j == n) pair[j] = x;
      }
    } else {
#pragma unroll 2
      for (int x = 2 * tt; x < DP; x += 8) {
#pragma unroll
        for (int j = 0; j < 3; ++j) {
          if (j >= nt) continue;
          const float2 r0 = ld_f2(qf + (ti[j] * 16 + g) * LD + x), r1 = ld_f2(qf + (ti[j] * 16 + 8 + g) * LD + x);
          float2 z = ld_f2(kf + (si[j] * 8 + g) * LD + x);
          if (ti[j] > si[j] / 2) {              // across blocks
            const float2 hi = ld_f2(ref + ti[j] * DP + x), lo = ld_f2(ref + si[j] / 2 * DP + x);
            z.x *= __expf(hi.x - lo.x), z.y *= __expf(hi.y - lo.y);
          }
          mma3(acc3[j], frag_a(r0.x, r1.x, r0.y, r1.y), z);
        }
      }
    }
    __syncthreads();                            // q, k and, with wild decays, the logs have been read
    for (int i = tid; i < kC * DP / 4; i += kThreads) {          // q e^L
      const int t = i / (DP / 4), x = i % (DP / 4) * 4;
      float4 y = ld_f4(qf + t * LD + x);
      const float4 l = ld_f4(wild ? lf + t * LD + x : ref + t / 16 * DP + x);
      y.x *= __expf(l.x), y.y *= __expf(l.y), y.z *= __expf(l.z), y.w *= __expf(l.w);
      st_f4(qf + t * LD + x, y);
    }
    rv.store(vs);
    if (wild) __syncthreads();
    for (int i = tid; i < kC * kAL; i += kThreads) am[i] = 0.f;
    __syncthreads();
  } else {
#pragma unroll
    for (int x = 0; x < DP; x += 32) {
      uint32_t b[4];
      if (warp < 4) ldsm4(b, ks + (warp * 8 + (lane & 7)) * LD + x + (lane >> 3) * 8);
#pragma unroll
      for (int j = 0; j < 3; ++j) {
        if (j >= nt) continue;
        if (warp >= 4) ldsm4(b, ks + (si[j] * 8 + (lane & 7)) * LD + x + (lane >> 3) * 8);
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          uint32_t r[4];
          ldsm4(r, tile16<DP>(qs, ti[j] * 16, x + h * 16));
          mma16816(acc3[j], r, b[2 * h], b[2 * h + 1]);
        }
      }
    }
  }
  if (MODE == kForget && wild) {
#pragma unroll
    for (int n = 0; n < kPairs; ++n) {
      const int i = n * kThreads + tid;
      if (i >= kC * (kC + 1) / 2) break;
      int t = (int)((sqrtf(8.f * i + 1.f) - 1.f) * 0.5f);
      while (t * (t + 1) / 2 > i) --t;
      while ((t + 1) * (t + 2) / 2 <= i) ++t;
      am[t * kAL + i - t * (t + 1) / 2] = pair[MODE == kForget ? n : 0];
    }
  } else {
#pragma unroll
    for (int j = 0; j < 3; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int t = ti[j] * 16 + g + (i >> 1) * 8, s = si[j] * 8 + 2 * tt + (i & 1);
        if (j >= nt || s > t) continue;
        float x = acc3[j][i];
        if constexpr (MODE != kForget) x *= a.g.q_mul * __expf(ls[t] - ls[s]) * fac[s];
        am[t * kAL + s] = x;
      }
  }
  // ---- outputs: row tiles `row(i)` x columns [n0, +16)
  const int n0 = warp % C::NW * 16, half = warp / C::NW;
  auto row = [&](int i) { return MT == 4 ? i : (i == 0 ? half : 3 - half); };      // 0 and 3, or 1 and 2: equal shares of A
  const bool live = v0 + n0 < e;
  float acc[MT][2][4] = {};
  if (live) {
    constexpr int GS = DP < 64 ? DP / 8 : 4;              // steps of 8 channels whose state is fetched ahead
    float2 nb[GS][2], b[GS][2];
    auto fetch = [&](int x0) {
#pragma unroll
      for (int s = 0; s < GS; ++s)
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          const int x = x0 + s * 8 + 2 * tt, col = v0 + n0 + j * 8 + g;
          const float* p = u + (size_t)x * ew + col;
          nb[s][j] = make_float2(0.f, 0.f);
          if (x < d && col < e) nb[s][j] = make_float2(p[0], p[ew]);            // d is a multiple of 8
        }
    };
    fetch(0);
#pragma unroll 1
    for (int x0 = 0; x0 < DP; x0 += GS * 8) {
#pragma unroll
      for (int s = 0; s < GS; ++s) b[s][0] = nb[s][0], b[s][1] = nb[s][1];
      if (x0 + GS * 8 < DP) fetch(x0 + GS * 8);
#pragma unroll
      for (int s = 0; s < GS; s += 2) {
        const int x = x0 + s * 8;
        if constexpr (MODE == kForget) {
#pragma unroll
          for (int h = 0; h < 2; ++h)
#pragma unroll
            for (int i = 0; i < MT; ++i) {
              const float2 r0 = ld_f2(qf + (row(i) * 16 + g) * LD + x + h * 8 + 2 * tt);
              const float2 r1 = ld_f2(qf + (row(i) * 16 + 8 + g) * LD + x + h * 8 + 2 * tt);
              const FragA f = frag_a(r0.x, r1.x, r0.y, r1.y);
#pragma unroll
              for (int j = 0; j < 2; ++j) mma3(acc[i][j], f, b[s + h][j]);
            }
        } else {
          uint32_t r[MT][4];
#pragma unroll
          for (int i = 0; i < MT; ++i) ldsm4(r[i], tile16<DP>(qs, row(i) * 16, x));
#pragma unroll
          for (int h = 0; h < 2; ++h)
#pragma unroll
            for (int j = 0; j < 2; ++j) {
              const Split y0 = split(b[s + h][j].x), y1 = split(b[s + h][j].y);
#pragma unroll
              for (int i = 0; i < MT; ++i) {
                const uint32_t r0 = r[i][2 * h], r1 = r[i][2 * h + 1];
                mma_tf32(acc[i][j], lo16(r0), lo16(r1), hi16(r0), hi16(r1), y0.lo, y1.lo);
                mma_tf32(acc[i][j], lo16(r0), lo16(r1), hi16(r0), hi16(r1), y0.hi, y1.hi);
              }
            }
        }
      }
    }
    if constexpr (MODE != kForget) {
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        const float f0 = a.g.q_mul * __expf(ls[row(i) * 16 + g]), f1 = a.g.q_mul * __expf(ls[row(i) * 16 + 8 + g]);
#pragma unroll
        for (int j = 0; j < 2; ++j) acc[i][j][0] *= f0, acc[i][j][1] *= f0, acc[i][j][2] *= f1, acc[i][j][3] *= f1;
      }
    }
  }
  __syncthreads();                        // A is complete
  if (live) {
#pragma unroll
    for (int s = 0; s < kC; s += 16) {
      uint32_t b[4];                      // columns n0 .. +8 (b0, b1), +8 .. +16 (b2, b3), 8 tokens each
      ldsm4_t(b, tile16<CW>(vs, s, n0));
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        if (row(i) < s / 16) continue;
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const float2 p0 = ld_f2(am + (row(i) * 16 + g) * kAL + s + h * 8 + 2 * tt);
          const float2 p1 = ld_f2(am + (row(i) * 16 + 8 + g) * kAL + s + h * 8 + 2 * tt);
          const FragA f = frag_a(p0.x, p1.x, p0.y, p1.y);
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            mma_tf32(acc[i][j], f.v[0].lo, f.v[1].lo, f.v[2].lo, f.v[3].lo, lo16(b[2 * j + h]), hi16(b[2 * j + h]));
            mma_tf32(acc[i][j], f.v[0].hi, f.v[1].hi, f.v[2].hi, f.v[3].hi, lo16(b[2 * j + h]), hi16(b[2 * j + h]));
          }
        }
      }
    }
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int t = row(i) * 16 + g + h * 8;
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
      for (int j = lane; j < DP; j += 32) x = fmaf(bf2f(qs[t * LD + j]), ns[j], x);
      for (int s = lane; s <= t; s += 32) y += am[t * kAL + s];
      x = warp_sum(fmaf(a.g.q_mul * __expf(ls[t]), x, y));
      if (lane == 0) a.g.out[((size_t)(t0 + t) * a.g.heads + head) * ew + e] = x;
    }
  }
}

template <int DP, int CW, int MODE>
int launch_chunks(const bf16* q, const bf16* k, const bf16* v, const ChunkArgs& a, int n_chunks, const int* segs, int n_segs,
                  cudaStream_t st) {
  using S = StateCfg<DP, CW, MODE>;
  using O = OutCfg<DP, CW, MODE>;
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(gla_chunk_state_kernel<DP, CW, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, S::SMEM) !=
            cudaSuccess ||
        cudaFuncSetAttribute(gla_chunk_out_kernel<DP, CW, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, O::SMEM) !=
            cudaSuccess)
      return 711;
    set = true;
  }
  const dim3 grid(n_chunks, a.g.heads, (a.g.e + CW - 1) / CW);
  dsv4_launch(gla_chunk_state_kernel<DP, CW, MODE>, grid, kThreads, S::SMEM, st, k, v, a);
  dsv4_launch(gla_chunk_carry_kernel<MODE == kForget>, dim3(n_segs, a.g.heads, (a.g.d * a.g.ew / 4 + 127) / 128), 128, 0, st, a, segs);
  dsv4_launch(gla_chunk_out_kernel<DP, CW, MODE>, grid, kThreads, O::SMEM, st, q, k, v, a);
  return (int)cudaGetLastError();
}
template <int DP, int MODE>
int dispatch_columns(const bf16* q, const bf16* k, const bf16* v, const ChunkArgs& a, int n_chunks, const int* segs, int n_segs,
                     cudaStream_t st) {
  return a.g.e <= 64 ? launch_chunks<DP, 64, MODE>(q, k, v, a, n_chunks, segs, n_segs, st)
                     : launch_chunks<DP, 128, MODE>(q, k, v, a, n_chunks, segs, n_segs, st);
}
template <int MODE>
int dispatch_chunks(const bf16* q, const bf16* k, const bf16* v, const ChunkArgs& a, int n_chunks, const int* segs, int n_segs,
                    cudaStream_t st) {
  if (a.g.d <= 32) return dispatch_columns<32, MODE>(q, k, v, a, n_chunks, segs, n_segs, st);
  if (a.g.d <= 64) return dispatch_columns<64, MODE>(q, k, v, a, n_chunks, segs, n_segs, st);
  return dispatch_columns<128, MODE>(q, k, v, a, n_chunks, segs, n_segs, st);
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
