// The gated delta rule of delta.cu for long prompt portions, in chunks of 32 tokens.  With L_t = sum_{j <= t} log g_j inside a
// chunk (per key channel) and S the state before it, the writes u_t solve a triangular system,
//
//   u_t + beta_t sum_{s < t} A_ts u_s = beta_t (v_t - S^T (k_t e^{L_t})),      A_ts = k_t . (k_s e^{L_t - L_s})
//
// so u = U0 - W S, where U0 and W solve it for the right sides beta v and beta (k e^L) and depend on the chunk alone;
//
//   o_t    = S^T (q_t e^{L_t}) + sum_{s <= t} B_ts u_s,                        B_ts = q_t . (k_s e^{L_t - L_s})
//   S_next = diag(e^{L_31}) S + sum_s (k_s e^{L_31 - L_s}) u_s^T.
//
//   delta_chunk_prep_kernel   every (chunk, head): A, B, W, U0, q e^L, k e^{L_31 - L}, e^{L_31}
//   delta_chunk_walk_kernel   every (request, head, 16 value columns): the chunks in sequence; columns of S are independent
// and head_norm_gate (delta.cu) behind them.
//
// The recurrence is a 32-bit computation.  Products run on the tensor cores in three TF32 terms: x = hi + lo with hi cut
// off to TF32's 11 bits, and hi hi' + hi lo' + lo hi' keeps about 21 bits of a product; sums are fp32.
//
// A and B are products of k e^{L - L_ref} and k e^{L_ref - L} with a reference inside each block of 16 tokens; the blocks'
// exponents may then be positive, which is safe up to e^60.  A chunk with decays beyond that takes its exponentials pair by
// pair on the CUDA cores.  log g is clamped at -40 per token (g below 1e-17).
//
// Fragments of m16n8k8 (lane = 4 g + t): A rows g, g + 8, B column g, C rows g, g + 8 and columns 2t, 2t + 1.  The order of the
// contraction index is free as long as A and B agree: with its places t, t + 4 standing for 2t, 2t + 1, a lane's two B values
// are neighbours in memory, and a C fragment is the A fragment of the next product as it is (c0, c2, c1, c3).
#include "delta.cuh"
#include "tf32.cuh"

namespace {

constexpr int kC = 32;            // tokens of a chunk
constexpr float kMinLog = -40.f;
constexpr float kSafe = 60.f;
constexpr int kAL = kC + 4;       // row stride of beta A in shared memory
constexpr int kTL = kC + 8;       // row stride of arrays read as B fragments (8 mod 32: conflict-free 8-byte reads)

__device__ __forceinline__ float2 ld_f2(const float* p) { return *reinterpret_cast<const float2*>(p); }

// ------------------------------------------------------------------ everything that depends on a chunk alone
struct PrepArgs {
  const float* q;         // [rows][kv_heads * d]
  const float* k;
  const float* rate;      // [rows][heads * d]
  const float* dt_bias;
  const float* a_log;
  int ld, at_b;           // p: step sizes' logits
  const int* chunks;      // [chunks][2]: first row, tokens
  float* w;               // [chunks][heads][kC][d]   W
  float* qd;              // [chunks][heads][kC][d]   q e^L
  float* kr;              // [chunks][heads][d][kC]   k e^{L_31 - L}
  float* u0;              // [chunks][heads][kC][e]
  float* b;               // [chunks][heads][kC][kC]  zero above the diagonal
  float* decay;           // [chunks][heads][d]       e^{L_31}
  int heads, group, d, e;
};

template <int DP>
struct PrepCfg {
  static constexpr int THREADS = 128;
  static constexpr int LD = DP + 8;
  static constexpr int SMEM = (3 * kC * LD + kC * kAL + kC * kTL + kC + 3 * DP) * 4;
};

template <typename T, int DP>
__global__ void __launch_bounds__(128, 3) delta_chunk_prep_kernel(const T* __restrict__ p, const T* __restrict__ v,
                                                                  const PrepArgs a) {
  pdl_entry();
  constexpr int LD = PrepCfg<DP>::LD, NT = PrepCfg<DP>::THREADS;
  extern __shared__ __align__(16) float sm[];
  float* ls = sm;                  // [kC][LD] inclusive log decays, later k e^{L_ref - L}
  float* qs = ls + kC * LD;        // [kC][LD] q, later q e^{L - L_ref}
  float* ks = qs + kC * LD;        // [kC][LD] k, later k e^{L - L_ref}
  float* am = ks + kC * LD;        // [kC][kAL] beta_t A_ts, zero from the diagonal on
  float* bm = am + kC * kAL;       // [kC][kTL] B_ts, zero above the diagonal
  float* beta = bm + kC * kTL;     // [kC]
  float* ref = beta + kC;          // [2][DP] L of the blocks' references
  float* gap = ref + 2 * DP;       // [DP] e^{L_ref1 - L_ref0}
  const int c = blockIdx.x, head = blockIdx.y, d = a.d, e = a.e, tid = threadIdx.x;
  const int t0 = a.chunks[c * 2], m = a.chunks[c * 2 + 1], kvh = head / a.group, nqk = a.heads / a.group * d;
  const float ea = expf(a.a_log[head]);
  const size_t ch = (size_t)c * a.heads + head;

#pragma unroll 4
  for (int i = tid; i < kC * DP / 4; i += NT) {     // tokens past the last one: k = q = 0, no decay
    const int t = i / (DP / 4), x = i % (DP / 4) * 4;
    const bool in = t < m && x < d;
    const float4 z = make_float4(0.f, 0.f, 0.f, 0.f);
    const size_t row = t0 + t;
    st_f4(qs + t * LD + x, in ? ld_f4(a.q + row * nqk + kvh * d + x) : z);
    st_f4(ks + t * LD + x, in ? ld_f4(a.k + row * nqk + kvh * d + x) : z);
    float4 g = z;
    if (in) {
      const float4 r = ld_f4(a.rate + row * a.heads * d + head * d + x), dt = ld_f4(a.dt_bias + head * d + x);
      auto decay = [&](float x, float y) {
        return fmaxf(sizeof(T) == 2 ? log_decay_fast(x, y, ea) : log_decay(x, y, ea), kMinLog);
      };
      g = make_float4(decay(r.x, dt.x), decay(r.y, dt.y), decay(r.z, dt.z), decay(r.w, dt.w));
    }
    st_f4(ls + t * LD + x, g);
  }
  if (tid < kC) beta[tid] = tid < m ? sigmoid_f(ld_f(p + (size_t)(t0 + tid) * a.ld + a.at_b + head)) : 0.f;
  for (int i = tid; i < kC * kAL; i += NT) am[i] = 0.f;
  for (int i = tid; i < kC * kTL; i += NT) bm[i] = 0.f;
  __syncthreads();
  bool wild = false;
  if (tid < DP) {
    float l[kC];
#pragma unroll
    for (int t = 0; t < kC; ++t) l[t] = ls[t * LD + tid];
#pragma unroll
    for (int t = 1; t < kC; ++t) l[t] += l[t - 1];
#pragma unroll
    for (int t = 0; t < kC; ++t) ls[t * LD + tid] = l[t];
    ref[tid] = l[7], ref[DP + tid] = l[23];
    gap[tid] = __expf(l[23] - l[7]);
    wild = fmaxf(fmaxf(l[0] - l[7], l[7] - l[15]), fmaxf(l[16] - l[23], l[23] - l[31])) > kSafe;
    if (tid < d) {
      a.decay[ch * d + tid] = expf(l[kC - 1]);
      float* kr = a.kr + (ch * d + tid) * kC;
#pragma unroll
      for (int t = 0; t < kC; t += 4)
        st_f4(kr + t, make_float4(ks[t * LD + tid] * __expf(l[kC - 1] - l[t]), ks[(t + 1) * LD + tid] * __expf(l[kC - 1] - l[t + 1]),
                                  ks[(t + 2) * LD + tid] * __expf(l[kC - 1] - l[t + 2]),
                                  ks[(t + 3) * LD + tid] * __expf(l[kC - 1] - l[t + 3])));
    }
  }
  wild = __syncthreads_or(wild);
  const int warp = tid >> 5, g = (tid & 31) >> 2, tt = tid & 3;
  if (!wild) {
#pragma unroll 2
    for (int i = tid; i < kC * DP / 4; i += NT) {
      const int t = i / (DP / 4), x = i % (DP / 4) * 4;
      const float4 q = ld_f4(qs + t * LD + x), k = ld_f4(ks + t * LD + x), l = ld_f4(ls + t * LD + x);
      const float4 r = ld_f4(ref + t / 16 * DP + x);
      if (x < d)
        st_f4(a.qd + (ch * kC + t) * d + x,
              make_float4(q.x * __expf(l.x), q.y * __expf(l.y), q.z * __expf(l.z), q.w * __expf(l.w)));
      const float4 f = make_float4(__expf(l.x - r.x), __expf(l.y - r.y), __expf(l.z - r.z), __expf(l.w - r.w));
      const float4 h = make_float4(__expf(r.x - l.x), __expf(r.y - l.y), __expf(r.z - l.z), __expf(r.w - l.w));
      st_f4(qs + t * LD + x, make_float4(q.x * f.x, q.y * f.y, q.z * f.z, q.w * f.w));
      st_f4(ks + t * LD + x, make_float4(k.x * f.x, k.y * f.y, k.z * f.z, k.w * f.w));
      st_f4(ls + t * LD + x, make_float4(k.x * h.x, k.y * h.y, k.z * h.z, k.w * h.w));
    }
    __syncthreads();
    // warps 0, 1: A, warps 2, 3: B.  The first of two takes tokens 16.. against sources 0..15 (across the references) and 0..15
    // against 0..7, the second tokens 16.. against 16.. and 0..15 against 8..15.
    const float* left = warp < 2 ? ks : qs;
    const int odd = warp & 1;
    float acc[3][4] = {};
#pragma unroll 2
    for (int x = 2 * tt; x < DP; x += 8) {
      const float2 lo0 = ld_f2(left + g * LD + x), lo1 = ld_f2(left + (g + 8) * LD + x);
      const float2 hi0 = ld_f2(left + (g + 16) * LD + x), hi1 = ld_f2(left + (g + 24) * LD + x);
      float2 s0 = ld_f2(ls + (odd * 16 + g) * LD + x), s1 = ld_f2(ls + (odd * 16 + 8 + g) * LD + x);
      const float2 s2 = ld_f2(ls + (odd * 8 + g) * LD + x);
      if (!odd) {
        const float2 f = ld_f2(gap + x);
        s0.x *= f.x, s0.y *= f.y, s1.x *= f.x, s1.y *= f.y;
      }
      const FragA fh = frag_a(hi0.x, hi1.x, hi0.y, hi1.y), fl = frag_a(lo0.x, lo1.x, lo0.y, lo1.y);
      mma3(acc[0], fh, s0);
      mma3(acc[1], fh, s1);
      mma3(acc[2], fl, s2);
    }
#pragma unroll
    for (int j = 0; j < 3; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int t = (j < 2 ? 16 : 0) + g + (i >> 1) * 8, s = (j < 2 ? odd * 16 + j * 8 : odd * 8) + 2 * tt + (i & 1);
        if (warp < 2) {
          if (s < t) am[t * kAL + s] = beta[t] * acc[j][i];
        } else if (s <= t) {
          bm[t * kTL + s] = acc[j][i];
        }
      }
  } else {
    for (int i = tid; i < kC * DP; i += NT) {
      const int t = i / DP, x = i % DP;
      if (x < d) a.qd[(ch * kC + t) * d + x] = qs[t * LD + x] * __expf(ls[t * LD + x]);
    }
    for (int i = tid; i < kC * (kC + 1) / 2; i += NT) {
      int t = (int)((sqrtf(8.f * i + 1.f) - 1.f) * 0.5f);        // i = t (t + 1) / 2 + s, s <= t
      while (t * (t + 1) / 2 > i) --t;
      while ((t + 1) * (t + 2) / 2 <= i) ++t;
      const int s = i - t * (t + 1) / 2;
      float aa = 0.f, bb = 0.f;
      for (int x = 0; x < d; ++x) {
        const float ke = ks[s * LD + x] * __expf(ls[t * LD + x] - ls[s * LD + x]);
        aa = fmaf(ks[t * LD + x], ke, aa), bb = fmaf(qs[t * LD + x], ke, bb);
      }
      if (s < t) am[t * kAL + s] = beta[t] * aa;
      bm[t * kTL + s] = bb;
    }
  }
  __syncthreads();
  for (int i = tid; i < kC * kC / 4; i += NT) {
    const int t = i / (kC / 4), s = i % (kC / 4) * 4;
    st_f4(a.b + (ch * kC + t) * kC + s, ld_f4(bm + t * kTL + s));
  }
  // the triangular system: right sides beta k e^L (d columns) and beta v (e columns), two columns per thread
  for (int col = 2 * tid; col < d + e; col += 2 * NT) {
    float x[kC], y[kC];
    if (col < d) {
      float2 f[2];
#pragma unroll
      for (int h = 0; h < 2; ++h)
        f[h] = wild ? make_float2(0.f, 0.f) : make_float2(expf(ref[h * DP + col]), expf(ref[h * DP + col + 1]));
#pragma unroll
      for (int t = 0; t < kC; ++t) {
        const float2 k = ld_f2(ks + t * LD + col);
        const float2 z = wild ? make_float2(__expf(ls[t * LD + col]), __expf(ls[t * LD + col + 1])) : f[t / 16];
        x[t] = beta[t] * k.x * z.x, y[t] = beta[t] * k.y * z.y;
      }
    } else {
      const T* vp = v + (size_t)t0 * a.heads * e + head * e + (col - d);
#pragma unroll
      for (int t = 0; t < kC; ++t) {
        x[t] = t < m ? ld_f(vp + (size_t)t * a.heads * e) : 0.f;
        y[t] = t < m ? ld_f(vp + (size_t)t * a.heads * e + 1) : 0.f;
      }
#pragma unroll
      for (int t = 0; t < kC; ++t) x[t] *= beta[t], y[t] *= beta[t];
    }
#pragma unroll
    for (int t = 1; t < kC; ++t) {
#pragma unroll
      for (int s = 0; s < t; s += 4) {
        const float4 f4 = ld_f4(am + t * kAL + s);     // zero from s = t on
        const float f[4] = {f4.x, f4.y, f4.z, f4.w};
#pragma unroll
        for (int h = 0; h < 4; ++h)
          if (s + h < t) x[t] = fmaf(-f[h], x[s + h], x[t]), y[t] = fmaf(-f[h], y[s + h], y[t]);
      }
    }
    float* dst = col < d ? a.w + ch * kC * d + col : a.u0 + ch * kC * e + col - d;
    const int step = col < d ? d : e;
#pragma unroll
    for (int t = 0; t < kC; ++t) *reinterpret_cast<float2*>(dst + (size_t)t * step) = make_float2(x[t], y[t]);
  }
}

// ------------------------------------------------------------------ the walk over the chunks
struct WalkArgs {
  const float *w, *qd, *kr, *u0, *b, *decay;
  float* state;           // [slots + 1][heads][d][e]
  float* raw;             // [rows][heads * e]
  const int* chunks;
  const int* segs;        // [n][4]: slot, first chunk, chunks, first row
  const int* seg_rows;    // [n + 1]
  const int* pos;
  int heads, d, e;
  ConvCols cols;
};

constexpr int kVB = 16;     // value columns per CTA: the rows of the products' tiles

template <int DP>
struct WalkCfg {
  static constexpr int LD = DP + 8;
  static constexpr int NW = DP == 128 ? 8 : 4;                    // warps
  static constexpr int KN = DP / 8 / NW;                          // groups of 8 keys per warp
  static constexpr int SMALL = kC * kTL + kC * kVB + DP;          // B, U0, decay: double buffered
  static constexpr int SMEM = (2 * kC * LD + DP * kTL + 2 * SMALL + NW * 8 * 128 + 4 * 128) * 4;
};

__device__ __forceinline__ void cp16(void* smem, const void* g) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(smem)), "l"(g) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void cp_wait_but_one() { asm volatile("cp.async.wait_group 1;" ::: "memory"); }

// One CTA per (request, head, 16 value columns), four or eight warps that share the keys.  All products are transposed: the
// 16 columns are the rows of every tile, so the state S^T of a warp's keys stays in registers as C fragments and enters the
// products W S and (q e^L) S as A fragments.  Their sums over the warps go through shared memory.  W and q e^L of the next
// chunk are fetched while this chunk's state is updated, and the other way round; a warp fetches its own keys.
template <typename T, int DP>
__global__ void __launch_bounds__(WalkCfg<DP>::NW * 32) delta_chunk_walk_kernel(const T* __restrict__ p, T* before, const WalkArgs a) {
  pdl_entry();
  using C = WalkCfg<DP>;
  constexpr int LD = C::LD, KN = C::KN, KW = KN * 8, NW = C::NW, NT = NW * 32;     // KW: keys per warp
  extern __shared__ __align__(16) float sm[];
  float* ws = sm;                        // [kC][LD] W
  float* qs = ws + kC * LD;              // [kC][LD] q e^L
  float* ks = qs + kC * LD;              // [DP][kTL] k e^{L_31 - L}, key major
  float* small = ks + DP * kTL;          // [2]: B [kC][kTL], U0 [kC][kVB], decay [DP]
  float4* red = reinterpret_cast<float4*>(small + 2 * C::SMALL);   // [warps][8][32 lanes] partial C fragments
  float4* us = red + NW * 8 * 32;        // [4][32 lanes] u as A fragments
  const int seg = blockIdx.x, head = blockIdx.y, v0 = blockIdx.z * kVB, tid = threadIdx.x, d = a.d, e = a.e;
  const int warp = tid >> 5, lane = tid & 31, g = lane >> 2, tt = lane & 3;
  const int slot = a.segs[seg * 4], c0 = a.segs[seg * 4 + 1], n = a.segs[seg * 4 + 2], row0 = a.segs[seg * 4 + 3];
  const bool fresh = a.pos[row0] == 0;
  float* sg = a.state + ((size_t)slot * a.heads + head) * d * e;
  const int key0 = warp * KW;

  auto fetch_wq = [&](int c) {
    if (c < n) {
      constexpr int Q = KW / 4, R = 32 / Q;        // 16-byte pieces per row of this warp, rows per pass
      const int t = lane / Q, x = key0 + lane % Q * 4;
      if (x < d) {
        const size_t src = (((size_t)(c0 + c) * a.heads + head) * kC + t) * d + x;
        const float *gw = a.w + src, *gq = a.qd + src;
        float *dw = ws + t * LD + x, *dq = qs + t * LD + x;
#pragma unroll
        for (int i = 0; i < kC / R; ++i, gw += R * d, gq += R * d) cp16(dw + i * R * LD, gw), cp16(dq + i * R * LD, gq);
      }
    }
    cp_commit();
  };
  auto fetch_rest = [&](int c) {
    if (c < n) {
      const size_t ch = (size_t)(c0 + c) * a.heads + head;
      const float* gk = a.kr + (ch * d + key0 + lane / 8) * kC + lane % 8 * 4;
      float* dk = ks + (key0 + lane / 8) * kTL + lane % 8 * 4;
#pragma unroll
      for (int i = 0; i < KW; i += 4)
        if (key0 + lane / 8 + i < d) cp16(dk + i * kTL, gk + i * kC);
      float* s = small + (c & 1) * C::SMALL;
#pragma unroll
      for (int i = 0; i < kC * kC / 4; i += NT)
        cp16(s + (tid + i) / 8 * kTL + tid % 8 * 4, a.b + ch * kC * kC + (tid + i) * 4);
      s += kC * kTL;
      if (tid < kC * kVB / 4) {
        const int t = tid / (kVB / 4), x = tid % (kVB / 4) * 4;
        if (v0 + x < e) cp16(s + t * kVB + x, a.u0 + (ch * kC + t) * e + v0 + x);
      }
      s += kC * kVB;
      if (tid < d / 4) cp16(s + tid * 4, a.decay + ch * d + tid * 4);
    }
    cp_commit();
  };
  // zero what the copies never fill: keys past d, columns past e
  for (int i = tid; i < 2 * kC * LD + DP * kTL + 2 * C::SMALL; i += NT) sm[i] = 0.f;
  __syncthreads();
  fetch_wq(0);
  fetch_rest(0);
  float st[KN][4];
#pragma unroll
  for (int k = 0; k < KN; ++k)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int key = key0 + k * 8 + 2 * tt + (i & 1), x = v0 + g + (i >> 1) * 8;
      st[k][i] = (!fresh && key < d && x < e) ? sg[(size_t)key * e + x] : 0.f;
    }

  for (int c = 0; c < n; ++c) {
    const float* bs = small + (c & 1) * C::SMALL;
    const float *u0 = bs + kC * kTL, *dec = u0 + kC * kVB;
    cp_wait_but_one();
    __syncwarp();
    float acc[8][4] = {};          // S^T (W^T | (q e^L)^T) over this warp's keys: 8 tokens each
#pragma unroll
    for (int k = 0; k < KN; ++k) {
      const FragA f = frag_a(st[k][0], st[k][2], st[k][1], st[k][3]);
#pragma unroll
      for (int j = 0; j < 8; ++j)
        mma3(acc[j], f, ld_f2((j < 4 ? ws : qs) + ((j & 3) * 8 + g) * LD + key0 + k * 8 + 2 * tt));
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) red[(warp * 8 + j) * 32 + lane] = make_float4(acc[j][0], acc[j][1], acc[j][2], acc[j][3]);
    __syncwarp();
    fetch_wq(c + 1);
    cp_wait_but_one();
    __syncthreads();
    // sums over the warps, eight tokens each: u = U0 - W S to everyone, (q e^L) S stays with the warp that makes the output
    const int tile = warp & 3;
    const bool makes_u = NW == 4 || warp < 4, makes_o = NW == 4 || warp >= 4;
    auto total = [&](int j) {
      float4 x = red[j * 32 + lane];
#pragma unroll
      for (int w = 1; w < NW; ++w) {
        const float4 y = red[(w * 8 + j) * 32 + lane];
        x.x += y.x, x.y += y.y, x.z += y.z, x.w += y.w;
      }
      return x;
    };
    float o[4] = {};
    if (makes_u) {
      const float4 x = total(tile);
      const float* up = u0 + (tile * 8 + 2 * tt) * kVB + g;
      us[tile * 32 + lane] = make_float4(up[0] - x.x, up[8] - x.z, up[kVB] - x.y, up[kVB + 8] - x.w);
    }
    if (makes_o) {
      const float4 y = total(4 + tile);
      o[0] = y.x, o[1] = y.y, o[2] = y.z, o[3] = y.w;
    }
    __syncthreads();
    FragA uf[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float4 u = us[j * 32 + lane];
      uf[j] = frag_a(u.x, u.y, u.z, u.w);
    }
#pragma unroll
    for (int k = 0; k < KN; ++k) {
      const float2 f = ld_f2(dec + key0 + k * 8 + 2 * tt);
      st[k][0] *= f.x, st[k][1] *= f.y, st[k][2] *= f.x, st[k][3] *= f.y;
#pragma unroll
      for (int j = 0; j < 4; ++j) mma3(st[k], uf[j], ld_f2(ks + (key0 + k * 8 + g) * kTL + j * 8 + 2 * tt));
    }
    if (makes_o) {
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (j <= tile) mma3(o, uf[j], ld_f2(bs + (tile * 8 + g) * kTL + j * 8 + 2 * tt));
    }
    __syncwarp();
    fetch_rest(c + 1);
    if (makes_o) {
      const int m = a.chunks[(c0 + c) * 2 + 1], t = tile * 8 + 2 * tt, x = v0 + g;
      float* out = a.raw + ((size_t)(a.chunks[(c0 + c) * 2] + t) * a.heads + head) * e + x;
      const int next = a.heads * e;
      if (t < m && x < e) out[0] = o[0];
      if (t + 1 < m && x < e) out[next] = o[1];
      if (t < m && x + 8 < e) out[8] = o[2];
      if (t + 1 < m && x + 8 < e) out[next + 8] = o[3];
    }
  }
#pragma unroll
  for (int k = 0; k < KN; ++k)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int key = key0 + k * 8 + 2 * tt + (i & 1), x = v0 + g + (i >> 1) * 8;
      if (key < d && x < e) sg[(size_t)key * e + x] = st[k][i];
    }
  if (blockIdx.z == 0)
    keep_conv_inputs(p, before + (size_t)slot * (a.cols.taps - 1) * (2 * a.cols.nqk + a.cols.nv), a.cols, row0,
                     a.seg_rows[seg + 1] - a.seg_rows[seg], fresh, head * NT + tid, a.heads * NT);
}

template <typename T, int DP>
int launch_chunks(const void* p, const void* v, void* before, const PrepArgs& a, const WalkArgs& w, int n_chunks, int n_segs,
                  cudaStream_t st) {
  using P = PrepCfg<DP>;
  using W = WalkCfg<DP>;
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(delta_chunk_prep_kernel<T, DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, P::SMEM) !=
            cudaSuccess ||
        cudaFuncSetAttribute(delta_chunk_walk_kernel<T, DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, W::SMEM) !=
            cudaSuccess)
      return 691;
    set = true;
  }
  dsv4_launch(delta_chunk_prep_kernel<T, DP>, dim3(n_chunks, a.heads), P::THREADS, P::SMEM, st, (const T*)p, (const T*)v, a);
  dsv4_launch(delta_chunk_walk_kernel<T, DP>, dim3(n_segs, a.heads, (a.e + kVB - 1) / kVB), W::NW * 32, W::SMEM, st, (const T*)p,
              (T*)before, w);
  return (int)cudaGetLastError();
}
template <typename T>
int dispatch_chunks(const void* p, const void* v, void* before, const PrepArgs& a, const WalkArgs& w, int n_chunks,
                    int n_segs, cudaStream_t st) {
  if (a.d <= 32) return launch_chunks<T, 32>(p, v, before, a, w, n_chunks, n_segs, st);
  if (a.d <= 64) return launch_chunks<T, 64>(p, v, before, a, w, n_chunks, n_segs, st);
  return launch_chunks<T, 128>(p, v, before, a, w, n_chunks, n_segs, st);
}

}  // namespace

// p, q, k, v, rate, ... as in dsv4_delta_scan; d, e multiples of 4, d <= 128.  chunks [n_chunks][2] = first row, tokens (at most
// 32; a request's chunks stand together), segs [n_segs][4] = slot, first chunk, chunks, first row.  Scratch: w, qd
// [n_chunks, heads, 32, d], kr [.., d, 32], u0 [.., 32, e], b [.., 32, 32], decay [.., d].  Leaves the outputs ahead of the norm
// in raw [rows, heads * e]; dsv4_head_norm_gate has to follow.
DSV4_API int dsv4_delta_chunked(const void* p, int ld, int at_k, int at_v, int at_b, int n_taps, const float* q, const float* k,
                                const void* v, const float* rate, const float* dt_bias, const float* a_log, float* state,
                                void* before, float* raw, const int* pos, const int* seg_off, const int* chunks, int n_chunks,
                                const int* segs, int n_segs, float* w, float* kr, float* qd, float* u0, float* b,
                                float* decay, int heads, int kv_heads, int d, int e, int fp32, cudaStream_t st) {
  if (n_chunks <= 0 || n_segs <= 0) return 0;
  if (heads < 1 || heads > 65535 || kv_heads < 1 || heads % kv_heads || d < 1 || d % 4 || e < 1 || e % 4 || d > 128) return 692;
  const PrepArgs a{q, k, rate, dt_bias, a_log, ld, at_b, chunks, w, qd, kr, u0, b, decay, heads, heads / kv_heads, d, e};
  const WalkArgs s{w, qd, kr, u0, b, decay, state, raw, chunks, segs, seg_off, pos, heads, d, e,
                   {ld, at_k, at_v, kv_heads * d, heads * e, n_taps}};
  return fp32 ? dispatch_chunks<float>(p, v, before, a, s, n_chunks, n_segs, st)
              : dispatch_chunks<__nv_bfloat16>(p, v, before, a, s, n_chunks, n_segs, st);
}
