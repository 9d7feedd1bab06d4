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
//   delta_chunk_walk_kernel   every (request, head, block of value columns): the chunks in sequence; columns of S are independent
// and head_norm_gate (delta.cu) behind them.  All of it in fp32 on the CUDA cores (the recurrence is a 32-bit computation).
//
// A and B are products of k e^{L - L_ref} and k e^{L_ref - L} with a reference inside each block of 16 tokens; the blocks'
// exponents may then be positive, which is safe up to e^60.  A block with decays beyond that takes its exponentials pair by
// pair.  log g is clamped at -40 per token (g below 1e-17).
#include "delta.cuh"

namespace {

constexpr int kC = 32;            // tokens of a chunk
constexpr float kMinLog = -40.f;
constexpr float kSafe = 60.f;
constexpr int kAL = kC + 4;       // row stride of A, B

struct PrepArgs {
  const float* q;         // [rows][kv_heads * d]
  const float* k;
  const float* rate;      // [rows][heads * d]
  const float* dt_bias;
  const float* a_log;
  int ld, at_b;           // p: step sizes' logits
  const int* chunks;      // [chunks][2]: first row, tokens
  float* w;               // [chunks][heads][kC][d]   W
  float* kr;              // [chunks][heads][kC][d]   k e^{L_31 - L}
  float* qd;              // [chunks][heads][kC][d]   q e^L
  float* u0;              // [chunks][heads][kC][e]
  float* b;               // [chunks][heads][kC][kC]
  float* decay;           // [chunks][heads][d]       e^{L_31}
  int heads, group, d, e;
};

template <int DP>
constexpr int prep_smem() { return (3 * kC * (DP + 4) + 2 * kC * kAL + kC + 2 * DP) * 4; }

template <typename T, int DP>
__global__ void __launch_bounds__(256, 2) delta_chunk_prep_kernel(const T* __restrict__ p, const T* __restrict__ v,
                                                               const PrepArgs a) {
  pdl_entry();
  constexpr int LD = DP + 4, NT = 256;
  extern __shared__ __align__(16) float sm[];
  float* ls = sm;                  // [kC][LD] inclusive log decays, later k e^{L_ref - L}
  float* qs = ls + kC * LD;        // [kC][LD] q, later q e^{L - L_ref}
  float* ks = qs + kC * LD;        // [kC][LD] k, later k e^{L - L_ref}
  float* am = ks + kC * LD;        // [kC][kAL] beta_t A_ts, zero from the diagonal on
  float* bm = am + kC * kAL;       // [kC][kAL] B_ts, zero above the diagonal
  float* beta = bm + kC * kAL;     // [kC]
  float* ref = beta + kC;          // [2][DP] L of the blocks' references
  const int c = blockIdx.x, head = blockIdx.y, d = a.d, e = a.e, tid = threadIdx.x;
  const int t0 = a.chunks[c * 2], m = a.chunks[c * 2 + 1], kvh = head / a.group, nqk = a.heads / a.group * d;
  const float ea = expf(a.a_log[head]);
  const size_t ch = (size_t)c * a.heads + head;

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
      g.x = fmaxf(log_decay(r.x, dt.x, ea), kMinLog), g.y = fmaxf(log_decay(r.y, dt.y, ea), kMinLog);
      g.z = fmaxf(log_decay(r.z, dt.z, ea), kMinLog), g.w = fmaxf(log_decay(r.w, dt.w, ea), kMinLog);
    }
    st_f4(ls + t * LD + x, g);
  }
  if (tid < kC) beta[tid] = tid < m ? sigmoid_f(ld_f(p + (size_t)(t0 + tid) * a.ld + a.at_b + head)) : 0.f;
  __syncthreads();
  bool wild = false;
  if (tid < DP) {
    float l = 0.f, first = 0.f, mid = 0.f;
#pragma unroll
    for (int t = 0; t < kC; ++t) {
      l += ls[t * LD + tid];
      ls[t * LD + tid] = l;
      if (t % 16 == 0) first = l;
      if (t % 16 == 7) {
        mid = l;
        ref[t / 16 * DP + tid] = l;
        wild |= first - l > kSafe;
      }
      if (t % 16 == 15) wild |= mid - l > kSafe;
    }
    if (tid < d) a.decay[ch * d + tid] = expf(l);
  }
  wild = __syncthreads_or(wild);

  for (int i = tid; i < kC * DP / 4; i += NT) {
    const int t = i / (DP / 4), x = i % (DP / 4) * 4;
    const float4 q = ld_f4(qs + t * LD + x), k = ld_f4(ks + t * LD + x), l = ld_f4(ls + t * LD + x);
    const float4 z = ld_f4(ls + (kC - 1) * LD + x);
    if (x < d) {
      st_f4(a.qd + (ch * kC + t) * d + x, make_float4(q.x * __expf(l.x), q.y * __expf(l.y), q.z * __expf(l.z), q.w * __expf(l.w)));
      st_f4(a.kr + (ch * kC + t) * d + x, make_float4(k.x * __expf(z.x - l.x), k.y * __expf(z.y - l.y),
                                                     k.z * __expf(z.z - l.z), k.w * __expf(z.w - l.w)));
    }
  }
  for (int i = tid; i < 2 * kC * kAL; i += NT) am[i] = 0.f;     // am and bm
  __syncthreads();
  if (!wild) {
    for (int i = tid; i < kC * DP / 4; i += NT) {
      const int t = i / (DP / 4), x = i % (DP / 4) * 4;
      const float4 q = ld_f4(qs + t * LD + x), k = ld_f4(ks + t * LD + x), l = ld_f4(ls + t * LD + x);
      const float4 r = ld_f4(ref + t / 16 * DP + x);
      const float4 f = make_float4(__expf(l.x - r.x), __expf(l.y - r.y), __expf(l.z - r.z), __expf(l.w - r.w));
      const float4 h = make_float4(__expf(r.x - l.x), __expf(r.y - l.y), __expf(r.z - l.z), __expf(r.w - l.w));
      st_f4(qs + t * LD + x, make_float4(q.x * f.x, q.y * f.y, q.z * f.z, q.w * f.w));
      st_f4(ks + t * LD + x, make_float4(k.x * f.x, k.y * f.y, k.z * f.z, k.w * f.w));
      st_f4(ls + t * LD + x, make_float4(k.x * h.x, k.y * h.y, k.z * h.z, k.w * h.w));
    }
    __syncthreads();
    // blocks of 16 x 16: (0, 0), (16, 16), (16, 0); 64 threads each, 2 tokens x 2 sources of A and of B per thread.  Between
    // the blocks the references' distance e^{L_ref1 - L_ref0} comes in between (never above one).
    if (tid < 192) {
      const int blk = tid >> 6, ti = tid >> 3 & 7, si = tid & 7;
      const int tb = (blk > 0 ? 16 : 0) + ti, sb = (blk == 1 ? 16 : 0) + si;
      float aa[2][2] = {}, bb[2][2] = {};
#pragma unroll 2
      for (int x = 0; x < DP; x += 4) {
        const float4 k0 = ld_f4(ks + tb * LD + x), k1 = ld_f4(ks + (tb + 8) * LD + x);
        const float4 q0 = ld_f4(qs + tb * LD + x), q1 = ld_f4(qs + (tb + 8) * LD + x);
        float4 s0 = ld_f4(ls + sb * LD + x), s1 = ld_f4(ls + (sb + 8) * LD + x);
        if (blk == 2) {
          const float4 r0 = ld_f4(ref + x), r1 = ld_f4(ref + DP + x);
          const float4 f = make_float4(__expf(r1.x - r0.x), __expf(r1.y - r0.y), __expf(r1.z - r0.z), __expf(r1.w - r0.w));
          s0 = make_float4(s0.x * f.x, s0.y * f.y, s0.z * f.z, s0.w * f.w);
          s1 = make_float4(s1.x * f.x, s1.y * f.y, s1.z * f.z, s1.w * f.w);
        }
        auto dot = [](float acc, const float4& u, const float4& w) {
          return fmaf(u.x, w.x, fmaf(u.y, w.y, fmaf(u.z, w.z, fmaf(u.w, w.w, acc))));
        };
        aa[0][0] = dot(aa[0][0], k0, s0), aa[0][1] = dot(aa[0][1], k0, s1);
        aa[1][0] = dot(aa[1][0], k1, s0), aa[1][1] = dot(aa[1][1], k1, s1);
        bb[0][0] = dot(bb[0][0], q0, s0), bb[0][1] = dot(bb[0][1], q0, s1);
        bb[1][0] = dot(bb[1][0], q1, s0), bb[1][1] = dot(bb[1][1], q1, s1);
      }
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          const int t = tb + i * 8, s = sb + j * 8;
          if (s < t) am[t * kAL + s] = beta[t] * aa[i][j];
          if (s <= t) bm[t * kAL + s] = bb[i][j];
        }
    }
  } else {
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
      bm[t * kAL + s] = bb;
    }
  }
  __syncthreads();
  for (int i = tid; i < kC * kC / 4; i += NT) {
    const int t = i / (kC / 4), s = i % (kC / 4) * 4;
    st_f4(a.b + (ch * kC + t) * kC + s, ld_f4(bm + t * kAL + s));
  }
  // the triangular system, one column of the right sides per thread
  for (int col = tid; col < d + e; col += NT) {
    float x[kC];
    if (col < d) {
      const float f0 = wild ? 0.f : expf(ref[col]), f1 = wild ? 0.f : expf(ref[DP + col]);
#pragma unroll
      for (int t = 0; t < kC; ++t)
        x[t] = beta[t] * ks[t * LD + col] * (wild ? __expf(ls[t * LD + col]) : t < 16 ? f0 : f1);
    } else {
      const T* vp = v + (size_t)t0 * a.heads * e + head * e + (col - d);
#pragma unroll
      for (int t = 0; t < kC; ++t) x[t] = t < m ? ld_f(vp + (size_t)t * a.heads * e) : 0.f;
#pragma unroll
      for (int t = 0; t < kC; ++t) x[t] *= beta[t];
    }
#pragma unroll
    for (int t = 1; t < kC; ++t) {
#pragma unroll
      for (int s = 0; s < t; s += 4) {
        const float4 f = ld_f4(am + t * kAL + s);     // zero from s = t on
        x[t] = fmaf(-f.x, x[s], x[t]);
        if (s + 1 < t) x[t] = fmaf(-f.y, x[s + 1], x[t]);
        if (s + 2 < t) x[t] = fmaf(-f.z, x[s + 2], x[t]);
        if (s + 3 < t) x[t] = fmaf(-f.w, x[s + 3], x[t]);
      }
    }
    float* dst = col < d ? a.w + ch * kC * d + col : a.u0 + ch * kC * e + col - d;
    const int step = col < d ? d : e;
#pragma unroll
    for (int t = 0; t < kC; ++t) dst[(size_t)t * step] = x[t];
  }
}

// ------------------------------------------------------------------ the walk over the chunks
struct WalkArgs {
  const float *w, *kr, *qd, *u0, *b, *decay;
  float* state;           // [slots + 1][heads][d][e]
  float* raw;             // [rows][heads * e]
  const int* chunks;
  const int* segs;        // [n][4]: slot, first chunk, chunks, first row
  const int* seg_rows;    // [n + 1]
  const int* pos;
  int heads, d, e;
  ConvCols cols;
};

template <int DP, int VB>
struct WalkCfg {
  static constexpr int RT = VB / 16;                         // rows per thread
  static constexpr int THREADS = 256;
  static constexpr int LD = DP + 4, US = kC + 4;
  static constexpr int STAGE = 3 * kC * LD + kC * kAL + kC * VB + DP;   // W, k e^.., q e^L, B, U0, decay
  static constexpr int SMEM = (2 * STAGE + VB * LD + VB * US) * 4;
};

__device__ __forceinline__ void cp16(void* smem, const void* g) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(smem)), "l"(g) : "memory");
}

// One CTA per (request, head, VB value columns); the state of these columns stays in shared memory, transposed.
template <typename T, int DP, int VB>
__global__ void __launch_bounds__(256) delta_chunk_walk_kernel(const T* __restrict__ p, T* before, const WalkArgs a) {
  pdl_entry();
  using C = WalkCfg<DP, VB>;
  constexpr int NT = C::THREADS, LD = C::LD, US = C::US, RT = C::RT, CG = VB / 2;
  extern __shared__ __align__(16) float sm[];
  float* st = sm + 2 * C::STAGE;     // [VB][LD] state, value column major
  float* us = st + VB * LD;          // [VB][US] u, value column major
  const int seg = blockIdx.x, head = blockIdx.y, v0 = blockIdx.z * VB, tid = threadIdx.x, d = a.d, e = a.e;
  const int slot = a.segs[seg * 4], c0 = a.segs[seg * 4 + 1], n = a.segs[seg * 4 + 2], row0 = a.segs[seg * 4 + 3];
  const bool fresh = a.pos[row0] == 0;
  float* sg = a.state + ((size_t)slot * a.heads + head) * d * e;

  auto fetch = [&](int c, int buf) {
    float* s = sm + buf * C::STAGE;
    const size_t ch = (size_t)(c0 + c) * a.heads + head;
    const int d4 = d / 4;
    for (int i = tid; i < kC * d4; i += NT) {
      const int t = i / d4, x = i % d4 * 4;
      const size_t src = (ch * kC + t) * d + x;
      cp16(s + t * LD + x, a.w + src);
      cp16(s + (kC + t) * LD + x, a.qd + src);
      cp16(s + (2 * kC + t) * LD + x, a.kr + src);
    }
    s += 3 * kC * LD;
    for (int i = tid; i < kC * kC / 4; i += NT) {
      const int t = i / (kC / 4), x = i % (kC / 4) * 4;
      cp16(s + t * kAL + x, a.b + (ch * kC + t) * kC + x);
    }
    s += kC * kAL;
    for (int i = tid; i < kC * VB / 4; i += NT) {
      const int t = i / (VB / 4), x = i % (VB / 4) * 4;
      if (v0 + x < e) cp16(s + t * VB + x, a.u0 + (ch * kC + t) * e + v0 + x);
    }
    s += kC * VB;
    for (int i = tid; i < d4; i += NT) cp16(s + i * 4, a.decay + ch * d + i * 4);
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  // zero what the copies never fill: channels past d, columns past e
  for (int i = tid; i < 2 * C::STAGE; i += NT) sm[i] = 0.f;
  __syncthreads();
  fetch(0, 0);
  for (int i = tid; i < DP * VB; i += NT) {
    const int key = i / VB, x = i % VB;
    st[x * LD + key] = (!fresh && key < d && v0 + x < e) ? sg[(size_t)key * e + v0 + x] : 0.f;
  }

  const int rg = tid / CG, cg = tid % CG;                 // rows rg + i * (32 / RT), columns cg and cg + CG
  constexpr int RS = kC / RT;
  constexpr int KG = DP / 4, ITEMS = KG * VB;             // state update: 4 keys x CPT columns per thread
  constexpr int CPT = ITEMS >= NT ? ITEMS / NT : 1;
  for (int c = 0; c < n; ++c) {
    const float* s = sm + (c & 1) * C::STAGE;
    if (c + 1 < n) fetch(c + 1, (c + 1) & 1);
    if (c + 1 < n)
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    else
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    const float *ws = s, *qs = s + kC * LD, *ks = s + 2 * kC * LD, *bs = s + 3 * kC * LD, *u0 = bs + kC * kAL;
    const float* dec = u0 + kC * VB;
    float pw[RT][2] = {}, pq[RT][2] = {};
#pragma unroll 2
    for (int x = 0; x < DP; x += 4) {
      const float4 s0 = ld_f4(st + cg * LD + x), s1 = ld_f4(st + (cg + CG) * LD + x);
#pragma unroll
      for (int i = 0; i < RT; ++i) {
        const float4 w = ld_f4(ws + (rg + i * RS) * LD + x), q = ld_f4(qs + (rg + i * RS) * LD + x);
        pw[i][0] = fmaf(w.x, s0.x, fmaf(w.y, s0.y, fmaf(w.z, s0.z, fmaf(w.w, s0.w, pw[i][0]))));
        pw[i][1] = fmaf(w.x, s1.x, fmaf(w.y, s1.y, fmaf(w.z, s1.z, fmaf(w.w, s1.w, pw[i][1]))));
        pq[i][0] = fmaf(q.x, s0.x, fmaf(q.y, s0.y, fmaf(q.z, s0.z, fmaf(q.w, s0.w, pq[i][0]))));
        pq[i][1] = fmaf(q.x, s1.x, fmaf(q.y, s1.y, fmaf(q.z, s1.z, fmaf(q.w, s1.w, pq[i][1]))));
      }
    }
#pragma unroll
    for (int i = 0; i < RT; ++i) {
      const int t = rg + i * RS;
      us[cg * US + t] = u0[t * VB + cg] - pw[i][0];
      us[(cg + CG) * US + t] = u0[t * VB + cg + CG] - pw[i][1];
    }
    __syncthreads();
#pragma unroll
    for (int x = 0; x < kC; x += 4) {
      const float4 u = ld_f4(us + cg * US + x), w = ld_f4(us + (cg + CG) * US + x);
#pragma unroll
      for (int i = 0; i < RT; ++i) {
        const float4 b = ld_f4(bs + (rg + i * RS) * kAL + x);
        pq[i][0] = fmaf(b.x, u.x, fmaf(b.y, u.y, fmaf(b.z, u.z, fmaf(b.w, u.w, pq[i][0]))));
        pq[i][1] = fmaf(b.x, w.x, fmaf(b.y, w.y, fmaf(b.z, w.z, fmaf(b.w, w.w, pq[i][1]))));
      }
    }
    const int t0 = a.chunks[(c0 + c) * 2], m = a.chunks[(c0 + c) * 2 + 1];
#pragma unroll
    for (int i = 0; i < RT; ++i) {
      const int t = rg + i * RS;
      if (t >= m) continue;
      float* o = a.raw + ((size_t)(t0 + t) * a.heads + head) * e + v0;
      if (v0 + cg < e) o[cg] = pq[i][0];
      if (v0 + cg + CG < e) o[cg + CG] = pq[i][1];
    }
    if (tid < ITEMS / CPT) {
      const int key = tid % KG * 4, x0 = tid / KG * CPT;
      const float4 g = ld_f4(dec + key);
      float4 acc[CPT];
#pragma unroll
      for (int j = 0; j < CPT; ++j) {
        acc[j] = ld_f4(st + (x0 + j) * LD + key);
        acc[j].x *= g.x, acc[j].y *= g.y, acc[j].z *= g.z, acc[j].w *= g.w;
      }
#pragma unroll 2
      for (int t = 0; t < kC; t += 4) {
        float4 kk[4];
#pragma unroll
        for (int h = 0; h < 4; ++h) kk[h] = ld_f4(ks + (t + h) * LD + key);
#pragma unroll
        for (int j = 0; j < CPT; ++j) {
          const float4 u = ld_f4(us + (x0 + j) * US + t);
          const float uu[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
          for (int h = 0; h < 4; ++h) {
            acc[j].x = fmaf(kk[h].x, uu[h], acc[j].x), acc[j].y = fmaf(kk[h].y, uu[h], acc[j].y);
            acc[j].z = fmaf(kk[h].z, uu[h], acc[j].z), acc[j].w = fmaf(kk[h].w, uu[h], acc[j].w);
          }
        }
      }
#pragma unroll
      for (int j = 0; j < CPT; ++j) st_f4(st + (x0 + j) * LD + key, acc[j]);
    }
    __syncthreads();     // the state is complete; the stage may be filled again
  }
  for (int i = tid; i < DP * VB; i += NT) {
    const int key = i / VB, x = i % VB;
    if (key < d && v0 + x < e) sg[(size_t)key * e + v0 + x] = st[x * LD + key];
  }
  if (blockIdx.z == 0)
    keep_conv_inputs(p, before + (size_t)slot * (a.cols.taps - 1) * (2 * a.cols.nqk + a.cols.nv), a.cols, row0,
                     a.seg_rows[seg + 1] - a.seg_rows[seg], fresh, head * NT + tid, a.heads * NT);
}

template <typename T, int DP, int VB>
int launch_walk(const void* p, void* before, const WalkArgs& a, int n_segs, cudaStream_t st) {
  using C = WalkCfg<DP, VB>;
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(delta_chunk_walk_kernel<T, DP, VB>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM) !=
        cudaSuccess)
      return 690;
    set = true;
  }
  dsv4_launch(delta_chunk_walk_kernel<T, DP, VB>, dim3(n_segs, a.heads, (a.e + VB - 1) / VB), C::THREADS, C::SMEM, st,
              (const T*)p, (T*)before, a);
  return (int)cudaGetLastError();
}
template <typename T, int DP>
int launch_chunks(const void* p, const void* v, void* before, const PrepArgs& a, const WalkArgs& w, int n_chunks, int n_segs,
                  int vb, cudaStream_t st) {
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(delta_chunk_prep_kernel<T, DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, prep_smem<DP>()) !=
        cudaSuccess)
      return 691;
    set = true;
  }
  dsv4_launch(delta_chunk_prep_kernel<T, DP>, dim3(n_chunks, a.heads), 256, prep_smem<DP>(), st, (const T*)p, (const T*)v, a);
  return vb == 16 ? launch_walk<T, DP, 16>(p, before, w, n_segs, st) : launch_walk<T, DP, 32>(p, before, w, n_segs, st);
}
template <typename T>
int dispatch_chunks(const void* p, const void* v, void* before, const PrepArgs& a, const WalkArgs& w, int n_chunks,
                    int n_segs, int vb, cudaStream_t st) {
  if (a.d <= 32) return launch_chunks<T, 32>(p, v, before, a, w, n_chunks, n_segs, vb, st);
  if (a.d <= 64) return launch_chunks<T, 64>(p, v, before, a, w, n_chunks, n_segs, vb, st);
  return launch_chunks<T, 128>(p, v, before, a, w, n_chunks, n_segs, vb, st);
}

}  // namespace

// p, q, k, v, rate, ... as in dsv4_delta_scan; d, e multiples of 4, d <= 128.  chunks [n_chunks][2] = first row, tokens (at most
// 32; a request's chunks stand together), segs [n_segs][4] = slot, first chunk, chunks, first row.  Scratch: w, kr, qd
// [n_chunks, heads, 32, d], u0 [.., 32, e], b [.., 32, 32], decay [.., d].  vb: value columns per CTA of the walk (16, 32).
// Leaves the outputs ahead of the norm in raw [rows, heads * e]; dsv4_head_norm_gate has to follow.
DSV4_API int dsv4_delta_chunked(const void* p, int ld, int at_k, int at_v, int at_b, int n_taps, const float* q, const float* k,
                                const void* v, const float* rate, const float* dt_bias, const float* a_log, float* state,
                                void* before, float* raw, const int* pos, const int* seg_off, const int* chunks, int n_chunks,
                                const int* segs, int n_segs, float* w, float* kr, float* qd, float* u0, float* b,
                                float* decay, int heads, int kv_heads, int d, int e, int vb, int fp32, cudaStream_t st) {
  if (n_chunks <= 0 || n_segs <= 0) return 0;
  if (heads < 1 || heads > 65535 || kv_heads < 1 || heads % kv_heads || d < 1 || d % 4 || e < 1 || e % 4 || d > 128) return 692;
  if (vb != 16 && vb != 32) return 693;
  const PrepArgs a{q, k, rate, dt_bias, a_log, ld, at_b, chunks, w, kr, qd, u0, b, decay, heads, heads / kv_heads, d, e};
  const WalkArgs s{w, kr, qd, u0, b, decay, state, raw, chunks, segs, seg_off, pos, heads, d, e,
                   {ld, at_k, at_v, kv_heads * d, heads * e, n_taps}};
  return fp32 ? dispatch_chunks<float>(p, v, before, a, s, n_chunks, n_segs, vb, st)
              : dispatch_chunks<__nv_bfloat16>(p, v, before, a, s, n_chunks, n_segs, vb, st);
}
