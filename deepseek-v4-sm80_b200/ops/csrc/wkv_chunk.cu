// The recurrence of wkv.cu for long prompt portions, in chunks of 32 tokens.  With L_t = sum_{j <= t} log w_j inside a
// chunk (per key channel, L_{-1} = 0) and S the state before it,
//
//   o_t    = (r_t e^{L_{t-1}})^T S + sum_{s < t} A_ts v_s + (r_t . u k_t) v_t,     A_ts = r_t . (k_s e^{L_{t-1} - L_s})
//   S_next = diag(e^{L_31}) S + sum_s (k_s e^{L_31 - L_s}) v_s^T
//
// so that only the carry S -> S_next runs in sequence:
//   wkv_chunk_state_kernel   every (chunk, head): its own contribution U = sum_s (k_s e^{L_31 - L_s}) v_s^T and e^{L_31}
//   wkv_chunk_carry_kernel   per state element: walks a request's chunks, leaves the state before each chunk in U's place
//   wkv_chunk_out_kernel     every (chunk, head): the outputs, with head norm and gate
// All of it in fp32 on the CUDA cores (the recurrence is a 32-bit computation).  Every exponent is a difference that is
// never positive: A is split at token 16, its off-diagonal block goes through L_15, the two diagonal blocks take their
// exponentials pair by pair.  log w is clamped at -60 (w below 1e-26).
#include "vec.cuh"

namespace {

constexpr int kC = 32;          // tokens of a chunk
constexpr float kMinLog = -60.f;

struct ChunkArgs {
  int ld;               // row stride of p: 4 heads d, columns r | k | v | g
  const float* a;       // [rows, heads d] decay logits
  const float* w0;      // [heads d]
  const float* u;
  const float* gain;
  const int* chunks;    // [chunks][2]: first row, tokens
  float* us;            // [chunks][heads][d][d] contributions, then states
  float* decay;         // [chunks][heads][d]
  int heads, d;
  float eps;
};

// Threads are laid out as 8 row groups x DP / 4 groups of four value columns.
template <int DP>
struct ChunkCfg {
  static constexpr int CG = DP / 4, THREADS = 8 * CG;
  static constexpr int LD = DP + 4;                    // row stride of the [token][channel] arrays
  static constexpr int SMEM_STATE = (2 * kC * LD + kC * DP) * 4;
  // the state moves into the space of log decays, r and k once A is complete, where it fits
  static constexpr bool ALIAS = DP * DP <= 3 * kC * LD;
  static constexpr int SMEM_OUT = (3 * kC * LD + kC * DP + (ALIAS ? 0 : DP * DP) + kC * (kC + 4) + DP * (kC + 4)) * 4;
};

// Inclusive running sums of log w over the chunk's tokens, one channel per thread (channels past d stay zero).
template <int DP>
__device__ __forceinline__ void log_decays(const ChunkArgs& a, int t0, int m, int head, float* ls) {
  constexpr int LD = ChunkCfg<DP>::LD;
  const int hd = a.heads * a.d;
  if ((int)threadIdx.x < DP) {
    const int e = threadIdx.x;
    const bool in = e < a.d;
    const float w0 = in ? a.w0[head * a.d + e] : 0.f;
    const float* ap = a.a + (size_t)t0 * hd + head * a.d + e;
    float v[kC];
#pragma unroll
    for (int t = 0; t < kC; ++t) v[t] = (in && t < m) ? ap[(size_t)t * hd] : 0.f;
    float l = 0.f;
#pragma unroll
    for (int t = 0; t < kC; ++t) {
      if (in && t < m) l += fmaxf(-expf(v[t] + w0), kMinLog);
      ls[t * LD + e] = l;
    }
  }
}
// Columns [q * heads d + head d, +d) of the chunk's rows as fp32 [kC][ld], zeros past d and past the last token.
template <typename T, int DP>
__device__ __forceinline__ void load_rows(const T* p, const ChunkArgs& a, int t0, int m, int head, int q, float* dst,
                                          int ld) {
  constexpr int N = kC * DP / 4 / ChunkCfg<DP>::THREADS;   // 4
  const T* src = p + (size_t)t0 * a.ld + (size_t)q * a.heads * a.d + head * a.d;
  if (a.d % 4 == 0) {
    float4 v[N];
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int i = threadIdx.x + n * ChunkCfg<DP>::THREADS, t = i / (DP / 4), e = i % (DP / 4) * 4;
      v[n] = (t < m && e < a.d) ? ld_f4(src + (size_t)t * a.ld + e) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int i = threadIdx.x + n * ChunkCfg<DP>::THREADS, t = i / (DP / 4), e = i % (DP / 4) * 4;
      *reinterpret_cast<float4*>(dst + t * ld + e) = v[n];
    }
  } else {
    for (int i = threadIdx.x; i < kC * DP; i += ChunkCfg<DP>::THREADS) {
      const int t = i / DP, e = i % DP;
      dst[t * ld + e] = (t < m && e < a.d) ? ld_f(src + (size_t)t * a.ld + e) : 0.f;
    }
  }
}

template <typename T, int DP>
__global__ void __launch_bounds__(ChunkCfg<DP>::THREADS) wkv_chunk_state_kernel(const T* __restrict__ p,
                                                                                const ChunkArgs a) {
  pdl_entry();
  using C = ChunkCfg<DP>;
  constexpr int LD = C::LD, KR = DP / 8;     // keys per thread
  extern __shared__ __align__(16) float cs[];
  float *ls = cs, *ks = ls + kC * LD, *vs = ks + kC * LD;
  const int c = blockIdx.x, head = blockIdx.y, d = a.d, tid = threadIdx.x;
  const int t0 = a.chunks[c * 2], m = a.chunks[c * 2 + 1];
  load_rows<T, DP>(p, a, t0, m, head, 1, ks, LD);
  load_rows<T, DP>(p, a, t0, m, head, 2, vs, DP);
  log_decays<DP>(a, t0, m, head, ls);
  __syncthreads();
  for (int i = tid; i < kC * DP; i += C::THREADS) {
    const int t = i / DP, e = i % DP;
    ks[t * LD + e] *= __expf(ls[(kC - 1) * LD + e] - ls[t * LD + e]);
  }
  __syncthreads();
  const int rg = tid / C::CG, cg = tid % C::CG;
  float acc[KR][4] = {};
#pragma unroll 4
  for (int t = 0; t < kC; ++t) {
    const float4 v = *reinterpret_cast<const float4*>(vs + t * DP + cg * 4);
#pragma unroll
    for (int i = 0; i < KR; i += 4) {
      const float4 k = *reinterpret_cast<const float4*>(ks + t * LD + rg * KR + i);
      const float kk[4] = {k.x, k.y, k.z, k.w};
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        acc[i + j][0] = fmaf(kk[j], v.x, acc[i + j][0]), acc[i + j][1] = fmaf(kk[j], v.y, acc[i + j][1]);
        acc[i + j][2] = fmaf(kk[j], v.z, acc[i + j][2]), acc[i + j][3] = fmaf(kk[j], v.w, acc[i + j][3]);
      }
    }
  }
  float* u = a.us + ((size_t)c * a.heads + head) * d * d;
#pragma unroll
  for (int i = 0; i < KR; ++i) {
    const int k = rg * KR + i;
    if (k >= d) break;
    if (d % 4 == 0) {
      if (cg * 4 < d) *reinterpret_cast<float4*>(u + (size_t)k * d + cg * 4) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
    } else {
      for (int j = 0; j < 4; ++j)
        if (cg * 4 + j < d) u[(size_t)k * d + cg * 4 + j] = acc[i][j];
    }
  }
  if (tid < d) a.decay[((size_t)c * a.heads + head) * d + tid] = expf(ls[(kC - 1) * LD + tid]);
}

// One thread per W consecutive state elements of one key (W = 4 when d allows).  segs: [n][4] = slot, first chunk, chunks,
// first row.
template <int W>
__global__ void __launch_bounds__(128) wkv_chunk_carry_kernel(float* __restrict__ us, const float* __restrict__ decay,
                                                              float* __restrict__ state, float* __restrict__ prev,
                                                              const float* __restrict__ tail, int width,
                                                              const int* __restrict__ segs, const int* __restrict__ pos,
                                                              const int* __restrict__ seg_rows, int heads, int d) {
  pdl_entry();
  const int seg = blockIdx.x, head = blockIdx.y, e = (blockIdx.z * 128 + threadIdx.x) * W;
  const int slot = segs[seg * 4], c0 = segs[seg * 4 + 1], n = segs[seg * 4 + 2], row = segs[seg * 4 + 3];
  const size_t dd = (size_t)d * d, step = (size_t)heads * dd, pstep = (size_t)heads * d;
  if (e < d * d) {
    float* st = state + ((size_t)slot * heads + head) * dd + e;
    float s[W] = {};
    if (pos[row] != 0) ld_w<W>(st, s);
    float* u = us + ((size_t)c0 * heads + head) * dd + e;
    const float* w = decay + ((size_t)c0 * heads + head) * d + e / d;
    constexpr int B = 8;
    for (int c = 0; c < n; c += B) {
      float uv[B][W], wv[B];
#pragma unroll
      for (int j = 0; j < B; ++j)
        if (c + j < n) ld_w<W>(u + (c + j) * step, uv[j]), wv[j] = w[(c + j) * pstep];
#pragma unroll
      for (int j = 0; j < B; ++j)
        if (c + j < n) {
          st_w<W>(u + (c + j) * step, s);
#pragma unroll
          for (int q = 0; q < W; ++q) s[q] = fmaf(wv[j], s[q], uv[j][q]);
        }
    }
    st_w<W>(st, s);
  }
  if (seg_rows[seg + 1] - seg_rows[seg] > 1 && blockIdx.z == 0) {  // the token shift's last row (wkv.cu: shift_mix_kernel)
    const int per = (width + heads - 1) / heads;
    for (int i = head * per + threadIdx.x; i < min((head + 1) * per, width); i += 128)
      prev[(size_t)slot * width + i] = tail[(size_t)slot * width + i];
  }
}

template <typename T, int DP>
__global__ void __launch_bounds__(ChunkCfg<DP>::THREADS) wkv_chunk_out_kernel(const T* __restrict__ p,
                                                                              T* __restrict__ y, const ChunkArgs a) {
  pdl_entry();
  using C = ChunkCfg<DP>;
  constexpr int LD = C::LD, TL = kC + 4;
  extern __shared__ __align__(16) float os[];
  float* ls = os;                    // [kC][LD] inclusive log decays
  float* rs = ls + kC * LD;          // [kC][LD] r
  float* ks = rs + kC * LD;          // [kC][LD] k
  float* vs = ks + kC * LD;          // [kC][DP]
  float* at = vs + kC * DP;          // [kC (s)][TL (t)] A transposed
  float* rt = at + kC * TL;          // [DP][TL] r e^{L_{t-1}} transposed
  float* ss = C::ALIAS ? ls : rt + DP * TL;  // [DP][DP] state before the chunk
  const int c = blockIdx.x, head = blockIdx.y, d = a.d, tid = threadIdx.x, hd = a.heads * d;
  const int t0 = a.chunks[c * 2], m = a.chunks[c * 2 + 1];
  load_rows<T, DP>(p, a, t0, m, head, 0, rs, LD);
  load_rows<T, DP>(p, a, t0, m, head, 1, ks, LD);
  load_rows<T, DP>(p, a, t0, m, head, 2, vs, DP);
  constexpr int NS = DP * DP / 4 / C::THREADS;
  const float* sg = a.us + ((size_t)c * a.heads + head) * d * d;
  float4 sv[NS];                     // in flight while A is computed
  if (d == DP) {
#pragma unroll
    for (int n = 0; n < NS; ++n) sv[n] = reinterpret_cast<const float4*>(sg)[tid + n * C::THREADS];
  }
  log_decays<DP>(a, t0, m, head, ls);
  for (int i = tid; i < kC * TL; i += C::THREADS) at[i] = 0.f;
  __syncthreads();
  // r e^{L_{t-1}}, key-major
  for (int i = tid; i < kC * DP; i += C::THREADS) {
    const int t = i % kC, e = i / kC;
    rt[e * TL + t] = rs[t * LD + e] * (t > 0 ? __expf(ls[(t - 1) * LD + e]) : 1.f);
  }
  // A inside the two diagonal blocks of 16 tokens, the pair's own exponent per channel; s == t is the bonus
  for (int i = tid; i < 2 * 136; i += C::THREADS) {
    int q = i % 136, t = 0;
    while ((t + 1) * (t + 2) / 2 <= q) ++t;          // q = t (t + 1) / 2 + s, s <= t
    const int s = q - t * (t + 1) / 2, b = i / 136 * 16;
    const float *rp = rs + (b + t) * LD, *kp = ks + (b + s) * LD;
    float acc = 0.f;
    if (s == t) {
      const float* up = a.u + head * d;
      if (d % 4 == 0) {
#pragma unroll 4
        for (int e = 0; e < d; e += 4) {
          const float4 r = *reinterpret_cast<const float4*>(rp + e), k = *reinterpret_cast<const float4*>(kp + e);
          const float4 u = *reinterpret_cast<const float4*>(up + e);
          acc = fmaf(r.x * u.x, k.x, fmaf(r.y * u.y, k.y, fmaf(r.z * u.z, k.z, fmaf(r.w * u.w, k.w, acc))));
        }
      } else {
        for (int e = 0; e < d; ++e) acc = fmaf(rp[e] * up[e], kp[e], acc);
      }
    } else {
      const float *lt = ls + (b + t - 1) * LD, *lp = ls + (b + s) * LD;
#pragma unroll 4
      for (int e = 0; e < DP; e += 4) {
        const float4 r = *reinterpret_cast<const float4*>(rp + e), k = *reinterpret_cast<const float4*>(kp + e);
        const float4 x = *reinterpret_cast<const float4*>(lt + e), z = *reinterpret_cast<const float4*>(lp + e);
        acc = fmaf(r.x * k.x, __expf(x.x - z.x), acc);
        acc = fmaf(r.y * k.y, __expf(x.y - z.y), acc);
        acc = fmaf(r.z * k.z, __expf(x.z - z.z), acc);
        acc = fmaf(r.w * k.w, __expf(x.w - z.w), acc);
      }
    }
    at[(b + s) * TL + b + t] = acc;
  }
  __syncthreads();
  // off-diagonal block through L_15: tokens 16..31 against 0..15.  r and k of those tokens are rescaled in place (rs is not
  // needed any more, rt has its own copy).
  for (int i = tid; i < 16 * DP; i += C::THREADS) {
    const int t = i / DP, e = i % DP;
    const float l15 = ls[15 * LD + e];
    rs[(16 + t) * LD + e] *= __expf(ls[(15 + t) * LD + e] - l15);
    ks[t * LD + e] *= __expf(l15 - ls[t * LD + e]);
  }
  __syncthreads();
  for (int i = tid; i < 256; i += C::THREADS) {
    const int t = i / 16, s = i % 16;
    const float *rp = rs + (16 + t) * LD, *kp = ks + s * LD;
    float acc = 0.f;
#pragma unroll 4
    for (int e = 0; e < DP; e += 4) {
      const float4 r = *reinterpret_cast<const float4*>(rp + e), k = *reinterpret_cast<const float4*>(kp + e);
      acc = fmaf(r.x, k.x, fmaf(r.y, k.y, fmaf(r.z, k.z, fmaf(r.w, k.w, acc))));
    }
    at[s * TL + 16 + t] = acc;
  }
  __syncthreads();
  if (d == DP) {
#pragma unroll
    for (int n = 0; n < NS; ++n) reinterpret_cast<float4*>(ss)[tid + n * C::THREADS] = sv[n];
  } else {
    for (int i = tid; i < DP * DP; i += C::THREADS) {
      const int k = i / DP, e = i % DP;
      ss[i] = (k < d && e < d) ? sg[(size_t)k * d + e] : 0.f;
    }
  }
  __syncthreads();
  // o: four tokens x four value columns per thread
  const int rg = tid / C::CG, cg = tid % C::CG;
  float o[4][4] = {};
  auto rank1 = [&](const float* left, const float* right) {
    const float4 x = *reinterpret_cast<const float4*>(left + rg * 4);
    const float4 v = *reinterpret_cast<const float4*>(right + cg * 4);
    const float xx[4] = {x.x, x.y, x.z, x.w}, vv[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) o[i][j] = fmaf(xx[i], vv[j], o[i][j]);
  };
#pragma unroll 8
  for (int k = 0; k < DP; ++k) rank1(rt + k * TL, ss + k * DP);
#pragma unroll 8
  for (int s = 0; s < kC; ++s) rank1(at + s * TL, vs + s * DP);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int t = rg * 4 + i;
    float q = o[i][0] * o[i][0] + o[i][1] * o[i][1] + o[i][2] * o[i][2] + o[i][3] * o[i][3];
#pragma unroll
    for (int off = C::CG / 2; off > 0; off >>= 1) q += __shfl_xor_sync(0xffffffffu, q, off);
    if (t >= m) continue;
    const float inv = 1.f / sqrtf(q / d + a.eps);
    const T* gp = p + (size_t)(t0 + t) * a.ld + 3 * hd + head * d + cg * 4;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int e = cg * 4 + j;
      if (e >= d) break;
      const float g = ld_f(gp + j);
      o[i][j] *= inv * a.gain[head * d + e] * (g / (1.f + expf(-g)));
    }
    T* dst = y + (size_t)(t0 + t) * hd + head * d + cg * 4;
    if (d % 4 == 0) {
      if (cg * 4 < d) st_f4(dst, make_float4(o[i][0], o[i][1], o[i][2], o[i][3]));
    } else {
      for (int j = 0; j < 4; ++j)
        if (cg * 4 + j < d) st_f(dst + j, o[i][j]);
    }
  }
}

template <typename T, int DP>
int launch_chunks(const void* p, void* y, const ChunkArgs& a, int n_chunks, float* state, float* prev, const float* tail,
                  int width, const int* segs, int n_segs, const int* pos, const int* seg_rows, cudaStream_t st) {
  using C = ChunkCfg<DP>;
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(wkv_chunk_state_kernel<T, DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM_STATE) !=
            cudaSuccess ||
        cudaFuncSetAttribute(wkv_chunk_out_kernel<T, DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM_OUT) !=
            cudaSuccess)
      return 627;
    set = true;
  }
  const dim3 grid(n_chunks, a.heads);
  dsv4_launch(wkv_chunk_state_kernel<T, DP>, grid, C::THREADS, C::SMEM_STATE, st, (const T*)p, a);
  if (a.d % 4 == 0)
    dsv4_launch(wkv_chunk_carry_kernel<4>, dim3(n_segs, a.heads, (a.d * a.d / 4 + 127) / 128), 128, 0, st, a.us, a.decay,
                state, prev, tail, width, segs, pos, seg_rows, a.heads, a.d);
  else
    dsv4_launch(wkv_chunk_carry_kernel<1>, dim3(n_segs, a.heads, (a.d * a.d + 127) / 128), 128, 0, st, a.us, a.decay,
                state, prev, tail, width, segs, pos, seg_rows, a.heads, a.d);
  dsv4_launch(wkv_chunk_out_kernel<T, DP>, grid, C::THREADS, C::SMEM_OUT, st, (const T*)p, (T*)y, a);
  return (int)cudaGetLastError();
}
template <typename T>
int dispatch_chunks(const void* p, void* y, const ChunkArgs& a, int n_chunks, float* state, float* prev,
                    const float* tail, int width, const int* segs, int n_segs, const int* pos, const int* seg_rows,
                    cudaStream_t st) {
  if (a.d <= 32) return launch_chunks<T, 32>(p, y, a, n_chunks, state, prev, tail, width, segs, n_segs, pos, seg_rows, st);
  if (a.d <= 64) return launch_chunks<T, 64>(p, y, a, n_chunks, state, prev, tail, width, segs, n_segs, pos, seg_rows, st);
  if (a.d <= 128) return launch_chunks<T, 128>(p, y, a, n_chunks, state, prev, tail, width, segs, n_segs, pos, seg_rows, st);
  return 625;
}

}  // namespace

// Arguments as in dsv4_wkv_scan; chunks [n_chunks][2] = first row, tokens (at most 32; a request's chunks stand together),
// segs [n_segs][4] = slot, first chunk, chunks, first row; us [n_chunks, heads, d, d] and decay [n_chunks, heads, d] scratch.
DSV4_API int dsv4_wkv_chunked(const void* p, const float* a, const float* w0, const float* u, const float* gain,
                              float* state, float* prev, const float* tail, int width, const int* pos,
                              const int* seg_off, const int* chunks, int n_chunks, const int* segs, int n_segs,
                              float* us, float* decay, int heads, int d, float eps, void* y, int fp32, cudaStream_t st) {
  if (n_chunks <= 0 || n_segs <= 0) return 0;
  if (heads < 1 || heads > 65535 || d < 1) return 626;
  const ChunkArgs c{4 * heads * d, a, w0, u, gain, chunks, us, decay, heads, d, eps};
  return fp32 ? dispatch_chunks<float>(p, y, c, n_chunks, state, prev, tail, width, segs, n_segs, pos, seg_off, st)
              : dispatch_chunks<__nv_bfloat16>(p, y, c, n_chunks, state, prev, tail, width, segs, n_segs, pos, seg_off, st);
}
