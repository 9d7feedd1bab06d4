// Recurrent time mixing with a per-channel decay and a bonus for the current token ("wkv"): the token shift in front of
// the projections, and the recurrence with its per-head norm and gate behind them.
//
//   o_t = (S_{t-1} + diag(u) k_t v_t^T)^T r_t,     S_t = diag(w_t) S_{t-1} + k_t v_t^T,     w_t = exp(-exp(a_t + w0))
//   y_t = o_t / rms(o_t) * gain * silu(g_t)        (per head; S is [key, value])
//
// State per request slot, fp32: S [heads][d][d] and the previous token's normed row.  A request at position 0 starts
// from zeros whatever its slot held before.
#include "vec.cuh"

namespace {

// ------------------------------------------------------------------ norm + token shift + mixes
// h = x / rms(x) * gain of this row and of the row before it (the slot's saved row for the first row of a portion,
// zeros at position 0);  out[t][m] = h + (h' - h) * mu[m] for the n_mix mixes.  A request's last row goes to the slot:
// directly if it is also the first one, else to `tail` (other CTAs may still have to read the slot), from where
// wkv_scan_kernel moves it.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) shift_mix_kernel(const float* __restrict__ x, const float* __restrict__ gain,
                                                        float eps, const float* __restrict__ mu, int n_mix,
                                                        float* __restrict__ prev, float* __restrict__ tail,
                                                        const int* __restrict__ slots, const int* __restrict__ pos,
                                                        T* __restrict__ out, int rows, int d) {
  pdl_entry();
  __shared__ float sh[32];
  constexpr int W = VEC ? 4 : 1;   // columns per access
  const int t = blockIdx.x, tid = threadIdx.x;
  const bool first = seg_first(slots, pos, t), last = seg_last(slots, pos, t, rows);
  const float* xc = x + (size_t)t * d;
  const float* xp = xc - d;  // only read when !first
  float sc = 0.f, sp = 0.f;
#pragma unroll 2
  for (int i = tid * W; i < d; i += 256 * W) {
    float v[W], q[W];
    ld_w<W>(xc + i, v);
    if (!first) ld_w<W>(xp + i, q);
#pragma unroll
    for (int j = 0; j < W; ++j) {
      sc += v[j] * v[j];
      if (!first) sp += q[j] * q[j];
    }
  }
  const float rc = 1.f / sqrtf(cta_sum(sc, sh) / d + eps);
  const float rp = first ? 0.f : 1.f / sqrtf(cta_sum(sp, sh) / d + eps);
  const bool fresh = pos[t] == 0;
  float* ps = prev + (size_t)slots[t] * d;
  float* ts = tail + (size_t)slots[t] * d;
#pragma unroll 2
  for (int i = tid * W; i < d; i += 256 * W) {
    float g[W], h[W], hp[W], m[W], r[W];
    ld_w<W>(gain + i, g);
    ld_w<W>(xc + i, h);
    if (!first)
      ld_w<W>(xp + i, hp);
    else if (!fresh)
      ld_w<W>(ps + i, hp);
#pragma unroll
    for (int j = 0; j < W; ++j) {
      h[j] *= rc * g[j];
      hp[j] = (first ? (fresh ? 0.f : hp[j]) : hp[j] * rp * g[j]) - h[j];
    }
    T* o = out + (size_t)t * n_mix * d + i;
    for (int n = 0; n < n_mix; ++n) {
      ld_w<W>(mu + (size_t)n * d + i, m);
#pragma unroll
      for (int j = 0; j < W; ++j) r[j] = h[j] + hp[j] * m[j];
      st_w<W>(o + (size_t)n * d, r);
    }
    if (last) st_w<W>((first ? ps : ts) + i, h);
  }
}

// ------------------------------------------------------------------ recurrence
struct ScanArgs {
  int ld;               // row stride of the projections: 4 heads d, columns r | k | v | g
  const float* a;       // [rows, heads d] decay logits
  const float* w0;      // [heads d]
  const float* u;       // [heads d]
  const float* gain;    // [heads d]
  float* state;         // [slots + 1][heads][d][d]
  float* prev;          // [slots + 1][width] saved rows of the token shift, and where they wait
  const float* tail;
  int width;
  const int* slots;
  const int* pos;
  const int* seg_off;   // [segments + 1] or null: segment s is row s
  int heads, d;
  float eps;
};

constexpr int kTC = 16;  // tokens staged at a time
constexpr int kKK = 16;  // keys per thread
constexpr int kVV = 2;   // value columns per thread
constexpr int kGS = kKK + 4;  // floats between two key groups in shared memory (keeps 16-byte reads conflict-free)

__device__ __forceinline__ void cp_async16(void* smem, const void* g) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(smem)), "l"(g) : "memory");
}

template <int DP>
struct ScanCfg {
  static constexpr int G = DP / kKK;                       // threads that share a pair of value columns
  static constexpr int ACTIVE = DP / kVV * G;
  static constexpr int THREADS = ACTIVE < 32 ? 32 : ACTIVE;
  static size_t smem(int esz) {  // staged r, k, w, v, o + raw ring of two
    return sizeof(float) * kTC * (3 * G * kGS + 2 * DP + 1) + 2 * (size_t)kTC * DP * (4 * esz + 4) + 16;
  }
};

// One CTA per (segment, head).  The state sits in registers: a thread owns kKK keys x kVV value columns; the sum over
// keys of o is a shuffle over the G neighbouring threads of a column pair.  Tokens are staged kTC at a time, the next
// kTC arrive with cp.async meanwhile.
template <typename T, int DP>
__global__ void __launch_bounds__(ScanCfg<DP>::THREADS) wkv_scan_kernel(const T* __restrict__ p, T* __restrict__ y,
                                                                        const ScanArgs a) {
  pdl_entry();
  using C = ScanCfg<DP>;
  constexpr int G = C::G, NT = C::THREADS;
  extern __shared__ __align__(16) uint8_t scan_smem[];
  const int d = a.d, hd = a.heads * d;
  float* rs = reinterpret_cast<float*>(scan_smem);   // [kTC][G * kGS]
  float* ks = rs + kTC * G * kGS;
  float* ws = ks + kTC * G * kGS;
  float* vs = ws + kTC * G * kGS;                    // [kTC][DP]
  float* os = vs + kTC * DP;                         // [kTC][DP]
  float* bonus = os + kTC * DP;                      // [kTC]
  float* raw_a = bonus + kTC;                        // [2][kTC][DP]
  T* raw = reinterpret_cast<T*>(raw_a + 2 * kTC * DP);  // [2][4][kTC][DP]
  const int seg = blockIdx.x, head = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int t0 = a.seg_off ? a.seg_off[seg] : seg, t1 = a.seg_off ? a.seg_off[seg + 1] : seg + 1;
  const int n = t1 - t0;
  if (n <= 0) return;
  const int slot = a.slots[t0];
  const int g = tid % G, col = tid / G * kVV;
  const bool live = tid < C::ACTIVE && col < d;
  const bool aligned = d % 8 == 0;

  auto fetch = [&](int c0, int buf) {  // rows t0 + c0 .. of the five inputs into raw buffer `buf`
    const int m = min(kTC, n - c0);
    if (aligned) {
      const int pc = d * (int)sizeof(T) / 16, ac = d / 4;
      for (int i = tid; i < m * (4 * pc + ac); i += NT) {
        const int tok = i / (4 * pc + ac), j = i % (4 * pc + ac);
        if (j < 4 * pc) {
          const int q = j / pc, e = j % pc * (16 / (int)sizeof(T));
          cp_async16(raw + (((size_t)buf * 4 + q) * kTC + tok) * DP + e,
                     p + (size_t)(t0 + c0 + tok) * a.ld + q * hd + head * d + e);
        } else {
          const int e = (j - 4 * pc) * 4;
          cp_async16(raw_a + ((size_t)buf * kTC + tok) * DP + e, a.a + (size_t)(t0 + c0 + tok) * hd + head * d + e);
        }
      }
    } else {
      for (int i = tid; i < m * 5 * d; i += NT) {
        const int tok = i / (5 * d), q = i / d % 5, e = i % d;
        if (q < 4)
          raw[(((size_t)buf * 4 + q) * kTC + tok) * DP + e] = p[(size_t)(t0 + c0 + tok) * a.ld + q * hd + head * d + e];
        else
          raw_a[((size_t)buf * kTC + tok) * DP + e] = a.a[(size_t)(t0 + c0 + tok) * hd + head * d + e];
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0, 0);

  float s[kKK][kVV];
  float* st = a.state + ((size_t)slot * a.heads + head) * d * d;
  const bool fresh = a.pos[t0] == 0;
#pragma unroll
  for (int i = 0; i < kKK; ++i) {
    const int key = g * kKK + i;
#pragma unroll
    for (int j = 0; j < kVV; ++j)
      s[i][j] = (live && !fresh && key < d && col + j < d) ? st[(size_t)key * d + col + j] : 0.f;
  }

  for (int c0 = 0, it = 0; c0 < n; c0 += kTC, ++it) {
    const int m = min(kTC, n - c0), buf = it & 1;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    // raw -> staged fp32 (keys and columns past d are zero: they never touch the state)
    const T* rb = raw + (size_t)buf * 4 * kTC * DP;
    for (int i = tid; i < m * DP; i += NT) {
      const int tok = i / DP, e = i % DP;
      const bool in = e < d;
      const int at = tok * G * kGS + e / kKK * kGS + e % kKK;
      rs[at] = in ? ld_f(rb + (0 * kTC + tok) * DP + e) : 0.f;
      ks[at] = in ? ld_f(rb + (1 * kTC + tok) * DP + e) : 0.f;
      vs[tok * DP + e] = in ? ld_f(rb + (2 * kTC + tok) * DP + e) : 0.f;
      ws[at] = in ? expf(-expf(raw_a[((size_t)buf * kTC + tok) * DP + e] + a.w0[head * d + e])) : 0.f;
    }
    for (int tok = warp; tok < m; tok += NT / 32) {
      float b = 0.f;
      for (int e = lane; e < d; e += 32)
        b += ld_f(rb + (0 * kTC + tok) * DP + e) * a.u[head * d + e] * ld_f(rb + (1 * kTC + tok) * DP + e);
      b = warp_sum(b);
      if (lane == 0) bonus[tok] = b;
    }
    __syncthreads();
    if (c0 + kTC < n) fetch(c0 + kTC, buf ^ 1);
    for (int tok = 0; tok < m; ++tok) {
      const float* rp = rs + tok * G * kGS + g * kGS;
      const float* kp = ks + tok * G * kGS + g * kGS;
      const float* wp = ws + tok * G * kGS + g * kGS;
      float v[kVV], o[kVV];
#pragma unroll
      for (int j = 0; j < kVV; ++j) v[j] = col + j < DP ? vs[tok * DP + col + j] : 0.f, o[j] = 0.f;
#pragma unroll
      for (int i = 0; i < kKK; i += 4) {
        const float4 r4 = *reinterpret_cast<const float4*>(rp + i);
        const float4 k4 = *reinterpret_cast<const float4*>(kp + i);
        const float4 w4 = *reinterpret_cast<const float4*>(wp + i);
        const float rr[4] = {r4.x, r4.y, r4.z, r4.w}, kk[4] = {k4.x, k4.y, k4.z, k4.w}, ww[4] = {w4.x, w4.y, w4.z, w4.w};
#pragma unroll
        for (int q = 0; q < 4; ++q)
#pragma unroll
          for (int j = 0; j < kVV; ++j) {
            o[j] = fmaf(rr[q], s[i + q][j], o[j]);
            s[i + q][j] = fmaf(ww[q], s[i + q][j], kk[q] * v[j]);
          }
      }
#pragma unroll
      for (int j = 0; j < kVV; ++j) {
#pragma unroll
        for (int off = 1; off < G; off <<= 1) o[j] += __shfl_xor_sync(0xffffffffu, o[j], off);
      }
      if (live && g == 0) {
        const float b = bonus[tok];
#pragma unroll
        for (int j = 0; j < kVV; ++j) os[tok * DP + col + j] = o[j] + b * v[j];
      }
    }
    __syncthreads();
    for (int tok = warp; tok < m; tok += NT / 32) {
      float q = 0.f;
      for (int e = lane; e < d; e += 32) q += os[tok * DP + e] * os[tok * DP + e];
      const float inv = 1.f / sqrtf(warp_sum(q) / d + a.eps);
      for (int e = lane; e < d; e += 32) {
        const float gt = ld_f(rb + (3 * kTC + tok) * DP + e);
        st_f(y + (size_t)(t0 + c0 + tok) * hd + head * d + e,
             os[tok * DP + e] * inv * a.gain[head * d + e] * (gt / (1.f + expf(-gt))));
      }
    }
  }
  if (live) {
#pragma unroll
    for (int i = 0; i < kKK; ++i) {
      const int key = g * kKK + i;
#pragma unroll
      for (int j = 0; j < kVV; ++j)
        if (key < d && col + j < d) st[(size_t)key * d + col + j] = s[i][j];
    }
  }
  if (n > 1) {  // the token shift's last row was parked by shift_mix_kernel; the heads share the copy
    const int per = (a.width + a.heads - 1) / a.heads;
    for (int i = head * per + tid; i < min((head + 1) * per, a.width); i += NT)
      a.prev[(size_t)slot * a.width + i] = a.tail[(size_t)slot * a.width + i];
  }
}

template <typename T>
void launch_shift(const float* x, const float* gain, float eps, const float* mu, int n_mix, float* prev, float* tail,
                  const int* slots, const int* pos, void* out, int rows, int d, cudaStream_t st) {
  if (d % 4 == 0)
    dsv4_launch(shift_mix_kernel<T, true>, rows, 256, 0, st, x, gain, eps, mu, n_mix, prev, tail, slots, pos, (T*)out,
                rows, d);
  else
    dsv4_launch(shift_mix_kernel<T, false>, rows, 256, 0, st, x, gain, eps, mu, n_mix, prev, tail, slots, pos, (T*)out,
                rows, d);
}

template <typename T, int DP>
int launch_scan(const void* p, void* y, const ScanArgs& a, int segs, cudaStream_t st) {
  const size_t smem = ScanCfg<DP>::smem(sizeof(T));
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(wkv_scan_kernel<T, DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) !=
        cudaSuccess)
      return 621;
    set = true;
  }
  dsv4_launch(wkv_scan_kernel<T, DP>, dim3(segs, a.heads), ScanCfg<DP>::THREADS, smem, st, (const T*)p, (T*)y, a);
  return (int)cudaGetLastError();
}
template <typename T>
int dispatch_scan(const void* p, void* y, const ScanArgs& a, int segs, cudaStream_t st) {
  if (a.d <= 16) return launch_scan<T, 16>(p, y, a, segs, st);
  if (a.d <= 32) return launch_scan<T, 32>(p, y, a, segs, st);
  if (a.d <= 64) return launch_scan<T, 64>(p, y, a, segs, st);
  if (a.d <= 128) return launch_scan<T, 128>(p, y, a, segs, st);
  return 620;
}

}  // namespace

DSV4_API int dsv4_shift_mix(const float* x, const float* gain, float eps, const float* mu, int n_mix, float* prev,
                            float* tail, const int* slots, const int* pos, void* out, int rows, int d, int fp32,
                            cudaStream_t st) {
  if (rows <= 0) return 0;
  if (n_mix < 1) return 622;
  if (fp32)
    launch_shift<float>(x, gain, eps, mu, n_mix, prev, tail, slots, pos, out, rows, d, st);
  else
    launch_shift<__nv_bfloat16>(x, gain, eps, mu, n_mix, prev, tail, slots, pos, out, rows, d, st);
  return (int)cudaGetLastError();
}

// p: [rows, 4 heads d] projections r | k | v | g;  a: [rows, heads d];  y: [rows, heads d].  segs: segments (seg_off
// given) or rows.  d <= 128.
DSV4_API int dsv4_wkv_scan(const void* p, const float* a, const float* w0, const float* u, const float* gain,
                           float* state, float* prev, const float* tail, int width, const int* slots, const int* pos,
                           const int* seg_off, int segs, int heads, int d, float eps, void* y, int fp32,
                           cudaStream_t st) {
  if (segs <= 0) return 0;
  if (heads < 1 || heads > 65535 || d < 1) return 623;
  const ScanArgs s{4 * heads * d, a, w0, u, gain, state, prev, tail, width, slots, pos, seg_off, heads, d, eps};
  return fp32 ? dispatch_scan<float>(p, y, s, segs, st) : dispatch_scan<__nv_bfloat16>(p, y, s, segs, st);
}
