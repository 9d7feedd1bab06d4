// Latent attention over a paged cache of latents: all heads of a token read the same row c_j (K = V = c_j, `rank` values), because
// the per-head up-projections of keys and values are absorbed into the query and into the output:
// score = (W_uk^T q) . c_j * scale,   o_lat = sum_j softmax_j c_j,   o = W_uv o_lat.
//
// Positions, where a design has them, turn `rot` further values of every query head and one part r_j that all heads share: a cache
// row is then [c_j | r_j], the score (W_uk^T q . c_j + q_r . r_j) * scale, and the values are still c_j.  With a window, position i
// sees the keys i - window + 1 .. i only.
//
// q and o are [T][heads][rank].  The (token, head) rows of a request are consecutive, and all of them see a prefix of the
// same keys, so a CTA takes M = 16 .. 64 consecutive rows of one request -- heads of one token in decode, several tokens
// in prefill -- and streams the request's latents once for all of them.  Position i sees every j <= i (of its window).
//   S phase : 8 warps share the M x 64 score tile (mma.sync m16n8k16, bf16 in, fp32 accumulate)
//   softmax : online (max, sum) per row in fp32, probabilities to shared memory as bf16
//   PV phase: warp w owns rank / 8 output columns of all M rows in registers
// Latent rows are fetched with cp.async into 128B-swizzled shared memory, double buffered.  grid.y splits the keys of a
// row tile when the row tiles alone leave SMs idle; latent_merge_kernel adds the partial results in split order.
//
// latent_attn_row_kernel computes the same with one warp per row on the CUDA cores, in fp32 throughout: models served in
// 32-bit floats, and ranks the tensor-core kernel does not take.
#include "mma16.cuh"

namespace {

struct LatArgs {
  const int* slots;
  const int* pos;
  const int* page_table;
  int ld_pt;
  const int* seg_off;    // [nseg + 1] row ranges of the requests, or null: every row is a request's only one
  int nseg;
  const int* num_valid;  // rows (tokens) >= *num_valid are padding, or null
  int rows;              // tokens
  int heads, rank;
  int rot;               // further values of a cache row and of a query head, which only the score reads
  const void* q_rot;     // [T] rows of stride ld_rot: head h's at h * rot
  int ld_rot;
  int window;            // > 0: position i sees the keys i - window + 1 .. i
  float scale;
  int nsplit;
  float* part_acc;       // [T * heads][nsplit][rank]
  float* part_ml;        // [T * heads][nsplit][2]
};

// ------------------------------------------------------------------ latent norm + store
// cache[out_loc[t]] = x[t] / rms(x[t]) * gain.  One warp per token.
template <typename T>
__global__ void __launch_bounds__(128) latent_store_kernel(const T* __restrict__ x, int ldx,
                                                           const float* __restrict__ gain, float eps,
                                                           T* __restrict__ cache, const int* __restrict__ out_loc,
                                                           int rows, int rank) {
  pdl_entry();
  const int t = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (t >= rows) return;
  const T* r = x + (size_t)t * ldx;
  float ss = 0.f;
  for (int i = lane; i < rank; i += 32) {
    const float v = ld_f(r + i);
    ss += v * v;
  }
  const float sc = 1.f / sqrtf(warp_sum(ss) / rank + eps);
  const int loc = out_loc[t];
  if (loc < 0) return;
  for (int i = lane; i < rank; i += 32) st_f(cache + (size_t)loc * rank + i, ld_f(r + i) * sc * gain[i]);
}

// ------------------------------------------------------------------ norm, rotation, store
struct LatStoreArgs {
  int ld;                // row stride of p
  int at_rot, at_c;      // columns: the heads' unrotated parts from 0, their parts that turn, then latent | shared part that turns
  const float* gain;     // [rank]
  float eps;
  const float* freq;     // [rot / 2]: neighbouring values turn by position * freq
  float mul;             // factor of cos and sin
  const int *pos, *out_loc;
  int heads, dim, rot, rank;
};

// One CTA per token.  cache row = [x / rms(x) * gain | turned part]; the queries' parts turn in place (`whole` null) or go, behind
// the unrotated ones, to whole [T][heads][dim + rot].  Four values at a time where every size is a multiple of four: the latent and a
// first share of the queries' turned parts then wait in registers while angles and squares are summed up.
__device__ __forceinline__ float4 turn4(const float4& v, const float2* cs) {
  const float4 r = *reinterpret_cast<const float4*>(cs);      // two pairs
  return make_float4(v.x * r.x - v.y * r.y, v.y * r.x + v.x * r.y, v.z * r.z - v.w * r.w, v.w * r.z + v.z * r.w);
}
constexpr int kLatThreads = 128;
template <typename T>
__global__ void __launch_bounds__(kLatThreads) latent_rotate_store4_kernel(T* p, T* __restrict__ cache, T* __restrict__ whole,
                                                                           const LatStoreArgs a) {
  pdl_entry();
  extern __shared__ __align__(16) float2 lat_cs[];
  __shared__ float sh[32];
  const int t = blockIdx.x, tid = threadIdx.x, loc = a.out_loc[t], wide = a.dim + a.rot, r4 = a.rot / 4, c4 = a.rank / 4;
  T* row = p + (size_t)t * a.ld;
  const T* x = row + a.at_c;
  T* q = row + a.at_rot;
  const int nq = a.heads * r4;
  float4 lat = make_float4(0.f, 0.f, 0.f, 0.f), mine = lat;
  if (tid < c4) lat = ld_f4(x + tid * 4);
  if (tid < nq) mine = ld_f4(q + tid * 4);
  for (int i = tid; i < a.rot / 2; i += kLatThreads) {
    float s, c;
    sincosf((float)a.pos[t] * a.freq[i], &s, &c);
    lat_cs[i] = make_float2(c * a.mul, s * a.mul);
  }
  float ss = lat.x * lat.x + lat.y * lat.y + lat.z * lat.z + lat.w * lat.w;
  for (int i = tid + kLatThreads; i < c4; i += kLatThreads) {
    const float4 v = ld_f4(x + i * 4);
    ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  if (whole)                                       // the unrotated parts, next to their heads' turned ones
    for (int i = tid; i < a.heads * (a.dim / 4); i += kLatThreads) {
      const int h = i / (a.dim / 4);
      st_f4(whole + ((size_t)t * a.heads + h) * wide + (i - h * (a.dim / 4)) * 4, ld_f4(row + i * 4));
    }
  const float sc = 1.f / sqrtf(cta_sum(ss, sh) / a.rank + a.eps);    // its barriers also publish lat_cs
  if (loc >= 0) {
    T* dst = cache + (size_t)loc * (a.rank + a.rot);
    for (int i = tid; i < c4; i += kLatThreads) {
      const float4 v = i == tid ? lat : ld_f4(x + i * 4), g = ld_f4(a.gain + i * 4);
      st_f4(dst + i * 4, make_float4(v.x * sc * g.x, v.y * sc * g.y, v.z * sc * g.z, v.w * sc * g.w));
    }
    for (int i = tid; i < r4; i += kLatThreads) st_f4(dst + a.rank + i * 4, turn4(ld_f4(x + a.rank + i * 4), lat_cs + 2 * i));
  }
  for (int i = tid; i < nq; i += kLatThreads) {
    const int h = i / r4, k = i - h * r4;
    st_f4(whole ? whole + ((size_t)t * a.heads + h) * wide + a.dim + 4 * k : q + 4 * i,
          turn4(i == tid ? mine : ld_f4(q + 4 * i), lat_cs + 2 * k));
  }
}

template <typename T>
__global__ void __launch_bounds__(256) latent_rotate_store_kernel(T* p, T* __restrict__ cache, T* __restrict__ whole,
                                                                  const LatStoreArgs a) {
  pdl_entry();
  extern __shared__ __align__(16) float2 lat_cs[];
  __shared__ float sh[32];
  const int t = blockIdx.x, loc = a.out_loc[t], half = a.rot / 2, wide = a.dim + a.rot;
  T* row = p + (size_t)t * a.ld;
  for (int i = threadIdx.x; i < half; i += 256) {
    float s, c;
    sincosf((float)a.pos[t] * a.freq[i], &s, &c);
    lat_cs[i] = make_float2(c * a.mul, s * a.mul);
  }
  const T* x = row + a.at_c;
  float ss = 0.f;
  for (int i = threadIdx.x; i < a.rank; i += 256) {
    const float v = ld_f(x + i);
    ss += v * v;
  }
  const float sc = 1.f / sqrtf(cta_sum(ss, sh) / a.rank + a.eps);    // its barriers also publish lat_cs
  if (loc >= 0) {
    T* dst = cache + (size_t)loc * (a.rank + a.rot);
    for (int i = threadIdx.x; i < a.rank; i += 256) st_f(dst + i, ld_f(x + i) * sc * a.gain[i]);
    for (int i = threadIdx.x; i < half; i += 256) {
      const float u = ld_f(x + a.rank + 2 * i), v = ld_f(x + a.rank + 2 * i + 1);
      const float2 cs = lat_cs[i];
      st_f(dst + a.rank + 2 * i, u * cs.x - v * cs.y);
      st_f(dst + a.rank + 2 * i + 1, v * cs.x + u * cs.y);
    }
  }
  T* q = row + a.at_rot;
  for (int i = threadIdx.x; i < a.heads * half; i += 256) {
    const int h = i / half, k = i - h * half;
    const float u = ld_f(q + 2 * i), v = ld_f(q + 2 * i + 1);
    const float2 cs = lat_cs[k];
    T* dst = whole ? whole + ((size_t)t * a.heads + h) * wide + a.dim + 2 * k : q + 2 * i;
    st_f(dst, u * cs.x - v * cs.y);
    st_f(dst + 1, v * cs.x + u * cs.y);
  }
  if (whole)
    for (int i = threadIdx.x; i < a.heads * a.dim; i += 256) {
      const int h = i / a.dim;
      whole[((size_t)t * a.heads + h) * wide + (i - h * a.dim)] = row[i];
    }
}

// ------------------------------------------------------------------ row tiles
// Which M consecutive (token, head) rows tile `b` covers: rows [row0, row1) of the request whose last token is t_last.
template <int M>
__device__ __forceinline__ bool find_tile(const LatArgs& a, int b, int& row0, int& row1) {
  const int lane = threadIdx.x & 31;
  if (!a.seg_off) {
    const int tpt = (a.heads + M - 1) / M;
    const int t = b / tpt;
    if (t >= a.rows) return false;
    row0 = t * a.heads + (b % tpt) * M;
    row1 = min(row0 + M, (t + 1) * a.heads);
    return true;
  }
  int base = 0;
  for (int s0 = 0; s0 < a.nseg; s0 += 32) {  // every warp does the same prefix sum over the requests' tile counts
    const int s = s0 + lane;
    int lo = 0, hi = 0;
    if (s < a.nseg) lo = a.seg_off[s] * a.heads, hi = a.seg_off[s + 1] * a.heads;
    const int cnt = (hi - lo + M - 1) / M;
    int inc = cnt;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int v = __shfl_up_sync(0xffffffffu, inc, o);
      if (lane >= o) inc += v;
    }
    const unsigned in = __ballot_sync(0xffffffffu, b < base + inc);
    if (in) {
      const int w = __ffs(in) - 1;
      const int first = __shfl_sync(0xffffffffu, base + inc - cnt, w);
      const int rlo = __shfl_sync(0xffffffffu, lo, w), rhi = __shfl_sync(0xffffffffu, hi, w);
      row0 = rlo + (b - first) * M;
      row1 = min(row0 + M, rhi);
      return true;
    }
    base += __shfl_sync(0xffffffffu, inc, 31);
  }
  return false;
}

// ------------------------------------------------------------------ tensor-core kernel
constexpr int kKT = 64;   // keys per tile
constexpr int kSP = kKT + 4;  // floats per score row

template <int RP, int MT>
struct LatCfg {
  static constexpr int M = MT * 16;
  static constexpr int RG = MT == 4 ? 2 : 1;       // warp row groups of the S phase
  static constexpr int WM = MT / RG;               // m16 tiles per warp
  static constexpr int KG = 8 / RG;                // key groups
  static constexpr int WN = kKT / KG / 8;          // n8 tiles per warp
  static constexpr int DW = RP / 8;                // output columns per warp
  static constexpr int NT = DW / 8;
  static constexpr int SMEM = M * RP * 2 + 2 * kKT * RP * 2 + M * kSP * 4 + M * kKT * 2 + 5 * M * 4;
};

template <int RP, int MT>
__global__ void __launch_bounds__(256) latent_attn_kernel(const __nv_bfloat16* __restrict__ q,
                                                          const __nv_bfloat16* __restrict__ cache,
                                                          __nv_bfloat16* __restrict__ o, const LatArgs a) {
  pdl_entry();
  using C = LatCfg<RP, MT>;
  constexpr int M = C::M, WM = C::WM, WN = C::WN, NT = C::NT;
  extern __shared__ __align__(128) uint8_t lat_smem[];
  __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(lat_smem);  // [M][RP] swizzled
  __nv_bfloat16* kv = qs + M * RP;                                 // [2][kKT][RP] swizzled
  float* ss = reinterpret_cast<float*>(kv + 2 * kKT * RP);         // [M][kSP]
  __nv_bfloat16* pb = reinterpret_cast<__nv_bfloat16*>(ss + M * kSP);  // [M][kKT] swizzled
  float* ms = reinterpret_cast<float*>(pb + M * kKT);
  float* ls = ms + M;
  float* alpha = ls + M;
  int* see = reinterpret_cast<int*>(alpha + M);                    // end of the keys the row sees
  int* from = see + M;                                             // and their beginning

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int split = blockIdx.y, R = a.rank, rch = R / 8, W = R + a.rot, wch = W / 8;
  int row0, row1;
  if (!find_tile<M>(a, blockIdx.x, row0, row1)) return;
  if (a.num_valid && row0 / a.heads >= *a.num_valid) return;
  const int t_last = (row1 - 1) / a.heads;
  const int key0 = a.window ? max(0, a.pos[row0 / a.heads] - a.window + 1) : 0;   // first key; keys are counted from there
  const int keys = a.pos[t_last] + 1 - key0;   // up to the tile's last token
  const int* pt = a.page_table + (size_t)a.slots[t_last] * a.ld_pt + key0;

  const int ktiles = (keys + kKT - 1) / kKT;
  const int per = (ktiles + a.nsplit - 1) / a.nsplit;
  const int kt0 = split * per, kt1 = min(kt0 + per, ktiles);
  if (kt0 >= kt1) {  // nothing for this split: an empty partial
    if (a.nsplit > 1)
      for (int r = row0 + tid; r < row1; r += 256) {
        float* ml = a.part_ml + ((size_t)r * a.nsplit + split) * 2;
        ml[0] = -1e30f, ml[1] = 0.f;
      }
    return;
  }

  for (int i = tid; i < M * (RP / 8); i += 256) {
    const int r = i / (RP / 8), c = i % (RP / 8);
    uint4 v = make_uint4(0, 0, 0, 0);
    if (row0 + r < row1 && c < wch)
      v = c < rch ? reinterpret_cast<const uint4*>(q + (size_t)(row0 + r) * R)[c]
                  : reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(a.q_rot) +
                                                   (size_t)((row0 + r) / a.heads) * a.ld_rot + (row0 + r) % a.heads * a.rot)[c - rch];
    reinterpret_cast<uint4*>(qs + r * RP)[swz(r, c)] = v;
  }
  if (tid < M) {
    ms[tid] = -1e30f, ls[tid] = 0.f;
    see[tid] = row0 + tid < row1 ? a.pos[(row0 + tid) / a.heads] + 1 - key0 : 0;
    from[tid] = a.window ? max(0, see[tid] - a.window) : 0;
  }

  // four threads fetch one latent row
  const int fk = tid >> 2, fp = tid & 3;
  auto key_loc = [&](int kt) {
    const int key = kt * kKT + fk;
    return (kt < kt1 && key < keys) ? pt[key] : -1;
  };
  auto issue = [&](int loc, int buf) {
    __nv_bfloat16* dst = kv + ((size_t)buf * kKT + fk) * RP;
    const __nv_bfloat16* src = cache + (size_t)max(loc, 0) * W;
#pragma unroll
    for (int c = fp; c < RP / 8; c += 4) {
      const bool in = loc >= 0 && c < wch;
      cpa16_zfill(dst + swz(fk, c) * 8, in ? src + c * 8 : cache, in);
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
  const float sc2 = a.scale * 1.4426950408889634f;  // scores in powers of two
  const int rg = warp / C::KG, kg = warp % C::KG;
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
    const __nv_bfloat16* kb = kv + (size_t)buf * kKT * RP;
    // ---- scores: rows [rg * WM * 16, +WM * 16) x keys [kg * WN * 8, +WN * 8)
    {
      float s[2][WM][WN][4] = {};
#pragma unroll 2
      for (int ks = 0; ks < RP / 16; ks += 2) {
        uint32_t bf[WN][4];
#pragma unroll
        for (int j = 0; j < WN; ++j) {
          const int br = (kg * WN + j) * 8 + (lane & 7);
          ldsm4(bf[j], kb + br * RP + swz(br, ks * 2 + (lane >> 3)) * 8);
        }
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
          for (int i = 0; i < WM; ++i) {
            const int ar = (rg * WM + i) * 16 + (lane & 15);
            uint32_t af[4];
            ldsm4(af, qs + ar * RP + swz(ar, (ks + h) * 2 + (lane >> 4)) * 8);
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
    // ---- online softmax
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
#pragma unroll
      for (int i = 0; i < PER; ++i) {
        v[i] = i < lim && i >= low ? v[i] : -INFINITY;
        mx = fmaxf(mx, v[i]);
      }
#pragma unroll
      for (int off = TPR / 2; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
      const float m_old = ms[r], m_new = fmaxf(m_old, mx);
      float sum = 0.f;
      __align__(16) __nv_bfloat16 e[PER];
#pragma unroll
      for (int i = 0; i < PER; ++i) {
        e[i] = f2bf(exp2f(v[i] - m_new));
        sum += bf2f(e[i]);   // the weights as they enter the product add up to what they are divided by
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
        const float al = exp2f(m_old - m_new);
        alpha[r] = al;
        ms[r] = m_new;
        ls[r] = ls[r] * al + sum;
      }
    }
    __syncthreads();
    // ---- o += P C: all rows, output columns [warp * DW, +DW)
    if (warp * C::DW < R) {
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
#pragma unroll
        for (int j = 0; j < NT; j += 2) {
          uint32_t vf[4];
          ldsm4_t(vf, kb + vr * RP + swz(vr, warp * (C::DW / 8) + j + (lane >> 4)) * 8);
#pragma unroll
          for (int i = 0; i < MT; ++i) {
            mma16816(acc[i][j], pf[i], vf[0], vf[1]);
            mma16816(acc[i][j + 1], pf[i], vf[2], vf[3]);
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
      const int r = i * 16 + (lane >> 2) + half * 8, row = row0 + r;
      if (row >= row1) continue;
      const float inv = 1.f / ls[r];
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        const int c = warp * C::DW + j * 8 + (lane & 3) * 2;
        if (c >= R) continue;
        const float x = acc[i][j][half * 2], y = acc[i][j][half * 2 + 1];
        if (a.nsplit > 1)
          *reinterpret_cast<float2*>(a.part_acc + ((size_t)row * a.nsplit + split) * R + c) = make_float2(x, y);
        else
          *reinterpret_cast<__nv_bfloat162*>(o + (size_t)row * R + c) = __floats2bfloat162_rn(x * inv, y * inv);
      }
    }
  if (a.nsplit > 1 && tid < M && row0 + tid < row1) {
    float* ml = a.part_ml + ((size_t)(row0 + tid) * a.nsplit + split) * 2;
    ml[0] = ms[tid], ml[1] = ls[tid];
  }
}

// o[row] = sum_s acc_s 2^(m_s - M) / sum_s l_s 2^(m_s - M)
__global__ void __launch_bounds__(128) latent_merge_kernel(__nv_bfloat16* __restrict__ o, const LatArgs a) {
  pdl_entry();
  const int row = blockIdx.x, n = a.nsplit;
  if (a.num_valid && row / a.heads >= *a.num_valid) return;
  const float* ml = a.part_ml + (size_t)row * n * 2;
  float mx = -1e30f, l = 0.f;
  for (int s = 0; s < n; ++s) mx = fmaxf(mx, ml[s * 2]);
  for (int s = 0; s < n; ++s) l += ml[s * 2 + 1] * exp2f(ml[s * 2] - mx);
  const float inv = 1.f / l;
  for (int c = threadIdx.x; c < a.rank; c += 128) {
    float v = 0.f;
    for (int s = 0; s < n; ++s)
      if (ml[s * 2 + 1] > 0.f) v = fmaf(a.part_acc[((size_t)row * n + s) * a.rank + c], exp2f(ml[s * 2] - mx), v);
    o[(size_t)row * a.rank + c] = f2bf(v * inv);
  }
}

// ------------------------------------------------------------------ one warp per row, fp32 arithmetic
template <typename T, int NI>
__global__ void __launch_bounds__(128) latent_attn_row_kernel(const T* __restrict__ q, const T* __restrict__ cache,
                                                              T* __restrict__ o, const LatArgs a) {
  pdl_entry();
  const int row = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31, R = a.rank;
  if (row >= a.rows * a.heads) return;
  const int t = row / a.heads;
  if (a.num_valid && t >= *a.num_valid) return;
  const int W = R + a.rot, key0 = a.window ? max(0, a.pos[t] - a.window + 1) : 0, keys = a.pos[t] + 1 - key0;
  const int* pt = a.page_table + (size_t)a.slots[t] * a.ld_pt + key0;
  const T* qr = static_cast<const T*>(a.q_rot) + (a.rot ? (size_t)t * a.ld_rot + row % a.heads * a.rot : 0);
  float qv[NI], acc[NI];
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int c = i * 32 + lane;
    qv[i] = c < R ? ld_f(q + (size_t)row * R + c) * a.scale : c < W ? ld_f(qr + c - R) * a.scale : 0.f;
    acc[i] = 0.f;
  }
  float m = -1e30f, l = 0.f;
  for (int k0 = 0; k0 < keys; k0 += 32) {
    const int mine = k0 + lane < keys ? pt[k0 + lane] : 0;
    const int n = min(32, keys - k0);
    for (int k = 0; k < n; ++k) {
      const T* c = cache + (size_t)__shfl_sync(0xffffffffu, mine, k) * W;
      float cv[NI], s = 0.f;
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        cv[i] = i * 32 + lane < W ? ld_f(c + i * 32 + lane) : 0.f;
        s = fmaf(qv[i], cv[i], s);
      }
      s = warp_sum(s);
      const float mn = fmaxf(m, s), al = expf(m - mn), p = expf(s - mn);
      l = l * al + p;
      m = mn;
#pragma unroll
      for (int i = 0; i < NI; ++i) acc[i] = fmaf(p, cv[i], acc[i] * al);
    }
  }
  const float inv = 1.f / l;
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int c = i * 32 + lane;
    if (c < R) st_f(o + (size_t)row * R + c, acc[i] * inv);
  }
}

// ctx[dst + j] = cache[page_table[slot][first + j]] for the keys of every listed request, zeros in the padding behind them.
// list: [segs][4] = slot, keys, first row of the copy, first key; rows [dst, dst of the next request) belong to a request.
__global__ void __launch_bounds__(128) latent_gather_kernel(const uint4* __restrict__ cache, uint4* __restrict__ ctx,
                                                            const int* __restrict__ list, int segs, int total,
                                                            const int* __restrict__ page_table, int ld_pt, int r8) {
  pdl_entry();
  const int row = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (row >= total) return;
  int lo = 0, hi = segs - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (list[mid * 4 + 2] <= row) lo = mid; else hi = mid - 1;
  }
  const int j = row - list[lo * 4 + 2];
  const bool in = j < list[lo * 4 + 1];
  const size_t src = in ? (size_t)page_table[(size_t)list[lo * 4] * ld_pt + list[lo * 4 + 3] + j] * r8 : 0;
  for (int i = lane; i < r8; i += 32) ctx[(size_t)row * r8 + i] = in ? cache[src + i] : make_uint4(0, 0, 0, 0);
}

template <int RP, int MT>
int launch_lat(const void* q, const void* cache, void* o, const LatArgs& a, int tiles, cudaStream_t st) {
  using C = LatCfg<RP, MT>;
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(latent_attn_kernel<RP, MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM) !=
        cudaSuccess)
      return 631;
    set = true;
  }
  dsv4_launch(latent_attn_kernel<RP, MT>, dim3(tiles, a.nsplit), 256, C::SMEM, st, (const __nv_bfloat16*)q,
              (const __nv_bfloat16*)cache, (__nv_bfloat16*)o, a);
  if (a.nsplit > 1)
    dsv4_launch(latent_merge_kernel, a.rows * a.heads, 128, 0, st, (__nv_bfloat16*)o, a);
  return (int)cudaGetLastError();
}
template <int RP>
int dispatch_lat(int m, const void* q, const void* cache, void* o, const LatArgs& a, int tiles, cudaStream_t st) {
  switch (m) {
    case 16: return launch_lat<RP, 1>(q, cache, o, a, tiles, st);
    case 32: return launch_lat<RP, 2>(q, cache, o, a, tiles, st);
    case 64:
      if constexpr (RP <= 512) return launch_lat<RP, 4>(q, cache, o, a, tiles, st);
      return 632;
    default: return 632;
  }
}
template <typename T>
int launch_row(const void* q, const void* cache, void* o, const LatArgs& a, cudaStream_t st) {
  const int grid = (a.rows * a.heads + 3) / 4;
  const T *tq = (const T*)q, *tc = (const T*)cache;
  const int w = a.rank + a.rot;
  if (w <= 128)
    dsv4_launch(latent_attn_row_kernel<T, 4>, grid, 128, 0, st, tq, tc, (T*)o, a);
  else if (w <= 256)
    dsv4_launch(latent_attn_row_kernel<T, 8>, grid, 128, 0, st, tq, tc, (T*)o, a);
  else if (w <= 512)
    dsv4_launch(latent_attn_row_kernel<T, 16>, grid, 128, 0, st, tq, tc, (T*)o, a);
  else if (w <= 1024)
    dsv4_launch(latent_attn_row_kernel<T, 32>, grid, 128, 0, st, tq, tc, (T*)o, a);
  else
    return 633;
  return (int)cudaGetLastError();
}

}  // namespace

DSV4_API int dsv4_latent_store(const void* x, int ldx, const float* gain, float eps, void* cache, const int* out_loc,
                               int rows, int rank, int fp32, cudaStream_t st) {
  if (rows <= 0) return 0;
  const int grid = (rows + 3) / 4;
  if (fp32)
    dsv4_launch(latent_store_kernel<float>, grid, 128, 0, st, (const float*)x, ldx, gain, eps, (float*)cache, out_loc,
                rows, rank);
  else
    dsv4_launch(latent_store_kernel<__nv_bfloat16>, grid, 128, 0, st, (const __nv_bfloat16*)x, ldx, gain, eps,
                (__nv_bfloat16*)cache, out_loc, rows, rank);
  return (int)cudaGetLastError();
}

// p [rows, ld]: the heads' unrotated parts (heads x dim) from column 0, the parts that turn (heads x rot, even) at at_rot, latent |
// shared part that turns (rank + rot) at at_c; cache [locations, rank + rot].  whole [rows, heads, dim + rot] or null: see above.
DSV4_API int dsv4_latent_rotate_store(void* p, int ld, int at_rot, int at_c, const float* gain, float eps, const float* freq,
                                      float mul, const int* pos, const int* out_loc, void* cache, void* whole, int rows,
                                      int heads, int dim, int rot, int rank, int fp32, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (rot < 2 || rot % 2 || rot > 8192 || !freq) return 637;
  const LatStoreArgs a{ld, at_rot, at_c, gain, eps, freq, mul, pos, out_loc, heads, dim, rot, rank};
  const bool fours = ld % 4 == 0 && at_rot % 4 == 0 && at_c % 4 == 0 && dim % 4 == 0 && rot % 4 == 0 && rank % 4 == 0 &&
                     ((uintptr_t)p & 15) == 0;
  auto go = [&](auto kern, int threads, auto type) {
    using T = decltype(type);
    dsv4_launch(kern, rows, threads, rot * 4, st, (T*)p, (T*)cache, (T*)whole, a);
  };
  using B = __nv_bfloat16;
  if (fp32)
    fours ? go(latent_rotate_store4_kernel<float>, kLatThreads, float()) : go(latent_rotate_store_kernel<float>, 256, float());
  else
    fours ? go(latent_rotate_store4_kernel<B>, kLatThreads, B()) : go(latent_rotate_store_kernel<B>, 256, B());
  return (int)cudaGetLastError();
}

// q_rot [rows] of stride ld_rot, heads x rot: the part of the score that positions turn (rot 0: none); cache [locations, rank + rot].
// m: rows per CTA (16, 32 or 64; 0 = the one-warp-per-row kernel), tiles: row tiles of that height over all requests.
// nsplit > 1 needs part_acc [T * heads, nsplit, rank] and part_ml [T * heads, nsplit, 2].
DSV4_API int dsv4_latent_attention(const void* q, const void* cache, void* o, const int* slots, const int* pos,
                                   const int* page_table, int ld_pt, const int* seg_off, int nseg,
                                   const int* num_valid, int rows, int heads, int rank, const void* q_rot, int ld_rot,
                                   int rot, int window, float scale, int m, int tiles, int nsplit, float* part_acc,
                                   float* part_ml, int fp32, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (nsplit < 1 || nsplit > 65535 || (nsplit > 1 && (!part_acc || !part_ml))) return 634;
  if (rot < 0 || (rot && !q_rot) || window < 0) return 638;
  const LatArgs a{slots, pos, page_table, ld_pt, seg_off, nseg, num_valid, rows, heads, rank, rot, q_rot, ld_rot, window, scale,
                  nsplit, part_acc, part_ml};
  if (m == 0) return fp32 ? launch_row<float>(q, cache, o, a, st) : launch_row<__nv_bfloat16>(q, cache, o, a, st);
  if (fp32 || rank % 8 || rot % 8 || ld_rot % 8) return 635;
  const int w = rank + rot;
  if (w <= 128) return dispatch_lat<128>(m, q, cache, o, a, tiles, st);
  if (w <= 256) return dispatch_lat<256>(m, q, cache, o, a, tiles, st);
  if (w <= 384) return dispatch_lat<384>(m, q, cache, o, a, tiles, st);
  if (w <= 512) return dispatch_lat<512>(m, q, cache, o, a, tiles, st);
  if (w <= 640) return dispatch_lat<640>(m, q, cache, o, a, tiles, st);
  return 636;
}

DSV4_API int dsv4_latent_gather(const void* cache, void* ctx, const int* list, int segs, int total,
                                const int* page_table, int ld_pt, int rank, cudaStream_t st) {
  if (total <= 0) return 0;
  if (rank % 8 || segs < 1) return 650;
  dsv4_launch(latent_gather_kernel, (total + 3) / 4, 128, 0, st, (const uint4*)cache, (uint4*)ctx, list, segs, total,
              page_table, ld_pt, rank / 8);
  return (int)cudaGetLastError();
}
