// Causal multi-head attention of long prompt portions on tcgen05 over keys and values that lie side by side: gathered from
// a paged cache (grouped_attn.cu: kv_gather, several query heads to a key head, optionally capped scores, a bias by distance
// (a table, or falling with the distance) and a sink, or sigmoids of the scores as weights), or expanded from cached latents
// (latent_attn.cu).  With a window an item's keys begin at the first one that its first query sees (rounded down).
//
// For latents, the absorbed form (latent_attn.cu) multiplies every (query, key) pair over the whole latent rank, twice.  For
// a portion of many tokens it is cheaper to expand the request's latents once,  K = C W_uk^T  and  V^T = W_uv C^T  (two
// plain projections; the second one comes out with the keys contiguous, which is the K-major operand of the PV product),
// and to run ordinary attention over `dim` and `vdim` per head.
//
// One CTA: one head, 256 consecutive queries of one request as two 128-row tiles that share every key / value tile (128
// keys).  The tensor core works on one tile while the softmax warps work on the other:
//   warp 0      TMA producer: Q once, then K and V^T tiles through two-stage rings
//   warp 1      tcgen05.mma issuer:  S_t = Q_t K^T,  O_t += P_t V  (P_t is read from tensor memory)
//   warps 2-5   softmax of tile 0, warps 6-9 of tile 1: one thread per row; P_t overwrites S_t in place as bf16
// Tensor memory: S0 | S1 | O0 | O1, 128 columns each.  O stays there; it is rescaled only when a row's maximum has grown by
// more than 2^8 since the last time (the sums stay far from overflow, the quotient does not depend on it).
#include "mma16.cuh"

namespace {

constexpr int kQT = 128;                     // queries per tile, keys per tile
constexpr int kBlk = kQT * 128;              // bytes of a [128 rows][64 elements] operand block
constexpr int kFThreads = 320;
constexpr int kColO = 256;

struct FlashArgs {
  const int* items;     // [n_items][5]: first query row, queries, context position of the first, first key row, keys
  int heads, group, dim, vdim, ldo;   // group: query heads that share a key head
  float scale2;         // scale * log2(e)
  // capped scores (CAP): in powers of two, cap2 tanh(s c) for the raw product s
  float c, cap2;
  float small;          // |s| up to here: s (p0 + p1 s^2 + p2 s^4 + p3 s^6), an odd polynomial
  float p0, p1, p2, p3;
  const float* sink;    // [heads] or null
  const float* rel;     // [heads][n_rel] (kCappedBias)
  int n_rel;
  const float* slope;   // [heads] (kSloped)
  const float* wbias;   // [heads] (kSigmoid)
  int window;           // > 0: a query sees its own position and the window - 1 before it
  const float2* turn;   // [rows][vdim / 2] cos and sin: results are turned back (vdim is a multiple of 32); or null
  const __nv_bfloat16* gate;   // [rows] of stride ld_gate, one per head: results times its sigmoid; or null
  int ld_gate;
};

struct FlashBars {
  uint64_t q_full, k_full[2], k_empty[2], v_full[2], v_empty[2], s_full[2], p_ready[2], o_full[2];
  uint32_t tmem;
  int abort_flag;
};

constexpr int kWin = 160;                    // distances between a warp's 32 queries and a tile's 128 keys (159)
constexpr int kBiasBytes = 8 * kWin * 4;

template <int NB>     // 64-wide blocks of dim
struct FlashCfg {
  static constexpr int kQ = 2 * NB * kBlk, kK = NB * kBlk, kV = 2 * kBlk;
  static constexpr int kSmem = kQ + 2 * (kK + kV) + kBiasBytes + 1024 + (int)sizeof(FlashBars);
};

// What happens to a score between the product and the softmax.
enum ScoreMode : int { kScaled = 0, kCapped = 1, kCappedBias = 2, kSloped = 3, kSigmoid = 4 };

template <int NB, int MODE>
__global__ void __launch_bounds__(kFThreads, 1)
flash_attn_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                  const __grid_constant__ CUtensorMap tmV, __nv_bfloat16* __restrict__ out, const FlashArgs a) {
  using C = FlashCfg<NB>;
  extern __shared__ uint8_t fsm_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(fsm_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* qs = smem;                       // [2 tiles][NB] blocks
  uint8_t* ks = qs + C::kQ;                 // [2 stages][NB] blocks
  uint8_t* vs = ks + 2 * C::kK;             // [2 stages][2] blocks of [vdim rows][64 keys]
  float* wins = reinterpret_cast<float*>(vs + 2 * C::kV);   // [8 warps][kWin] bias by distance
  FlashBars* b = reinterpret_cast<FlashBars*>(wins + 8 * kWin);
  volatile int* abort_flag = &b->abort_flag;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int head = blockIdx.x, kv_head = head / a.group;

  if (threadIdx.x == 0) {
    mbar_init(&b->q_full, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&b->k_full[i], 1), mbar_init(&b->k_empty[i], 1);
      mbar_init(&b->v_full[i], 1), mbar_init(&b->v_empty[i], 1);
      mbar_init(&b->s_full[i], 1), mbar_init(&b->o_full[i], 1);
      mbar_init(&b->p_ready[i], 128);
    }
    b->abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tmQ);
    tma_prefetch_desc(&tmK);
    tma_prefetch_desc(&tmV);
  }
  if (warp == 1) {
    tmem_alloc(&b->tmem, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = b->tmem;
  pdl_wait();
  pdl_launch_dependents();
  const int* it = a.items + blockIdx.y * 5;
  const int q0 = it[0], nq = it[1], pos0 = it[2], kv0 = it[3], nkeys = it[4];
  const int n = (nkeys + kQT - 1) / kQT;    // key tiles: every key the last query sees
  const int vp = (a.vdim + 15) & ~15;       // columns of the PV product
  const uint32_t v_bytes = 2u * (uint32_t)vp * 128u;

  if (warp == 0) {
    if (lane == 0) {
      mbar_expect_tx(&b->q_full, C::kQ);
      for (int t = 0; t < 2; ++t)
        for (int j = 0; j < NB; ++j) tma_load_3d(qs + (t * NB + j) * kBlk, &tmQ, &b->q_full, j * 64, head, q0 + t * kQT);
      for (int i = 0; i < n; ++i) {
        const int s = i & 1;
        const uint32_t ph = ((i >> 1) & 1) ^ 1;
        if (i >= 2 && !mbar_wait<32>(&b->k_empty[s], ph, abort_flag, 81)) break;
        mbar_expect_tx(&b->k_full[s], C::kK);
        for (int j = 0; j < NB; ++j)
          tma_load_3d(ks + s * C::kK + j * kBlk, &tmK, &b->k_full[s], j * 64, kv_head, kv0 + i * kQT);
        if (i >= 2 && !mbar_wait<32>(&b->v_empty[s], ph, abort_flag, 82)) break;
        mbar_expect_tx(&b->v_full[s], v_bytes);
        for (int j = 0; j < 2; ++j)
          tma_load_3d(vs + s * C::kV + j * kBlk, &tmV, &b->v_full[s], kv0 + i * kQT + j * 64, 0, kv_head);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t kIdS = umma_idesc(128, kQT, 1, 1);
      const uint32_t id_o = umma_idesc(128, vp, 1, 1);
      auto scores = [&](int t, int i) {
        const uint8_t* kt = ks + (i & 1) * C::kK;
#pragma unroll
        for (int k = 0; k < NB * 4; ++k)
          umma_f16(tmem + t * 128, umma_desc_k128(qs + (t * NB + k / 4) * kBlk, (k & 3) * 32),
                   umma_desc_k128(kt + k / 4 * kBlk, (k & 3) * 32), kIdS, k > 0);
      };
      auto values = [&](int t, int i) {
        const uint8_t* vt = vs + (i & 1) * C::kV;
#pragma unroll
        for (int k = 0; k < 8; ++k)
          umma_f16_ta(tmem + kColO + t * 128, tmem + t * 128 + k * 8,
                      umma_desc_k128(vt + k / 4 * kBlk, (k & 3) * 32), id_o, i > 0 || k > 0);
      };
      bool ok = mbar_wait(&b->q_full, 0, abort_flag, 83) && mbar_wait(&b->k_full[0], 0, abort_flag, 84);
      tc_fence_after();
      if (ok) {
        for (int t = 0; t < 2; ++t) {
          scores(t, 0);
          umma_commit(&b->s_full[t]);
        }
        umma_commit(&b->k_empty[0]);
      }
      for (int i = 0; i < n && ok; ++i) {
        const bool more = i + 1 < n;
        ok = mbar_wait(&b->v_full[i & 1], (i >> 1) & 1, abort_flag, 85);
        for (int t = 0; t < 2 && ok; ++t) {
          ok = mbar_wait(&b->p_ready[t], i & 1, abort_flag, 86);
          if (!ok) break;
          tc_fence_after();
          values(t, i);
          if (more) {
            // S_t may only be written now: P_t, which sits on it, has been consumed by the product before (MMAs of one
            // thread run in order)
            if (t == 0) ok = mbar_wait(&b->k_full[(i + 1) & 1], ((i + 1) >> 1) & 1, abort_flag, 87);
            if (!ok) break;
            tc_fence_after();
            scores(t, i + 1);
            umma_commit(&b->s_full[t]);
          } else {
            umma_commit(&b->o_full[t]);
          }
        }
        if (ok) {
          umma_commit(&b->v_empty[i & 1]);
          if (more) umma_commit(&b->k_empty[(i + 1) & 1]);
        }
      }
    }
  } else {
    const int t = (warp - 2) >> 2, quarter = warp & 3;
    const int row = t * kQT + quarter * 32 + lane;            // query within the item
    const uint32_t lane_base = (uint32_t)(quarter * 32) << 16;
    const uint32_t sp = tmem + t * 128 + lane_base, op = tmem + kColO + t * 128 + lane_base;
    const int last = row < nq ? pos0 + row : -1;              // last key the row sees
    const int first_masked = (pos0 + t * kQT + quarter * 32 + 1) / kQT;  // key tiles before it are seen whole by the warp
    const float sc = MODE == kScaled || MODE == kSigmoid ? a.scale2 : 1.f;        // the other modes leave scores in powers of two
    float* win = wins + (warp - 2) * kWin;
    const float* rel = MODE == kCappedBias ? a.rel + (size_t)head * a.n_rel : nullptr;
    const float rel_far = MODE == kCappedBias ? rel[a.n_rel - 1] * kLog2e : 0.f;
    const float slope2 = MODE == kSloped ? a.slope[head] * kLog2e : 0.f;
    const float wb2 = MODE == kSigmoid ? a.wbias[head] * kLog2e : 0.f;
    // key tiles from here on are past the window's edge of all of the warp's queries
    const int edge_end = a.window ? (pos0 + t * kQT + quarter * 32 + 31 - a.window) / kQT : -1;
    float m = -1e30f, l = 0.f;
    bool ok = true;
    for (int i = 0; i < n; ++i) {
      const int base = pos0 + t * kQT + quarter * 32 - i * kQT;   // distance of the warp's first query and the tile's first key
      const bool all_far = base - (kQT - 1) >= a.n_rel - 1;
      if (MODE == kCappedBias && !all_far) {
        __syncwarp();
#pragma unroll
        for (int x = 0; x < kWin; x += 32)
          win[x + lane] = rel[max(min(base - (kQT - 1) + x + lane, a.n_rel - 1), 0)] * kLog2e;
        __syncwarp();
      }
      ok = mbar_wait<16>(&b->s_full[t], i & 1, abort_flag, 88);
      if (!ok) break;
      tc_fence_after();
      float s[kQT];
      float big = 0.f;
#pragma unroll
      for (int c = 0; c < kQT; c += 32) {
        uint32_t r[32];
        tmem_ld_32x32(sp + c, r);
        tmem_ld_wait();
#pragma unroll
        for (int j = 0; j < 32; ++j) s[c + j] = __uint_as_float(r[j]);
        if (MODE == kCapped || MODE == kCappedBias) {
#pragma unroll
          for (int j = 0; j < 32; ++j) big = fmaxf(big, fabsf(s[c + j]));
        }
      }
      if (MODE == kSloped) {
        const float from = slope2 * (float)(i * kQT - pos0 - row);      // minus the distance of the tile's first key
#pragma unroll
        for (int j = 0; j < kQT; ++j) s[j] = fmaf(s[j], a.scale2, fmaf(slope2, (float)j, from));
      }
      if (MODE == kCapped || MODE == kCappedBias) {
        const bool small = __all_sync(0xffffffffu, big <= a.small);
        const float e = 2.f * kLog2e * a.c;
#pragma unroll
        for (int c = 0; c < kQT; c += 32) {
          float* x = s + c;
          if (small) {
#pragma unroll
            for (int j = 0; j < 32; ++j) {
              const float y = x[j] * x[j];
              x[j] *= fmaf(fmaf(fmaf(a.p3, y, a.p2), y, a.p1), y, a.p0);
            }
          } else {
#pragma unroll
            for (int j = 0; j < 32; ++j) x[j] = softcap_ex2(x[j], e, a.cap2);
          }
          if (MODE == kCappedBias) {
            if (all_far) {
#pragma unroll
              for (int j = 0; j < 32; ++j) x[j] += rel_far;
            } else {
#pragma unroll
              for (int j = 0; j < 32; ++j) x[j] += win[kQT - 1 + lane - c - j];
            }
          }
        }
      }
      if (i >= first_masked || row >= nq) {
        const int lim = last - i * kQT;
#pragma unroll
        for (int j = 0; j < kQT; ++j)
          if (j > lim) s[j] = -INFINITY;
      }
      if (i <= edge_end) {
        const int low = pos0 + row - a.window - i * kQT;
#pragma unroll
        for (int j = 0; j < kQT; ++j)
          if (j <= low) s[j] = -INFINITY;
      }
      if constexpr (MODE == kSigmoid) {
        // 1 / a and 1 / b from one reciprocal: b / (a b), a / (a b); weights below 2^-60 count as 2^-60, masked ones as 0
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          uint32_t pk[16];
#pragma unroll
          for (int j = 0; j < 16; ++j) {
            const float x0 = s[c * 32 + 2 * j], x1 = s[c * 32 + 2 * j + 1];
            const float e0 = 1.f + ex2(fminf(-fmaf(x0, sc, wb2), 60.f)), e1 = 1.f + ex2(fminf(-fmaf(x1, sc, wb2), 60.f));
            const float q = rcp_approx(e0 * e1);
            const __nv_bfloat162 p = __floats2bfloat162_rn(x0 == -INFINITY ? 0.f : e1 * q, x1 == -INFINITY ? 0.f : e0 * q);
            pk[j] = *reinterpret_cast<const uint32_t*>(&p);
          }
          tmem_st_32x16(sp + c * 16, pk);
        }
        tmem_st_wait();
        tc_fence_before();
        mbar_arrive(&b->p_ready[t]);
        continue;
      }
      float mx = s[0];
#pragma unroll
      for (int j = 1; j < kQT; ++j) mx = fmaxf(mx, s[j]);
      mx *= sc;
      const bool grow = mx > m + 8.f;
      if (__any_sync(0xffffffffu, grow)) {
        const float mn = grow ? mx : m, f = ex2(m - mn);
        m = mn;
        l *= f;
        if (i > 0) {
#pragma unroll 1
          for (int c = 0; c < vp; c += 16) {
            uint32_t r[16];
            tmem_ld_32x16(op + c, r);
            tmem_ld_wait();
#pragma unroll
            for (int j = 0; j < 16; ++j) r[j] = __float_as_uint(__uint_as_float(r[j]) * f);
            tmem_st_32x16(op + c, r);
          }
        }
      }
      float sum0 = 0.f, sum1 = 0.f;
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        uint32_t pk[16];
#pragma unroll
        for (int j = 0; j < 16; ++j) {
          const float p0 = ex2(fmaf(s[c * 32 + 2 * j], sc, -m)), p1 = ex2(fmaf(s[c * 32 + 2 * j + 1], sc, -m));
          sum0 += p0, sum1 += p1;
          const __nv_bfloat162 p = __floats2bfloat162_rn(p0, p1);
          pk[j] = *reinterpret_cast<const uint32_t*>(&p);
        }
        tmem_st_32x16(sp + c * 16, pk);
      }
      l += sum0 + sum1;
      tmem_st_wait();
      tc_fence_before();
      mbar_arrive(&b->p_ready[t]);
    }
    if (ok && mbar_wait<16>(&b->o_full[t], 0, abort_flag, 89)) {
      tc_fence_after();
      float f = 1.f;
      if (a.sink) {            // one more term of the sum, without a key or a value
        const float s2 = a.sink[head] * kLog2e, mm = fmaxf(m, s2);
        f = ex2(m - mm);
        l = l * f + ex2(s2 - mm);
      }
      float inv = MODE == kSigmoid ? 1.f : f / l;
      if (a.gate && row < nq) inv *= sigmoid_f(bf2f(a.gate[(size_t)(q0 + row) * a.ld_gate + head]));
      __nv_bfloat16* dst = out + (size_t)(q0 + row) * a.ldo + head * a.vdim;
      if (a.turn) {            // column c of the first half meets its partner in the second
        const int half = a.vdim / 2;
        const float2* turn = a.turn + (size_t)(q0 + row) * half;
#pragma unroll 1
        for (int c = 0; c < half; c += 16) {
          uint32_t u[16], v[16];
          tmem_ld_32x16(op + c, u);
          tmem_ld_32x16(op + half + c, v);
          tmem_ld_wait();
          if (row < nq) {
            uint4 o0[2], o1[2];
            __nv_bfloat162 *p0 = reinterpret_cast<__nv_bfloat162*>(o0), *p1 = reinterpret_cast<__nv_bfloat162*>(o1);
#pragma unroll
            for (int j = 0; j < 8; ++j) {
              const float4 cs = *reinterpret_cast<const float4*>(turn + c + 2 * j);       // two pairs
              const float ua = __uint_as_float(u[2 * j]), ub = __uint_as_float(u[2 * j + 1]);
              const float va = __uint_as_float(v[2 * j]), vb = __uint_as_float(v[2 * j + 1]);
              p0[j] = __floats2bfloat162_rn((ua * cs.x + va * cs.y) * inv, (ub * cs.z + vb * cs.w) * inv);
              p1[j] = __floats2bfloat162_rn((va * cs.x - ua * cs.y) * inv, (vb * cs.z - ub * cs.w) * inv);
            }
#pragma unroll
            for (int h = 0; h < 2; ++h) {
              reinterpret_cast<uint4*>(dst + c)[h] = o0[h];
              reinterpret_cast<uint4*>(dst + half + c)[h] = o1[h];
            }
          }
        }
      } else {
#pragma unroll 1
        for (int c = 0; c < vp; c += 16) {
          uint32_t r[16];
          tmem_ld_32x16(op + c, r);
          tmem_ld_wait();
          if (row < nq) {
#pragma unroll
            for (int h = 0; h < 2; ++h) {
              if (c + h * 8 >= a.vdim) break;      // vdim is a multiple of 8
              uint4 u;
              __nv_bfloat162* p = reinterpret_cast<__nv_bfloat162*>(&u);
#pragma unroll
              for (int j = 0; j < 4; ++j)
                p[j] = __floats2bfloat162_rn(__uint_as_float(r[h * 8 + 2 * j]) * inv,
                                             __uint_as_float(r[h * 8 + 2 * j + 1]) * inv);
              *reinterpret_cast<uint4*>(dst + c + h * 8) = u;
            }
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem, 512);
}

template <int NB, int MODE>
int launch_flash(const CUtensorMap& q, const CUtensorMap& k, const CUtensorMap& v, void* out, const FlashArgs& a,
                 int n_items, cudaStream_t st) {
  using C = FlashCfg<NB>;
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(flash_attn_kernel<NB, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::kSmem) !=
        cudaSuccess)
      return 655;
    set = true;
  }
  dsv4_launch(flash_attn_kernel<NB, MODE>, dim3(a.heads, n_items), kFThreads, C::kSmem, st, q, k, v, (__nv_bfloat16*)out, a);
  return (int)cudaGetLastError();
}
template <int NB>
int dispatch_flash(int mode, const CUtensorMap& q, const CUtensorMap& k, const CUtensorMap& v, void* out,
                   const FlashArgs& a, int n_items, cudaStream_t st) {
  if (mode == kScaled) return launch_flash<NB, kScaled>(q, k, v, out, a, n_items, st);
  if (mode == kCapped) return launch_flash<NB, kCapped>(q, k, v, out, a, n_items, st);
  if (mode == kSloped) return launch_flash<NB, kSloped>(q, k, v, out, a, n_items, st);
  if (mode == kSigmoid) return launch_flash<NB, kSigmoid>(q, k, v, out, a, n_items, st);
  return launch_flash<NB, kCappedBias>(q, k, v, out, a, n_items, st);
}

}  // namespace

// q: bf16 [rows, heads * dim] (row stride ldq), k: [kv_rows, kv_heads * dim], vt: [kv_heads * vdim, kv_rows] (row stride
// kv_rows), out: [rows, heads * vdim]; query head h reads key head h / (heads / kv_heads).  items as in FlashArgs, at most 256
// queries each; first key rows are multiples of 8.  Scores: cap tanh(q.k scale / cap) (cap 0: q.k scale), plus rel[h,
// min(distance, n_rel - 1)] if rel is given; or, without cap and rel, less slope[h] * distance.  sink [heads] or null adds e^sink
// to the sum of a row's weights.  wbias [heads]: weights are sigmoid(score + wbias) instead, without cap, rel, slope and sink.
// window: keys further back are not seen; items then begin with the first key their first query sees, or before it.  turn, gate:
// as in FlashArgs.
DSV4_API int dsv4_flash_attention(const void* q, int ldq, const void* k, const void* vt, void* out, const int* items,
                                  int n_items, int rows, int kv_rows, int heads, int kv_heads, int dim, int vdim,
                                  float scale, float cap, const float* sink, const float* rel, int n_rel,
                                  const float* slope, const float* wbias, int window, const float* turn, const void* gate,
                                  int ld_gate, cudaStream_t st) {
  if (n_items <= 0) return 0;
  if (dim % 8 || vdim % 8 || ldq % 8 || kv_rows % 8 || dim < 8 || dim > 128 || vdim < 8 || vdim > 128 || n_items > 65535)
    return 651;
  if (kv_heads < 1 || heads % kv_heads || (rel && n_rel < 1) || (slope && (rel || cap > 0.f))) return 656;
  if ((wbias && (slope || rel || cap > 0.f || sink)) || window < 0 || (turn && vdim % 32)) return 657;
  CUtensorMap tq, tk, tv;
  if (dsv4_make_tmap_3d(&tq, q, dim, heads, rows, (uint64_t)dim * 2, (uint64_t)ldq * 2, 64, 1, kQT)) return 652;
  if (dsv4_make_tmap_3d(&tk, k, dim, kv_heads, kv_rows, (uint64_t)dim * 2, (uint64_t)kv_heads * dim * 2, 64, 1, kQT)) return 653;
  const int vp = (vdim + 15) & ~15;
  if (dsv4_make_tmap_3d(&tv, vt, kv_rows, vdim, kv_heads, (uint64_t)kv_rows * 2, (uint64_t)vdim * kv_rows * 2, 64, vp)) return 654;
  FlashArgs a{items, heads, heads / kv_heads, dim, vdim, heads * vdim, scale * kLog2e};
  a.sink = sink, a.rel = rel, a.n_rel = rel ? n_rel : 0, a.slope = slope, a.wbias = wbias, a.window = window;
  a.turn = reinterpret_cast<const float2*>(turn), a.gate = (const __nv_bfloat16*)gate, a.ld_gate = ld_gate;
  if (cap > 0.f) {
    // tanh x = x - x^3 / 3 + 2 x^5 / 15 - 17 x^7 / 315 + ..., to 2e-6 relative for x up to 0.3
    const float c = scale / cap, cap2 = cap * kLog2e, c2 = c * c;
    a.c = c, a.cap2 = cap2, a.small = 0.3f / fabsf(c);
    a.p0 = cap2 * c, a.p1 = -a.p0 * c2 / 3.f, a.p2 = a.p0 * c2 * c2 * (2.f / 15.f), a.p3 = a.p0 * c2 * c2 * c2 * (-17.f / 315.f);
  } else {
    a.small = INFINITY, a.p0 = a.scale2;      // only reached with a bias
  }
  const int mode = wbias ? kSigmoid : slope ? kSloped : rel ? kCappedBias : cap > 0.f ? kCapped : kScaled;
  return dim <= 64 ? dispatch_flash<1>(mode, tq, tk, tv, out, a, n_items, st)
                   : dispatch_flash<2>(mode, tq, tk, tv, out, a, n_items, st);
}
