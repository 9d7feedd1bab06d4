// Routed experts with bf16 weights: a grouped tcgen05 GEMM over the route plan of moe.cu.
//
//   D[row, route] = W_e[row, :] . X[route, :]
// "swap-AB" as in moe_mx.cu: 128 weight rows on the TMEM lanes, up to NT routes of one expert on N, so an expert with a
// handful of routes costs a narrow instruction instead of a padded 128-row one.
//   MODE 1: the tile holds 128 gate rows and the 128 matching up rows as two accumulators; the epilogue writes
//           silu(gate) * up in expert order (position), the operand of the second GEMM.
//   MODE 2: 128 output rows; the epilogue writes them to the route's own row.  The weighted sum over a token's routes
//           belongs to the kernel that adds it to the residual stream (residual.cu).
// Persistent: a CTA per SM walks the (tile, row tile) items, row tiles of a tile side by side, with the accumulators double
// buffered in tensor memory so that an epilogue (narrow, transposing stores) runs under the next item's MMAs.
// Warp roles (192 threads): warp 0 TMA producer, warp 1 tcgen05.mma issuer, warps 2-5 epilogue.  Weight tensor maps are
// 3-D (k, row, expert [x gate / up]), so a row or k count that does not fill its tile is zero-filled and never reads the
// next expert.
#include "vec.cuh"

namespace {

struct GroupedArgs {
  const int* hdr;           // [0] tiles, [1] routes
  const int* tiles;         // [max_tiles][3]
  const int* sorted_route;  // position -> route
  int max_tiles, routes, experts;
  int N, K, ldo;            // rows per expert (MODE 1: of gate), reduction length, output row stride
};

template <int NT, int MODE>
struct GroupedCfg {
  static constexpr int kABytes = 128 * 128 * (MODE == 1 ? 2 : 1);
  static constexpr int kBBytes = NT * 128;
  static constexpr int kStageBytes = kABytes + kBBytes;
  static constexpr int kFit = 200 * 1024 / kStageBytes;
  static constexpr int kStages = kFit > 8 ? 8 : kFit;
  static constexpr int kSmem = kStages * kStageBytes + 1024 + 256;
  static constexpr int kAcc = NT < 32 ? 32 : NT;               // tensor-memory columns of one accumulator
  static constexpr int kSet = (MODE == 1 ? 2 : 1) * kAcc;      // of an item
  static constexpr int kCols = 2 * kSet;                       // double buffered
};

// item -> expert, first position, routes, first weight row; false: past the plan (or a plan from other sizes)
struct GroupedItem {
  int e, pos0, cnt, r0;
};
template <int NT>
__device__ __forceinline__ bool grouped_item(const GroupedArgs& g, int id, int row_tiles, int ntiles, GroupedItem& it) {
  const int t = id / row_tiles;
  if (t >= ntiles) return false;
  it.e = g.tiles[t * 3], it.pos0 = g.tiles[t * 3 + 1], it.cnt = g.tiles[t * 3 + 2];
  it.r0 = (id - t * row_tiles) * 128;
  return it.e >= 0 && it.e < g.experts && it.pos0 >= 0 && it.cnt >= 1 && it.cnt <= NT && it.pos0 + it.cnt <= g.routes;
}

template <int NT, int MODE>
__global__ void __launch_bounds__(192, 1) moe_bf16_gemm_kernel(const __grid_constant__ CUtensorMap tmA,
                                                               const __grid_constant__ CUtensorMap tmB,
                                                               __nv_bfloat16* __restrict__ out, const GroupedArgs g) {
  using C = GroupedCfg<NT, MODE>;
  constexpr int S = C::kStages;
  constexpr uint32_t kIdesc = umma_idesc(128, NT, 1, 1);
  extern __shared__ uint8_t gsm_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(gsm_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + S * C::kStageBytes);
  uint64_t *empty = full + S, *tfull = empty + S, *tempty = tfull + 2;
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(tempty + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_holder + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  if (threadIdx.x == 0) {
    for (int i = 0; i < S; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 1);
    }
    for (int i = 0; i < 2; ++i) mbar_init(&tfull[i], 1), mbar_init(&tempty[i], 4);
    *abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tmA);
    tma_prefetch_desc(&tmB);
  }
  if (warp == 1) {
    tmem_alloc(tmem_holder, C::kCols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_holder;
  pdl_wait();
  pdl_launch_dependents();
  const int row_tiles = (g.N + 127) / 128, nkt = (g.K + 63) / 64;
  int ntiles = g.hdr[0];
  if (ntiles > g.max_tiles) {
    if (threadIdx.x == 0) dsv4_set_error(DSV4_ERR_BAD_INDEX, 61, ntiles);
    ntiles = 0;
  }
  GroupedItem w;

  if (warp == 0) {
    if (lane == 0) {
      int i = 0;
      bool ok = true;
      for (int id = blockIdx.x; ok && grouped_item<NT>(g, id, row_tiles, ntiles, w); id += gridDim.x) {
        for (int k = 0; k < nkt; ++k, ++i) {
          const int s = i % S;
          if (i >= S && !mbar_wait<32>(&empty[s], ((i / S) & 1) ^ 1, abort_flag, 71)) {
            ok = false;
            break;
          }
          uint8_t* st = smem + s * C::kStageBytes;
          mbar_expect_tx(&full[s], C::kStageBytes);
          if (MODE == 1) {
            tma_load_3d(st, &tmA, &full[s], k * 64, w.r0, 2 * w.e);
            tma_load_3d(st + 128 * 128, &tmA, &full[s], k * 64, w.r0, 2 * w.e + 1);
          } else {
            tma_load_3d(st, &tmA, &full[s], k * 64, w.r0, w.e);
          }
          tma_load_2d(st + C::kABytes, &tmB, &full[s], k * 64, w.pos0);
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      int i = 0, n = 0;
      bool ok = true;
      for (int id = blockIdx.x; ok && grouped_item<NT>(g, id, row_tiles, ntiles, w); id += gridDim.x, ++n) {
        const uint32_t d = tmem + (n & 1) * C::kSet;
        if (n >= 2 && !mbar_wait(&tempty[n & 1], ((n >> 1) & 1) ^ 1, abort_flag, 74)) break;
        tc_fence_after();
        for (int k = 0; k < nkt; ++k, ++i) {
          const int s = i % S;
          if (!mbar_wait(&full[s], (i / S) & 1, abort_flag, 72)) {
            ok = false;
            break;
          }
          tc_fence_after();
          const uint8_t* st = smem + s * C::kStageBytes;
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const uint64_t bd = umma_desc_k128(st + C::kABytes, j * 32);
            umma_f16(d, umma_desc_k128(st, j * 32), bd, kIdesc, k > 0 || j > 0);
            if (MODE == 1) umma_f16(d + C::kAcc, umma_desc_k128(st + 128 * 128, j * 32), bd, kIdesc, k > 0 || j > 0);
          }
          umma_commit(&empty[s]);
        }
        if (ok) umma_commit(&tfull[n & 1]);
      }
    }
  } else {
    const int q = warp & 3;
    int n = 0;
    for (int id = blockIdx.x; grouped_item<NT>(g, id, row_tiles, ntiles, w); id += gridDim.x, ++n) {
      const uint32_t d0 = tmem + (n & 1) * C::kSet + ((uint32_t)(q * 32) << 16);
      const int orow = w.r0 + q * 32 + lane;
      if (!mbar_wait<64>(&tfull[n & 1], (n >> 1) & 1, abort_flag, 73)) break;
      tc_fence_after();
#pragma unroll 1
      for (int c0 = 0; c0 < NT; c0 += 16) {
        if (c0 >= w.cnt) break;
        uint32_t a[16], b[16];
        tmem_ld_32x16(d0 + c0, a);
        if (MODE == 1) tmem_ld_32x16(d0 + C::kAcc + c0, b);
        int route = 0;
        if (MODE == 2 && lane < 16 && c0 + lane < w.cnt) route = g.sorted_route[w.pos0 + c0 + lane];
        tmem_ld_wait();
#pragma unroll
        for (int c = 0; c < 16; ++c) {
          const int r = MODE == 1 ? w.pos0 + c0 + c : __shfl_sync(0xffffffffu, route, c);
          if (orow < g.N && c0 + c < w.cnt) {
            float v = __uint_as_float(a[c]);
            if (MODE == 1) v = v / (1.f + expf(-v)) * __uint_as_float(b[c]);
            out[(size_t)r * g.ldo + orow] = f2bf(v);
          }
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&tempty[n & 1]);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem, C::kCols);
}

// xs[pos] = x[sorted_route[pos] / topk], rows of d8 16-byte pieces
__global__ void __launch_bounds__(128) moe_gather_rows_kernel(const uint4* __restrict__ x, uint4* __restrict__ xs,
                                                              const int* __restrict__ hdr,
                                                              const int* __restrict__ sorted_route, int topk, int d8,
                                                              int routes) {
  pdl_entry();
  const int pos = blockIdx.x;
  if (pos >= hdr[1]) return;
  const int r = sorted_route[pos];
  if (r < 0 || r >= routes) {
    if (threadIdx.x == 0) dsv4_set_error(DSV4_ERR_BAD_INDEX, 62, pos);
    return;
  }
  for (int i = threadIdx.x; i < d8; i += 128) xs[(size_t)pos * d8 + i] = x[(size_t)(r / topk) * d8 + i];
}

template <int NT, int MODE>
int launch_grouped(const CUtensorMap& tmA, const void* xs, void* out, const GroupedArgs& g, int sms, cudaStream_t st) {
  using C = GroupedCfg<NT, MODE>;
  CUtensorMap tmB;
  if (dsv4_make_tmap_2d(&tmB, xs, 1, g.K, g.routes, (uint64_t)g.K * 2, 64, NT, 3)) return 642;
  auto kern = moe_bf16_gemm_kernel<NT, MODE>;
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, C::kSmem) != cudaSuccess) return 643;
    set = true;
  }
  const long long items = (long long)((g.N + 127) / 128) * g.max_tiles;
  dsv4_launch(kern, (unsigned)(items < sms ? items : sms), 192, C::kSmem, st, tmA, tmB, (__nv_bfloat16*)out, g);
  return (int)cudaGetLastError();
}
template <int MODE>
int dispatch_grouped(int nt, const CUtensorMap& tmA, const void* xs, void* out, const GroupedArgs& g, int sms,
                     cudaStream_t st) {
  switch (nt) {
    case 16: return launch_grouped<16, MODE>(tmA, xs, out, g, sms, st);
    case 32: return launch_grouped<32, MODE>(tmA, xs, out, g, sms, st);
    case 64: return launch_grouped<64, MODE>(tmA, xs, out, g, sms, st);
    case 128: return launch_grouped<128, MODE>(tmA, xs, out, g, sms, st);
    default: return 644;
  }
}

}  // namespace

DSV4_API int dsv4_moe_gather_rows(const void* x, void* xs, const int* plan, int routes, int max_tiles, int topk, int d,
                                  cudaStream_t st) {
  if (routes <= 0) return 0;
  if (d % 8) return 640;
  dsv4_launch(moe_gather_rows_kernel, routes, 128, 0, st, (const uint4*)x, (uint4*)xs, plan, plan + 4 + 3 * max_tiles,
              topk, d / 8, routes);
  return (int)cudaGetLastError();
}

// mode 1: w [experts][2][N][K] (gate, up), x = rows in expert order [routes, K] -> out [routes, N] in expert order;
// mode 2: w [experts][N][K], x = act [routes, K] -> out [routes, N], row = route.  nt: the plan's routes per tile.
DSV4_API int dsv4_moe_bf16_gemm(int mode, int nt, const void* w, const void* x, const int* plan, int routes,
                                int max_tiles, void* out, int experts, int N, int K, int sms, cudaStream_t st) {
  if (routes <= 0) return 0;
  if (K % 8 || max_tiles < 1 || sms < 1 || (mode != 1 && mode != 2)) return 645;
  CUtensorMap tmA;
  if (dsv4_make_tmap_3d(&tmA, w, K, N, (uint64_t)experts * (mode == 1 ? 2 : 1), (uint64_t)K * 2, (uint64_t)N * K * 2, 64,
                        128))
    return 641;
  const int* tiles = plan + 4;
  const GroupedArgs g{plan, tiles, tiles + 3 * max_tiles, max_tiles, routes, experts, N, K, N};
  return mode == 1 ? dispatch_grouped<1>(nt, tmA, x, out, g, sms, st) : dispatch_grouped<2>(nt, tmA, x, out, g, sms, st);
}
