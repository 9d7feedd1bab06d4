// Routed experts with bf16 weights: a grouped tcgen05 GEMM over the route plan of moe.cu.
//
//   D[row, route] = W_e[row, :] . X[route, :]
// "swap-AB" as in moe_mx.cu: 128 weight rows on the TMEM lanes, up to NT routes of one expert on N, so an expert with a
// handful of routes costs a narrow instruction instead of a padded 128-row one.
//   MODE 1: the tile holds 128 gate rows and the 128 matching up rows as two accumulators; the epilogue writes
//           silu(gate) * up in expert order (position), the operand of the second GEMM.
//   MODE 2: 128 output rows; the epilogue writes them to the route's own row.  The weighted sum over a token's routes
//           belongs to the kernel that adds it to the residual stream (residual.cu).
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
  static constexpr int kStages = MODE == 1 ? 4 : (NT >= 128 ? 5 : 6);
  static constexpr int kSmem = kStages * kStageBytes + 1024 + 256;
  static constexpr int kAcc = NT < 32 ? 32 : NT;          // tensor-memory columns between the two accumulators
  static constexpr int kCols = (MODE == 1 ? 2 : 1) * kAcc;
};

template <int NT, int MODE>
__global__ void __launch_bounds__(192) moe_bf16_gemm_kernel(const __grid_constant__ CUtensorMap tmA,
                                                            const __grid_constant__ CUtensorMap tmB,
                                                            __nv_bfloat16* __restrict__ out, const GroupedArgs g) {
  using C = GroupedCfg<NT, MODE>;
  constexpr int S = C::kStages;
  constexpr uint32_t kIdesc = umma_idesc(128, NT, 1, 1);
  extern __shared__ uint8_t gsm_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(gsm_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + S * C::kStageBytes);
  uint64_t* empty = full + S;
  uint64_t* tfull = empty + S;
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(tfull + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_holder + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  if (threadIdx.x == 0) {
    for (int i = 0; i < S; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 1);
    }
    mbar_init(tfull, 1);
    *abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tmA);
    tma_prefetch_desc(&tmB);
  }
  pdl_wait();
  pdl_launch_dependents();
  // the plan decides whether this CTA has work: uniform over the CTA, before tensor memory is taken
  const int ntiles = g.hdr[0];
  if ((int)blockIdx.y >= ntiles) return;
  const int e = g.tiles[blockIdx.y * 3], pos0 = g.tiles[blockIdx.y * 3 + 1], cnt = g.tiles[blockIdx.y * 3 + 2];
  if (ntiles > g.max_tiles || e < 0 || e >= g.experts || pos0 < 0 || cnt < 1 || cnt > NT || pos0 + cnt > g.routes) {
    if (threadIdx.x == 0) dsv4_set_error(DSV4_ERR_BAD_INDEX, 61, e);  // a plan from other sizes
    return;
  }
  if (warp == 1) {
    tmem_alloc(tmem_holder, C::kCols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_holder;
  const int nkt = (g.K + 63) / 64, r0 = blockIdx.x * 128;

  if (warp == 0) {
    if (lane == 0) {
      for (int i = 0; i < nkt; ++i) {
        const int s = i % S;
        if (i >= S && !mbar_wait<32>(&empty[s], ((i / S) & 1) ^ 1, abort_flag, 71)) break;
        uint8_t* st = smem + s * C::kStageBytes;
        mbar_expect_tx(&full[s], C::kStageBytes);
        if (MODE == 1) {
          tma_load_3d(st, &tmA, &full[s], i * 64, r0, 2 * e);
          tma_load_3d(st + 128 * 128, &tmA, &full[s], i * 64, r0, 2 * e + 1);
        } else {
          tma_load_3d(st, &tmA, &full[s], i * 64, r0, e);
        }
        tma_load_2d(st + C::kABytes, &tmB, &full[s], i * 64, pos0);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      for (int i = 0; i < nkt; ++i) {
        const int s = i % S;
        if (!mbar_wait(&full[s], (i / S) & 1, abort_flag, 72)) break;
        tc_fence_after();
        const uint8_t* st = smem + s * C::kStageBytes;
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          const uint64_t bd = umma_desc_k128(st + C::kABytes, k * 32);
          umma_f16(tmem, umma_desc_k128(st, k * 32), bd, kIdesc, i > 0 || k > 0);
          if (MODE == 1) umma_f16(tmem + C::kAcc, umma_desc_k128(st + 128 * 128, k * 32), bd, kIdesc, i > 0 || k > 0);
        }
        umma_commit(&empty[s]);
      }
      umma_commit(tfull);
    }
  } else {
    const int q = warp & 3;
    const uint32_t d0 = tmem + ((uint32_t)(q * 32) << 16);
    const int orow = r0 + q * 32 + lane;
    if (mbar_wait<64>(tfull, 0, abort_flag, 73)) {
      tc_fence_after();
#pragma unroll 1
      for (int c0 = 0; c0 < NT; c0 += 16) {
        if (c0 >= cnt) break;
        uint32_t a[16], b[16];
        tmem_ld_32x16(d0 + c0, a);
        if (MODE == 1) tmem_ld_32x16(d0 + C::kAcc + c0, b);
        tmem_ld_wait();
        if (orow < g.N) {
#pragma unroll
          for (int c = 0; c < 16; ++c) {
            if (c0 + c >= cnt) break;
            float v = __uint_as_float(a[c]);
            size_t r = pos0 + c0 + c;
            if (MODE == 1)
              v = v / (1.f + expf(-v)) * __uint_as_float(b[c]);
            else
              r = g.sorted_route[r];
            out[r * g.ldo + orow] = f2bf(v);
          }
        }
      }
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
int launch_grouped(const CUtensorMap& tmA, const void* xs, void* out, const GroupedArgs& g, cudaStream_t st) {
  using C = GroupedCfg<NT, MODE>;
  CUtensorMap tmB;
  if (dsv4_make_tmap_2d(&tmB, xs, 1, g.K, g.routes, (uint64_t)g.K * 2, 64, NT, 3)) return 642;
  auto kern = moe_bf16_gemm_kernel<NT, MODE>;
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, C::kSmem) != cudaSuccess) return 643;
    set = true;
  }
  dsv4_launch(kern, dim3((g.N + 127) / 128, g.max_tiles), 192, C::kSmem, st, tmA, tmB, (__nv_bfloat16*)out, g);
  return (int)cudaGetLastError();
}
template <int MODE>
int dispatch_grouped(int nt, const CUtensorMap& tmA, const void* xs, void* out, const GroupedArgs& g, cudaStream_t st) {
  switch (nt) {
    case 16: return launch_grouped<16, MODE>(tmA, xs, out, g, st);
    case 32: return launch_grouped<32, MODE>(tmA, xs, out, g, st);
    case 64: return launch_grouped<64, MODE>(tmA, xs, out, g, st);
    case 128: return launch_grouped<128, MODE>(tmA, xs, out, g, st);
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
                                int max_tiles, void* out, int experts, int N, int K, cudaStream_t st) {
  if (routes <= 0) return 0;
  if (K % 8 || max_tiles < 1 || max_tiles > 65535 || (mode != 1 && mode != 2)) return 645;
  CUtensorMap tmA;
  if (dsv4_make_tmap_3d(&tmA, w, K, N, (uint64_t)experts * (mode == 1 ? 2 : 1), (uint64_t)K * 2, (uint64_t)N * K * 2, 64,
                        128))
    return 641;
  const int* tiles = plan + 4;
  const GroupedArgs g{plan, tiles, tiles + 3 * max_tiles, max_tiles, routes, experts, N, K, N};
  return mode == 1 ? dispatch_grouped<1>(nt, tmA, x, out, g, st) : dispatch_grouped<2>(nt, tmA, x, out, g, st);
}
