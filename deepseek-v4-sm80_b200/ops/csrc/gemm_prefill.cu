// bf16 projections of many rows:  out[M,N] = act(X[M,K] W[N,K]^T), the persistent counterpart of gemm_tcgen05.cu for
// problems with at least about one 128 x 256 tile per SM.  One CTA per SM walks the output tiles; the accumulator is double
// buffered in tensor memory (2 x 256 columns), so a tile's epilogue runs under the next tile's MMAs.
//   warp 0 TMA producer (4 stages of 64 K elements), warp 1 tcgen05.mma issuer, warps 2-5 epilogue
// Batches as in gemm_tcgen05.cu (batch b: A columns b K .., W rows b N .., output columns b N ..).
#include "vec.cuh"

namespace {

constexpr int kPM = 128, kPN = 256, kPStages = 4;
constexpr int kPA = kPM * 128, kPB = kPN * 128, kPStage = kPA + kPB;
constexpr int kPSmem = kPStages * kPStage + 1024 + 256;
constexpr int kGroupM = 16;   // row tiles that share a column of weight tiles before the next column

struct BigArgs {
  int M, N, K, ldo, batches, accumulate, act;
  float limit;          // of kActClampGate
  int mt, nt;
};

__device__ __forceinline__ void big_tile(const BigArgs& g, int id, int& m, int& n, int& b) {
  const int per = g.mt * g.nt;
  b = id / per;
  const int r = id % per, gid = r / (kGroupM * g.nt), m_first = gid * kGroupM;
  const int rows = min(kGroupM, g.mt - m_first), in = r - gid * kGroupM * g.nt;
  m = m_first + in % rows;
  n = in / rows;
}

template <typename OutT>
__global__ void __launch_bounds__(192, 1) gemm_prefill_kernel(const __grid_constant__ CUtensorMap tmA,
                                                              const __grid_constant__ CUtensorMap tmB,
                                                              OutT* __restrict__ out, const BigArgs g) {
  extern __shared__ uint8_t bsm_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(bsm_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + kPStages * kPStage);
  uint64_t *empty = full + kPStages, *tfull = empty + kPStages, *tempty = tfull + 2;
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(tempty + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_holder + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int i = 0; i < kPStages; ++i) mbar_init(&full[i], 1), mbar_init(&empty[i], 1);
    for (int i = 0; i < 2; ++i) mbar_init(&tfull[i], 1), mbar_init(&tempty[i], 4);
    *abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tmA);
    tma_prefetch_desc(&tmB);
  }
  if (warp == 1) {
    tmem_alloc(tmem_holder, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_holder;
  pdl_wait();
  pdl_launch_dependents();
  const int total = g.mt * g.nt * g.batches, nkt = (g.K + 63) / 64;

  if (warp == 0) {
    if (lane == 0) {
      int i = 0;
      bool ok = true;
      for (int id = blockIdx.x; id < total && ok; id += gridDim.x) {
        int m, n, b;
        big_tile(g, id, m, n, b);
        for (int k = 0; k < nkt; ++k, ++i) {
          const int s = i % kPStages;
          if (i >= kPStages && !mbar_wait<20>(&empty[s], ((i / kPStages) & 1) ^ 1, abort_flag, 91)) { ok = false; break; }
          uint8_t* st = smem + s * kPStage;
          mbar_expect_tx(&full[s], kPStage);
          tma_load_2d(st, &tmA, &full[s], b * g.K + k * 64, m * kPM);
          tma_load_2d(st + kPA, &tmB, &full[s], k * 64, b * g.N + n * kPN);
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t kIdesc = umma_idesc(128, kPN, 1, 1);
      int i = 0, it = 0;
      bool ok = true;
      for (int id = blockIdx.x; id < total && ok; id += gridDim.x, ++it) {
        const int acc = it & 1;
        if (it >= 2 && !mbar_wait(&tempty[acc], ((it >> 1) & 1) ^ 1, abort_flag, 92)) break;
        tc_fence_after();
        for (int k = 0; k < nkt; ++k, ++i) {
          const int s = i % kPStages;
          if (!mbar_wait(&full[s], (i / kPStages) & 1, abort_flag, 93)) { ok = false; break; }
          tc_fence_after();
          const uint8_t* st = smem + s * kPStage;
#pragma unroll
          for (int j = 0; j < 4; ++j)
            umma_f16(tmem + acc * kPN, umma_desc_k128(st, j * 32), umma_desc_k128(st + kPA, j * 32), kIdesc, k > 0 || j > 0);
          umma_commit(&empty[s]);
        }
        if (ok) umma_commit(&tfull[acc]);
      }
    }
  } else {
    const int q = warp & 3;
    int it = 0;
    for (int id = blockIdx.x; id < total; id += gridDim.x, ++it) {
      const int acc = it & 1;
      int m, n, b;
      big_tile(g, id, m, n, b);
      if (!mbar_wait<40>(&tfull[acc], (it >> 1) & 1, abort_flag, 94)) break;
      tc_fence_after();
      const int row = m * kPM + q * 32 + lane;
      const uint32_t d0 = tmem + acc * kPN + ((uint32_t)(q * 32) << 16);
      const bool gated = gated_act(g.act);
      OutT* dst = out + (size_t)row * g.ldo + (gated ? (size_t)n * (kPN / 2) : (size_t)b * g.N + n * kPN);
      const int cols = min(kPN, g.N - n * kPN);
      const bool vec = ((uintptr_t)dst & 15) == 0;
#pragma unroll 1
      for (int c = 0; c < cols; c += 32) {
        uint32_t r[32];
        tmem_ld_32x32(d0 + c, r);
        tmem_ld_wait();
        if (row >= g.M) continue;
        float v[32];
#pragma unroll
        for (int j = 0; j < 32; ++j) v[j] = __uint_as_float(r[j]);
        if (gated) {
          gate_block(v, g.act, g.limit);
          st_f16x(dst + c / 2, v);
          continue;
        }
        if (g.act) {
#pragma unroll
          for (int j = 0; j < 32; ++j) v[j] = gemm_act(v[j], g.act);
        }
        if (vec && cols - c >= 32) {
          if (g.accumulate) {
            float4 o[8];
#pragma unroll
            for (int j = 0; j < 8; ++j) o[j] = ld_f4(dst + c + 4 * j);
#pragma unroll
            for (int j = 0; j < 8; ++j) v[4 * j] += o[j].x, v[4 * j + 1] += o[j].y, v[4 * j + 2] += o[j].z, v[4 * j + 3] += o[j].w;
          }
          if constexpr (sizeof(OutT) == 4) {
#pragma unroll
            for (int j = 0; j < 8; ++j) st_f4(dst + c + 4 * j, make_float4(v[4 * j], v[4 * j + 1], v[4 * j + 2], v[4 * j + 3]));
          } else {
#pragma unroll
            for (int j = 0; j < 4; ++j) {
              uint4 u;
              __nv_bfloat162* p = reinterpret_cast<__nv_bfloat162*>(&u);
#pragma unroll
              for (int e = 0; e < 4; ++e) p[e] = __floats2bfloat162_rn(v[8 * j + 2 * e], v[8 * j + 2 * e + 1]);
              reinterpret_cast<uint4*>(dst + c)[j] = u;
            }
          }
        } else {
#pragma unroll
          for (int j = 0; j < 32; ++j)
            if (c + j < cols) {
              if (g.accumulate) v[j] += ld_f(dst + c + j);
              st_f(dst + c + j, v[j]);
            }
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&tempty[acc]);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem, 512);
}

template <typename OutT>
int launch_big(const CUtensorMap& a, const CUtensorMap& b, void* out, const BigArgs& g, int sms, cudaStream_t st) {
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(gemm_prefill_kernel<OutT>, cudaFuncAttributeMaxDynamicSharedMemorySize, kPSmem) != cudaSuccess)
      return 663;
    set = true;
  }
  const int total = g.mt * g.nt * g.batches;
  dsv4_launch(gemm_prefill_kernel<OutT>, total < sms ? total : sms, 192, kPSmem, st, a, b, (OutT*)out, g);
  return (int)cudaGetLastError();
}

}  // namespace

DSV4_API int dsv4_gemm_prefill(const void* x, const void* w, void* out, int M, int N, int K, int ldx, int ldw, int ldo,
                               int out_fp32, int accumulate, int act, float limit, int batches, int sms, cudaStream_t st) {
  if (M <= 0 || N <= 0) return 0;
  if (K % 8 || ldx % 8 || ldw % 8 || batches < 1 || sms < 1) return 660;
  if (gated_act(act) && (N % 32 || ldo % 16 || batches != 1 || accumulate)) return 664;
  CUtensorMap ta, tb;
  if (dsv4_make_tmap_2d(&ta, x, 1, (uint64_t)K * batches, M, (uint64_t)ldx * 2, 64, kPM, 3)) return 661;
  if (dsv4_make_tmap_2d(&tb, w, 1, K, (uint64_t)N * batches, (uint64_t)ldw * 2, 64, kPN, 3)) return 662;
  const BigArgs g{M, N, K, ldo, batches, accumulate, act, limit, (M + kPM - 1) / kPM, (N + kPN - 1) / kPN};
  return out_fp32 ? launch_big<float>(ta, tb, out, g, sms, st) : launch_big<__nv_bfloat16>(ta, tb, out, g, sms, st);
}
