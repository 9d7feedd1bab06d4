// Projections on the CUDA cores: out = act(x w^T), true fp32 multiply-adds.  Two uses: models served in 32-bit floats
// (fp32 activations, the tensor cores have no such format), and bf16 operands whose rows do not start on 16 bytes and
// therefore cannot be fetched by TMA.  Plain, batched over column groups, or grouped by expert with the route plan of
// moe.cu (then the activation row of a route is x[route / a_div] and its result goes to out[route]).
#include "vec.cuh"

namespace {

constexpr int kTM = 64, kTN = 64, kTK = 16;

struct SimtArgs {
  int M, N, K, ldx, ldw, ldo;
  int a_col_pb, b_row_pb, out_col_pb;  // batch offsets: x columns, w rows, out columns
  int accumulate, act;
  // grouped by expert
  const int* plan_hdr;      // [0] tiles, [1] routes; null: plain
  const int* tiles;         // [max_tiles][3]: expert, first position, routes
  const int* sorted_route;  // position -> route
  int a_div, routes, experts;
  long long w_stride;       // elements between the weights of two experts
};

template <typename TX, typename TO>
__global__ void __launch_bounds__(256) simt_gemm_kernel(const TX* __restrict__ x, const __nv_bfloat16* __restrict__ w,
                                                        TO* __restrict__ out, const SimtArgs g) {
  pdl_entry();
  __shared__ float as[kTK][kTM + 4];
  __shared__ float bs[kTK][kTN + 4];
  const int n0 = blockIdx.x * kTN, batch = blockIdx.z, tid = threadIdx.x;
  int rows, row0 = blockIdx.y * kTM;
  const __nv_bfloat16* wb = w;
  if (g.plan_hdr) {
    const int nt = g.plan_hdr[0];
    if ((int)blockIdx.y >= nt) return;
    const int e = g.tiles[blockIdx.y * 3];
    row0 = g.tiles[blockIdx.y * 3 + 1];
    rows = g.tiles[blockIdx.y * 3 + 2];
    if (e < 0 || e >= g.experts || row0 < 0 || rows > kTM || row0 + rows > g.routes) {  // a plan from other sizes
      if (tid == 0) dsv4_set_error(DSV4_ERR_BAD_INDEX, 51, e);
      return;
    }
    wb += (size_t)e * g.w_stride;
  } else {
    rows = min(kTM, g.M - row0);
  }
  wb += (size_t)batch * g.b_row_pb * g.ldw;
  // loader: thread -> one row of the tile, four consecutive k
  const int lr = tid >> 2, lk = (tid & 3) * 4;
  const TX* xr = nullptr;
  if (lr < rows) {
    int ar = row0 + lr;
    if (g.plan_hdr) ar = g.sorted_route[ar] / g.a_div;
    xr = x + (size_t)ar * g.ldx + (size_t)batch * g.a_col_pb;
  }
  const __nv_bfloat16* wr = n0 + lr < g.N ? wb + (size_t)(n0 + lr) * g.ldw : nullptr;
  const int tm = (tid >> 4) * 4, tn = (tid & 15) * 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < g.K; k0 += kTK) {
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int k = k0 + lk + j;
      as[lk + j][lr] = (xr && k < g.K) ? ld_f(xr + k) : 0.f;
      bs[lk + j][lr] = (wr && k < g.K) ? bf2f(wr[k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kTK; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&as[k][tm]);
      const float4 b = *reinterpret_cast<const float4*>(&bs[k][tn]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    if (tm + i >= rows) continue;
    int orow = row0 + tm + i;
    if (g.plan_hdr) orow = g.sorted_route[orow];
    TO* o = out + (size_t)orow * g.ldo + (size_t)batch * g.out_col_pb;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tn + j;
      if (n >= g.N) continue;
      float v = gemm_act(acc[i][j], g.act);
      if (g.accumulate) v += ld_f(o + n);
      st_f(o + n, v);
    }
  }
}

template <typename TX>
int launch_simt(const void* x, const void* w, void* out, const SimtArgs& g, int out_fp32, int grid_y, int batches,
                cudaStream_t st) {
  const dim3 grid((g.N + kTN - 1) / kTN, grid_y, batches);
  if (out_fp32)
    dsv4_launch(simt_gemm_kernel<TX, float>, grid, 256, 0, st, (const TX*)x, (const __nv_bfloat16*)w, (float*)out, g);
  else
    dsv4_launch(simt_gemm_kernel<TX, __nv_bfloat16>, grid, 256, 0, st, (const TX*)x, (const __nv_bfloat16*)w,
                (__nv_bfloat16*)out, g);
  return (int)cudaGetLastError();
}

}  // namespace

// x (bf16 or fp32) [M, K], w bf16 [N, K], out bf16 or fp32; batches and act as in dsv4_gemm_bf16.
DSV4_API int dsv4_gemm_simt(const void* x, const void* w, void* out, int M, int N, int K, int ldx, int ldw, int ldo,
                            int x_fp32, int out_fp32, int accumulate, int act, int batches, cudaStream_t st) {
  if (M <= 0 || N <= 0) return 0;
  if ((M + kTM - 1) / kTM > 65535) return 610;
  const SimtArgs g{M, N, K, ldx, ldw, ldo, K, N, N, accumulate, act, nullptr, nullptr, nullptr, 1, 0, 0, 0};
  const int b = batches < 1 ? 1 : batches;
  return x_fp32 ? launch_simt<float>(x, w, out, g, out_fp32, (M + kTM - 1) / kTM, b, st)
                : launch_simt<__nv_bfloat16>(x, w, out, g, out_fp32, (M + kTM - 1) / kTM, b, st);
}

// Grouped by expert: plan is the buffer of dsv4_moe_plan (built with 64 routes per tile), w bf16 [experts, N, K].
DSV4_API int dsv4_moe_gemm_simt(const void* x, const void* w, void* out, const int* plan, int routes, int max_tiles,
                                int experts, int N, int K, int a_div, int fp32, cudaStream_t st) {
  if (routes <= 0 || N <= 0) return 0;
  if (max_tiles > 65535) return 611;
  const int* tiles = plan + 4;
  const int* sorted = tiles + 3 * max_tiles;
  const SimtArgs g{routes, N, K, K, K, N, 0, 0, 0, 0, 0, plan, tiles, sorted, a_div, routes, experts, (long long)N * K};
  return fp32 ? launch_simt<float>(x, w, out, g, 1, max_tiles, 1, st)
              : launch_simt<__nv_bfloat16>(x, w, out, g, 0, max_tiles, 1, st);
}
