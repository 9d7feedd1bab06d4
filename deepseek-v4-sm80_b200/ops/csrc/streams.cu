// Residual streams with constant mixing weights (hyper-connections) of models that keep them in 32-bit floats: a layer reads a
// weighted sum of the streams, and its output goes back into all of them while they mix.
//
//   y   = sub + sum_k w_k e_k + w_id h        (sub-layer: a projection's output, chosen experts, experts that pass h on)
//   x_t <- sum_s mix[s, t] x_s + out[t] y     (all streams at once, from the old ones)
//   u   = sum_s in[s] x_s,   h' = u / rms(u) * gain
//
// One kernel does the three lines between two sub-layers, so every stream is read and written once per sub-layer.  x is
// [rows][streams][d]; a thread owns whole coordinates (of all streams), which makes the update safe in place.
#include "vec.cuh"

namespace {

constexpr int kMaxStreams = 16;

struct StreamArgs {
  float* x;                   // [rows][streams][d], updated in place if keep
  const long long* rows_idx;  // not null: output row r belongs to token rows_idx[r], and the streams are left alone
  const float* post;          // out [streams] | mix [from][to]; null: nothing comes in
  const float* sub;           // [rows][d] or null
  const float* wts;           // [rows][topk] weights of the chosen experts
  const int* eidx;            // [rows][topk]: expert ids; negative: none, n_experts and up: the input h itself
  int topk, n_experts;        // topk 0: no experts
  const float* pre;           // in [streams] | gain; null: no output
  float eps;
  int streams, d, keep;
};

__device__ __forceinline__ void fma4(float4& a, float w, const float4& v) {
  a.x = fmaf(w, v.x, a.x), a.y = fmaf(w, v.y, a.y), a.z = fmaf(w, v.z, a.z), a.w = fmaf(w, v.w, a.w);
}

// S streams (0: any number up to kMaxStreams), NT threads, NV x 4 coordinates per thread; NV = 0: any d, one coordinate at a time
// and u in shared memory.
template <typename T, int S, int NV, int NT>
__global__ void __launch_bounds__(NT, S > 0 && NV == 1 ? 1024 / NT : 1) stream_norm_kernel(const StreamArgs a, const T* __restrict__ erows,
                                                          const T* __restrict__ h, T* __restrict__ out) {
  pdl_entry();
  constexpr int SM = S ? S : kMaxStreams;
  __shared__ float sh[32], post[kMaxStreams * (kMaxStreams + 1)], pre[kMaxStreams + 1], ew[32];
  __shared__ int ei[32];
  extern __shared__ float rest[];
  const int r = blockIdx.x, d = a.d, ns = S ? S : a.streams;
  const size_t tok = a.rows_idx ? (size_t)a.rows_idx[r] : r;
  for (int i = threadIdx.x; a.post && i < ns * (ns + 1); i += NT) post[i] = a.post[i];
  for (int i = threadIdx.x; a.pre && i <= ns; i += NT) pre[i] = a.pre[i];
  if ((int)threadIdx.x < a.topk) {
    const int e = a.eidx[tok * a.topk + threadIdx.x];
    ei[threadIdx.x] = e, ew[threadIdx.x] = e < 0 ? 0.f : a.wts[tok * a.topk + threadIdx.x];
  }
  __syncthreads();
  float w_id = 0.f;           // weight of the input itself
  for (int k = 0; k < a.topk; ++k)
    if (ei[k] >= a.n_experts) w_id += ew[k];
  float* x = a.x + tok * ns * d;
  const T *er = erows + tok * a.topk * d, *hr = h + tok * d;
  float ss = 0.f;
  if constexpr (NV > 0) {
    float4 u[NV];
#pragma unroll
    for (int n = 0; n < NV; ++n) {
      const int i = (n * NT + (int)threadIdx.x) * 4;
      u[n] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (i >= d) continue;
      float4 s[SM];
#pragma unroll
      for (int j = 0; j < SM; ++j)
        if (S || j < ns) s[j] = ld_f4(x + (size_t)j * d + i);
      if (a.post) {
        float4 y = a.sub ? ld_f4(a.sub + tok * d + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        if (a.topk) {
          const float4 id = w_id != 0.f ? ld_f4(hr + i) : make_float4(0.f, 0.f, 0.f, 0.f);
          for (int k0 = 0; k0 < a.topk; k0 += 4) {         // four rows in flight
            float4 e[4];
#pragma unroll
            for (int k = 0; k < 4; ++k) {
              const bool runs = k0 + k < a.topk && (unsigned)ei[k0 + k] < (unsigned)a.n_experts;
              e[k] = runs ? ld_f4(er + (size_t)(k0 + k) * d + i) : make_float4(0.f, 0.f, 0.f, 0.f);
            }
#pragma unroll
            for (int k = 0; k < 4; ++k)
              if (k0 + k < a.topk) fma4(y, ew[k0 + k], e[k]);
          }
          fma4(y, w_id, id);
        }
#pragma unroll
        for (int j = 0; j < SM; ++j) {
          if (!S && j >= ns) continue;
          const float o = post[j];
          float4 t = make_float4(o * y.x, o * y.y, o * y.z, o * y.w);
#pragma unroll
          for (int q = 0; q < SM; ++q)
            if (S || q < ns) fma4(t, post[ns + q * ns + j], s[q]);
          if (a.keep) st_f4(x + (size_t)j * d + i, t);
          if (a.pre) fma4(u[n], pre[j], t);
        }
      } else if (a.pre) {
#pragma unroll
        for (int j = 0; j < SM; ++j)
          if (S || j < ns) fma4(u[n], pre[j], s[j]);
      }
      ss += (u[n].x * u[n].x + u[n].y * u[n].y) + (u[n].z * u[n].z + u[n].w * u[n].w);
    }
    if (!a.pre) return;
    const float sc = pre[ns] / sqrtf(cta_sum(ss, sh) / d + a.eps);
#pragma unroll
    for (int n = 0; n < NV; ++n) {
      const int i = (n * NT + (int)threadIdx.x) * 4;
      if (i < d) st_f4(out + (size_t)r * d + i, make_float4(u[n].x * sc, u[n].y * sc, u[n].z * sc, u[n].w * sc));
    }
  } else {
    for (int i = threadIdx.x; i < d; i += NT) {
      float s[SM], u = 0.f;
#pragma unroll
      for (int j = 0; j < SM; ++j)
        if (S || j < ns) s[j] = x[(size_t)j * d + i];
      if (a.post) {
        float y = a.sub ? a.sub[tok * d + i] : 0.f;
        for (int k = 0; k < a.topk; ++k)
          if ((unsigned)ei[k] < (unsigned)a.n_experts) y = fmaf(ew[k], ld_f(er + (size_t)k * d + i), y);
        if (w_id != 0.f) y = fmaf(w_id, ld_f(hr + i), y);
        for (int j = 0; j < ns; ++j) {
          float t = post[j] * y;
#pragma unroll
          for (int q = 0; q < SM; ++q)
            if (S || q < ns) t = fmaf(post[ns + q * ns + j], s[q], t);
          if (a.keep) x[(size_t)j * d + i] = t;
          if (a.pre) u = fmaf(pre[j], t, u);
        }
      } else if (a.pre) {
#pragma unroll
        for (int j = 0; j < SM; ++j)
          if (S || j < ns) u = fmaf(pre[j], s[j], u);
      }
      if (a.pre) rest[i] = u;
      ss += u * u;
    }
    if (!a.pre) return;
    const float sc = pre[ns] / sqrtf(cta_sum(ss, sh) / d + a.eps);
    for (int i = threadIdx.x; i < d; i += NT) st_f(out + (size_t)r * d + i, rest[i] * sc);   // what the thread wrote itself
  }
}

template <typename T, int S>
int launch_streams(const StreamArgs& a, const void* erows, const void* h, void* out, int rows, cudaStream_t st) {
  auto go = [&](auto kern, int threads, size_t smem) {
    dsv4_launch(kern, rows, threads, smem, st, a, (const T*)erows, (const T*)h, (T*)out);
  };
  if (a.d % 4 || a.d > 8192) {
    if (a.d > 8192 + 2048) return 611;       // u in 40 KB of shared memory
    go(stream_norm_kernel<T, S, 0, 256>, 256, (size_t)a.d * 4);
  } else if (a.d <= 1024)
    go(stream_norm_kernel<T, S, 1, 256>, 256, 0);
  else if (a.d <= 2048)
    go(stream_norm_kernel<T, S, 1, 512>, 512, 0);
  else if (a.d <= 4096)
    go(stream_norm_kernel<T, S, 2, 512>, 512, 0);
  else
    go(stream_norm_kernel<T, S, 4, 512>, 512, 0);
  return (int)cudaGetLastError();
}
template <typename T>
int dispatch_streams(const StreamArgs& a, const void* erows, const void* h, void* out, int rows, cudaStream_t st) {
  switch (a.streams) {
    case 1: return launch_streams<T, 1>(a, erows, h, out, rows, st);
    case 2: return launch_streams<T, 2>(a, erows, h, out, rows, st);
    case 3: return launch_streams<T, 3>(a, erows, h, out, rows, st);
    case 4: return launch_streams<T, 4>(a, erows, h, out, rows, st);
    default: return launch_streams<T, 0>(a, erows, h, out, rows, st);
  }
}

}  // namespace

// See StreamArgs.  erows [rows * topk, d] and h [rows, d]: activations (fp32: their type), needed when topk > 0; out [n, d] for
// pre.  rows: output rows (rows_idx given: n of them, keep must be 0).
DSV4_API int dsv4_stream_norm(float* x, const long long* rows_idx, const float* post, const float* sub, const void* erows,
                              const float* wts, const int* eidx, int topk, int n_experts, const void* h, const float* pre,
                              float eps, int keep, void* out, int rows, int streams, int d, int fp32, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (streams < 1 || streams > kMaxStreams || topk < 0 || topk > 32) return 612;
  if ((rows_idx && keep) || (pre && !out) || (topk > 0 && (!erows || !wts || !eidx || !h))) return 613;
  const StreamArgs a{x, rows_idx, post, sub, wts, eidx, topk, n_experts, pre, eps, streams, d, keep};
  return fp32 ? dispatch_streams<float>(a, erows, h, out, rows, st)
              : dispatch_streams<__nv_bfloat16>(a, erows, h, out, rows, st);
}
