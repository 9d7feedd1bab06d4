// The residual stream of models that keep it in 32-bit floats: embedding gather, and RMSNorm fused with whatever is
// added to the stream right before it (a projection's output, a learned vector, the weighted outputs of the chosen
// experts).  T is the activation type the next projection reads (bf16, or fp32 for models served in 32-bit).
#include "vec.cuh"

namespace {

// x[t] = embed[id] * mul (+ pos_w[pos[t]]) (+ pair_w[row of the token and the one before it]), `copies` times side by side,
// also as activations (x0, may be null).  feedback as in embed_kernel: the token of row t is feedback[slots[t]] and is written to
// ids[t].
struct EmbedArgs {
  float mul;
  const __nv_bfloat16* pos_w;   // [n_pos][d] learned position vectors, or null
  const int* pos;
  int n_pos, copies, d;
  // A vector per pair of tokens: row (before * mul_before + id * mul_id) mod buckets, row `buckets` at the start of a sequence.
  // tokens: the cached sequences' tokens by location; every row adds its own.
  const __nv_bfloat16* pair_w;  // [buckets + 1][d] or null
  unsigned buckets, mul_before, mul_id;      // the factors are below buckets
  int* tokens;
  const int* out_loc;
  const int* page_table;
  int ld_pt;
};
template <typename T>
__global__ void __launch_bounds__(256) embed_residual_kernel(int* __restrict__ ids, const int* __restrict__ feedback,
                                                             const int* __restrict__ slots,
                                                             const __nv_bfloat16* __restrict__ w,
                                                             float* __restrict__ x, T* __restrict__ x0, const EmbedArgs a) {
  pdl_entry();
  const int d = a.d;
  const int t = blockIdx.x;
  int id;
  if (feedback) {
    id = feedback[slots[t]];
    if (threadIdx.x == 0) ids[t] = id;
  } else {
    id = ids[t];
  }
  const __nv_bfloat16* src = w + (size_t)id * d;
  const __nv_bfloat16* at = nullptr;
  if (a.pos_w) {
    const int p = a.pos[t];
    if (p >= a.n_pos && threadIdx.x == 0) dsv4_set_error(DSV4_ERR_BAD_INDEX, 60, p);
    at = a.pos_w + (size_t)min(p, a.n_pos - 1) * d;
  }
  const __nv_bfloat16* pair = nullptr;
  if (a.pair_w) {
    const int p = a.pos[t], slot = slots[t], loc = a.out_loc[t];
    unsigned row = a.buckets;
    if (p > 0) {
      // rows of one request stand together; what an earlier forward ran is in the cache (decode rows only have that)
      const bool here = !feedback && t > 0 && slots[t - 1] == slot && a.pos[t - 1] + 1 == p;
      const int before = here ? ids[t - 1] : a.tokens[a.page_table[(size_t)slot * a.ld_pt + p - 1]];
      row = (unsigned)(((unsigned long long)before * a.mul_before + (unsigned long long)id * a.mul_id) % a.buckets);
    }
    pair = a.pair_w + (size_t)row * d;
    if (threadIdx.x == 0 && loc >= 0) a.tokens[loc] = id;
  }
  if (d % 4 == 0) {
    for (int i = threadIdx.x * 4; i < d; i += blockDim.x * 4) {
      float4 v = ld_f4(src + i);
      v.x *= a.mul, v.y *= a.mul, v.z *= a.mul, v.w *= a.mul;
      if (at) {
        const float4 p = ld_f4(at + i);
        v.x += p.x, v.y += p.y, v.z += p.z, v.w += p.w;
      }
      if (pair) {
        const float4 p = ld_f4(pair + i);
        v.x += p.x, v.y += p.y, v.z += p.z, v.w += p.w;
      }
      for (int c = 0; c < a.copies; ++c) st_f4(x + ((size_t)t * a.copies + c) * d + i, v);
      if (x0) st_f4(x0 + (size_t)t * d + i, v);
    }
    return;
  }
  for (int i = threadIdx.x; i < d; i += blockDim.x) {
    const float v = bf2f(src[i]) * a.mul + (at ? bf2f(at[i]) : 0.f) + (pair ? bf2f(pair[i]) : 0.f);
    for (int c = 0; c < a.copies; ++c) x[((size_t)t * a.copies + c) * d + i] = v;
    if (x0) st_f(x0 + (size_t)t * d + i, v);
  }
}

struct NormArgs {
  float* x;             // [rows, d] stream (row stride d), updated in place when something is added
  const long long* rows_idx;  // not null: output row r belongs to stream row rows_idx[r] (only `sub` may be added then, and the
                              // stream is left alone)
  const float* sub;     // a sub-layer's output [rows, d]: (sub + sub_bias) / rms * sub_gain is added first; or null
  const float* sub_bias;      // [d] or null
  const float* sub_gain;      // [d]
  const float* add;     // [rows, d] or null
  const float* add2;    // [rows, d] or null
  const float* vec;     // [d] or null
  const float* wts;     // [rows, topk]: weights of the expert rows below
  const int* eidx;      // [rows, topk]: expert ids, negative = no expert ran for this place
  int topk;             // 0: no expert rows
  const float* gain;    // [d]; null: no norm, only the additions (out, if given, receives the sum as activations)
  float eps, mul;       // out = x / rms(x) * gain * mul
  int d;
};

// One CTA per row.  NV > 0: the row stays in registers between the two passes, NV x 4 values per thread.
template <typename T, int NV>
__global__ void __launch_bounds__(256) residual_norm_kernel(const NormArgs a, const T* __restrict__ erows,
                                                            T* __restrict__ out) {
  pdl_entry();
  __shared__ float sh[32];
  const int r = blockIdx.x, d = a.d;
  const size_t src = (size_t)(a.rows_idx ? a.rows_idx[r] : r) * d;
  const bool adds = a.sub || a.add || a.add2 || a.vec || a.topk > 0;
  float ss = 0.f;
  if constexpr (NV > 0) {
    float4 keep[NV];
    float4 y[NV];
#pragma unroll
    for (int n = 0; n < NV; ++n) {          // everything in flight before the first sum
      const int i = (n * 256 + threadIdx.x) * 4;
      if (i >= d) continue;
      keep[n] = ld_f4(a.x + src + i);
      if (a.sub) y[n] = ld_f4(a.sub + src + i);
    }
    float sub_sc = 0.f;
    if (a.sub) {
      float s2 = 0.f;
#pragma unroll
      for (int n = 0; n < NV; ++n) {
        const int i = (n * 256 + threadIdx.x) * 4;
        if (i >= d) continue;
        if (a.sub_bias) {
          const float4 u = ld_f4(a.sub_bias + i);
          y[n].x += u.x, y[n].y += u.y, y[n].z += u.z, y[n].w += u.w;
        }
        s2 += y[n].x * y[n].x + y[n].y * y[n].y + y[n].z * y[n].z + y[n].w * y[n].w;
      }
      sub_sc = 1.f / sqrtf(cta_sum(s2, sh) / d + a.eps);
    }
#pragma unroll
    for (int n = 0; n < NV; ++n) {
      const int i = (n * 256 + threadIdx.x) * 4;
      if (i >= d) continue;
      float4 v = keep[n];
      if (adds) {
        if (a.sub) {
          const float4 g = ld_f4(a.sub_gain + i);
          v.x += y[n].x * sub_sc * g.x, v.y += y[n].y * sub_sc * g.y, v.z += y[n].z * sub_sc * g.z, v.w += y[n].w * sub_sc * g.w;
        }
        if (a.add) {
          const float4 u = *reinterpret_cast<const float4*>(a.add + src + i);
          v.x += u.x, v.y += u.y, v.z += u.z, v.w += u.w;
        }
        if (a.add2) {
          const float4 u = *reinterpret_cast<const float4*>(a.add2 + src + i);
          v.x += u.x, v.y += u.y, v.z += u.z, v.w += u.w;
        }
        if (a.vec) {
          const float4 u = *reinterpret_cast<const float4*>(a.vec + i);
          v.x += u.x, v.y += u.y, v.z += u.z, v.w += u.w;
        }
        if (a.topk > 0) {
          float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
          for (int k = 0; k < a.topk; ++k) {
            if (a.eidx[r * a.topk + k] < 0) continue;
            const float w = a.wts[r * a.topk + k];
            const float4 u = ld_f4(erows + ((size_t)r * a.topk + k) * d + i);
            s.x += w * u.x, s.y += w * u.y, s.z += w * u.z, s.w += w * u.w;
          }
          v.x += s.x, v.y += s.y, v.z += s.z, v.w += s.w;
        }
        if (!a.rows_idx) *reinterpret_cast<float4*>(a.x + src + i) = v;
      }
      keep[n] = v;
      if (!a.gain && out) st_f4(out + (size_t)r * d + i, v);
      ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    if (!a.gain) return;
    ss = cta_sum(ss, sh);
    const float sc = a.mul / sqrtf(ss / d + a.eps);
#pragma unroll
    for (int n = 0; n < NV; ++n) {
      const int i = (n * 256 + threadIdx.x) * 4;
      if (i >= d) continue;
      const float4 g = *reinterpret_cast<const float4*>(a.gain + i);
      st_f4(out + (size_t)r * d + i,
            make_float4(keep[n].x * sc * g.x, keep[n].y * sc * g.y, keep[n].z * sc * g.z, keep[n].w * sc * g.w));
    }
  } else {
    extern __shared__ float row[];      // d floats if there is a sub: the sum, which the stream does not always take
    float sub_sc = 0.f;
    if (a.sub) {
      float s2 = 0.f;
      for (int i = threadIdx.x; i < d; i += 256) {
        const float v = a.sub[src + i] + (a.sub_bias ? a.sub_bias[i] : 0.f);
        s2 += v * v;
      }
      sub_sc = 1.f / sqrtf(cta_sum(s2, sh) / d + a.eps);
    }
    for (int i = threadIdx.x; i < d; i += 256) {
      float v = a.x[src + i];
      if (adds) {
        if (a.sub) v += (a.sub[src + i] + (a.sub_bias ? a.sub_bias[i] : 0.f)) * sub_sc * a.sub_gain[i];
        if (a.add) v += a.add[src + i];
        if (a.add2) v += a.add2[src + i];
        if (a.vec) v += a.vec[i];
        float s = 0.f;
        for (int k = 0; k < a.topk; ++k)
          if (a.eidx[r * a.topk + k] >= 0)
            s += a.wts[r * a.topk + k] * ld_f(erows + ((size_t)r * a.topk + k) * d + i);
        v += s;
        if (!a.rows_idx) a.x[src + i] = v;
        if (a.sub) row[i] = v;
      }
      if (!a.gain && out) st_f(out + (size_t)r * d + i, v);
      ss += v * v;
    }
    if (!a.gain) return;
    ss = cta_sum(ss, sh);
    const float sc = a.mul / sqrtf(ss / d + a.eps);
    for (int i = threadIdx.x; i < d; i += 256)  // each thread re-reads what it wrote itself
      st_f(out + (size_t)r * d + i, (a.sub ? row[i] : a.x[src + i]) * sc * a.gain[i]);
  }
}

// silu(gate) * up: gu [rows, 2 f] (gate columns first) -> out [rows, f]
template <typename T>
__global__ void __launch_bounds__(256) silu_mul_kernel(const T* __restrict__ gu, T* __restrict__ out, long long total,
                                                       int f) {
  pdl_entry();
  const long long i = blockIdx.x * 256ll + threadIdx.x;
  if (i >= total) return;
  const long long r = i / f;
  const int c = (int)(i % f);
  const float g = ld_f(gu + r * 2 * f + c), u = ld_f(gu + r * 2 * f + f + c);
  st_f(out + i, g / (1.f + expf(-g)) * u);
}

// ------------------------------------------------------------------ layer norms around the sub-layers
struct LayerNormArgs {
  float* x;                   // [rows, d] stream, updated in place if keep
  const long long* rows_idx;  // not null: output row r belongs to stream row rows_idx[r], and the stream is left alone
  const float *sub, *sub_w, *sub_b;  // a sub-layer's output [rows, d], normed and added; or null
  const void* add;            // activations [rows, d], added; or null
  const float *w, *b;         // norm of the sum; null: no output
  float eps;
  int d, keep;
};

// Mean and 1 / standard deviation of a row of d values of which this thread holds NV x 4 (or walks every 256th); two passes:
// the deviations are summed around the mean itself.
template <int NV>
__device__ __forceinline__ float2 row_stats(const float4 (&v)[NV], int d, float eps, float* sh) {
  float s = 0.f;
#pragma unroll
  for (int n = 0; n < NV; ++n)
    if ((n * 256 + (int)threadIdx.x) * 4 < d) s += (v[n].x + v[n].y) + (v[n].z + v[n].w);
  const float mean = cta_sum(s, sh) / d;
  float q = 0.f;
#pragma unroll
  for (int n = 0; n < NV; ++n)
    if ((n * 256 + (int)threadIdx.x) * 4 < d) {
      const float a = v[n].x - mean, b = v[n].y - mean, c = v[n].z - mean, e = v[n].w - mean;
      q += (a * a + b * b) + (c * c + e * e);
    }
  return make_float2(mean, 1.f / sqrtf(cta_sum(q, sh) / d + eps));
}
__device__ __forceinline__ float4 norm4(const float4& v, const float2& st, const float4& w, const float4& b) {
  return make_float4((v.x - st.x) * st.y * w.x + b.x, (v.y - st.x) * st.y * w.y + b.y, (v.z - st.x) * st.y * w.z + b.z,
                     (v.w - st.x) * st.y * w.w + b.w);
}

// x += N(sub; sub_w, sub_b);  x += add;  out = N(x; w, b).  One CTA per row, the row stays in registers (NV x 4 values per
// thread); NV = 0: any d, the sum passes through `out_row` in shared memory.
template <typename T, int NV>
__global__ void __launch_bounds__(256) residual_layer_norm_kernel(const LayerNormArgs a, T* __restrict__ out) {
  pdl_entry();
  __shared__ float sh[32];
  extern __shared__ float rest[];
  const int r = blockIdx.x, d = a.d;
  const size_t src = (size_t)(a.rows_idx ? a.rows_idx[r] : r) * d;
  const T* add = a.add ? static_cast<const T*>(a.add) + src : nullptr;
  if constexpr (NV > 0) {
    float4 x[NV], y[NV];
#pragma unroll
    for (int n = 0; n < NV; ++n) {
      const int i = (n * 256 + threadIdx.x) * 4;
      x[n] = y[n] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (i >= d) continue;
      x[n] = ld_f4(a.x + src + i);
      if (a.sub) y[n] = ld_f4(a.sub + src + i);
    }
    if (a.sub) {
      const float2 st = row_stats<NV>(y, d, a.eps, sh);
#pragma unroll
      for (int n = 0; n < NV; ++n) {
        const int i = (n * 256 + threadIdx.x) * 4;
        if (i >= d) continue;
        const float4 v = norm4(y[n], st, ld_f4(a.sub_w + i), ld_f4(a.sub_b + i));
        x[n].x += v.x, x[n].y += v.y, x[n].z += v.z, x[n].w += v.w;
      }
    }
#pragma unroll
    for (int n = 0; n < NV; ++n) {
      const int i = (n * 256 + threadIdx.x) * 4;
      if (i >= d) continue;
      if (add) {
        const float4 v = ld_f4(add + i);
        x[n].x += v.x, x[n].y += v.y, x[n].z += v.z, x[n].w += v.w;
      }
      if (a.keep) st_f4(a.x + src + i, x[n]);
    }
    if (!a.w) return;
    const float2 st = row_stats<NV>(x, d, a.eps, sh);
#pragma unroll
    for (int n = 0; n < NV; ++n) {
      const int i = (n * 256 + threadIdx.x) * 4;
      if (i < d) st_f4(out + (size_t)r * d + i, norm4(x[n], st, ld_f4(a.w + i), ld_f4(a.b + i)));
    }
  } else {
    auto stats = [&](const float* v) {
      float s = 0.f, q = 0.f;
      for (int i = threadIdx.x; i < d; i += 256) s += v[i];
      const float mean = cta_sum(s, sh) / d;
      for (int i = threadIdx.x; i < d; i += 256) q += (v[i] - mean) * (v[i] - mean);
      return make_float2(mean, 1.f / sqrtf(cta_sum(q, sh) / d + a.eps));
    };
    float2 st = make_float2(0.f, 0.f);
    if (a.sub) st = stats(a.sub + src);
    for (int i = threadIdx.x; i < d; i += 256) {   // every thread only reads back what it wrote itself
      float v = a.x[src + i];
      if (a.sub) v += (a.sub[src + i] - st.x) * st.y * a.sub_w[i] + a.sub_b[i];
      if (add) v += ld_f(add + i);
      if (a.keep) a.x[src + i] = v;
      rest[i] = v;
    }
    if (!a.w) return;
    st = stats(rest);
    for (int i = threadIdx.x; i < d; i += 256) st_f(out + (size_t)r * d + i, (rest[i] - st.x) * st.y * a.w[i] + a.b[i]);
  }
}

template <typename T>
int launch_layer_norm(const LayerNormArgs& a, void* out, int rows, cudaStream_t st) {
  auto go = [&](auto kern, size_t smem) { dsv4_launch(kern, rows, 256, smem, st, a, (T*)out); };
  if (a.d % 4 || a.d > 8192) {
    if (a.d > 11264) return 606;       // the row in 44 KB of shared memory
    go(residual_layer_norm_kernel<T, 0>, (size_t)a.d * 4);
  } else if (a.d <= 1024)
    go(residual_layer_norm_kernel<T, 1>, 0);
  else if (a.d <= 2048)
    go(residual_layer_norm_kernel<T, 2>, 0);
  else if (a.d <= 4096)
    go(residual_layer_norm_kernel<T, 4>, 0);
  else
    go(residual_layer_norm_kernel<T, 8>, 0);
  return (int)cudaGetLastError();
}

// gate(z) * up behind a projection without the gated epilogue: gu [rows, 2 f] in alternating blocks of 16 columns
template <typename T>
__global__ void __launch_bounds__(256) gate_mul_kernel(const T* __restrict__ gu, T* __restrict__ out, long long total, int f,
                                                       int act, float limit) {
  pdl_entry();
  const long long i = blockIdx.x * 256ll + threadIdx.x;
  if (i >= total) return;
  const int c = (int)(i % f);
  const T* g = gu + i / f * 2 * f + c / kGateBlock * 2 * kGateBlock + c % kGateBlock;
  st_f(out + i, gate_mul(ld_f(g), ld_f(g + kGateBlock), act, limit));
}

template <typename T>
int launch_norm(const NormArgs& a, const void* erows, void* out, int rows, cudaStream_t st) {
  auto go = [&](auto kern, size_t smem = 0) { dsv4_launch(kern, rows, 256, smem, st, a, (const T*)erows, (T*)out); };
  if (a.d % 4 || a.d > 8192) {
    if (a.sub && a.d > 11264) return 608;      // the row in 44 KB of shared memory
    go(residual_norm_kernel<T, 0>, a.sub ? (size_t)a.d * 4 : 0);
  } else if (a.d <= 1024)
    go(residual_norm_kernel<T, 1>);
  else if (a.d <= 2048)
    go(residual_norm_kernel<T, 2>);
  else if (a.d <= 4096)
    go(residual_norm_kernel<T, 4>);
  else
    go(residual_norm_kernel<T, 8>);
  return (int)cudaGetLastError();
}

}  // namespace

// fp32: the activation type (0 = bf16, 1 = fp32).  x [t, copies, d].  pair_w [buckets + 1, d]: see EmbedArgs.
DSV4_API int dsv4_embed_residual(int* ids, const int* feedback, const int* slots, const void* w, float* x, void* x0,
                                 float mul, const void* pos_w, const int* pos, int n_pos, int copies, const void* pair_w,
                                 int buckets, int mul_before, int mul_id, int* tokens, const int* out_loc,
                                 const int* page_table, int ld_pt, int t, int d, int fp32, cudaStream_t st) {
  if (t <= 0) return 0;
  if ((feedback && !slots) || (pos_w && (!pos || n_pos < 1)) || copies < 1) return 600;
  if (pair_w && (buckets < 1 || mul_before < 0 || mul_id < 0 || mul_before >= buckets || mul_id >= buckets || !tokens ||
                 !out_loc || !page_table || !pos || !slots))
    return 609;
  const EmbedArgs a{mul, (const __nv_bfloat16*)pos_w, pos, n_pos, copies, d, (const __nv_bfloat16*)pair_w, (unsigned)buckets,
                    (unsigned)mul_before, (unsigned)mul_id, tokens, out_loc, page_table, ld_pt};
  if (fp32)
    dsv4_launch(embed_residual_kernel<float>, t, 256, 0, st, ids, feedback, slots, (const __nv_bfloat16*)w, x,
                (float*)x0, a);
  else
    dsv4_launch(embed_residual_kernel<__nv_bfloat16>, t, 256, 0, st, ids, feedback, slots, (const __nv_bfloat16*)w, x,
                (__nv_bfloat16*)x0, a);
  return (int)cudaGetLastError();
}

// x (+= N(sub + sub_bias) * sub_gain + add + add2 + vec + sum_k wts[k] * erows[k]);  out = x / rms(x) * gain * mul.  rows_idx
// (nothing but sub is added then): gathers the rows first and leaves x alone.
DSV4_API int dsv4_residual_norm(float* x, const long long* rows_idx, const float* sub, const float* sub_bias,
                                const float* sub_gain, const float* add, const float* add2, const float* vec,
                                const void* erows, const float* wts, const int* eidx, int topk, const float* gain, float eps,
                                float mul, void* out, int rows, int d, int fp32, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (rows_idx && (add || add2 || vec || topk)) return 601;
  if (topk > 0 && (!erows || !wts || !eidx)) return 602;
  if ((gain && !out) || (sub && !sub_gain)) return 603;
  const NormArgs a{x, rows_idx, sub, sub_bias, sub_gain, add, add2, vec, wts, eidx, topk, gain, eps, mul, d};
  return fp32 ? launch_norm<float>(a, erows, out, rows, st) : launch_norm<__nv_bfloat16>(a, erows, out, rows, st);
}

DSV4_API int dsv4_silu_mul(const void* gu, void* out, int rows, int f, int fp32, cudaStream_t st) {
  if (rows <= 0) return 0;
  const long long total = (long long)rows * f;
  const unsigned grid = (unsigned)((total + 255) / 256);
  if (fp32)
    dsv4_launch(silu_mul_kernel<float>, grid, 256, 0, st, (const float*)gu, (float*)out, total, f);
  else
    dsv4_launch(silu_mul_kernel<__nv_bfloat16>, grid, 256, 0, st, (const __nv_bfloat16*)gu, (__nv_bfloat16*)out, total,
                f);
  return (int)cudaGetLastError();
}

// x (+= N(sub; sub_w, sub_b)) (+= add);  out = N(x; w, b), N the layer norm of a row.  add and out: activations.  With
// rows_idx the rows are gathered first and x is left alone.
DSV4_API int dsv4_residual_layer_norm(float* x, const long long* rows_idx, const float* sub, const float* sub_w,
                                      const float* sub_b, const void* add, const float* w, const float* b, float eps,
                                      int keep, void* out, int rows, int d, int fp32, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (rows_idx && keep) return 604;
  if ((w && !out) || (sub && (!sub_w || !sub_b)) || (w && !b)) return 605;
  const LayerNormArgs a{x, rows_idx, sub, sub_w, sub_b, add, w, b, eps, d, keep};
  return fp32 ? launch_layer_norm<float>(a, out, rows, st) : launch_layer_norm<__nv_bfloat16>(a, out, rows, st);
}

DSV4_API int dsv4_gate_mul(const void* gu, void* out, int rows, int f, int act, float limit, int fp32, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (f % kGateBlock || !gated_act(act)) return 607;
  const long long total = (long long)rows * f;
  const unsigned grid = (unsigned)((total + 255) / 256);
  if (fp32)
    dsv4_launch(gate_mul_kernel<float>, grid, 256, 0, st, (const float*)gu, (float*)out, total, f, act, limit);
  else
    dsv4_launch(gate_mul_kernel<__nv_bfloat16>, grid, 256, 0, st, (const __nv_bfloat16*)gu, (__nv_bfloat16*)out, total, f,
                act, limit);
  return (int)cudaGetLastError();
}
