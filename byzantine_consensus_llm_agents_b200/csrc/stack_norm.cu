// Row-wise kernels of layer stacks:
//   embed_norm      x = scale * E[ids] (+ P[positions] or sinusoids), normed or not;  xn = rmsnorm(x) * w (or x)
//   sandwich_norm   x += rmsnorm(delta) * w_post (or += delta);  xn = rmsnorm(x) * w_next (or x)
//                   delta may have a bias and rows of a second source (a token's experts, weighted or not) added
//   rows_norm       xn[i] = rmsnorm(x[rows[i]]) * w
//   poly_norm       PolyNorm activation: a N(z) + b N(z^2) + c N(z^3) + e, N = division by the row's RMS
// `delta` and `z` arrive as fp32 split-K slabs of the projection in front.  Decode-sized launches spread a
// row over a cluster of eight CTAs (sums exchanged through distributed shared memory), prompt-sized ones
// give a row to one CTA.  All arithmetic is fp32; only what feeds the next product is rounded.
#include "stack_common.cuh"
#include "kernels.h"

namespace bcg {

constexpr int kRowT = 256;          // threads per CTA
constexpr int kRowCluster = 8;
constexpr int kClusterMaxRows = 128;

template <typename T, int V>
__global__ void __launch_bounds__(kRowT)
embed_norm_kernel(const EmbedArgs a, const float* __restrict__ w, float* __restrict__ residual, T* __restrict__ xn, int d,
                  float eps) {
  __shared__ RowSum<kRowT, 1, 1> sh;
  pdl_launch_dependents();
  pdl_wait();
  const long long t = blockIdx.x, row = a.ids[t];
  for (int i = blockIdx.x * kRowT + threadIdx.x; i < a.n_zero; i += gridDim.x * kRowT) a.zero[i] = 0;
  const __nv_bfloat16* pos = nullptr;
  if (a.pos_embed) pos = a.pos_embed + static_cast<long long>(min(a.positions[t], a.n_pos - 1)) * d;
  const double at = a.pos_turns ? a.positions[t] : 0;
  float ss[1] = {0.f};
  for (int v = threadIdx.x * V; v < d; v += kRowT * V) {
    Vec<V> x = load_vec<V>(a.embed + row * d + v);
#pragma unroll
    for (int k = 0; k < V; ++k) x.x[k] *= a.scale;
    if (pos) x.add(load_vec<V>(pos + v));
    if (a.pos_turns) {
      // whole turns are taken off in double precision: the angle is exact at any position
#pragma unroll
      for (int k = 0; k < V; ++k) {
        const double turns = at * a.pos_turns[(v + k) >> 1];
        const float half = static_cast<float>(2.0 * (turns - rint(turns)));
        x.x[k] += ((v + k) & 1) ? cospif(half) : sinpif(half);
      }
    }
    store_vec<V>(residual + t * d + v, x);      // read again below by the same thread
    ss[0] += x.sumsq();
  }
  row_sum<kRowT, 1, 1>(sh, ss, 0);
  float inv = rsqrtf(ss[0] / static_cast<float>(d) + eps);
  if (a.norm) {
    ss[0] = 0.f;
    for (int v = threadIdx.x * V; v < d; v += kRowT * V) {
      Vec<V> x = load_vec<V>(residual + t * d + v);
      const Vec<V> ww = load_vec<V>(a.norm + v);
#pragma unroll
      for (int k = 0; k < V; ++k) x.x[k] *= inv * ww.x[k];
      store_vec<V>(residual + t * d + v, x);
      ss[0] += x.sumsq();
    }
    row_sum<kRowT, 1, 1>(sh, ss, 1);
    inv = rsqrtf(ss[0] / static_cast<float>(d) + eps);
  }
  for (int v = threadIdx.x * V; v < d; v += kRowT * V) {
    Vec<V> x = load_vec<V>(residual + t * d + v);
    if (w) {
      const Vec<V> ww = load_vec<V>(w + v);
#pragma unroll
      for (int k = 0; k < V; ++k) x.x[k] *= inv * ww.x[k];
    }
    store_vec<V>(xn + t * d + v, x);
  }
}

template <typename T, int V, int CL>
__global__ void __launch_bounds__(kRowT)
sandwich_norm_kernel(float* __restrict__ residual, const float* __restrict__ delta, int n_partials,
                     long long partial_stride, const float* __restrict__ w_post, const float* __restrict__ w_next,
                     T* __restrict__ xn, int d, float eps, const NormExtra extra) {
  extern __shared__ float4 stage_raw[];   // this CTA's part of the row
  float* stage = reinterpret_cast<float*>(stage_raw);
  __shared__ RowSum<kRowT, CL, 1> sh;
  pdl_launch_dependents();
  pdl_wait();
  const long long t = CL > 1 ? blockIdx.y : blockIdx.x;
  const int per = (d / V + CL - 1) / CL * V;
  const int v0 = (CL > 1 ? static_cast<int>(blockIdx.x) : 0) * per, v1 = min(d, v0 + per);
  const float inv_d = 1.0f / static_cast<float>(d);
  float ss[1] = {0.f};
  for (int v = v0 + threadIdx.x * V; v < v1; v += kRowT * V) {
    Vec<V> y;
    if (delta) {
      y = slab_sum_vec<V>(delta + t * d + v, n_partials, partial_stride);
    } else {
#pragma unroll
      for (int k = 0; k < V; ++k) y.x[k] = 0.f;
    }
    if (extra.bias) y.add(load_vec<V>(extra.bias + v));
    for (int k = 0; k < extra.per_row; ++k) {
      const Vec<V> row = slab_sum_vec<V>(extra.rows + static_cast<long long>(extra.index[t * extra.per_row + k]) * d + v,
                                         extra.n_partials, extra.partial_stride);
      const float f = extra.weight ? extra.weight[t * extra.per_row + k] : 1.0f;
#pragma unroll
      for (int j = 0; j < V; ++j) y.x[j] = fmaf(f, row.x[j], y.x[j]);
    }
    store_vec<V>(stage + v - v0, y);
    ss[0] += y.sumsq();
  }
  float inv = 1.0f;
  if (w_post) {
    row_sum<kRowT, CL, 1>(sh, ss, 0);
    inv = rsqrtf(ss[0] * inv_d + eps);
  }
  ss[0] = 0.f;
  for (int v = v0 + threadIdx.x * V; v < v1; v += kRowT * V) {
    const Vec<V> y = load_vec<V>(stage + v - v0);
    Vec<V> x = load_vec<V>(residual + t * d + v);
    if (w_post) {
      const Vec<V> ww = load_vec<V>(w_post + v);
#pragma unroll
      for (int k = 0; k < V; ++k) x.x[k] = fmaf(y.x[k], inv * ww.x[k], x.x[k]);
    } else {
#pragma unroll
      for (int k = 0; k < V; ++k) x.x[k] += y.x[k];
    }
    store_vec<V>(residual + t * d + v, x);
    store_vec<V>(stage + v - v0, x);
    if (!w_next && xn) store_vec<V>(xn + t * d + v, x);
    ss[0] += x.sumsq();
  }
  if (w_next) {
    row_sum<kRowT, CL, 1>(sh, ss, 1);
    const float inv2 = rsqrtf(ss[0] * inv_d + eps);
    for (int v = v0 + threadIdx.x * V; v < v1; v += kRowT * V) {
      Vec<V> x = load_vec<V>(stage + v - v0);
      const Vec<V> ww = load_vec<V>(w_next + v);
#pragma unroll
      for (int k = 0; k < V; ++k) x.x[k] *= inv2 * ww.x[k];
      store_vec<V>(xn + t * d + v, x);
    }
  }
  row_sum_exit<CL>();
}

template <typename T, int V>
__global__ void __launch_bounds__(kRowT)
rows_norm_kernel(const float* __restrict__ residual, const int* __restrict__ rows, const float* __restrict__ w,
                 T* __restrict__ xn, int d, float eps) {
  __shared__ RowSum<kRowT, 1, 1> sh;
  pdl_launch_dependents();
  pdl_wait();
  const long long t = blockIdx.x, src = rows[t];
  float ss[1] = {0.f};
  for (int v = threadIdx.x * V; v < d; v += kRowT * V) ss[0] += load_vec<V>(residual + src * d + v).sumsq();
  row_sum<kRowT, 1, 1>(sh, ss, 0);
  const float inv = rsqrtf(ss[0] / static_cast<float>(d) + eps);
  for (int v = threadIdx.x * V; v < d; v += kRowT * V) {
    Vec<V> x = load_vec<V>(residual + src * d + v);
    const Vec<V> ww = load_vec<V>(w + v);
#pragma unroll
    for (int k = 0; k < V; ++k) x.x[k] *= inv * ww.x[k];
    store_vec<V>(xn + t * d + v, x);
  }
}

template <typename T, int V, int CL>
__global__ void __launch_bounds__(kRowT)
poly_norm_kernel(const float* __restrict__ z, int n_partials, long long partial_stride,
                 const float* __restrict__ coef, T* __restrict__ out, int ff, float eps) {
  extern __shared__ float4 stage_raw[];
  float* stage = reinterpret_cast<float*>(stage_raw);
  __shared__ RowSum<kRowT, CL, 3> sh;
  pdl_launch_dependents();
  pdl_wait();
  const long long t = CL > 1 ? blockIdx.y : blockIdx.x;
  const int per = (ff / V + CL - 1) / CL * V;
  const int v0 = (CL > 1 ? static_cast<int>(blockIdx.x) : 0) * per, v1 = min(ff, v0 + per);
  float s[3] = {0.f, 0.f, 0.f};   // sums of z^2, z^4, z^6
  for (int v = v0 + threadIdx.x * V; v < v1; v += kRowT * V) {
    const Vec<V> x = slab_sum_vec<V>(z + t * ff + v, n_partials, partial_stride);
    store_vec<V>(stage + v - v0, x);
#pragma unroll
    for (int k = 0; k < V; ++k) {
      const float x2 = x.x[k] * x.x[k], x4 = x2 * x2;
      s[0] += x2;
      s[1] += x4;
      s[2] = fmaf(x4, x2, s[2]);
    }
  }
  row_sum<kRowT, CL, 3>(sh, s, 0);
  const float inv_f = 1.0f / static_cast<float>(ff);
  const float a = coef[0] * rsqrtf(s[0] * inv_f + eps), b = coef[1] * rsqrtf(s[1] * inv_f + eps),
              c = coef[2] * rsqrtf(s[2] * inv_f + eps), e = coef[3];
  for (int v = v0 + threadIdx.x * V; v < v1; v += kRowT * V) {
    Vec<V> x = load_vec<V>(stage + v - v0);
#pragma unroll
    for (int k = 0; k < V; ++k) x.x[k] = fmaf(x.x[k], fmaf(x.x[k], fmaf(x.x[k], c, b), a), e);
    store_vec<V>(out + t * ff + v, x);
  }
  row_sum_exit<CL>();
}

// calls FN<type, vector width>(...) for the activation dtype and the row width
#define BCG_BY_TYPE(FN, WIDTH, DTYPE, ...)                                   \
  do {                                                                       \
    if ((DTYPE) == BCG_DT_F32)                                               \
      return (WIDTH) % 4 ? FN<float, 1>(__VA_ARGS__) : FN<float, 4>(__VA_ARGS__); \
    return (WIDTH) % 4 ? FN<__nv_bfloat16, 1>(__VA_ARGS__) : FN<__nv_bfloat16, 4>(__VA_ARGS__); \
  } while (0)

template <typename T, int V>
static int embed_t(const EmbedArgs& a, const float* w, float* residual, void* xn, int T_rows, int d, float eps,
                   cudaStream_t st) {
  BCG_CUDA_CHECK(launch_k(embed_norm_kernel<T, V>, dim3(T_rows), dim3(kRowT), 0, st, a, w, residual, static_cast<T*>(xn), d,
                          eps));
  return BCG_OK;
}
int embed_norm(const EmbedArgs& a, const float* w, float* residual, void* xn, int act_dtype, int T, int d, float eps,
               cudaStream_t st) {
  BCG_BY_TYPE(embed_t, d, act_dtype, a, w, residual, xn, T, d, eps, st);
}

template <typename T, int V>
static int rows_t(const float* residual, const int* rows, const float* w, void* xn, int n, int d, float eps,
                  cudaStream_t st) {
  BCG_CUDA_CHECK(launch_k(rows_norm_kernel<T, V>, dim3(n), dim3(kRowT), 0, st, residual, rows, w, static_cast<T*>(xn),
                          d, eps));
  return BCG_OK;
}
int rows_norm(const float* residual, const int* rows, const float* w, void* xn, int act_dtype, int n, int d,
              float eps, cudaStream_t st) {
  BCG_BY_TYPE(rows_t, d, act_dtype, residual, rows, w, xn, n, d, eps, st);
}

// One row per cluster (decode) or per CTA; shared memory stages a CTA's part of the row.
static bool row_cluster(int rows, int width) { return rows <= kClusterMaxRows && width >= 1024; }
static size_t row_stage(bool cluster, int width, int v) {
  return static_cast<size_t>(cluster ? (width / v + kRowCluster - 1) / kRowCluster * v : width) * 4;
}

template <typename T, int V>
static int sandwich_t(float* residual, const float* delta, int n_partials, long long stride, const float* w_post,
                      const float* w_next, void* xn, int T_rows, int d, float eps, const NormExtra& extra,
                      cudaStream_t st) {
  const bool cl = row_cluster(T_rows, d);
  const size_t sm = row_stage(cl, d, V);
  T* x = static_cast<T*>(xn);
  if (cl) {
    BCG_CUDA_CHECK(launch_cluster(sandwich_norm_kernel<T, V, kRowCluster>, dim3(kRowCluster, T_rows), dim3(kRowT),
                                  kRowCluster, sm, st, residual, delta, n_partials, stride, w_post, w_next, x, d, eps, extra));
  } else {
    BCG_TRY(ensure_dynamic_smem(reinterpret_cast<const void*>(sandwich_norm_kernel<T, V, 1>), 200 * 1024));
    BCG_CUDA_CHECK(launch_k(sandwich_norm_kernel<T, V, 1>, dim3(T_rows), dim3(kRowT), sm, st, residual, delta, n_partials,
                            stride, w_post, w_next, x, d, eps, extra));
  }
  return BCG_OK;
}
int sandwich_norm(float* residual, const float* delta, int n_partials, long long partial_stride,
                  const float* w_post, const float* w_next, void* xn, int act_dtype, int T, int d, float eps,
                  const NormExtra& extra, cudaStream_t st) {
  if (!residual || (!delta && extra.per_row <= 0) || T <= 0 || d <= 0 || d > 51200 || n_partials < 1 || (w_next && !xn)) {
    set_last_error("bcg_sandwich_norm", "bad argument (d <= 51200)");
    return BCG_ERR_ARG;
  }
  BCG_BY_TYPE(sandwich_t, d, act_dtype, residual, delta, n_partials, partial_stride, w_post, w_next, xn, T, d, eps, extra,
              st);
}

template <typename T, int V>
static int poly_t(const float* z, int n_partials, long long stride, const float* coef, void* out, int T_rows, int ff,
                  float eps, cudaStream_t st) {
  const bool cl = row_cluster(T_rows, ff);
  const size_t sm = row_stage(cl, ff, V);
  T* o = static_cast<T*>(out);
  if (cl) {
    BCG_CUDA_CHECK(launch_cluster(poly_norm_kernel<T, V, kRowCluster>, dim3(kRowCluster, T_rows), dim3(kRowT), kRowCluster,
                                  sm, st, z, n_partials, stride, coef, o, ff, eps));
  } else {
    BCG_TRY(ensure_dynamic_smem(reinterpret_cast<const void*>(poly_norm_kernel<T, V, 1>), 200 * 1024));
    BCG_CUDA_CHECK(launch_k(poly_norm_kernel<T, V, 1>, dim3(T_rows), dim3(kRowT), sm, st, z, n_partials, stride, coef, o,
                            ff, eps));
  }
  return BCG_OK;
}
int poly_norm(const float* z, int n_partials, long long partial_stride, const float* coef, void* out, int act_dtype,
              int T, int ff, float eps, cudaStream_t st) {
  if (!z || !coef || !out || T <= 0 || ff <= 0 || ff > 51200 || n_partials < 1) {
    set_last_error("bcg_poly_norm", "bad argument (ff <= 51200)");
    return BCG_ERR_ARG;
  }
  BCG_BY_TYPE(poly_t, ff, act_dtype, z, n_partials, partial_stride, coef, out, T, ff, eps, st);
}

}  // namespace bcg
