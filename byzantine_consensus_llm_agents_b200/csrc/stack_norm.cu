// Row-wise kernels of layer stacks:
//   embed_norm      x = E[ids];  xn = rmsnorm(x) * w
//   sandwich_norm   x += rmsnorm(delta) * w_post (or += delta);  xn = rmsnorm(x) * w_next
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

template <typename T>
__global__ void __launch_bounds__(kRowT)
embed_norm_kernel(const int* __restrict__ ids, const __nv_bfloat16* __restrict__ embed, const float* __restrict__ w,
                  float* __restrict__ residual, T* __restrict__ xn, int d, float eps) {
  __shared__ RowSum<kRowT, 1, 1> sh;
  pdl_launch_dependents();
  pdl_wait();
  const long long t = blockIdx.x, row = ids[t];
  const int nvec = d >> 2;
  float ss[1] = {0.f};
  for (int v = threadIdx.x; v < nvec; v += kRowT) {
    const uint2 raw = *reinterpret_cast<const uint2*>(embed + row * d + v * 4);
    const float4 x = make_float4(bf16lo(raw.x), bf16hi(raw.x), bf16lo(raw.y), bf16hi(raw.y));
    *reinterpret_cast<float4*>(residual + t * d + v * 4) = x;
    ss[0] += x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
  }
  row_sum<kRowT, 1, 1>(sh, ss, 0);
  const float inv = rsqrtf(ss[0] / static_cast<float>(d) + eps);
  for (int v = threadIdx.x; v < nvec; v += kRowT) {
    const uint2 raw = *reinterpret_cast<const uint2*>(embed + row * d + v * 4);
    const float4 ww = *reinterpret_cast<const float4*>(w + v * 4);
    store4(xn + t * d + v * 4, bf16lo(raw.x) * inv * ww.x, bf16hi(raw.x) * inv * ww.y, bf16lo(raw.y) * inv * ww.z,
           bf16hi(raw.y) * inv * ww.w);
  }
}

template <typename T, int CL>
__global__ void __launch_bounds__(kRowT)
sandwich_norm_kernel(float* __restrict__ residual, const float* __restrict__ delta, int n_partials,
                     long long partial_stride, const float* __restrict__ w_post, const float* __restrict__ w_next,
                     T* __restrict__ xn, int d, float eps) {
  extern __shared__ float4 stage[];   // this CTA's part of the row
  __shared__ RowSum<kRowT, CL, 1> sh;
  pdl_launch_dependents();
  pdl_wait();
  const long long t = CL > 1 ? blockIdx.y : blockIdx.x;
  const int nvec = d >> 2, per = (nvec + CL - 1) / CL;
  const int v0 = (CL > 1 ? static_cast<int>(blockIdx.x) : 0) * per, v1 = min(nvec, v0 + per);
  const float inv_d = 1.0f / static_cast<float>(d);
  float ss[1] = {0.f};
  for (int v = v0 + threadIdx.x; v < v1; v += kRowT) {
    const float4 y = slab_sum4(delta + t * d + v * 4, n_partials, partial_stride);
    stage[v - v0] = y;
    ss[0] += y.x * y.x + y.y * y.y + y.z * y.z + y.w * y.w;
  }
  float inv = 1.0f;
  if (w_post) {
    row_sum<kRowT, CL, 1>(sh, ss, 0);
    inv = rsqrtf(ss[0] * inv_d + eps);
  }
  ss[0] = 0.f;
  for (int v = v0 + threadIdx.x; v < v1; v += kRowT) {
    float4 y = stage[v - v0];
    if (w_post) {
      const float4 ww = *reinterpret_cast<const float4*>(w_post + v * 4);
      y.x *= inv * ww.x; y.y *= inv * ww.y; y.z *= inv * ww.z; y.w *= inv * ww.w;
    }
    float4 x = *reinterpret_cast<const float4*>(residual + t * d + v * 4);
    x.x += y.x; x.y += y.y; x.z += y.z; x.w += y.w;
    *reinterpret_cast<float4*>(residual + t * d + v * 4) = x;
    stage[v - v0] = x;
    ss[0] += x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
  }
  if (w_next) {
    row_sum<kRowT, CL, 1>(sh, ss, 1);
    const float inv2 = rsqrtf(ss[0] * inv_d + eps);
    for (int v = v0 + threadIdx.x; v < v1; v += kRowT) {
      const float4 x = stage[v - v0];
      const float4 ww = *reinterpret_cast<const float4*>(w_next + v * 4);
      store4(xn + t * d + v * 4, x.x * inv2 * ww.x, x.y * inv2 * ww.y, x.z * inv2 * ww.z, x.w * inv2 * ww.w);
    }
  }
  row_sum_exit<CL>();
}

template <typename T>
__global__ void __launch_bounds__(kRowT)
rows_norm_kernel(const float* __restrict__ residual, const int* __restrict__ rows, const float* __restrict__ w,
                 T* __restrict__ xn, int d, float eps) {
  __shared__ RowSum<kRowT, 1, 1> sh;
  pdl_launch_dependents();
  pdl_wait();
  const long long t = blockIdx.x, src = rows[t];
  const int nvec = d >> 2;
  float ss[1] = {0.f};
  for (int v = threadIdx.x; v < nvec; v += kRowT) {
    const float4 x = *reinterpret_cast<const float4*>(residual + src * d + v * 4);
    ss[0] += x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
  }
  row_sum<kRowT, 1, 1>(sh, ss, 0);
  const float inv = rsqrtf(ss[0] / static_cast<float>(d) + eps);
  for (int v = threadIdx.x; v < nvec; v += kRowT) {
    const float4 x = *reinterpret_cast<const float4*>(residual + src * d + v * 4);
    const float4 ww = *reinterpret_cast<const float4*>(w + v * 4);
    store4(xn + t * d + v * 4, x.x * inv * ww.x, x.y * inv * ww.y, x.z * inv * ww.z, x.w * inv * ww.w);
  }
}

template <typename T, int CL>
__global__ void __launch_bounds__(kRowT)
poly_norm_kernel(const float* __restrict__ z, int n_partials, long long partial_stride,
                 const float* __restrict__ coef, T* __restrict__ out, int ff, float eps) {
  extern __shared__ float4 stage[];
  __shared__ RowSum<kRowT, CL, 3> sh;
  pdl_launch_dependents();
  pdl_wait();
  const long long t = CL > 1 ? blockIdx.y : blockIdx.x;
  const int nvec = ff >> 2, per = (nvec + CL - 1) / CL;
  const int v0 = (CL > 1 ? static_cast<int>(blockIdx.x) : 0) * per, v1 = min(nvec, v0 + per);
  float s[3] = {0.f, 0.f, 0.f};   // sums of z^2, z^4, z^6
  auto add = [&](float x) {
    const float x2 = x * x, x4 = x2 * x2;
    s[0] += x2;
    s[1] += x4;
    s[2] = fmaf(x4, x2, s[2]);
  };
  for (int v = v0 + threadIdx.x; v < v1; v += kRowT) {
    const float4 x = slab_sum4(z + t * ff + v * 4, n_partials, partial_stride);
    stage[v - v0] = x;
    add(x.x); add(x.y); add(x.z); add(x.w);
  }
  row_sum<kRowT, CL, 3>(sh, s, 0);
  const float inv_f = 1.0f / static_cast<float>(ff);
  const float a = coef[0] * rsqrtf(s[0] * inv_f + eps), b = coef[1] * rsqrtf(s[1] * inv_f + eps),
              c = coef[2] * rsqrtf(s[2] * inv_f + eps), e = coef[3];
  auto act = [&](float x) { return fmaf(x, fmaf(x, fmaf(x, c, b), a), e); };
  for (int v = v0 + threadIdx.x; v < v1; v += kRowT) {
    const float4 x = stage[v - v0];
    store4(out + t * ff + v * 4, act(x.x), act(x.y), act(x.z), act(x.w));
  }
  row_sum_exit<CL>();
}

int embed_norm(const int* ids, const void* embed, const float* w, float* residual, void* xn, int act_dtype, int T,
               int d, float eps, cudaStream_t st) {
  const auto* e = static_cast<const __nv_bfloat16*>(embed);
  if (act_dtype == BCG_DT_F32)
    BCG_CUDA_CHECK(launch_k(embed_norm_kernel<float>, dim3(T), dim3(kRowT), 0, st, ids, e, w, residual,
                            static_cast<float*>(xn), d, eps));
  else
    BCG_CUDA_CHECK(launch_k(embed_norm_kernel<__nv_bfloat16>, dim3(T), dim3(kRowT), 0, st, ids, e, w, residual,
                            static_cast<__nv_bfloat16*>(xn), d, eps));
  return BCG_OK;
}

int rows_norm(const float* residual, const int* rows, const float* w, void* xn, int act_dtype, int n, int d,
              float eps, cudaStream_t st) {
  if (act_dtype == BCG_DT_F32)
    BCG_CUDA_CHECK(launch_k(rows_norm_kernel<float>, dim3(n), dim3(kRowT), 0, st, residual, rows, w,
                            static_cast<float*>(xn), d, eps));
  else
    BCG_CUDA_CHECK(launch_k(rows_norm_kernel<__nv_bfloat16>, dim3(n), dim3(kRowT), 0, st, residual, rows, w,
                            static_cast<__nv_bfloat16*>(xn), d, eps));
  return BCG_OK;
}

// One row per cluster (decode) or per CTA; KERNEL is a template over <T, CL>.
#define BCG_LAUNCH_ROWS(KERNEL, T_ROWS, WIDTH, TYPE, ...)                                                           \
  do {                                                                                                              \
    if ((T_ROWS) <= kClusterMaxRows && (WIDTH) >= 1024) {                                                           \
      const size_t _sm = static_cast<size_t>(((WIDTH) / 4 + kRowCluster - 1) / kRowCluster) * 16;                   \
      BCG_CUDA_CHECK(launch_cluster(KERNEL<TYPE, kRowCluster>, dim3(kRowCluster, T_ROWS), dim3(kRowT), kRowCluster, \
                                    _sm, st, __VA_ARGS__));                                                         \
    } else {                                                                                                        \
      const size_t _sm = static_cast<size_t>(WIDTH) * 4;                                                            \
      BCG_TRY(ensure_dynamic_smem(reinterpret_cast<const void*>(KERNEL<TYPE, 1>), 200 * 1024));                     \
      BCG_CUDA_CHECK(launch_k(KERNEL<TYPE, 1>, dim3(T_ROWS), dim3(kRowT), _sm, st, __VA_ARGS__));                   \
    }                                                                                                               \
  } while (0)

int sandwich_norm(float* residual, const float* delta, int n_partials, long long partial_stride,
                  const float* w_post, const float* w_next, void* xn, int act_dtype, int T, int d, float eps,
                  cudaStream_t st) {
  if (!residual || !delta || T <= 0 || d <= 0 || (d % 4) || d > 51200 || n_partials < 1 || (w_next && !xn)) {
    set_last_error("bcg_sandwich_norm", "bad argument (d must be a multiple of 4, <= 51200)");
    return BCG_ERR_ARG;
  }
  if (act_dtype == BCG_DT_F32)
    BCG_LAUNCH_ROWS(sandwich_norm_kernel, T, d, float, residual, delta, n_partials, partial_stride, w_post, w_next,
                    static_cast<float*>(xn), d, eps);
  else
    BCG_LAUNCH_ROWS(sandwich_norm_kernel, T, d, __nv_bfloat16, residual, delta, n_partials, partial_stride, w_post,
                    w_next, static_cast<__nv_bfloat16*>(xn), d, eps);
  return BCG_OK;
}

int poly_norm(const float* z, int n_partials, long long partial_stride, const float* coef, void* out, int act_dtype,
              int T, int ff, float eps, cudaStream_t st) {
  if (!z || !coef || !out || T <= 0 || ff <= 0 || (ff % 4) || ff > 51200 || n_partials < 1) {
    set_last_error("bcg_poly_norm", "bad argument (ff must be a multiple of 4, <= 51200)");
    return BCG_ERR_ARG;
  }
  if (act_dtype == BCG_DT_F32)
    BCG_LAUNCH_ROWS(poly_norm_kernel, T, ff, float, z, n_partials, partial_stride, coef, static_cast<float*>(out), ff,
                    eps);
  else
    BCG_LAUNCH_ROWS(poly_norm_kernel, T, ff, __nv_bfloat16, z, n_partials, partial_stride, coef,
                    static_cast<__nv_bfloat16*>(out), ff, eps);
  return BCG_OK;
}

}  // namespace bcg
