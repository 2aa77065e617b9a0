// out fp32 [M, ldo] = X [M, ldx] * W bf16 [N, ldw]^T on CUDA cores, fp32 FMA throughout: the product of
// fp32 activations, and of bf16 ones whose shape TMA cannot address.  64 x 64 tiles, 4 x 4 per thread.
// With row counts: rows sorted by group, blockIdx.z = group, W = the groups' matrices one after another.
#include "moe.cuh"
#include "stack_common.cuh"
#include "kernels.h"

namespace bcg {

constexpr int kSgT = 64, kSgK = 16;

template <typename T>
__global__ void __launch_bounds__(256)
gemm_simt_kernel(const T* __restrict__ X, const __nv_bfloat16* __restrict__ W, float* __restrict__ out, int M, int N,
                 int K, long long ldx, long long ldw, long long ldo, const int* __restrict__ counts) {
  __shared__ float xs[kSgK][kSgT + 4], wsm[kSgK][kSgT + 4];
  pdl_launch_dependents();
  pdl_wait();
  if (counts) {
    M = counts[blockIdx.z];
    if (static_cast<int>(blockIdx.y) * kSgT >= M) return;
    const long long row0 = expert_offset(counts, blockIdx.z, threadIdx.x & 31);
    X += row0 * ldx;
    out += row0 * ldo;
    W += static_cast<long long>(blockIdx.z) * N * ldw;
  }
  const int n0 = blockIdx.x * kSgT, m0 = blockIdx.y * kSgT;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const int lk = threadIdx.x & 15, lr = threadIdx.x >> 4;   // loader: k within the slice, row (four turns)
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += kSgK) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = lr + 16 * i, k = k0 + lk;
      xs[lk][r] = (m0 + r < M && k < K) ? to_f32<T>(X[(m0 + r) * ldx + k]) : 0.f;
      wsm[lk][r] = (n0 + r < N && k < K) ? __bfloat162float(W[(n0 + r) * ldw + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kSgK; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&xs[k][ty * 4]);
      const float4 b = *reinterpret_cast<const float4*>(&wsm[k][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (m0 + ty * 4 + i < M && n0 + tx * 4 + j < N)
        out[(m0 + ty * 4 + i) * ldo + n0 + tx * 4 + j] = acc[i][j];
}

int gemm_any(const void* X, int x_dtype, const void* W, float* out, int M, int N, int K, long long ldx,
             long long ldw, long long ldo, cudaStream_t st) {
  if (!X || !W || !out || M <= 0 || N <= 0 || K <= 0 || (M + kSgT - 1) / kSgT > 65535) {
    set_last_error("bcg_gemm_any", "null pointer, non-positive dimension or M too large");
    return BCG_ERR_ARG;
  }
  const dim3 grid((N + kSgT - 1) / kSgT, (M + kSgT - 1) / kSgT);
  const auto* w = static_cast<const __nv_bfloat16*>(W);
  if (x_dtype == BCG_DT_F32)
    BCG_CUDA_CHECK(launch_k(gemm_simt_kernel<float>, grid, dim3(256), 0, st, static_cast<const float*>(X), w, out, M,
                            N, K, ldx, ldw, ldo, nullptr));
  else
    BCG_CUDA_CHECK(launch_k(gemm_simt_kernel<__nv_bfloat16>, grid, dim3(256), 0, st,
                            static_cast<const __nv_bfloat16*>(X), w, out, M, N, K, ldx, ldw, ldo, nullptr));
  return BCG_OK;
}

int gemm_any_grouped(const void* X, int x_dtype, const void* W, float* out, int N, int K, const GemmGroups& g,
                     cudaStream_t st) {
  if (!X || !W || !out || N <= 0 || K <= 0 || !g.counts || g.n_groups <= 0 || g.n_groups > 65535 || g.max_rows <= 0 ||
      (g.max_rows + kSgT - 1) / kSgT > 65535) {
    set_last_error("bcg_gemm_any", "bad grouped product");
    return BCG_ERR_ARG;
  }
  const dim3 grid((N + kSgT - 1) / kSgT, (g.max_rows + kSgT - 1) / kSgT, g.n_groups);
  const auto* w = static_cast<const __nv_bfloat16*>(W);
  if (x_dtype == BCG_DT_F32)
    BCG_CUDA_CHECK(launch_k(gemm_simt_kernel<float>, grid, dim3(256), 0, st, static_cast<const float*>(X), w, out, 0, N, K,
                            K, K, N, g.counts));
  else
    BCG_CUDA_CHECK(launch_k(gemm_simt_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, static_cast<const __nv_bfloat16*>(X),
                            w, out, 0, N, K, K, K, N, g.counts));
  return BCG_OK;
}

}  // namespace bcg
