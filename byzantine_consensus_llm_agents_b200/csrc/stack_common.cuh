// Helpers shared by the layer-stack kernels: activations of either dtype, split-K slabs, row reductions
// that may span a thread-block cluster.
#pragma once
#include <cooperative_groups.h>

#include "common.cuh"

namespace bcg {

template <typename T>
__device__ __forceinline__ float to_f32(T v);
template <>
__device__ __forceinline__ float to_f32<float>(float v) { return v; }
template <>
__device__ __forceinline__ float to_f32<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T from_f32(float v);
template <>
__device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

__device__ __forceinline__ void store4(float* p, float a, float b, float c, float d) {
  *reinterpret_cast<float4*>(p) = make_float4(a, b, c, d);
}
__device__ __forceinline__ void store4(__nv_bfloat16* p, float a, float b, float c, float d) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(a, b), pack_bf16(c, d));
}

__device__ __forceinline__ float sigmoid_f32(float x) { return __fdividef(1.0f, 1.0f + expf(-x)); }

// fp32 split-K slabs summed in index order; four loads in flight per thread.
__device__ __forceinline__ float slab_sum(const float* p, int n, long long stride) {
  float acc = p[0];
  for (int s = 1; s < n; s += 4) {
    float v[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) v[i] = p[min(s + i, n - 1) * stride];
#pragma unroll
    for (int i = 0; i < 4; ++i)
      if (s + i < n) acc += v[i];
  }
  return acc;
}
// V consecutive floats: 4 (vector access, widths that are multiples of 4) or 1 (any width).
template <int V>
struct Vec {
  float x[V];
  __device__ __forceinline__ float sumsq() const {
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < V; ++i) s += x[i] * x[i];
    return s;
  }
  __device__ __forceinline__ void add(const Vec& o) {
#pragma unroll
    for (int i = 0; i < V; ++i) x[i] += o.x[i];
  }
};
template <int V>
__device__ __forceinline__ Vec<V> load_vec(const float* p) {
  Vec<V> v;
  if constexpr (V == 4) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    v.x[0] = f.x; v.x[1] = f.y; v.x[2] = f.z; v.x[3] = f.w;
  } else {
    v.x[0] = *p;
  }
  return v;
}
template <int V>
__device__ __forceinline__ Vec<V> load_vec(const __nv_bfloat16* p) {
  Vec<V> v;
  if constexpr (V == 4) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    v.x[0] = bf16lo(raw.x); v.x[1] = bf16hi(raw.x); v.x[2] = bf16lo(raw.y); v.x[3] = bf16hi(raw.y);
  } else {
    v.x[0] = __bfloat162float(*p);
  }
  return v;
}
template <int V, typename T>
__device__ __forceinline__ void store_vec(T* p, const Vec<V>& v) {
  if constexpr (V == 4) store4(p, v.x[0], v.x[1], v.x[2], v.x[3]);
  else *p = from_f32<T>(v.x[0]);
}
template <int V>
__device__ __forceinline__ Vec<V> slab_sum_vec(const float* p, int n, long long stride) {
  Vec<V> acc = load_vec<V>(p);
  for (int s = 1; s < n; s += 8) {
    Vec<V> v[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] = load_vec<V>(p + min(s + i, n - 1) * stride);
#pragma unroll
    for (int i = 0; i < 8; ++i)
      if (s + i < n) {
#pragma unroll
        for (int k = 0; k < V; ++k) acc.x[k] += v[i].x[k];
      }
  }
  return acc;
}

// Sum of N values over the THREADS x CL threads that share a row (CL CTAs of one cluster); fixed order, so a
// row's result does not depend on its neighbours.  `slot` must be a fresh 0, 1, ... per call in a kernel.
// Before a kernel with CL > 1 ends, every thread must pass row_sum_exit<CL>().
template <int THREADS, int CL, int N>
struct RowSum {
  float warp[N][THREADS / 32];
  float cta[2][N];
};
template <int THREADS, int CL, int N>
__device__ __forceinline__ void row_sum(RowSum<THREADS, CL, N>& sh, float (&v)[N], int slot) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
#pragma unroll
  for (int k = 0; k < N; ++k) {
    v[k] = warp_sum(v[k]);
    if (lane == 0) sh.warp[k][warp] = v[k];
  }
  __syncthreads();
#pragma unroll
  for (int k = 0; k < N; ++k) {
    float t = 0.f;
#pragma unroll
    for (int i = 0; i < THREADS / 32; ++i) t += sh.warp[k][i];
    v[k] = t;
  }
  if constexpr (CL > 1) {
    namespace cg = cooperative_groups;
    cg::cluster_group cluster = cg::this_cluster();
    if (threadIdx.x < N) {
      float mine = v[0];
#pragma unroll
      for (int k = 1; k < N; ++k)
        if (static_cast<int>(threadIdx.x) == k) mine = v[k];
      sh.cta[slot & 1][threadIdx.x] = mine;
    }
    cluster.sync();
#pragma unroll
    for (int k = 0; k < N; ++k) {
      float t = 0.f;
#pragma unroll
      for (int i = 0; i < CL; ++i) t += *cluster.map_shared_rank(&sh.cta[slot & 1][k], i);
      v[k] = t;
    }
  } else {
    __syncthreads();
  }
}
template <int CL>
__device__ __forceinline__ void row_sum_exit() {
  if constexpr (CL > 1) cooperative_groups::this_cluster().sync();
}

template <typename... KArgs, typename... Args>
inline cudaError_t launch_cluster(void (*kernel)(KArgs...), dim3 grid, dim3 block, int cluster_x, size_t smem,
                                  cudaStream_t stream, Args&&... args) {
  prefer_max_smem_carveout(reinterpret_cast<const void*>(kernel));
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = (launch_flags() & 1) ? 1 : 0;
  attr[1].id = cudaLaunchAttributeClusterDimension;
  attr[1].val.clusterDim.x = cluster_x;
  attr[1].val.clusterDim.y = 1;
  attr[1].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = cluster_x > 1 ? 2 : 1;
  return cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);
}

#define BCG_TRY(expr)              \
  do {                             \
    int _rc = (expr);              \
    if (_rc != BCG_OK) return _rc; \
  } while (0)

}  // namespace bcg
