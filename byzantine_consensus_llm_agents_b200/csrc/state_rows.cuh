// What kernels with a recurrent fp32 state [rows][n] per head share: gates, the rows of a state over groups of lanes.
#pragma once
#include "attn_tcgen05.cuh"
#include "mma_sync.cuh"
#include "stack_common.cuh"

namespace bcg {

constexpr float kSsLog2e = 1.4426950408889634f;

__device__ __forceinline__ float softplus_f32(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
// rounded once near 1: a state that decays slowly would drift with the error of exp
__device__ __forceinline__ float decay_f32(float x) { return 1.0f + expm1f(x); }

__device__ __forceinline__ void bulk_store_1d(void* gdst, const void* smem_src, uint32_t bytes) {
  asm volatile("cp.async.bulk.global.shared::cta.bulk_group [%0], [%1], %2;" ::"l"(gdst), "r"(smem_u32(smem_src)), "r"(bytes) : "memory");
  asm volatile("cp.async.bulk.commit_group;" ::: "memory");
}

constexpr int kSsThreads = 256, kSsRows = 64;     // threads and state rows of a CTA

// Rows of a head's state over groups of lanes: a group holds a row's entries, four (or twice four) per lane, and every
// kPass-th row of the CTA's block.
template <int NP>
struct StateRows {
  static constexpr int kLanes = NP / 4 < 32 ? NP / 4 : 32, kQ = NP / (4 * kLanes), kPass = kSsThreads / kLanes,
                       kR = kSsRows / kPass;
  static_assert(kR <= kLanes, "lane r of a group finishes its row r");
  float s[kR][kQ][4];

  static __device__ __forceinline__ int lane() { return threadIdx.x % kLanes; }
  static __device__ __forceinline__ int row(int r) { return r * kPass + static_cast<int>(threadIdx.x) / kLanes; }
  static __device__ __forceinline__ int entry(int q) { return (q * kLanes + lane()) * 4; }
  __device__ __forceinline__ void zero() {
#pragma unroll
    for (int r = 0; r < kR; ++r)
#pragma unroll
      for (int q = 0; q < kQ; ++q)
#pragma unroll
        for (int i = 0; i < 4; ++i) s[r][q][i] = 0.f;
  }
  // st: [rows][n], `rows` of them valid
  __device__ __forceinline__ void load(const float* st, int rows, int n) {
#pragma unroll
    for (int r = 0; r < kR; ++r)
#pragma unroll
      for (int q = 0; q < kQ; ++q) {
        const int e = entry(q);
        const float* p = st + static_cast<long long>(row(r)) * n + e;
        if (row(r) < rows && e < n && n % 4 == 0) {
          const float4 v = *reinterpret_cast<const float4*>(p);
          s[r][q][0] = v.x; s[r][q][1] = v.y; s[r][q][2] = v.z; s[r][q][3] = v.w;
        } else {
#pragma unroll
          for (int i = 0; i < 4; ++i) s[r][q][i] = row(r) < rows && e + i < n ? p[i] : 0.f;
        }
      }
  }
  __device__ __forceinline__ void store(float* st, int rows, int n) const {
#pragma unroll
    for (int r = 0; r < kR; ++r)
#pragma unroll
      for (int q = 0; q < kQ; ++q) {
        const int e = entry(q);
        float* p = st + static_cast<long long>(row(r)) * n + e;
        if (row(r) >= rows) continue;
        if (e < n && n % 4 == 0) {
          *reinterpret_cast<float4*>(p) = make_float4(s[r][q][0], s[r][q][1], s[r][q][2], s[r][q][3]);
        } else {
#pragma unroll
          for (int i = 0; i < 4; ++i)
            if (e + i < n) p[i] = s[r][q][i];
        }
      }
  }
  // The row of the group whose output a lane ends up with, and whether it is the lane to write it.
  static __device__ __forceinline__ int mine() { return lane() / (kLanes / kR); }
  static __device__ __forceinline__ bool writes() { return lane() % (kLanes / kR) == 0; }
  // One token: v(r) = step * x of row r, b / c the lane's entries of B and C.  Returns S^T C of row mine().
  template <typename F>
  __device__ __forceinline__ float token(float keep, F v, const float (&b)[kQ][4], const float (&c)[kQ][4]) {
    float y[kR];
#pragma unroll
    for (int r = 0; r < kR; ++r) {
      const float vr = v(r);
      y[r] = 0.f;
#pragma unroll
      for (int q = 0; q < kQ; ++q)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          s[r][q][i] = fmaf(keep, s[r][q][i], vr * b[q][i]);
          y[r] = fmaf(s[r][q][i], c[q][i], y[r]);
        }
    }
    return gather(y);
  }
  // The sums over a group's lanes; every lane gets row mine()'s.  Half of the rows change sides at every exchange.
  static __device__ __forceinline__ float gather(float (&y)[kR]) {
    int m = kLanes / 2;
#pragma unroll
    for (int w = kR / 2; w > 0; w >>= 1, m >>= 1) {
      const bool up = lane() & m;
#pragma unroll
      for (int r = 0; r < w; ++r) {
        const float other = __shfl_xor_sync(0xffffffffu, up ? y[r] : y[r + w], m);
        y[r] = (up ? y[r + w] : y[r]) + other;
      }
    }
#pragma unroll
    for (; m > 0; m >>= 1) y[0] += __shfl_xor_sync(0xffffffffu, y[0], m);
    return y[0];
  }
  // token() on a state in shared memory, row by row, n a multiple of 4.  FULL: all rows, n = NP.
  template <bool FULL, typename F>
  static __device__ __forceinline__ float token_in_place(float* st, int rows, int n, bool fresh, float keep, F v,
                                                         const float (&b)[kQ][4], const float (&c)[kQ][4]) {
    const int pitch = FULL ? NP : n;
    float y[kR];
#pragma unroll
    for (int r = 0; r < kR; ++r) {
      y[r] = 0.f;
      if (!FULL && row(r) >= rows) continue;
      const float vr = v(r);
#pragma unroll
      for (int q = 0; q < kQ; ++q) {
        if (!FULL && entry(q) >= n) continue;
        float4* p = reinterpret_cast<float4*>(st + row(r) * pitch + entry(q));
        float4 s = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *p;
        s.x = fmaf(keep, s.x, vr * b[q][0]);
        s.y = fmaf(keep, s.y, vr * b[q][1]);
        s.z = fmaf(keep, s.z, vr * b[q][2]);
        s.w = fmaf(keep, s.w, vr * b[q][3]);
        *p = s;
        y[r] = fmaf(s.w, c[q][3], fmaf(s.z, c[q][2], fmaf(s.y, c[q][1], fmaf(s.x, c[q][0], y[r]))));
      }
    }
    return gather(y);
  }
};

}  // namespace bcg
