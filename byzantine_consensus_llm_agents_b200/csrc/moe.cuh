// Routing of a mixture of experts: which experts a token uses, with which weights, and its place among an
// expert's rows.
#pragma once
#include "stack_common.cuh"
#include "kernels.h"

namespace bcg {

struct MoeRoute {
  int experts, top, col;     // logits are columns col.. of the projection
  int* expert;               // [T][top]
  int* rank;                 // [T][top] place among the expert's rows
  float* weight;             // [T][top]
  int* counts;               // [experts] rows per expert, zero before the step
  const float* bias;         // [experts] added to the logits, or NULL
  bool softmax;              // weights are the softmax over the chosen logits, else their sigmoids
};

__host__ inline MoeRoute moe_route(const bcg_layer* l, const bcg_stack_ws* ws) {
  MoeRoute r;
  r.experts = l->experts;
  r.top = l->top;
  r.col = l->router_col;
  r.expert = ws->moe_expert;
  r.rank = ws->moe_rank;
  r.weight = ws->moe_weight;
  r.counts = ws->moe_counts + l->moe_counts_at;
  r.bias = l->router_bias;
  r.softmax = l->ff_kind == BCG_FF_EXPERTS;
  return r;
}

// fp32 <-> unsigned integers of the same order
__device__ __forceinline__ uint32_t ordered_bits(float v) {
  const uint32_t b = __float_as_uint(v);
  return b & 0x80000000u ? ~b : b | 0x80000000u;
}
__device__ __forceinline__ float from_ordered(uint32_t k) {
  return __uint_as_float(k & 0x80000000u ? k & 0x7fffffffu : ~k);
}

// Shared memory of route_tokens, in words: a key per expert and warp, two counters per expert.
__host__ __device__ constexpr int route_words(int experts, int threads) { return experts * (threads / 32 + 2); }

// One warp, one token: the `top` experts with the largest logits (the sigmoid is monotone; ties go to the lower
// index), weighted by their sigmoid scores or by the softmax over the chosen ones.  keys: the warp's shared memory, one word per expert.
// counters: rows of every expert so far.
__device__ __forceinline__ void route_token(const MoeRoute& r, const float* row, int n_partials, long long pstride, int t,
                                            uint32_t* keys, int* counters, int lane) {
  for (int e = lane; e < r.experts; e += 32) keys[e] = ordered_bits(slab_sum(row + r.col + e, n_partials, pstride) + (r.bias ? r.bias[e] : 0.f));
  uint32_t best;      // the lane's best expert that is still free (key 0: none)
  int at;
  auto scan = [&]() {
    best = 0;
    at = lane < r.experts ? lane : 0x7fffffff;
    for (int e = lane; e < r.experts; e += 32)
      if (keys[e] > best) {
        best = keys[e];
        at = e;
      }
  };
  __syncwarp();
  scan();
  int mine = 0;              // lane k keeps choice k: the counters are then touched side by side
  uint32_t key = 0;
  float first = 0.f, sum = 0.f;      // largest logit, this lane's exponentials
  for (int k = 0; k < r.top; ++k) {
    const uint32_t top = __reduce_max_sync(0xffffffffu, best);
    if (k == 0) first = from_ordered(top);
    const int e = __reduce_min_sync(0xffffffffu, best == top ? at : 0x7fffffff);
    if (e % 32 == lane) {
      keys[e] = 0;
      scan();
    }
    if (k % 32 == lane) {
      mine = e;
      key = top;
    }
    if (k % 32 == 31 || k == r.top - 1) {
      const int i = t * r.top + (k & ~31) + lane;
      if (lane <= k % 32) {
        r.expert[i] = mine;
        const float z = from_ordered(key), w = r.softmax ? expf(z - first) : 1.0f / (1.0f + expf(-z));
        r.weight[i] = w;
        sum += w;
        r.rank[i] = atomicAdd(counters + mine, 1);
      }
    }
  }
  if (r.softmax) {
    sum = warp_sum(sum);
    for (int k = lane; k < r.top; k += 32) r.weight[t * r.top + k] /= sum;
  }
}

// One CTA: tokens t0 .. t1.  With more than one token per warp, rows are numbered inside the CTA first, so that a
// global counter is touched once per CTA.
template <int THREADS>
__device__ __forceinline__ void route_tokens(const MoeRoute& r, const float* proj, int n_partials, long long pstride,
                                             long long ld, int t0, int t1, uint32_t* mem) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (t1 - t0 <= THREADS / 32) {
    if (t0 + warp < t1)
      route_token(r, proj + (t0 + warp) * ld, n_partials, pstride, t0 + warp, mem + warp * r.experts, r.counts, lane);
    return;
  }
  int* local = reinterpret_cast<int*>(mem + THREADS / 32 * r.experts);
  int* base = local + r.experts;
  for (int e = threadIdx.x; e < r.experts; e += THREADS) local[e] = 0;
  __syncthreads();
  for (int t = t0 + warp; t < t1; t += THREADS / 32)
    route_token(r, proj + t * ld, n_partials, pstride, t, mem + warp * r.experts, local, lane);
  __syncthreads();
  for (int e = threadIdx.x; e < r.experts; e += THREADS) base[e] = local[e] ? atomicAdd(r.counts + e, local[e]) : 0;
  __syncthreads();
  for (int i = t0 * r.top + threadIdx.x; i < t1 * r.top; i += THREADS) r.rank[i] += base[r.expert[i]];
}

// First row of an expert's rows: the counts in front of it.  A whole warp calls this.
__device__ __forceinline__ int expert_offset(const int* counts, int expert, int lane) {
  int sum = 0;
  for (int e = lane; e < expert; e += 32) sum += counts[e];
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
  return sum;
}

// Gated unit of an expert: gate from above, linear part from both sides clamped.
__device__ __forceinline__ float clamped_glu(float g, float u, float limit, float alpha) {
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return g / (1.0f + expf(-alpha * g)) * (u + 1.0f);
}
// 0.5 z (1 + tanh(y)) = z / (1 + exp(-2 y)), y = sqrt(2 / pi) (z + 0.044715 z^3)
__device__ __forceinline__ float gelu_tanh(float z) {
  return z / (1.0f + expf(-1.5957691216057308f * fmaf(0.044715f * z * z, z, z)));
}
__device__ __forceinline__ float gelu_erf(float z) { return 0.5f * z * (1.0f + erff(z * 0.70710678118654752f)); }

}  // namespace bcg
