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
  return r;
}

// One CTA, one token: the `top` experts with the largest logits (the sigmoid is monotone; ties go to the lower
// index), weighted by their sigmoid scores.  scores: shared memory, one float per expert.
template <int THREADS>
__device__ __forceinline__ void route_token(const MoeRoute& r, const float* row, int n_partials, long long pstride, int t,
                                            float* scores) {
  for (int e = threadIdx.x; e < r.experts; e += THREADS) scores[e] = slab_sum(row + r.col + e, n_partials, pstride);
  __syncthreads();
  if (threadIdx.x >= 32) return;
  const int lane = threadIdx.x;
  for (int k = 0; k < r.top; ++k) {
    float best = -INFINITY;
    int at = 0x7fffffff;
    for (int e = lane; e < r.experts; e += 32)
      if (scores[e] > best || at == 0x7fffffff) {
        best = scores[e];
        at = e;
      }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float other = __shfl_xor_sync(0xffffffffu, best, o);
      const int oat = __shfl_xor_sync(0xffffffffu, at, o);
      if (other > best || (other == best && oat < at)) {
        best = other;
        at = oat;
      }
    }
    if (lane == 0) {
      const int i = t * r.top + k;
      r.expert[i] = at;
      r.rank[i] = atomicAdd(r.counts + at, 1);
      r.weight[i] = 1.0f / (1.0f + expf(-best));
      scores[at] = -INFINITY;      // not chosen again: top <= experts leaves another one, or all are taken
    }
    __syncwarp();
  }
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

}  // namespace bcg
