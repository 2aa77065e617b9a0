// Mixture of experts: T tokens, `top` experts each.
//   (parallel layers: routing happens in the kernel that reads the input projection: moe.cuh)
//   expert_in      other layers: routing, and the shared expert's unit of split-K slabs
//   moe_scatter    rows of the normed stream -> rows sorted by expert
//   grouped GEMM   every expert's gate and up matrices over its rows (gemm_tcgen05.cu; CUDA cores for fp32)
//   moe_unit       gated unit or gelu of split-K slabs (prompts: in the GEMM's epilogue)
//   grouped GEMM   down matrices, fp32 rows; the norm kernel adds a token's rows, weighted or not, to its residual
// Gated experts: the routing weight scales an expert's input.  Its products are linear in that input, so the weight is
// applied to the fp32 accumulators of gate and up instead of the bf16 operand.
#include "moe.cuh"

namespace bcg {

constexpr int kMoeThreads = 128;

// A warp per (token, choice).  UNIT: bytes copied at a time.
template <typename UNIT>
__global__ void __launch_bounds__(kMoeThreads)
moe_scatter_kernel(const UNIT* __restrict__ x, UNIT* __restrict__ out, const MoeRoute r, int* __restrict__ row_of,
                   float* __restrict__ row_weight, int n, int units) {
  pdl_launch_dependents();
  pdl_wait();
  const int i = (blockIdx.x * kMoeThreads + threadIdx.x) >> 5, lane = threadIdx.x & 31;
  if (i >= n) return;
  const int row = expert_offset(r.counts, r.expert[i], lane) + r.rank[i];
  if (lane == 0) {
    row_of[i] = row;
    row_weight[row] = r.weight[i];
  }
  const UNIT* src = x + static_cast<long long>(i / r.top) * units;
  UNIT* dst = out + static_cast<long long>(row) * units;
#pragma unroll 4
  for (int c = lane; c < units; c += 32) dst[c] = src[c];
}

// z: slabs of [rows][2 * ff_ld], 16 gate columns beside 16 up columns, or, without gates, [rows][ff_ld]; a warp-wide run of
// columns per thread group.
template <typename T, int UNIT>
__global__ void __launch_bounds__(kMoeThreads)
moe_unit_kernel(const float* __restrict__ z, int n_partials, long long pstride, const float* __restrict__ row_weight,
                T* __restrict__ out, int ff_ld, float limit, float alpha) {
  pdl_launch_dependents();
  pdl_wait();
  const long long row = blockIdx.x;
  const float w = row_weight ? row_weight[row] : 1.f;
  const float* src = z + row * (UNIT == BCG_EPI_GELU ? 1 : 2) * ff_ld;
  for (int c = (blockIdx.y * kMoeThreads + threadIdx.x) * 4; c < ff_ld; c += gridDim.y * kMoeThreads * 4) {
    Vec<4> y;
    if constexpr (UNIT == BCG_EPI_GELU) {
      y = slab_sum_vec<4>(src + c, n_partials, pstride);
#pragma unroll
      for (int k = 0; k < 4; ++k) y.x[k] = gelu_erf(w * y.x[k]);
    } else {
      const float* p = src + (c >> 4) * 32 + (c & 15);
      const Vec<4> g = slab_sum_vec<4>(p, n_partials, pstride), u = slab_sum_vec<4>(p + 16, n_partials, pstride);
#pragma unroll
      for (int k = 0; k < 4; ++k)
        y.x[k] = UNIT == BCG_EPI_GLU ? clamped_glu(w * g.x[k], w * u.x[k], limit, alpha) : gelu_tanh(w * g.x[k]) * (w * u.x[k]);
    }
    store_vec<4>(out + row * ff_ld + c, y);
  }
}

template <typename T>
static int unit_t(const float* z, int n_partials, long long pstride, const float* row_weight, void* out, dim3 grid, int ff_ld, int unit,
                  float limit, float alpha, cudaStream_t st) {
  T* o = static_cast<T*>(out);
  const dim3 block(kMoeThreads);
  if (unit == BCG_EPI_GLU)
    BCG_CUDA_CHECK(launch_k(moe_unit_kernel<T, BCG_EPI_GLU>, grid, block, 0, st, z, n_partials, pstride, row_weight, o, ff_ld, limit, alpha));
  else if (unit == BCG_EPI_GELU_GLU)
    BCG_CUDA_CHECK(launch_k(moe_unit_kernel<T, BCG_EPI_GELU_GLU>, grid, block, 0, st, z, n_partials, pstride, row_weight, o, ff_ld, limit, alpha));
  else
    BCG_CUDA_CHECK(launch_k(moe_unit_kernel<T, BCG_EPI_GELU>, grid, block, 0, st, z, n_partials, pstride, row_weight, o, ff_ld, limit, alpha));
  return BCG_OK;
}

int unit_rows(const float* z, int n_partials, long long pstride, const float* row_weight, void* out, int act_dtype, int rows,
              int ff_ld, int unit, float limit, float alpha, cudaStream_t st) {
  if (!z || !out || rows <= 0 || ff_ld <= 0 || ff_ld % 16 || n_partials < 1) {
    set_last_error("bcg feed-forward unit", "bad argument (ff % 16)");
    return BCG_ERR_ARG;
  }
  const int per = rows <= 1024 ? (ff_ld + kMoeThreads * 4 - 1) / (kMoeThreads * 4) : 1;
  const dim3 grid(rows, per);
  return act_dtype == BCG_DT_F32 ? unit_t<float>(z, n_partials, pstride, row_weight, out, grid, ff_ld, unit, limit, alpha, st)
                                 : unit_t<__nv_bfloat16>(z, n_partials, pstride, row_weight, out, grid, ff_ld, unit, limit, alpha, st);
}

// ------------------------------------------------------------------------------------------- layers that are not parallel
constexpr int kExpertInThreads = 256;

// grid: `blocks` CTAs per token for the shared expert's columns, then the routing CTAs (`route_tokens_per` tokens each)
template <typename T>
__global__ void __launch_bounds__(kExpertInThreads)
expert_in_kernel(const float* __restrict__ proj, int n_partials, long long pstride, long long ld, const MoeRoute route, int route_tokens_per,
                 int n_tokens, int blocks, int act_from, int ff, T* __restrict__ act) {
  extern __shared__ uint32_t route_mem[];
  pdl_launch_dependents();
  pdl_wait();
  const int split = static_cast<int>(blockIdx.x) - n_tokens * blocks;
  if (split >= 0) {
    const int t0 = split * route_tokens_per;
    route_tokens<kExpertInThreads>(route, proj, n_partials, pstride, ld, t0, min(t0 + route_tokens_per, n_tokens), route_mem);
    return;
  }
  const long long t = blockIdx.x / blocks;
  for (int c = (static_cast<int>(blockIdx.x % blocks) * kExpertInThreads + threadIdx.x) * 4; c < ff; c += blocks * kExpertInThreads * 4) {
    Vec<4> x = slab_sum_vec<4>(proj + t * ld + act_from + c, n_partials, pstride);
#pragma unroll
    for (int k = 0; k < 4; ++k) x.x[k] = gelu_erf(x.x[k]);
    store_vec<4>(act + t * ff + c, x);
  }
}

int expert_in(const bcg_stack* m, const bcg_layer* l, const bcg_stack_ws* ws, int T, int n_partials, long long pstride, long long ld,
              bool with_act, cudaStream_t st) {
  const int ff = with_act ? l->ff : 0;
  const int blocks = ff == 0 ? 0 : T <= 128 ? (ff + kExpertInThreads * 4 - 1) / (kExpertInThreads * 4) : 1;
  const int per = T <= 128 ? kExpertInThreads / 32 : kExpertInThreads / 8;
  const dim3 grid(T * blocks + (T + per - 1) / per);
  const size_t sm = static_cast<size_t>(route_words(l->experts, kExpertInThreads)) * 4;
  if (sm > 48 * 1024 || l->top > l->experts || l->n_router < l->experts || l->n_router % 4 || l->ff % 16 || !l->router_bias) {
    set_last_error("bcg_experts", "at most 1,200 experts with a bias, shared sizes in multiples of 16");
    return BCG_ERR_UNSUPPORTED;
  }
  const MoeRoute r = moe_route(l, ws);
  if (m->act_dtype == BCG_DT_F32)
    BCG_CUDA_CHECK(launch_k(expert_in_kernel<float>, grid, dim3(kExpertInThreads), sm, st, ws->proj, n_partials, pstride, ld, r, per, T,
                            blocks, l->n_router, ff, static_cast<float*>(ws->act)));
  else
    BCG_CUDA_CHECK(launch_k(expert_in_kernel<__nv_bfloat16>, grid, dim3(kExpertInThreads), sm, st, ws->proj, n_partials, pstride, ld, r,
                            per, T, blocks, l->n_router, ff, static_cast<__nv_bfloat16*>(ws->act)));
  return BCG_OK;
}

static bool moe_tensor(const bcg_stack* m, const bcg_layer* l, int T, int N, int K) {
  return m->act_dtype == BCG_DT_BF16 && K % 8 == 0 && (T <= 128 || N % 16 == 0) && l->experts <= kMaxGroups;
}

// A grouped product over the sorted rows; *splits slabs of [T * top][N] fp32 when epi is BCG_EPI_F32.
static int expert_gemm(const bcg_stack* m, const bcg_layer* l, const bcg_stack_ws* ws, int T, const void* x, const void* w,
                       void* out, long long cap, int N, int K, int epi, int* splits, cudaStream_t st) {
  const int rows = T * l->top;
  const bool tensor = moe_tensor(m, l, T, N, K);
  *splits = tensor ? moe_splits(T, l->top, N, K) : 1;
  if (epi == BCG_EPI_F32 && static_cast<long long>(*splits) * rows * N > cap) {
    set_last_error("bcg_experts", "expert scratch too small");
    return BCG_ERR_TOO_LARGE;
  }
  GemmGroups g = {};
  g.counts = ws->moe_counts + l->moe_counts_at;
  g.n_groups = l->experts;
  g.max_rows = T;
  g.row_weight = ws->moe_row_weight;
  g.glu_limit = l->glu_limit;
  g.glu_alpha = l->glu_alpha;
  if (tensor) return gemm_grouped(x, w, out, rows, N, K, epi, *splits, g, st);
  return gemm_any_grouped(x, m->act_dtype, w, static_cast<float*>(out), N, K, g, st);
}

// Split-K slabs of a grouped product: a function of the shapes a token meets, not of the batch.
int moe_splits(int T, int top, int N, int K) { return T <= 128 ? gemm_splits_for(1, top * N, K) : 1; }

int experts(const bcg_stack* m, const bcg_layer* l, const bcg_stack_ws* ws, int T, int* splits, cudaStream_t st) {
  const int rows = T * l->top, d = m->d_model, ff = l->expert_ld, size = m->act_dtype == BCG_DT_F32 ? 4 : 2;
  if (rows > ws->moe_rows_max) {
    set_last_error("bcg_experts", "more (token, choice) rows than the workspace holds");
    return BCG_ERR_TOO_LARGE;
  }
  const MoeRoute r = moe_route(l, ws);
  const int unit = l->ff_kind == BCG_FF_EXPERTS ? BCG_EPI_GELU : BCG_EPI_GLU, n_in = unit == BCG_EPI_GELU ? ff : 2 * ff;
  const dim3 grid((rows + kMoeThreads / 32 - 1) / (kMoeThreads / 32));
  if (d * size % 16 == 0)
    BCG_CUDA_CHECK(launch_k(moe_scatter_kernel<uint4>, grid, dim3(kMoeThreads), 0, st, static_cast<const uint4*>(ws->xn),
                            static_cast<uint4*>(ws->moe_x), r, ws->moe_row, ws->moe_row_weight, rows, d * size / 16));
  else
    BCG_CUDA_CHECK(launch_k(moe_scatter_kernel<uint16_t>, grid, dim3(kMoeThreads), 0, st,
                            static_cast<const uint16_t*>(ws->xn), static_cast<uint16_t*>(ws->moe_x), r, ws->moe_row,
                            ws->moe_row_weight, rows, d * size / 2));
  if (T > 128 && moe_tensor(m, l, T, n_in, d)) {
    int one;
    BCG_TRY(expert_gemm(m, l, ws, T, ws->moe_x, l->w_experts_in, ws->moe_h, 0, n_in, d, unit, &one, st));
  } else {
    int s;
    BCG_TRY(expert_gemm(m, l, ws, T, ws->moe_x, l->w_experts_in, ws->moe_proj, ws->moe_proj_floats, n_in, d, BCG_EPI_F32,
                        &s, st));
    BCG_TRY(unit_rows(ws->moe_proj, s, static_cast<long long>(rows) * n_in, unit == BCG_EPI_GLU ? ws->moe_row_weight : nullptr,
                      ws->moe_h, m->act_dtype, rows, ff, unit, l->glu_limit, l->glu_alpha, st));
  }
  return expert_gemm(m, l, ws, T, ws->moe_h, l->w_experts_out, ws->moe_out, ws->moe_out_floats, d, ff, BCG_EPI_F32, splits,
                     st);
}

}  // namespace bcg
