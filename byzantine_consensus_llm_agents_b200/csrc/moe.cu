// Mixture of experts: T tokens, `top` experts each.
//   (routing happens in the kernel that reads the input projection: moe.cuh)
//   moe_scatter    rows of the normed stream -> rows sorted by expert
//   grouped GEMM   every expert's gate and up matrices over its rows (gemm_tcgen05.cu; CUDA cores for fp32)
//   moe_glu        clamped gated unit of split-K slabs (prompts: in the GEMM's epilogue)
//   grouped GEMM   down matrices, fp32 rows; the norm kernel adds a token's rows to its residual
// The routing weight scales an expert's input.  Its products are linear in that input, so the weight is applied to
// the fp32 accumulators of gate and up instead of the bf16 operand.
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

// z: slabs of [rows][2 * ff_ld], 16 gate columns beside 16 up columns; a warp-wide run of columns per thread group.
template <typename T>
__global__ void __launch_bounds__(kMoeThreads)
moe_glu_kernel(const float* __restrict__ z, int n_partials, long long pstride, const float* __restrict__ row_weight,
               T* __restrict__ out, int ff_ld, float limit, float alpha) {
  pdl_launch_dependents();
  pdl_wait();
  const long long row = blockIdx.x;
  const float w = row_weight ? row_weight[row] : 1.f;
  const float* src = z + row * 2 * ff_ld;
  for (int c = (blockIdx.y * kMoeThreads + threadIdx.x) * 4; c < ff_ld; c += gridDim.y * kMoeThreads * 4) {
    const float* p = src + (c >> 4) * 32 + (c & 15);
    const Vec<4> g = slab_sum_vec<4>(p, n_partials, pstride), u = slab_sum_vec<4>(p + 16, n_partials, pstride);
    Vec<4> y;
#pragma unroll
    for (int k = 0; k < 4; ++k) y.x[k] = clamped_glu(w * g.x[k], w * u.x[k], limit, alpha);
    store_vec<4>(out + row * ff_ld + c, y);
  }
}

int clamped_glu_rows(const float* z, int n_partials, long long pstride, const float* row_weight, void* out, int act_dtype,
                     int rows, int ff_ld, float limit, float alpha, cudaStream_t st) {
  if (!z || !out || rows <= 0 || ff_ld <= 0 || ff_ld % 16 || n_partials < 1) {
    set_last_error("bcg_clamped_glu", "bad argument (ff % 16)");
    return BCG_ERR_ARG;
  }
  const int per = rows <= 1024 ? (ff_ld + kMoeThreads * 4 - 1) / (kMoeThreads * 4) : 1;
  const dim3 grid(rows, per);
  if (act_dtype == BCG_DT_F32)
    BCG_CUDA_CHECK(launch_k(moe_glu_kernel<float>, grid, dim3(kMoeThreads), 0, st, z, n_partials, pstride, row_weight,
                            static_cast<float*>(out), ff_ld, limit, alpha));
  else
    BCG_CUDA_CHECK(launch_k(moe_glu_kernel<__nv_bfloat16>, grid, dim3(kMoeThreads), 0, st, z, n_partials, pstride, row_weight,
                            static_cast<__nv_bfloat16*>(out), ff_ld, limit, alpha));
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
  const dim3 grid((rows + kMoeThreads / 32 - 1) / (kMoeThreads / 32));
  if (d * size % 16 == 0)
    BCG_CUDA_CHECK(launch_k(moe_scatter_kernel<uint4>, grid, dim3(kMoeThreads), 0, st, static_cast<const uint4*>(ws->xn),
                            static_cast<uint4*>(ws->moe_x), r, ws->moe_row, ws->moe_row_weight, rows, d * size / 16));
  else
    BCG_CUDA_CHECK(launch_k(moe_scatter_kernel<uint16_t>, grid, dim3(kMoeThreads), 0, st,
                            static_cast<const uint16_t*>(ws->xn), static_cast<uint16_t*>(ws->moe_x), r, ws->moe_row,
                            ws->moe_row_weight, rows, d * size / 2));
  if (T > 128 && moe_tensor(m, l, T, 2 * ff, d)) {
    int one;
    BCG_TRY(expert_gemm(m, l, ws, T, ws->moe_x, l->w_experts_in, ws->moe_h, 0, 2 * ff, d, BCG_EPI_GLU, &one, st));
  } else {
    int s;
    BCG_TRY(expert_gemm(m, l, ws, T, ws->moe_x, l->w_experts_in, ws->moe_proj, ws->moe_proj_floats, 2 * ff, d, BCG_EPI_F32,
                        &s, st));
    BCG_TRY(clamped_glu_rows(ws->moe_proj, s, static_cast<long long>(rows) * 2 * ff, ws->moe_row_weight, ws->moe_h,
                             m->act_dtype, rows, ff, l->glu_limit, l->glu_alpha, st));
  }
  return expert_gemm(m, l, ws, T, ws->moe_h, l->w_experts_out, ws->moe_out, ws->moe_out_floats, d, ff, BCG_EPI_F32, splits,
                     st);
}

}  // namespace bcg
