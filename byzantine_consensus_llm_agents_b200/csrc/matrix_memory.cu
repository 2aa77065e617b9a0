// Matrix memory with exponential gates over ragged sequences, per head a state S [vdim][dim], a normalizer n [dim] and a running
// maximum m of the log gates, all fp32:
//     m' = max(f + m, i),   S <- exp(f + m - m') S + exp(i - m') v k^T,   n likewise with k alone,
//     o = S q / (max(|n . q|, exp(-m')) + 1e-6),   q scaled by dim^(-1/2);
//     i = cap tanh((z_i + b_i) / cap),  f = logsigmoid(cap tanh((z_f + b_f) / cap));
// then every head's o by its root mean square, times a weight and the sigmoid of an output gate.  A state is stored as
// [vdim + 1][dim] per head, n behind S; every block of 64 rows keeps its own copy of m, so that no CTA waits for another's.
//
//   memory_in      projection slabs -> q | k | v | output gate as activations, heads padded to multiples of 8 columns
//   memory_scan    portions token by token in fp32: the fp32 engine's kernel
//   memory_norm    denominators, head norms and output gates
#include "state_rows.cuh"
#include "kernels.h"

namespace bcg {

struct MemArgs {
  const float* proj;         // rows q | k | v | output gate, from column gate_col on input gates | forget gates
  int n_partials;
  long long pstride, ld;
  int gate_col;
  const float *bias, *norm;  // [2 heads], [heads * vdim]
  const int *positions, *slot_map, *seq_start, *state_slots;
  float *state, *top, *den;  // top: the running maxima
  void *x, *y;               // act [T][x_ld()], [T][heads * vdim]
  int heads, dim, vdim, n_tokens;
  float cap, scale, eps;

  __host__ __device__ int k_pad() const { return (dim + 7) / 8 * 8; }
  __host__ __device__ int v_pad() const { return (vdim + 7) / 8 * 8; }
  __host__ __device__ int x_ld() const { return 2 * heads * (k_pad() + v_pad()); }
  __host__ __device__ int blocks() const { return (vdim + kSsRows - 1) / kSsRows; }
  __host__ __device__ int inner() const { return heads * vdim; }
  __device__ __forceinline__ int q_col(int h) const { return h * k_pad(); }
  __device__ __forceinline__ int k_col(int h) const { return (heads + h) * k_pad(); }
  __device__ __forceinline__ int v_col(int h) const { return 2 * heads * k_pad() + h * v_pad(); }
  __device__ __forceinline__ int g_col(int h) const { return 2 * heads * k_pad() + (heads + h) * v_pad(); }
  __device__ __forceinline__ int first_of(int s) const { return seq_start ? seq_start[s] : s; }
  __device__ __forceinline__ int end_of(int s) const { return seq_start ? seq_start[s + 1] : s + 1; }
  __device__ __forceinline__ float* state_of(int slot, int h) const {
    return state + (static_cast<long long>(slot) * heads + h) * (vdim + 1) * dim;
  }
  __device__ __forceinline__ float* top_of(int slot, int h, int block) const {
    return top + (static_cast<long long>(slot) * heads + h) * blocks() + block;
  }
};

struct LogGates {
  float in, keep;
};
__device__ __forceinline__ LogGates log_gates(const MemArgs& a, float zi, float zf, int h) {
  LogGates g;
  g.in = a.cap * tanhf((zi + a.bias[h]) / a.cap);
  g.keep = -softplus_f32(-a.cap * tanhf((zf + a.bias[a.heads + h]) / a.cap));
  return g;
}
__device__ __forceinline__ LogGates load_gates(const MemArgs& a, long long t, int h) {
  const float* p = a.proj + t * a.ld + a.gate_col + h;
  return log_gates(a, slab_sum(p, a.n_partials, a.pstride), slab_sum(p + a.heads, a.n_partials, a.pstride), h);
}

// One step of the running maximum: what the old state and the new summand are multiplied by.
struct GateStep {
  float keep, add, top;
  __device__ __forceinline__ GateStep(float top0, const LogGates& g) {
    const float kept = g.keep + top0;
    top = fmaxf(kept, g.in);
    keep = decay_f32(kept - top);
    add = expf(g.in - top);
  }
};
__device__ __forceinline__ float denominator(float nq, float top) { return fmaxf(fabsf(nq), expf(-top)) + 1e-6f; }

// ------------------------------------------------------------------------------------------- inputs
constexpr int kMiThreads = 256;

template <typename T, int V>
__global__ void __launch_bounds__(kMiThreads)
memory_in_kernel(const MemArgs a, int blocks) {
  pdl_launch_dependents();
  pdl_wait();
  const long long t = blockIdx.x / blocks;
  const float* row = a.proj + t * a.ld;
  T* out = static_cast<T*>(a.x) + t * a.x_ld();
  const int nk = 2 * a.heads * a.dim, n = nk + 2 * a.heads * a.vdim;
  for (int c = (static_cast<int>(blockIdx.x % blocks) * kMiThreads + threadIdx.x) * V; c < n; c += blocks * kMiThreads * V) {
    const int e = c - nk;
    const int to = e < 0 ? c / a.dim * a.k_pad() + c % a.dim : 2 * a.heads * a.k_pad() + e / a.vdim * a.v_pad() + e % a.vdim;
    store_vec<V>(out + to, slab_sum_vec<V>(row + c, a.n_partials, a.pstride));
  }
}

// ------------------------------------------------------------------------------------------- token by token
template <typename T, int NP>
__global__ void __launch_bounds__(kSsThreads)
memory_scan_kernel(const MemArgs a) {
  using S = StateRows<NP>;
  const int h = blockIdx.x, block = blockIdx.y, p0 = block * kSsRows, sq = blockIdx.z;
  const int rows = min(kSsRows, a.vdim - p0), N = a.dim;
  pdl_launch_dependents();
  pdl_wait();
  const int t0 = a.first_of(sq), t1 = a.end_of(sq);
  if (t1 <= t0 || a.slot_map[t0] < 0) return;
  const int slot = a.state_slots[sq];
  float* st = a.state_of(slot, h) + static_cast<long long>(p0) * N;
  float* norm_row = a.state_of(slot, h) + static_cast<long long>(a.vdim) * N;
  const bool fresh = a.positions[t0] == 0;
  S s;
  float n[S::kQ][4], top = 0.f;      // block 0 has the normalizer
#pragma unroll
  for (int q = 0; q < S::kQ; ++q)
#pragma unroll
    for (int i = 0; i < 4; ++i) n[q][i] = !fresh && block == 0 && S::entry(q) + i < N ? norm_row[S::entry(q) + i] : 0.f;
  if (fresh) {
    s.zero();
  } else {
    s.load(st, rows, N);
    top = *a.top_of(slot, h, block);
  }
  const T* base = static_cast<const T*>(a.x);
  float v[S::kR], k[S::kQ][4], q[S::kQ][4];
  LogGates g;
  auto fetch = [&](int t) {
    const T* tok = base + static_cast<long long>(t) * a.x_ld();
    g = load_gates(a, t, h);
#pragma unroll
    for (int r = 0; r < S::kR; ++r) v[r] = S::row(r) < rows ? to_f32<T>(tok[a.v_col(h) + p0 + S::row(r)]) : 0.f;
#pragma unroll
    for (int j = 0; j < S::kQ; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int e = S::entry(j) + i;
        k[j][i] = e < N ? to_f32<T>(tok[a.k_col(h) + e]) : 0.f;
        q[j][i] = e < N ? a.scale * to_f32<T>(tok[a.q_col(h) + e]) : 0.f;
      }
  };
  fetch(t0);
  for (int t = t0; t < t1; ++t) {
    const GateStep step(top, g);
    top = step.top;
    float add[S::kR], kk[S::kQ][4], qq[S::kQ][4], nq = 0.f;
#pragma unroll
    for (int r = 0; r < S::kR; ++r) add[r] = step.add * v[r];
#pragma unroll
    for (int j = 0; j < S::kQ; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        kk[j][i] = k[j][i];
        qq[j][i] = q[j][i];
        n[j][i] = fmaf(step.keep, n[j][i], step.add * kk[j][i]);
        nq = fmaf(n[j][i], qq[j][i], nq);
      }
    if (t + 1 < t1) fetch(t + 1);
    const float y = s.token(step.keep, [&](int r) { return add[r]; }, kk, qq);
    const int p = S::row(S::mine());
    if (S::writes() && p < rows) static_cast<T*>(a.y)[static_cast<long long>(t) * a.inner() + h * a.vdim + p0 + p] = from_f32<T>(y);
    if (block == 0) {
#pragma unroll
      for (int m = S::kLanes / 2; m > 0; m >>= 1) nq += __shfl_xor_sync(0xffffffffu, nq, m);
      if (threadIdx.x == 0) a.den[static_cast<long long>(t) * a.heads + h] = denominator(nq, top);
    }
  }
  s.store(st, rows, N);
  if (threadIdx.x == 0) *a.top_of(slot, h, block) = top;
  if (block == 0 && threadIdx.x < S::kLanes) {
#pragma unroll
    for (int j = 0; j < S::kQ; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (S::entry(j) + i < N) norm_row[S::entry(j) + i] = n[j][i];
  }
}

// ------------------------------------------------------------------------------------------- norm
constexpr int kMnThreads = 256;

// A head of a token per warp.  GT: where the output gates are, activations of a.x (T) or columns of the projection's slabs (float, SLABS).
template <typename T, int V>
__global__ void __launch_bounds__(kMnThreads)
memory_norm_kernel(const MemArgs a, T* __restrict__ out, long long out_ld) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const long long unit = blockIdx.x * static_cast<long long>(kMnThreads / 32) + (threadIdx.x >> 5);
  if (unit >= static_cast<long long>(a.n_tokens) * a.heads) return;
  const long long t = unit / a.heads;
  const int h = static_cast<int>(unit % a.heads);
  const T* y = static_cast<const T*>(a.y) + t * a.inner() + h * a.vdim;
  const T* g = static_cast<const T*>(a.x) + t * a.x_ld() + a.g_col(h);
  const float* w = a.norm + h * a.vdim;
  float ss = 0.f;
  for (int c = lane * V; c < a.vdim; c += 32 * V) ss += load_vec<V>(y + c).sumsq();
  const float den = 1.0f / a.den[unit];
  const float f = den * rsqrtf(warp_sum(ss) * den * den / static_cast<float>(a.vdim) + a.eps);
  T* dst = out + t * out_ld + h * a.vdim;
  for (int c = lane * V; c < a.vdim; c += 32 * V) {
    Vec<V> o = load_vec<V>(y + c);
    const Vec<V> gate = load_vec<V>(g + c), ww = load_vec<V>(w + c);
#pragma unroll
    for (int k = 0; k < V; ++k) o.x[k] *= f * ww.x[k] * sigmoid_f32(gate.x[k]);
    store_vec<V>(dst + c, o);
  }
}

// ------------------------------------------------------------------------------------------- launches
template <typename T>
static int run_t(const MemArgs& a, int n_seqs, bool one_token, int mode, void* out, long long out_ld, cudaStream_t st) {
  const bool wide = ((a.dim | a.vdim) & 3) == 0 && a.ld % 4 == 0 && a.pstride % 4 == 0;
  const int n = 2 * a.heads * (a.dim + a.vdim);
  const int blocks = a.n_tokens <= 128 ? (n + kMiThreads * 4 - 1) / (kMiThreads * 4) : 1;
  const dim3 in_grid(static_cast<unsigned>(a.n_tokens * blocks));
  if (wide) BCG_CUDA_CHECK(launch_k(memory_in_kernel<T, 4>, in_grid, dim3(kMiThreads), 0, st, a, blocks));
  else BCG_CUDA_CHECK(launch_k(memory_in_kernel<T, 1>, in_grid, dim3(kMiThreads), 0, st, a, blocks));
  const dim3 grid(a.heads, a.blocks(), n_seqs);
  if (a.dim <= 32) BCG_CUDA_CHECK(launch_k(memory_scan_kernel<T, 32>, grid, dim3(kSsThreads), 0, st, a));
  else if (a.dim <= 64) BCG_CUDA_CHECK(launch_k(memory_scan_kernel<T, 64>, grid, dim3(kSsThreads), 0, st, a));
  else if (a.dim <= 128) BCG_CUDA_CHECK(launch_k(memory_scan_kernel<T, 128>, grid, dim3(kSsThreads), 0, st, a));
  else BCG_CUDA_CHECK(launch_k(memory_scan_kernel<T, 256>, grid, dim3(kSsThreads), 0, st, a));
  const dim3 norm_grid(static_cast<unsigned>((static_cast<long long>(a.n_tokens) * a.heads + kMnThreads / 32 - 1) / (kMnThreads / 32)));
  T* o = static_cast<T*>(out);
  if (a.vdim % 4 == 0 && out_ld % 4 == 0) BCG_CUDA_CHECK(launch_k(memory_norm_kernel<T, 4>, norm_grid, dim3(kMnThreads), 0, st, a, o, out_ld));
  else BCG_CUDA_CHECK(launch_k(memory_norm_kernel<T, 1>, norm_grid, dim3(kMnThreads), 0, st, a, o, out_ld));
  return BCG_OK;
}

int matrix_memory(const bcg_stack* m, const bcg_layer* l, const bcg_stack_ws* ws, const bcg_step_batch* b, int n_partials,
                  long long pstride, long long ld, int mode, cudaStream_t st) {
  if (!l->mem_bias || !l->mem_norm || !l->mem_state || !l->mem_max || !ws->ssm_x || !ws->ssm_y || !ws->mem_den || !b->state_slots ||
      l->heads <= 0 || l->dim <= 0 || l->dim > 256 || l->vdim <= 0 || l->vdim > 65535 * kSsRows || l->gate_cap <= 0.f || b->n_seqs > 65535) {
    set_last_error("bcg_matrix_memory", "bad layer (1..256 key channels) or too many sequences");
    return BCG_ERR_ARG;
  }
  MemArgs a = {};
  a.proj = ws->proj;
  a.n_partials = n_partials;
  a.pstride = pstride;
  a.ld = ld;
  a.gate_col = l->gate_col;
  a.bias = l->mem_bias;
  a.norm = l->mem_norm;
  a.positions = b->positions;
  a.slot_map = b->slot_map;
  a.seq_start = b->seq_start;
  a.state_slots = b->state_slots;
  a.state = l->mem_state;
  a.top = l->mem_max;
  a.den = ws->mem_den;
  a.x = ws->ssm_x;
  a.y = ws->ssm_y;
  a.heads = l->heads;
  a.dim = l->dim;
  a.vdim = l->vdim;
  a.n_tokens = b->T;
  a.cap = l->gate_cap;
  a.scale = 1.0f / sqrtf(static_cast<float>(l->dim));
  a.eps = m->eps;
  const bool one = b->T == b->n_seqs;
  return m->act_dtype == BCG_DT_F32 ? run_t<float>(a, b->n_seqs, one, mode, ws->mix, l->mix_ld, st)
                                    : run_t<__nv_bfloat16>(a, b->n_seqs, one, mode, ws->mix, l->mix_ld, st);
}

}  // namespace bcg
