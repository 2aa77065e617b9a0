// Matrix memory with exponential gates over ragged sequences, per head a state S [vdim][dim], a normalizer n [dim] and a running
// maximum m of the log gates, all fp32:
//     m' = max(f + m, i),   S <- exp(f + m - m') S + exp(i - m') v k^T,   n likewise with k alone,
//     o = S q / (max(|n . q|, exp(-m')) + 1e-6),   q scaled by dim^(-1/2);
//     i = cap tanh((z_i + b_i) / cap),  f = logsigmoid(cap tanh((z_f + b_f) / cap));
// then every head's o by its root mean square, times a weight and the sigmoid of an output gate.  A state is stored as
// [vdim + 1][dim] per head, n behind S; every block of 64 rows keeps its own copy of m, so that no CTA waits for another's.
//
//   memory_in      projection slabs -> q | k | v | output gate as activations, heads padded to multiples of 8 columns
//                  (long bf16 launches: the product writes them itself where no head needs padding)
//   chunks         portions (bf16): chunks of 64 tokens on tensor cores (state_chunk.cuh).  With c_t the running sum of f in a chunk,
//                  a_t = i_t - c_t and M_t the running maximum of a and the chunk's first m, m_t = c_t + M_t, so that all
//                  weights are exp(a_j - M_i), exp(m - M_i) and exp(a_j - M_last): no difference of large sums
//   memory_scan    portions token by token in fp32: the fp32 engine's kernel
//   memory_stream  single tokens: states pass through shared memory once, operands come straight from the slabs
//   memory_norm    denominators, head norms and output gates
#include "state_chunk.cuh"
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
  // what state_chunk.cuh asks for
  __device__ __forceinline__ int in_col(int h) const { return k_col(h); }
  __device__ __forceinline__ int out_col(int h) const { return q_col(h); }
  __device__ __forceinline__ int row_col(int h) const { return v_col(h); }
  __device__ __forceinline__ int entries() const { return dim; }
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

// ------------------------------------------------------------------------------------------- chunks
// Scalars of a chunk: -M | -a, both in log2 units | exp(-m) | exp(a - M_last) | first m in log2 units, exp(first m - M_last).
struct MemoryRule {
  using Args = MemArgs;
  static constexpr bool kNormalized = true;
  static constexpr int kScalars = 4 * kChTok + 4;
  const MemArgs& a;
  const int h, t0, t1, block;
  float zi[2], zf[2], top;    // gates of tokens 2 lane, 2 lane + 1 of the next chunk; running maximum in front of it
  __device__ __forceinline__ MemoryRule(const MemArgs& a_, int h_, int t0_, int t1_, int block_, bool fresh)
      : a(a_), h(h_), t0(t0_), t1(t1_), block(block_), zi{}, zf{}, top(0.f) {
    if (!fresh) top = *a.top_of(slot(), h, block);
  }
  __device__ __forceinline__ int slot() const { return a.state_slots[blockIdx.z]; }
  __device__ __forceinline__ void request(int chunk, int lane) {
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = t0 + chunk * kChTok + 2 * lane + e;
      const float* p = a.proj + static_cast<long long>(min(t, t1 - 1)) * a.ld + a.gate_col + h;
      zi[e] = slab_sum(p, a.n_partials, a.pstride);
      zf[e] = slab_sum(p + a.heads, a.n_partials, a.pstride);
    }
  }
  __device__ __forceinline__ void scalars(float* sc, int chunk, int lane) {
    float in[2], keep[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const LogGates g = log_gates(a, zi[e], zf[e], h);
      const bool there = t0 + chunk * kChTok + 2 * lane + e < t1;
      in[e] = there ? g.in : -INFINITY;
      keep[e] = there ? g.keep : 0.f;
    }
    float run = keep[0] + keep[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, run, o);
      if (lane >= o) run += v;
    }
    const float c1 = run, c0 = run - keep[1], a0 = in[0] - c0, a1 = in[1] - c1;
    float mx = fmaxf(a0, a1);
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, mx, o);
      if (lane >= o) mx = fmaxf(mx, v);
    }
    const float before = __shfl_up_sync(0xffffffffu, mx, 1);
    const float m0 = fmaxf(fmaxf(top, lane > 0 ? before : top), a0), m1 = fmaxf(m0, a1);
    const float last = __shfl_sync(0xffffffffu, m1, 31);
    *reinterpret_cast<float2*>(sc + 2 * lane) = make_float2(-m0 * kSsLog2e, -m1 * kSsLog2e);
    *reinterpret_cast<float2*>(sc + kChTok + 2 * lane) = make_float2(-a0 * kSsLog2e, -a1 * kSsLog2e);
    *reinterpret_cast<float2*>(sc + 2 * kChTok + 2 * lane) = make_float2(expf(-(c0 + m0)), expf(-(c1 + m1)));
    *reinterpret_cast<float2*>(sc + 3 * kChTok + 2 * lane) = make_float2(expf(a0 - last), expf(a1 - last));
    if (lane == 0) *reinterpret_cast<float2*>(sc + 4 * kChTok) = make_float2(top * kSsLog2e, decay_f32(top - last));
    top = __shfl_sync(0xffffffffu, run, 31) + last;
  }
  __device__ __forceinline__ float2 weights(const float* sc, float mi, int j) const {
    const float2 aj = *reinterpret_cast<const float2*>(sc + kChTok + j);
    return make_float2(a.scale * ex2_approx(mi - aj.x), a.scale * ex2_approx(mi - aj.y));
  }
  __device__ __forceinline__ float2 readout(const float* sc, int i) const {
    const float2 m = *reinterpret_cast<const float2*>(sc + i);
    const float m0 = sc[4 * kChTok];
    return make_float2(a.scale * ex2_approx(m0 + m.x), a.scale * ex2_approx(m0 + m.y));
  }
  __device__ __forceinline__ float keep(const float* sc) const { return sc[4 * kChTok + 1]; }
  __device__ __forceinline__ float skip() const { return 0.f; }
  // sum: row i of M; nc: n . q without the scale, n at the chunk's start
  __device__ __forceinline__ void denominator(const float* sc, int i, int first, float sum, float nc) const {
    const float r = fmaf(a.scale * ex2_approx(sc[4 * kChTok] + sc[i]), nc, sum);
    if (first + i < t1) a.den[static_cast<long long>(first + i) * a.heads + h] = fmaxf(fabsf(r), sc[2 * kChTok + i]) + 1e-6f;
  }
  __device__ __forceinline__ void finish(int, int, int, bool) const {
    if (threadIdx.x == 0) *a.top_of(slot(), h, block) = top;
  }
};

// ------------------------------------------------------------------------------------------- single tokens
// A column of the projection on the way: up to four slabs are requested ahead, value() is their sum.
struct SlabItem {
  const float* p;
  float v[4];
  __device__ __forceinline__ void request(const MemArgs& a, const float* p_) {
    p = p_;
#pragma unroll
    for (int q = 0; q < 4; ++q) v[q] = p && q < a.n_partials ? p[q * a.pstride] : 0.f;
  }
  __device__ __forceinline__ float value(const MemArgs& a) const {
    float x = (v[0] + v[1]) + (v[2] + v[3]);
    if (p)
      for (int q = 4; q < a.n_partials; ++q) x += p[q * a.pstride];
    return x;
  }
};

// A unit is 64 rows of a token's head (fewer at a head's end; the normalizer comes with a head's first ones), a CTA has consecutive
// ones: queries, keys and gates are made once per head.  Warps 0-7 compute, warp 8 moves states: a stage is filled, worked on in
// place, stored, and filled again once it has been read.  Rows of 16 bytes' multiple.
constexpr int kMtStages = 3, kMtThreads = kSsThreads + 32;
template <int NP>
struct MtCfg {
  static constexpr int kStage = (kSsRows + 1) * NP;                       // floats
  static constexpr int kGates = 2 * NP, kHead = kGates + 4;               // of a head: k | q | keep, add, exp(-m), m
  static constexpr int kSmem = (kMtStages * kStage + 2 * kSsRows + 2 * kHead) * 4 + 64;
  static constexpr int kCtasPerSm = NP <= 128 ? 2 : 1;
};

// A walk over units: blocks of rows first, then heads, then tokens.
struct MemWalk {
  int t, h, pb;
  __device__ __forceinline__ MemWalk(const MemArgs& a, int u) {
    const int r = u / a.blocks();
    pb = u - r * a.blocks();
    t = r / a.heads;
    h = r - t * a.heads;
  }
  __device__ __forceinline__ void next(const MemArgs& a) {
    if (++pb < a.blocks()) return;
    pb = 0;
    if (++h < a.heads) return;
    h = 0;
    ++t;
  }
  __device__ __forceinline__ int rows(const MemArgs& a) const { return min(kSsRows, a.vdim - pb * kSsRows); }
};

template <typename T, int NP>
__global__ void __launch_bounds__(kMtThreads, MtCfg<NP>::kCtasPerSm)
memory_stream_kernel(const MemArgs a, int n_units) {
  using S = StateRows<NP>;
  using C = MtCfg<NP>;
  constexpr int kItems = (2 * NP + kSsThreads - 1) / kSsThreads, kGateThread = kSsThreads - 1;
  extern __shared__ __align__(128) float st_raw[];
  float* vs = st_raw + kMtStages * C::kStage;                   // [2][rows]
  float* hs = vs + 2 * kSsRows;                                 // [2][head]
  uint64_t* full = reinterpret_cast<uint64_t*>(hs + 2 * C::kHead);   // [stages] a state has arrived
  uint64_t* done = full + kMtStages;                            // [stages] it has been worked on
  const int N = a.dim;
  const int u0 = static_cast<int>(static_cast<long long>(n_units) * blockIdx.x / gridDim.x);
  const int n = static_cast<int>(static_cast<long long>(n_units) * (blockIdx.x + 1) / gridDim.x) - u0;
  pdl_launch_dependents();
  if (threadIdx.x == 0) {
    for (int i = 0; i < kMtStages; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&done[i], kSsThreads);
    }
    fence_barrier_init();
  }
  __syncthreads();
  // States, slots and positions were written by earlier steps, which are complete before any kernel of this step starts.
  if (threadIdx.x >= kSsThreads) {
    if (threadIdx.x == kSsThreads) {
      MemWalk in(a, u0), out = in;
      auto state_of = [&](const MemWalk& u) { return a.state_of(a.state_slots[u.t], u.h); };
      for (int i = 0; i < n + kMtStages - 1; ++i) {
        if (i < n) {
          const uint32_t bytes = static_cast<uint32_t>(in.rows(a) * N * 4), extra = in.pb == 0 ? static_cast<uint32_t>(N * 4) : 0u;
          const float* head = state_of(in);
          float* stage = st_raw + (i % kMtStages) * C::kStage;
          // the stage's previous state (unit i - stages) was stored a turn ago
          if (i >= kMtStages) asm volatile("cp.async.bulk.wait_group.read 0;" ::: "memory");
          mbar_arrive_expect_tx(&full[i % kMtStages], bytes + extra);
          bulk_load_1d(stage, head + static_cast<long long>(in.pb) * kSsRows * N, bytes, &full[i % kMtStages]);
          if (extra) bulk_load_1d(stage + kSsRows * NP, head + static_cast<long long>(a.vdim) * N, extra, &full[i % kMtStages]);
          in.next(a);
        }
        const int j = i - (kMtStages - 1);
        if (j >= 0) {
          float* head = state_of(out);
          const float* stage = st_raw + (j % kMtStages) * C::kStage;
          const bool idle = a.slot_map[out.t] < 0;
          mbar_wait(&done[j % kMtStages], (j / kMtStages) & 1);
          if (!idle) {
            bulk_store_1d(head + static_cast<long long>(out.pb) * kSsRows * N, stage, static_cast<uint32_t>(out.rows(a) * N * 4));
            if (out.pb == 0) bulk_store_1d(head + static_cast<long long>(a.vdim) * N, stage + kSsRows * NP, static_cast<uint32_t>(N * 4));
          }
          out.next(a);
        }
      }
      asm volatile("cp.async.bulk.wait_group 0;" ::: "memory");
    }
    return;
  }
  const int tid = static_cast<int>(threadIdx.x);
  MemWalk u(a, u0);
  SlabItem v, kq[kItems], gi, gf;   // threads up to kSsRows have a value, all have some of k and q, one has the gates
  float top = 0.f;
  auto v_request = [&](const MemWalk& w) {
    const float* row = a.proj + static_cast<long long>(w.t) * a.ld + 2 * a.heads * N + w.h * a.vdim + w.pb * kSsRows;
    v.request(a, tid < w.rows(a) ? row + tid : nullptr);
  };
  auto head_request = [&](const MemWalk& w) {
    const float* row = a.proj + static_cast<long long>(w.t) * a.ld;
#pragma unroll
    for (int j = 0; j < kItems; ++j) {
      const int e = tid + j * kSsThreads, c = e % NP;
      kq[j].request(a, e < 2 * NP && c < N ? row + (e < NP ? a.heads + w.h : w.h) * N + c : nullptr);
    }
    if (tid == kGateThread) {
      gi.request(a, row + a.gate_col + w.h);
      gf.request(a, row + a.gate_col + a.heads + w.h);
      top = a.positions[w.t] == 0 ? 0.f : *a.top_of(a.state_slots[w.t], w.h, w.pb);     // nobody else writes this copy
    }
  };
  pdl_wait();
  v_request(u);
  head_request(u);
  bool new_head = true;
  int side = 1;                     // of hs
  for (int i = 0; i < n; ++i) {
    float* vi = vs + (i & 1) * kSsRows;
    if (tid < kSsRows) vi[tid] = v.value(a);
    if (new_head) {
      side ^= 1;
      float* hd = hs + side * C::kHead;
#pragma unroll
      for (int j = 0; j < kItems; ++j) {
        const int e = tid + j * kSsThreads;
        if (e < 2 * NP) hd[e] = (e < NP ? 1.0f : a.scale) * kq[j].value(a);
      }
      if (tid == kGateThread) {
        const GateStep step(top, log_gates(a, gi.value(a), gf.value(a), u.h));
        *reinterpret_cast<float4*>(hd + C::kGates) = make_float4(step.keep, step.add, expf(-step.top), step.top);
      }
    }
    const bool idle = a.slot_map[u.t] < 0, fresh = a.positions[u.t] == 0;
    MemWalk w = u;
    new_head = false;
    if (i + 1 < n) {                // requested now, used a turn later
      w.next(a);
      new_head = w.pb == 0;
      v_request(w);
      if (new_head) head_request(w);
    }
    asm volatile("bar.sync 1, %0;" ::"n"(kSsThreads) : "memory");     // operands are there
    mbar_wait(&full[i % kMtStages], (i / kMtStages) & 1);
    if (!idle) {
      float* st = st_raw + (i % kMtStages) * C::kStage;
      const float* hd = hs + side * C::kHead;
      const float4 gates = *reinterpret_cast<const float4*>(hd + C::kGates);
      float k[S::kQ][4], q[S::kQ][4];
#pragma unroll
      for (int j = 0; j < S::kQ; ++j) {
        const float4 kv = *reinterpret_cast<const float4*>(hd + S::entry(j)), qv = *reinterpret_cast<const float4*>(hd + NP + S::entry(j));
        k[j][0] = kv.x; k[j][1] = kv.y; k[j][2] = kv.z; k[j][3] = kv.w;
        q[j][0] = qv.x; q[j][1] = qv.y; q[j][2] = qv.z; q[j][3] = qv.w;
      }
      const int rows = u.rows(a);
      auto add = [&](int r) { return gates.y * vi[S::row(r)]; };
      const float y = rows == kSsRows && N == NP ? S::template token_in_place<true>(st, rows, N, fresh, gates.x, add, k, q)
                                                 : S::template token_in_place<false>(st, rows, N, fresh, gates.x, add, k, q);
      const int p = S::row(S::mine());
      if (S::writes() && p < rows)
        static_cast<T*>(a.y)[static_cast<long long>(u.t) * a.inner() + u.h * a.vdim + u.pb * kSsRows + p] = from_f32<T>(y);
      if (u.pb == 0 && tid >= kSsThreads - 32) {       // the normalizer; groups of fewer than 32 lanes hold it several times
        float nq = 0.f;
        float4 x[S::kQ];
#pragma unroll
        for (int j = 0; j < S::kQ; ++j) {
          x[j] = make_float4(0.f, 0.f, 0.f, 0.f);
          if (S::entry(j) < N && !fresh) x[j] = *reinterpret_cast<const float4*>(st + kSsRows * NP + S::entry(j));
          x[j].x = fmaf(gates.x, x[j].x, gates.y * k[j][0]);
          x[j].y = fmaf(gates.x, x[j].y, gates.y * k[j][1]);
          x[j].z = fmaf(gates.x, x[j].z, gates.y * k[j][2]);
          x[j].w = fmaf(gates.x, x[j].w, gates.y * k[j][3]);
          nq = fmaf(x[j].w, q[j][3], fmaf(x[j].z, q[j][2], fmaf(x[j].y, q[j][1], fmaf(x[j].x, q[j][0], nq))));
        }
        __syncwarp();
#pragma unroll
        for (int j = 0; j < S::kQ; ++j)
          if (S::entry(j) < N && tid >= kSsThreads - S::kLanes) *reinterpret_cast<float4*>(st + kSsRows * NP + S::entry(j)) = x[j];
#pragma unroll
        for (int m = S::kLanes / 2; m > 0; m >>= 1) nq += __shfl_xor_sync(0xffffffffu, nq, m);
        if (tid == kGateThread) a.den[static_cast<long long>(u.t) * a.heads + u.h] = fmaxf(fabsf(nq), gates.z) + 1e-6f;
      }
      if (tid == kGateThread) *a.top_of(a.state_slots[u.t], u.h, u.pb) = gates.w;
      fence_proxy_async();
    }
    mbar_arrive(&done[i % kMtStages]);
    u = w;
  }
}

// ------------------------------------------------------------------------------------------- norm
constexpr int kMnThreads = 256;

__device__ __forceinline__ float sigmoid_fast(float x) { return __fdividef(1.0f, 1.0f + __expf(-x)); }

// A head of a token per warp.  SLABS: output gates are columns of the projection, else of a.x.  Up to NV vectors per lane stay in
// registers between the sum of squares and the output (NV = 0: any number, read twice).
template <typename T, int V, bool SLABS, int NV>
__global__ void __launch_bounds__(kMnThreads)
memory_norm_kernel(const MemArgs a, T* __restrict__ out, long long out_ld) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31, unit = blockIdx.x * (kMnThreads / 32) + (threadIdx.x >> 5);
  const int tok = unit / a.heads, h = unit - tok * a.heads;
  if (tok >= a.n_tokens) return;
  const long long t = tok;
  const T* y = static_cast<const T*>(a.y) + t * a.inner() + h * a.vdim;
  const T* g = static_cast<const T*>(a.x) + t * a.x_ld() + a.g_col(h);
  const float* slabs = a.proj + t * a.ld + 2 * a.heads * a.dim + (a.heads + h) * a.vdim;
  const float* w = a.norm + h * a.vdim;
  T* dst = out + t * out_ld + h * a.vdim;
  const float den = 1.0f / a.den[unit];
  auto gate_of = [&](int c) {
    if constexpr (SLABS) return slab_sum_vec<V>(slabs + c, a.n_partials, a.pstride);
    else return load_vec<V>(g + c);
  };
  auto finish = [&](Vec<V> o, const Vec<V>& gate, float f, int c) {
    const Vec<V> ww = load_vec<V>(w + c);
#pragma unroll
    for (int k = 0; k < V; ++k) o.x[k] *= f * ww.x[k] * (sizeof(T) == 2 ? sigmoid_fast(gate.x[k]) : sigmoid_f32(gate.x[k]));
    store_vec<V>(dst + c, o);
  };
  float ss = 0.f;
  Vec<V> o[NV > 0 ? NV : 1], gate[NV > 0 ? NV : 1];
  if constexpr (NV > 0) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * 32 + lane) * V;
      if (c < a.vdim) {
        o[i] = load_vec<V>(y + c);
        gate[i] = gate_of(c);
      } else {
        o[i] = Vec<V>{};
      }
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) ss += o[i].sumsq();
  } else {
    for (int c = lane * V; c < a.vdim; c += 32 * V) ss += load_vec<V>(y + c).sumsq();
  }
  const float f = den * rsqrtf(warp_sum(ss) * den * den / static_cast<float>(a.vdim) + a.eps);
  if constexpr (NV > 0) {
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if ((i * 32 + lane) * V < a.vdim) finish(o[i], gate[i], f, (i * 32 + lane) * V);
  } else {
    for (int c = lane * V; c < a.vdim; c += 32 * V) finish(load_vec<V>(y + c), gate_of(c), f, c);
  }
}

// ------------------------------------------------------------------------------------------- launches
template <typename T, int NP>
static int launch_stream(const MemArgs& a, int n_seqs, cudaStream_t st) {
  using C = MtCfg<NP>;
  const long long units = static_cast<long long>(n_seqs) * a.heads * a.blocks(), most = 148ll * C::kCtasPerSm;
  if (units > 0x7fffffff) {
    set_last_error("bcg_matrix_memory", "too many sequences");
    return BCG_ERR_TOO_LARGE;
  }
  BCG_TRY(ensure_dynamic_smem(reinterpret_cast<const void*>(memory_stream_kernel<T, NP>), C::kSmem));
  BCG_CUDA_CHECK(launch_k(memory_stream_kernel<T, NP>, dim3(static_cast<unsigned>(units < most ? units : most)), dim3(kMtThreads), C::kSmem, st,
                          a, static_cast<int>(units)));
  return BCG_OK;
}

template <typename T, int NP>
static int run_np(const MemArgs& a, int n_seqs, bool stream, bool chunks, cudaStream_t st) {
  const dim3 grid(a.heads, a.blocks(), n_seqs);
  if (stream) return launch_stream<T, NP>(a, n_seqs, st);
  if (chunks) return launch_chunks<(NP < 64 ? 64 : NP), MemoryRule>(a, grid, st);
  BCG_CUDA_CHECK(launch_k(memory_scan_kernel<T, NP>, grid, dim3(kSsThreads), 0, st, a));
  return BCG_OK;
}

template <typename T, int V, bool SLABS>
static int launch_norm(const MemArgs& a, void* out, long long out_ld, cudaStream_t st) {
  const dim3 grid(static_cast<unsigned>((static_cast<long long>(a.n_tokens) * a.heads + kMnThreads / 32 - 1) / (kMnThreads / 32)));
  T* o = static_cast<T*>(out);
  const dim3 block(kMnThreads);
  if (V == 4 && a.vdim <= 256) BCG_CUDA_CHECK(launch_k(memory_norm_kernel<T, V, SLABS, 2>, grid, block, 0, st, a, o, out_ld));
  else if (V == 4 && a.vdim <= 512) BCG_CUDA_CHECK(launch_k(memory_norm_kernel<T, V, SLABS, 4>, grid, block, 0, st, a, o, out_ld));
  else BCG_CUDA_CHECK(launch_k(memory_norm_kernel<T, V, SLABS, 0>, grid, block, 0, st, a, o, out_ld));
  return BCG_OK;
}

template <typename T>
static int run_t(const MemArgs& a, int n_seqs, bool one_token, int mode, bool split, void* out, long long out_ld, cudaStream_t st) {
  const bool wide = ((a.dim | a.vdim) & 3) == 0 && (split || a.ld % 4 == 0) && a.pstride % 4 == 0 && out_ld % 4 == 0;
  const bool stream = one_token && mode == 0 && !split && a.dim % 4 == 0, chunks = sizeof(T) == 2 && mode == 0;
  if (!stream && !split) {
    const int n = 2 * a.heads * (a.dim + a.vdim);
    const int blocks = a.n_tokens <= 128 ? (n + kMiThreads * 4 - 1) / (kMiThreads * 4) : 1;
    const dim3 grid(static_cast<unsigned>(a.n_tokens * blocks));
    if (wide) BCG_CUDA_CHECK(launch_k(memory_in_kernel<T, 4>, grid, dim3(kMiThreads), 0, st, a, blocks));
    else BCG_CUDA_CHECK(launch_k(memory_in_kernel<T, 1>, grid, dim3(kMiThreads), 0, st, a, blocks));
  }
  if (a.dim <= 32) BCG_TRY((run_np<T, 32>(a, n_seqs, stream, chunks, st)));
  else if (a.dim <= 64) BCG_TRY((run_np<T, 64>(a, n_seqs, stream, chunks, st)));
  else if (a.dim <= 128) BCG_TRY((run_np<T, 128>(a, n_seqs, stream, chunks, st)));
  else BCG_TRY((run_np<T, 256>(a, n_seqs, stream, chunks, st)));
  if (stream) return wide ? launch_norm<T, 4, true>(a, out, out_ld, st) : launch_norm<T, 1, true>(a, out, out_ld, st);
  return wide ? launch_norm<T, 4, false>(a, out, out_ld, st) : launch_norm<T, 1, false>(a, out, out_ld, st);
}

int matrix_memory(const bcg_stack* m, const bcg_layer* l, const bcg_stack_ws* ws, const bcg_step_batch* b, int n_partials,
                  long long pstride, long long ld, int mode, bool split, cudaStream_t st) {
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
  a.gate_col = split ? 0 : l->gate_col;
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
  return m->act_dtype == BCG_DT_F32 ? run_t<float>(a, b->n_seqs, one, mode, split, ws->mix, l->mix_ld, st)
                                    : run_t<__nv_bfloat16>(a, b->n_seqs, one, mode, split, ws->mix, l->mix_ld, st);
}

}  // namespace bcg
