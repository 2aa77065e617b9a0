// State-space mixer with one decay per head (state-space duality) over ragged sequences, state in fp32:
//     S <- exp(-rate * step) S + step * B x^T,      y = S^T C + skip * x,      step = softplus(. + bias),
// x, B and C behind a causal convolution per channel and silu; then  y * silu(z), an RMS norm in equal parts.
// A state is stored as [vdim][n] per head, rows of its n entries.
//
//   ssm_conv    projection slabs -> convolved x | B | C (activations, heads and groups padded to multiples of 8 columns)
//               and steps; the inputs ahead of a portion come from the convolution's state
//   chunks      portions (bf16): chunks of 64 tokens on tensor cores (state_chunk.cuh).  Inside a chunk the recurrence is a product,
//                   y_i = exp(c_i) S^T C_i + sum_{j <= i} exp(c_i - c_j) step_j (B_j . C_i) x_j,   c = running sum of -rate * step,
//               and the state moves once per chunk.  Everything is held transposed (rows = entries of a head's output), so
//               that the state stays in fp32 accumulators and becomes an operand without leaving the registers.  Weights (decays,
//               steps) are formed in fp32; what they add to the state enters its product as two bf16 halves (hi + lo),
//               what is only read out is rounded like any activation.
//   ssm_scan    portions token by token in fp32: the fp32 engine's kernel
//   ssm_token   one token per sequence (decode): convolution and recurrence in one kernel, a head per CTA; the states are
//               requested before the dependency wait
//   ssm_stream  the same with the states streamed through shared memory: a CTA has a list of heads, bulk copies of the
//               next ones' states in flight both ways, and the next one's operands requested a turn ahead
//   ssm_norm    gate and norm of the outputs
// The convolution's state moves on where nobody reads it any more: behind the chunks or the scan, and in ssm_norm for
// single tokens (whose B and C every head of a group convolves for itself).
#include "state_chunk.cuh"
#include "kernels.h"

namespace bcg {

struct SsmArgs {
  const float* proj;         // rows z | x | B | C | step from column col on, pitch ld
  int n_partials;
  long long pstride, ld;
  int col;
  const float *conv_w, *conv_b, *step_bias, *rate, *skip, *norm;
  const int *positions, *slot_map, *row_seq, *seq_start, *state_slots;
  float *state, *conv_state, *step;
  void *x, *y;
  int heads, vdim, n, groups, taps, parts, n_tokens;
  float eps;

  __host__ __device__ int inner() const { return heads * vdim; }
  __host__ __device__ int channels() const { return heads * vdim + 2 * groups * n; }
  __host__ __device__ int x_pad() const { return (vdim + 7) / 8 * 8; }
  __host__ __device__ int n_pad() const { return (n + 7) / 8 * 8; }
  __host__ __device__ int x_ld() const { return heads * x_pad() + 2 * groups * n_pad(); }
  __device__ __forceinline__ int x_col(int c) const {        // place of channel c in x
    if (c < inner()) return c / vdim * x_pad() + c % vdim;
    c -= inner();
    return heads * x_pad() + c / n * n_pad() + c % n;
  }
  __device__ __forceinline__ int b_col(int g) const { return heads * x_pad() + g * n_pad(); }
  __device__ __forceinline__ int c_col(int g) const { return heads * x_pad() + (groups + g) * n_pad(); }
  // what state_chunk.cuh asks for: columns of a head, entries of a state row, a head's state
  __device__ __forceinline__ int in_col(int h) const { return b_col(h / (heads / groups)); }
  __device__ __forceinline__ int out_col(int h) const { return c_col(h / (heads / groups)); }
  __device__ __forceinline__ int row_col(int h) const { return h * x_pad(); }
  __device__ __forceinline__ int entries() const { return n; }
  __device__ __forceinline__ float* state_of(int slot, int h) const { return state + (static_cast<long long>(slot) * heads + h) * vdim * n; }
  __device__ __forceinline__ const float* row(long long t) const { return proj + t * ld + col; }
  __device__ __forceinline__ int seq_of(int t) const { return row_seq ? row_seq[t] : t; }
  __device__ __forceinline__ int first_of(int s) const { return seq_start ? seq_start[s] : s; }
  __device__ __forceinline__ int end_of(int s) const { return seq_start ? seq_start[s + 1] : s + 1; }
};

__device__ __forceinline__ float silu_f32(float x) { return x * sigmoid_f32(x); }
// silu of what becomes an activation of type T: the short exponential where that is rounded to bf16
template <typename T>
__device__ __forceinline__ float silu_act(float x) {
  return sizeof(T) == 2 ? __fdividef(x, 1.0f + __expf(-x)) : silu_f32(x);
}
// ------------------------------------------------------------------------------------------- convolution
constexpr int kConvThreads = 128;

// V channels of the convolution's input at token t - k of the sequence that starts at token t0 of the step.
template <int V>
__device__ __forceinline__ Vec<V> conv_input(const SsmArgs& a, int c, int t, int k, int t0, int slot, bool fresh) {
  if (t - k >= t0) return slab_sum_vec<V>(a.row(t - k) + a.inner() + c, a.n_partials, a.pstride);
  Vec<V> x;
#pragma unroll
  for (int i = 0; i < V; ++i) x.x[i] = 0.f;
  if (!fresh)
    x = load_vec<V>(a.conv_state + (static_cast<long long>(slot) * (a.taps - 1) + (a.taps - 1) + (t - t0) - k) * a.channels() + c);
  return x;
}

constexpr int kConvAhead = 4;     // inputs in flight per thread

// TAPS: a window of inputs in registers; 0: any number of taps, every input loaded where it is used.  ONE: one slab.
template <typename T, int V, int TAPS, bool ONE>
__global__ void __launch_bounds__(kConvThreads, V == 4 ? 8 : 12)
ssm_conv_kernel(const SsmArgs a, int run, int conv_blocks) {
  pdl_launch_dependents();
  pdl_wait();
  const int r0 = blockIdx.y * run, r1 = min(a.n_tokens, r0 + run);
  if (static_cast<int>(blockIdx.x) >= conv_blocks) {
    const int h = (blockIdx.x - conv_blocks) * kConvThreads + threadIdx.x;
    if (h >= a.heads) return;
    for (int t = r0; t < r1; ++t)
      a.step[static_cast<long long>(t) * a.heads + h] =
          softplus_f32(slab_sum(a.row(t) + a.inner() + a.channels() + h, a.n_partials, a.pstride) + a.step_bias[h]);
    return;
  }
  const int c = (blockIdx.x * kConvThreads + threadIdx.x) * V, ch = a.channels(), x_ld = a.x_ld();
  if (c >= ch) return;
  T* out = static_cast<T*>(a.x) + a.x_col(c);
  const float* in = a.row(0) + a.inner() + c;
  const Vec<V> bias = load_vec<V>(a.conv_b + c);
  constexpr int W = TAPS > 0 ? TAPS : 1;
  Vec<V> w[W], hist[W];            // hist[k - 1]: input of token t - k
  if constexpr (TAPS > 0) {
#pragma unroll
    for (int k = 0; k < TAPS; ++k) w[k] = load_vec<V>(a.conv_w + static_cast<long long>(k) * ch + c);
  }
  for (int t = r0; t < r1;) {      // a sequence's part of the run
    const int s = a.seq_of(t), t0 = a.first_of(s), t_end = min(r1, a.end_of(s)), slot = a.state_slots[s];
    const bool fresh = a.positions[t0] == 0;
    if constexpr (TAPS > 1) {
#pragma unroll
      for (int k = 1; k < TAPS; ++k) hist[k - 1] = conv_input<V>(a, c, t, k, t0, slot, fresh);
    }
    for (; t < t_end; t += kConvAhead) {
      Vec<V> x[kConvAhead];
#pragma unroll
      for (int j = 0; j < kConvAhead; ++j) {
        const float* p = in + static_cast<long long>(min(t + j, t_end - 1)) * a.ld;
        x[j] = ONE ? load_vec<V>(p) : slab_sum_vec<V>(p, a.n_partials, a.pstride);
      }
#pragma unroll
      for (int j = 0; j < kConvAhead; ++j) {
        if (t + j >= t_end) break;
        Vec<V> y = bias;
        if constexpr (TAPS > 0) {
#pragma unroll
          for (int i = 0; i < V; ++i) {
#pragma unroll
            for (int k = TAPS - 1; k > 0; --k) y.x[i] = fmaf(w[TAPS - 1 - k].x[i], hist[k - 1].x[i], y.x[i]);
            y.x[i] = fmaf(w[TAPS - 1].x[i], x[j].x[i], y.x[i]);
          }
#pragma unroll
          for (int k = TAPS - 1; k > 1; --k) hist[k - 1] = hist[k - 2];
          if constexpr (TAPS > 1) hist[0] = x[j];
        } else {
          for (int k = a.taps - 1; k >= 0; --k) {
            const Vec<V> xk = k ? conv_input<V>(a, c, t + j, k, t0, slot, fresh) : x[j];
            const Vec<V> wk = load_vec<V>(a.conv_w + static_cast<long long>(a.taps - 1 - k) * ch + c);
#pragma unroll
            for (int i = 0; i < V; ++i) y.x[i] = fmaf(wk.x[i], xk.x[i], y.x[i]);
          }
        }
#pragma unroll
        for (int i = 0; i < V; ++i) y.x[i] = silu_act<T>(y.x[i]);
        store_vec<V>(out + static_cast<long long>(t + j) * x_ld, y);
      }
    }
    t = t_end;
  }
}

template <typename T, int V, bool ONE>
static int launch_conv(const SsmArgs& a, cudaStream_t st) {
  const int run = a.n_tokens <= 256 ? 1 : a.n_tokens <= 4096 ? 8 : 32;
  const int blocks = (a.channels() / V + kConvThreads - 1) / kConvThreads;
  const dim3 grid(blocks + (a.heads + kConvThreads - 1) / kConvThreads, (a.n_tokens + run - 1) / run);
  switch (a.taps) {
    case 2: BCG_CUDA_CHECK(launch_k(ssm_conv_kernel<T, V, 2, ONE>, grid, dim3(kConvThreads), 0, st, a, run, blocks)); break;
    case 3: BCG_CUDA_CHECK(launch_k(ssm_conv_kernel<T, V, 3, ONE>, grid, dim3(kConvThreads), 0, st, a, run, blocks)); break;
    case 4: BCG_CUDA_CHECK(launch_k(ssm_conv_kernel<T, V, 4, ONE>, grid, dim3(kConvThreads), 0, st, a, run, blocks)); break;
    default: BCG_CUDA_CHECK(launch_k(ssm_conv_kernel<T, V, 0, ONE>, grid, dim3(kConvThreads), 0, st, a, run, blocks));
  }
  return BCG_OK;
}

// The convolution's state of channel c behind the last token of sequence s: row r <- input n + r - (taps - 1) of the
// portion of n tokens, or old row n + r.
__device__ __forceinline__ void advance_conv(const SsmArgs& a, int s, int t0, int t1, bool fresh, int c) {
  const int keep = a.taps - 1, n = t1 - t0, ch = a.channels();
  float* cs = a.conv_state + static_cast<long long>(a.state_slots[s]) * keep * ch + c;
  for (int r = 0; r < keep; ++r) {
    const int i = n + r - keep;
    float x = 0.f;
    if (i >= 0) x = slab_sum(a.row(t0 + i) + a.inner() + c, a.n_partials, a.pstride);
    else if (!fresh) x = cs[static_cast<long long>(n + r) * ch];
    cs[static_cast<long long>(r) * ch] = x;
  }
}
// The channels that the CTA of head h and entries p0.. is in charge of: its own x, and its group's B and C where the head
// is the group's first.
__device__ __forceinline__ void advance_conv_of_head(const SsmArgs& a, int s, int t0, int t1, bool fresh, int h, int p0, int rows) {
  const int per = a.heads / a.groups, g = h / per;
  const int n = rows + (h % per == 0 && p0 == 0 ? 2 * a.n : 0);
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    const int e = i - rows;
    advance_conv(a, s, t0, t1, fresh, i < rows ? h * a.vdim + p0 + i : a.inner() + (e / a.n * a.groups + g) * a.n + e % a.n);
  }
}

// ------------------------------------------------------------------------------------------- single tokens
constexpr int kTapsAhead = 4;     // taps whose past inputs are requested ahead of time

// What is known of a token before its projections are.
struct TokenPlace {
  int t, h, slot;
  bool idle, fresh;
  __device__ __forceinline__ void load(const SsmArgs& a, int t_, int h_) {
    t = t_;
    h = h_;
    idle = a.slot_map[t] < 0;
    fresh = a.positions[t] == 0;
    slot = a.state_slots[t];
  }
};

// One channel of a single token's convolution (or its step) on the way: begin() requests weights and what earlier steps
// left, arrive() the projection (up to four slabs), value() is the sum behind its activation.
constexpr int kPadChannel = -1, kStepChannel = -2;
struct TokenChannel {
  int c;
  float past[kTapsAhead - 1], w[kTapsAhead], bias, v[4];

  __device__ __forceinline__ void begin(const SsmArgs& a, const TokenPlace& at, int c_) {
    c = c_;
    const int ch = a.channels(), tap0 = a.taps - kTapsAhead;     // w[kTapsAhead - 1] is the current token's
    const float* cw = a.conv_w + c;
    const float* cs = a.conv_state + static_cast<long long>(at.slot) * (a.taps - 1) * ch + c;
    const bool old = c >= 0 && !at.idle && !at.fresh;
#pragma unroll
    for (int j = 0; j < kTapsAhead; ++j) {
      w[j] = c >= 0 && tap0 + j >= 0 ? cw[(tap0 + j) * ch] : 0.f;
      if (j < kTapsAhead - 1) past[j] = old && tap0 + j >= 0 ? cs[(tap0 + j) * ch] : 0.f;
    }
    bias = c >= 0 ? a.conv_b[c] : c == kStepChannel ? a.step_bias[at.h] : 0.f;
  }
  __device__ __forceinline__ const float* source(const SsmArgs& a, const TokenPlace& at) const {
    return a.row(at.t) + a.inner() + (c == kStepChannel ? a.channels() + at.h : max(c, 0));
  }
  __device__ __forceinline__ void arrive(const SsmArgs& a, const TokenPlace& at) {
    const float* src = source(a, at);
#pragma unroll
    for (int q = 0; q < 4; ++q) v[q] = c != kPadChannel && q < a.n_partials ? src[q * a.pstride] : 0.f;
  }
  __device__ __forceinline__ float value(const SsmArgs& a, const TokenPlace& at) const {
    float in = (v[0] + v[1]) + (v[2] + v[3]);
    if (c == kPadChannel) return 0.f;
    for (int q = 4; q < a.n_partials; ++q) in += source(a, at)[q * a.pstride];
    if (c == kStepChannel) return softplus_f32(in + bias);
    float y = fmaf(w[kTapsAhead - 1], in, bias);
#pragma unroll
    for (int j = 0; j < kTapsAhead - 1; ++j) y = fmaf(w[j], past[j], y);
    if (!at.fresh)
      for (int j = 0; j < a.taps - kTapsAhead; ++j)
        y = fmaf(a.conv_w[static_cast<long long>(j) * a.channels() + c],
                 a.conv_state[(static_cast<long long>(at.slot) * (a.taps - 1) + j) * a.channels() + c], y);
    return silu_f32(y);
  }
};
// Channel of entry e of [B: NP | C: NP] of group g.
template <int NP>
__device__ __forceinline__ int bc_channel(const SsmArgs& a, int g, int e) {
  const int which = e / NP, k = e % NP;
  return e < 2 * NP && k < a.n ? a.inner() + (which * a.groups + g) * a.n + k : kPadChannel;
}

template <typename T, int NP>
__global__ void __launch_bounds__(kSsThreads, NP <= 128 ? 2 : 1)
ssm_token_kernel(const SsmArgs a) {
  using S = StateRows<NP>;
  constexpr int kItems = (kSsRows + 2 * NP + 1 + kSsThreads - 1) / kSsThreads;
  __shared__ float xbc[kItems * kSsThreads];        // x of the CTA's rows | B | C | step
  const int h = blockIdx.x, p0 = blockIdx.y * kSsRows, t = blockIdx.z;
  const int rows = min(kSsRows, a.vdim - p0), N = a.n;
  pdl_launch_dependents();
  // Positions, slots and states were written by earlier steps, which are complete before any kernel of this step
  // starts, so the states are on their way while the projections are finished.
  TokenPlace at;
  at.load(a, t, h);
  float* st = a.state + ((static_cast<long long>(at.slot) * a.heads + h) * a.vdim + p0) * N;
  S s;
  if (at.idle || at.fresh) s.zero();
  else s.load(st, rows, N);
  TokenChannel in[kItems];
#pragma unroll
  for (int k = 0; k < kItems; ++k) {
    const int i = threadIdx.x + k * kSsThreads, e = i - kSsRows;
    in[k].begin(a, at, e < 0 ? (i < rows ? h * a.vdim + p0 + i : kPadChannel)
                             : e == 2 * NP ? kStepChannel : bc_channel<NP>(a, h / (a.heads / a.groups), e));
  }
  pdl_wait();
  if (at.idle) return;
#pragma unroll
  for (int k = 0; k < kItems; ++k) in[k].arrive(a, at);
#pragma unroll
  for (int k = 0; k < kItems; ++k) xbc[threadIdx.x + k * kSsThreads] = in[k].value(a, at);
  __syncthreads();
  const float step = xbc[kSsRows + 2 * NP], keep = decay_f32(-a.rate[h] * step);
  float b[S::kQ][4], c[S::kQ][4];
#pragma unroll
  for (int q = 0; q < S::kQ; ++q)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      b[q][i] = xbc[kSsRows + S::entry(q) + i];
      c[q][i] = xbc[kSsRows + NP + S::entry(q) + i];
    }
  const float y = s.token(keep, [&](int r) { return step * xbc[S::row(r)]; }, b, c);
  s.store(st, rows, N);
  const int p = S::row(S::mine());
  if (S::writes() && p < rows)
    static_cast<T*>(a.y)[static_cast<long long>(t) * a.inner() + h * a.vdim + p0 + p] = from_f32<T>(fmaf(a.skip[h], xbc[p], y));
}

// State rows of 16 bytes' multiple, up to 128 entries.  A unit is 64 rows of a token's head (fewer at a head's end), a CTA
// has consecutive ones: B and C are made once per group.  Warps 0-7 compute, warp 8 moves states: a stage is filled, worked
// on in place, stored, and filled again once it has been read.
constexpr int kStStages = 3, kStThreads = kSsThreads + 32;
template <int NP>
struct StCfg {
  static constexpr int kStage = kSsRows * NP;                             // floats
  static constexpr int kX = kSsRows + 4, kBC = 2 * NP;                    // x and the step (16-byte multiple); B and C; two of each
  static constexpr int kSmem = (kStStages * kStage + 2 * kX + 2 * kBC) * 4 + 64;
};

// A walk over units: heads first, then blocks of rows, then tokens.
struct UnitWalk {
  int t, pb, h, in_group, g;
  __device__ __forceinline__ UnitWalk(const SsmArgs& a, int blocks, int u) {
    const int r = u / a.heads, per = a.heads / a.groups;
    h = u - r * a.heads;
    t = r / blocks;
    pb = r - t * blocks;
    g = h / per;
    in_group = h - g * per;
  }
  __device__ __forceinline__ void next(const SsmArgs& a, int blocks) {
    ++h;
    if (++in_group == a.heads / a.groups) {
      in_group = 0;
      ++g;
    }
    if (h == a.heads) {
      h = g = 0;
      if (++pb == blocks) {
        pb = 0;
        ++t;
      }
    }
  }
  __device__ __forceinline__ int rows(const SsmArgs& a) const { return min(kSsRows, a.vdim - pb * kSsRows); }
};

template <typename T, int NP>
__global__ void __launch_bounds__(kStThreads, 2)
ssm_stream_kernel(const SsmArgs a, int n_units) {
  using S = StateRows<NP>;
  using C = StCfg<NP>;
  constexpr int kItems = (C::kBC + kSsThreads - 1) / kSsThreads;
  extern __shared__ __align__(128) float st_raw[];
  float* xs = st_raw + kStStages * C::kStage;                   // [2][rows | step]
  float* bc = xs + 2 * C::kX;                                   // [2][B | C]
  uint64_t* full = reinterpret_cast<uint64_t*>(bc + 2 * C::kBC);   // [stages] a state has arrived
  uint64_t* done = full + kStStages;                            // [stages] it has been worked on
  const int N = a.n, blocks = (a.vdim + kSsRows - 1) / kSsRows;
  const int u0 = static_cast<int>(static_cast<long long>(n_units) * blockIdx.x / gridDim.x);
  const int n = static_cast<int>(static_cast<long long>(n_units) * (blockIdx.x + 1) / gridDim.x) - u0;
  pdl_launch_dependents();
  if (threadIdx.x == 0) {
    for (int i = 0; i < kStStages; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&done[i], kSsThreads);
    }
    fence_barrier_init();
  }
  __syncthreads();
  // States, slots and positions were written by earlier steps (see ssm_token).
  if (threadIdx.x >= kSsThreads) {
    if (threadIdx.x == kSsThreads) {
      UnitWalk in(a, blocks, u0), out = in;
      auto state_of = [&](const UnitWalk& u) {
        return a.state + ((static_cast<long long>(a.state_slots[u.t]) * a.heads + u.h) * a.vdim + u.pb * kSsRows) * N;
      };
      for (int i = 0; i < n + kStStages - 1; ++i) {
        if (i < n) {
          const uint32_t bytes = static_cast<uint32_t>(in.rows(a) * N * 4);
          const float* src = state_of(in);
          // the stage's previous state (unit i - stages) was stored a turn ago
          if (i >= kStStages) asm volatile("cp.async.bulk.wait_group.read 0;" ::: "memory");
          mbar_arrive_expect_tx(&full[i % kStStages], bytes);
          bulk_load_1d(st_raw + (i % kStStages) * C::kStage, src, bytes, &full[i % kStStages]);
          in.next(a, blocks);
        }
        const int j = i - (kStStages - 1);
        if (j >= 0) {
          float* dst = state_of(out);
          const bool idle = a.slot_map[out.t] < 0;
          mbar_wait(&done[j % kStStages], (j / kStStages) & 1);
          if (!idle) bulk_store_1d(dst, st_raw + (j % kStStages) * C::kStage, static_cast<uint32_t>(out.rows(a) * N * 4));
          out.next(a, blocks);
        }
      }
      asm volatile("cp.async.bulk.wait_group 0;" ::: "memory");
    }
    return;
  }
  UnitWalk u(a, blocks, u0);
  TokenPlace at, ahead;             // of this unit, of the next one
  TokenChannel x, group[kItems];    // threads up to kSsRows have an x channel or the step, all have some of B and C
  auto x_begin = [&](const UnitWalk& w, const TokenPlace& place) {
    const int tid = static_cast<int>(threadIdx.x);
    if (tid <= kSsRows)
      x.begin(a, place, tid == kSsRows ? kStepChannel : tid < w.rows(a) ? w.h * a.vdim + w.pb * kSsRows + tid : kPadChannel);
  };
  auto x_arrive = [&](const TokenPlace& place) {
    if (threadIdx.x <= kSsRows) x.arrive(a, place);
  };
  auto group_begin = [&](const UnitWalk& w, const TokenPlace& place) {
#pragma unroll
    for (int k = 0; k < kItems; ++k) group[k].begin(a, place, bc_channel<NP>(a, w.g, threadIdx.x + k * kSsThreads));
  };
  auto group_arrive = [&](const TokenPlace& place) {
#pragma unroll
    for (int k = 0; k < kItems; ++k) group[k].arrive(a, place);
  };
  at.load(a, u.t, u.h);
  x_begin(u, at);
  group_begin(u, at);
  float rate = a.rate[u.h], skip = a.skip[u.h];
  pdl_wait();
  x_arrive(at);
  group_arrive(at);
  bool new_group = true;
  int side = 1;                     // of bc
  for (int i = 0; i < n; ++i) {
    float* xi = xs + (i & 1) * C::kX;
    if (threadIdx.x <= kSsRows) xi[threadIdx.x] = x.value(a, at);
    if (new_group) {
      side ^= 1;
#pragma unroll
      for (int k = 0; k < kItems; ++k) {
        const int e = threadIdx.x + k * kSsThreads;
        if (e < C::kBC) bc[side * C::kBC + e] = group[k].value(a, at);
      }
    }
    UnitWalk w = u;
    float rate1 = rate, skip1 = skip;
    ahead = at;
    new_group = false;
    if (i + 1 < n) {                // requested now, used a turn later
      w.next(a, blocks);
      if (w.t != u.t) ahead.load(a, w.t, w.h);
      ahead.h = w.h;
      new_group = w.t != u.t || w.g != u.g;
      x_begin(w, ahead);
      x_arrive(ahead);
      if (new_group) {
        group_begin(w, ahead);
        group_arrive(ahead);
      }
      rate1 = a.rate[w.h];
      skip1 = a.skip[w.h];
    }
    asm volatile("bar.sync 1, %0;" ::"n"(kSsThreads) : "memory");     // operands are there
    mbar_wait(&full[i % kStStages], (i / kStStages) & 1);
    if (!at.idle) {
      float* st = st_raw + (i % kStStages) * C::kStage;
      const float step = xi[kSsRows], keep = decay_f32(-rate * step);
      float b[S::kQ][4], c[S::kQ][4];
#pragma unroll
      for (int q = 0; q < S::kQ; ++q) {
        const float4 bv = *reinterpret_cast<const float4*>(bc + side * C::kBC + S::entry(q));
        const float4 cv = *reinterpret_cast<const float4*>(bc + side * C::kBC + NP + S::entry(q));
        b[q][0] = bv.x; b[q][1] = bv.y; b[q][2] = bv.z; b[q][3] = bv.w;
        c[q][0] = cv.x; c[q][1] = cv.y; c[q][2] = cv.z; c[q][3] = cv.w;
      }
      const int rows = u.rows(a);
      auto v = [&](int r) { return step * xi[S::row(r)]; };
      const float y = rows == kSsRows && N == NP ? S::template token_in_place<true>(st, rows, N, at.fresh, keep, v, b, c)
                                                 : S::template token_in_place<false>(st, rows, N, at.fresh, keep, v, b, c);
      const int p = S::row(S::mine());
      if (S::writes() && p < rows)
        static_cast<T*>(a.y)[static_cast<long long>(u.t) * a.inner() + u.h * a.vdim + u.pb * kSsRows + p] = from_f32<T>(fmaf(skip, xi[p], y));
      fence_proxy_async();
    }
    mbar_arrive(&done[i % kStStages]);
    u = w;
    at = ahead;
    rate = rate1;
    skip = skip1;
  }
}

// Token by token over a portion whose convolution is done.
template <typename T, int NP>
__global__ void __launch_bounds__(kSsThreads)
ssm_scan_kernel(const SsmArgs a) {
  using S = StateRows<NP>;
  const int h = blockIdx.x, p0 = blockIdx.y * kSsRows, sq = blockIdx.z;
  const int rows = min(kSsRows, a.vdim - p0), N = a.n, g = h / (a.heads / a.groups), inner = a.inner();
  pdl_launch_dependents();
  pdl_wait();
  const int t0 = a.first_of(sq), t1 = a.end_of(sq);
  if (t1 <= t0 || a.slot_map[t0] < 0) return;
  float* st = a.state + ((static_cast<long long>(a.state_slots[sq]) * a.heads + h) * a.vdim + p0) * N;
  S s;
  const bool fresh = a.positions[t0] == 0;
  if (fresh) s.zero();
  else s.load(st, rows, N);
  const T* base = static_cast<const T*>(a.x);
  const float rate = a.rate[h], skip = a.skip[h];
  float x[S::kR], b[S::kQ][4], c[S::kQ][4], step;
  auto fetch = [&](int t) {
    const T* tok = base + static_cast<long long>(t) * a.x_ld();
    step = a.step[static_cast<long long>(t) * a.heads + h];
#pragma unroll
    for (int r = 0; r < S::kR; ++r) x[r] = S::row(r) < rows ? to_f32<T>(tok[h * a.x_pad() + p0 + S::row(r)]) : 0.f;
#pragma unroll
    for (int q = 0; q < S::kQ; ++q)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int e = S::entry(q) + i;
        b[q][i] = e < N ? to_f32<T>(tok[a.b_col(g) + e]) : 0.f;
        c[q][i] = e < N ? to_f32<T>(tok[a.c_col(g) + e]) : 0.f;
      }
  };
  fetch(t0);
  for (int t = t0; t < t1; ++t) {
    const float keep = decay_f32(-rate * step);
    float v[S::kR], bb[S::kQ][4], cc[S::kQ][4], mine = x[0];
#pragma unroll
    for (int r = 0; r < S::kR; ++r) {
      v[r] = step * x[r];
      if (S::mine() == r) mine = x[r];
    }
#pragma unroll
    for (int q = 0; q < S::kQ; ++q)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        bb[q][i] = b[q][i];
        cc[q][i] = c[q][i];
      }
    if (t + 1 < t1) fetch(t + 1);
    const float y = s.token(keep, [&](int r) { return v[r]; }, bb, cc);
    const int p = S::row(S::mine());
    if (S::writes() && p < rows)
      static_cast<T*>(a.y)[static_cast<long long>(t) * inner + h * a.vdim + p0 + p] = from_f32<T>(fmaf(skip, mine, y));
  }
  s.store(st, rows, N);
  advance_conv_of_head(a, sq, t0, t1, fresh, h, p0, rows);
}

// ------------------------------------------------------------------------------------------- chunks
// Scalars of a chunk: running sums of -rate * step in log2 units | steps | exp(sum) | step * exp(total - sum).
struct SsdRule {
  using Args = SsmArgs;
  static constexpr bool kNormalized = false;
  static constexpr int kScalars = 4 * kChTok;
  const SsmArgs& a;
  const int h, t0, t1;
  const float rate;
  float s0, s1;               // steps of tokens 2 lane, 2 lane + 1 of the next chunk
  __device__ __forceinline__ SsdRule(const SsmArgs& a_, int h_, int t0_, int t1_, int, bool) : a(a_), h(h_), t0(t0_), t1(t1_), rate(a_.rate[h_]), s0(0.f), s1(0.f) {}
  __device__ __forceinline__ float step_at(int t) const { return t < t1 ? a.step[static_cast<long long>(t) * a.heads + h] : 0.f; }
  __device__ __forceinline__ void request(int chunk, int lane) {
    s0 = step_at(t0 + chunk * kChTok + 2 * lane);
    s1 = step_at(t0 + chunk * kChTok + 2 * lane + 1);
  }
  __device__ __forceinline__ void scalars(float* sum2, int, int lane) {
    float *steps = sum2 + kChTok, *e_s = steps + kChTok, *w_s = e_s + kChTok;
    const float a0 = -rate * s0, a1 = -rate * s1;
    float run = a0 + a1;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, run, o);
      if (lane >= o) run += v;
    }
    const float total = __shfl_sync(0xffffffffu, run, 31);
    const float c1 = run, c0 = run - a1;
    *reinterpret_cast<float2*>(sum2 + 2 * lane) = make_float2(c0 * kSsLog2e, c1 * kSsLog2e);
    *reinterpret_cast<float2*>(steps + 2 * lane) = make_float2(s0, s1);
    *reinterpret_cast<float2*>(e_s + 2 * lane) = make_float2(expf(c0), expf(c1));
    *reinterpret_cast<float2*>(w_s + 2 * lane) = make_float2(s0 * expf(total - c0), s1 * expf(total - c1));
  }
  // exp(c_i - c_j) step_j of tokens j, j + 1; ci: entry i of the scalars
  __device__ __forceinline__ float2 weights(const float* sc, float ci, int j) const {
    const float2 cj = *reinterpret_cast<const float2*>(sc + j), sj = *reinterpret_cast<const float2*>(sc + kChTok + j);
    return make_float2(ex2_approx(ci - cj.x) * sj.x, ex2_approx(ci - cj.y) * sj.y);
  }
  __device__ __forceinline__ float2 readout(const float* sc, int i) const { return *reinterpret_cast<const float2*>(sc + 2 * kChTok + i); }
  // past the end steps are zero: the whole chunk's decay
  __device__ __forceinline__ float keep(const float* sc) const { return sc[3 * kChTok - 1]; }
  __device__ __forceinline__ float skip() const { return a.skip[h]; }
  __device__ __forceinline__ void finish(int sq, int p0, int rows, bool fresh) const {
    advance_conv_of_head(a, sq, t0, t1, fresh, h, p0, rows);
  }
};

// ------------------------------------------------------------------------------------------- norm
constexpr int kSnThreads = 256;

// A part of a token's outputs per CTA, or per cluster of CL.  ADVANCE: single tokens, the convolution's state moves on.
template <typename T, int V, int CL, bool ADVANCE>
__global__ void __launch_bounds__(kSnThreads)
ssm_norm_kernel(const SsmArgs a, T* __restrict__ out, long long out_ld) {
  extern __shared__ float4 stage_raw[];
  float* stage = reinterpret_cast<float*>(stage_raw);
  __shared__ RowSum<kSnThreads, CL, 1> sh;
  pdl_launch_dependents();
  pdl_wait();
  const int unit = blockIdx.x % (a.parts * CL), t = blockIdx.x / (a.parts * CL);
  const int part = unit / CL, inner = a.inner(), width = inner / a.parts;
  const int per = (width / V + CL - 1) / CL * V, v0 = unit % CL * per, v1 = min(width, v0 + per);
  const T* y = static_cast<const T*>(a.y) + static_cast<long long>(t) * inner + part * width;
  const float* z = a.row(t) + part * width;
  float ss[1] = {0.f};
  for (int v = v0 + threadIdx.x * V; v < v1; v += kSnThreads * V) {
    Vec<V> u = load_vec<V>(y + v);
    const Vec<V> g = slab_sum_vec<V>(z + v, a.n_partials, a.pstride);
#pragma unroll
    for (int k = 0; k < V; ++k) u.x[k] *= silu_act<T>(g.x[k]);
    store_vec<V>(stage + v - v0, u);
    ss[0] += u.sumsq();
  }
  row_sum<kSnThreads, CL, 1>(sh, ss, 0);
  const float inv = rsqrtf(ss[0] / static_cast<float>(width) + a.eps);
  for (int v = v0 + threadIdx.x * V; v < v1; v += kSnThreads * V) {
    Vec<V> x = load_vec<V>(stage + v - v0);
    const Vec<V> w = load_vec<V>(a.norm + part * width + v);
#pragma unroll
    for (int k = 0; k < V; ++k) x.x[k] *= inv * w.x[k];
    store_vec<V>(out + t * out_ld + part * width + v, x);
  }
  if constexpr (ADVANCE) {
    if (a.taps > 1 && a.slot_map[t] >= 0) {
      const int ch = a.channels();
      const bool fresh = a.positions[t] == 0;
      for (int c = unit * kSnThreads + threadIdx.x; c < ch; c += a.parts * CL * kSnThreads) advance_conv(a, t, t, t + 1, fresh, c);
    }
  }
  row_sum_exit<CL>();
}

// Prompts, one slab: a part of a token's outputs per warp, NV vectors of four per lane.
template <typename T, int NV>
__global__ void __launch_bounds__(kSnThreads, NV <= 8 ? 4 : 2)
ssm_norm_warp_kernel(const SsmArgs a, T* __restrict__ out, long long out_ld) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const long long unit = blockIdx.x * static_cast<long long>(kSnThreads / 32) + (threadIdx.x >> 5);
  if (unit >= static_cast<long long>(a.n_tokens) * a.parts) return;
  const long long t = unit / a.parts;
  const int inner = a.inner(), width = inner / a.parts, c0 = static_cast<int>(unit % a.parts) * width;
  const T* y = static_cast<const T*>(a.y) + t * inner + c0;
  const float* z = a.row(t) + c0;
  Vec<4> u[NV], g[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int v = min((i * 32 + lane) * 4, width - 4);
    u[i] = load_vec<4>(y + v);
    g[i] = load_vec<4>(z + v);
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
#pragma unroll
    for (int k = 0; k < 4; ++k) u[i].x[k] *= silu_act<T>(g[i].x[k]);
    if ((i * 32 + lane) * 4 < width) ss += u[i].sumsq();
  }
  const float inv = rsqrtf(warp_sum(ss) / static_cast<float>(width) + a.eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int v = (i * 32 + lane) * 4;
    if (v >= width) break;
    const Vec<4> w = load_vec<4>(a.norm + c0 + v);
#pragma unroll
    for (int k = 0; k < 4; ++k) u[i].x[k] *= inv * w.x[k];
    store_vec<4>(out + t * out_ld + c0 + v, u[i]);
  }
}

template <typename T, int V, int CL, bool ADVANCE>
static int launch_norm_cl(const SsmArgs& a, void* out, long long out_ld, cudaStream_t st) {
  const int width = a.inner() / a.parts;
  const dim3 grid(static_cast<unsigned>(static_cast<long long>(a.n_tokens) * a.parts * CL));
  const size_t sm = static_cast<size_t>((width / V + CL - 1) / CL * V) * 4;
  BCG_TRY(ensure_dynamic_smem(reinterpret_cast<const void*>(ssm_norm_kernel<T, V, CL, ADVANCE>), 200 * 1024));
  BCG_CUDA_CHECK(launch_cluster(ssm_norm_kernel<T, V, CL, ADVANCE>, grid, dim3(kSnThreads), CL, sm, st, a, static_cast<T*>(out), out_ld));
  return BCG_OK;
}

template <typename T, int V>
static int launch_norm(const SsmArgs& a, bool advance, void* out, long long out_ld, cudaStream_t st) {
  const int width = a.inner() / a.parts;
  if constexpr (V == 4) {
    if (!advance && a.n_partials == 1 && width <= 2048 && a.n_tokens > 128) {
      const dim3 grid(static_cast<unsigned>((static_cast<long long>(a.n_tokens) * a.parts + kSnThreads / 32 - 1) / (kSnThreads / 32)));
      T* o = static_cast<T*>(out);
      if (width <= 256) BCG_CUDA_CHECK(launch_k(ssm_norm_warp_kernel<T, 2>, grid, dim3(kSnThreads), 0, st, a, o, out_ld));
      else if (width <= 1024) BCG_CUDA_CHECK(launch_k(ssm_norm_warp_kernel<T, 8>, grid, dim3(kSnThreads), 0, st, a, o, out_ld));
      else BCG_CUDA_CHECK(launch_k(ssm_norm_warp_kernel<T, 16>, grid, dim3(kSnThreads), 0, st, a, o, out_ld));
      return BCG_OK;
    }
  }
  if (static_cast<long long>(a.n_tokens) * a.parts <= 64 && width >= 1024)      // few of them: a cluster each
    return advance ? launch_norm_cl<T, V, 8, true>(a, out, out_ld, st) : launch_norm_cl<T, V, 8, false>(a, out, out_ld, st);
  return advance ? launch_norm_cl<T, V, 1, true>(a, out, out_ld, st) : launch_norm_cl<T, V, 1, false>(a, out, out_ld, st);
}

// ------------------------------------------------------------------------------------------- launches
template <typename T, int NP>
static int run_np(const SsmArgs& a, int n_seqs, bool one_token, bool chunks, cudaStream_t st) {
  const int blocks = (a.vdim + kSsRows - 1) / kSsRows;
  const dim3 grid(a.heads, blocks, n_seqs);
  if (one_token && NP <= 128 && a.n % 4 == 0) {
    constexpr int P = NP <= 128 ? NP : 128;
    const long long units = static_cast<long long>(n_seqs) * a.heads * blocks;
    const int ctas = static_cast<int>(units < 2 * 148 ? units : 2 * 148);
    BCG_TRY(ensure_dynamic_smem(reinterpret_cast<const void*>(ssm_stream_kernel<T, P>), StCfg<P>::kSmem));
    BCG_CUDA_CHECK(launch_k(ssm_stream_kernel<T, P>, dim3(ctas), dim3(kStThreads), StCfg<P>::kSmem, st, a, static_cast<int>(units)));
  } else if (one_token) {
    BCG_CUDA_CHECK(launch_k(ssm_token_kernel<T, NP>, grid, dim3(kSsThreads), 0, st, a));
  } else if (chunks) {
    constexpr int P = NP < 64 ? 64 : NP;
    BCG_TRY((launch_chunks<P, SsdRule>(a, grid, st)));
  } else {
    BCG_CUDA_CHECK(launch_k(ssm_scan_kernel<T, NP>, grid, dim3(kSsThreads), 0, st, a));
  }
  return BCG_OK;
}

template <typename T>
static int run_t(const SsmArgs& a, int n_seqs, bool one_token, int mode, void* out, long long out_ld, cudaStream_t st) {
  const bool bf16 = sizeof(T) == 2;
  const bool wide = ((a.vdim | a.n | a.col) & 3) == 0 && a.ld % 4 == 0 && a.pstride % 4 == 0;
  const bool token = one_token && mode == 0, chunks = bf16 && mode == 0;
  if (!token) {
    if (!wide) BCG_TRY((launch_conv<T, 1, false>(a, st)));
    else if (a.n_partials == 1) BCG_TRY((launch_conv<T, 4, true>(a, st)));
    else BCG_TRY((launch_conv<T, 4, false>(a, st)));
  }
  if (a.n <= 32) BCG_TRY((run_np<T, 32>(a, n_seqs, token, chunks, st)));
  else if (a.n <= 64) BCG_TRY((run_np<T, 64>(a, n_seqs, token, chunks, st)));
  else if (a.n <= 128) BCG_TRY((run_np<T, 128>(a, n_seqs, token, chunks, st)));
  else BCG_TRY((run_np<T, 256>(a, n_seqs, token, chunks, st)));
  const int width = a.inner() / a.parts;
  if (width % 4 == 0 && out_ld % 4 == 0 && a.col % 4 == 0 && a.ld % 4 == 0 && a.pstride % 4 == 0)
    return launch_norm<T, 4>(a, token, out, out_ld, st);
  return launch_norm<T, 1>(a, token, out, out_ld, st);
}

int state_space(const bcg_stack* m, const bcg_layer* l, const bcg_stack_ws* ws, const bcg_step_batch* b, int n_partials,
                long long pstride, long long ld, int mode, cudaStream_t st) {
  if (!l->conv_w || !l->conv_b || !l->step_bias || !l->decay_rate || !l->skip || !l->ssm_norm || !l->ssm_state ||
      (l->ssm_taps > 1 && !l->conv_state) || !ws->ssm_x || !ws->ssm_step || !ws->ssm_y || !b->state_slots || l->ssm_n <= 0 ||
      l->ssm_n > 256 || l->ssm_vdim <= 0 || l->ssm_taps < 1 || l->ssm_groups <= 0 || l->ssm_heads % l->ssm_groups ||
      l->ssm_norm_parts <= 0 || (l->ssm_heads * l->ssm_vdim) % l->ssm_norm_parts || l->ssm_heads * l->ssm_vdim / l->ssm_norm_parts > 51200 || b->n_seqs > 65535) {
    set_last_error("bcg_state_space", "bad layer (1..256 state entries, groups and parts that divide) or too many sequences");
    return BCG_ERR_ARG;
  }
  SsmArgs a = {};
  a.proj = ws->proj;
  a.n_partials = n_partials;
  a.pstride = pstride;
  a.ld = ld;
  a.col = l->ssm_col;
  a.conv_w = l->conv_w;
  a.conv_b = l->conv_b;
  a.step_bias = l->step_bias;
  a.rate = l->decay_rate;
  a.skip = l->skip;
  a.norm = l->ssm_norm;
  a.positions = b->positions;
  a.slot_map = b->slot_map;
  a.row_seq = b->row_seq;
  a.seq_start = b->seq_start;
  a.state_slots = b->state_slots;
  a.state = l->ssm_state;
  a.conv_state = l->conv_state;
  a.step = ws->ssm_step;
  a.x = ws->ssm_x;
  a.y = ws->ssm_y;
  a.heads = l->ssm_heads;
  a.vdim = l->ssm_vdim;
  a.n = l->ssm_n;
  a.groups = l->ssm_groups;
  a.taps = l->ssm_taps;
  a.parts = l->ssm_norm_parts;
  a.n_tokens = b->T;
  a.eps = m->eps;
  const bool one = b->T == b->n_seqs;
  const int size = m->act_dtype == BCG_DT_F32 ? 4 : 2;
  void* out = static_cast<char*>(ws->mix) + static_cast<long long>(l->ssm_mix_col) * size;
  return size == 4 ? run_t<float>(a, b->n_seqs, one, mode, out, l->mix_ld, st)
                   : run_t<__nv_bfloat16>(a, b->n_seqs, one, mode, out, l->mix_ld, st);
}

}  // namespace bcg
