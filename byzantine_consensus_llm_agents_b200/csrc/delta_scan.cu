// Generalized delta rule over ragged sequences, state in fp32:
//     S <- diag(w) S - (a * u)(u^T S) + k v^T,     o = S^T r,      u = k / sqrt(|k|^2 + 1e-6),
//     w = exp(-exp(-1/2) sigmoid(decay + decay_bias)),  a = sigmoid(rate + rate_bias)   per key channel,
// followed per head by  o / rms(o) * out_norm * sigmoid(g).
//
// Columns of S evolve independently given (r, k, w, a, u), so a head is spread over threads by columns: a
// lane holds DIM/8 rows of CPT columns in registers (rows interleaved by fours over the warp's eight row
// groups), a warp 4*CPT columns, and the scan warps of a CTA - or of a cluster of CL CTAs - the whole head.
// Both products of a step read the old state,
//     o = (r*w)^T S - (r . (a*u)) (u^T S) + (r . k) v,
// so their reductions overlap and the state update is off the critical path.  Everything is fp32 FMA.
//
// Two kernels share this core:
//   delta_token   one token per sequence (decode): streams the state through registers; the state is
//                 requested before the dependency wait
//   delta_scan    portions of prompts: scan warps run the recurrence over a chunk of tokens without a barrier
//                 while preparation warps turn the next chunk's projections into operands (unit keys, gates,
//                 the two scalars) and finish the previous chunk's outputs.  Few (sequence, head) pairs take
//                 the many-CTA shape, many take the one-CTA shape.
#include "attn_tcgen05.cuh"
#include "stack_common.cuh"
#include "kernels.h"

namespace bcg {

constexpr float kDecayGain = 0.60653065971263342f;   // exp(-1/2)

struct DeltaArgs {
  const float* proj;       // rows r | k | v | g | rate, pitch ld
  int n_partials;
  long long pstride, ld;
  const float* decay;      // [T, heads * dim] slabs
  int d_partials;
  long long dstride;
  const float *decay_bias, *rate_bias, *out_norm;
  const int *positions, *slot_map, *seq_start, *state_slots;
  float* state;
  int heads, dim;
  float eps;
};

// tanh of the low-rank decay input: [T, rank] activations of the decay projection
template <typename T>
__global__ void __launch_bounds__(256)
delta_low_kernel(const float* __restrict__ proj, int n_partials, long long pstride, long long ld, long long col0,
                 T* __restrict__ low, int T_rows, int rank) {
  pdl_launch_dependents();
  pdl_wait();
  const long long i = static_cast<long long>(blockIdx.x) * 256 + threadIdx.x;
  if (i >= static_cast<long long>(T_rows) * rank) return;
  const long long t = i / rank;
  low[i] = from_f32<T>(tanhf(slab_sum(proj + t * ld + col0 + (i - t * rank), n_partials, pstride)));
}

// ------------------------------------------------------------------------------------------- core
// One lane's share of a head's state: rows q*32 + rg*4 + {0..3}, q < DP/32, of columns col .. col + CPT - 1.
template <int DP, int CPT>
struct StateTile {
  static constexpr int kQ = DP / 32;
  uint64_t s[CPT][kQ * 2];

  __device__ __forceinline__ void zero() {
#pragma unroll
    for (int c = 0; c < CPT; ++c)
#pragma unroll
      for (int i = 0; i < kQ * 2; ++i) s[c][i] = 0ull;
  }
  // st: the head's [D, D] state; vec: D is a multiple of CPT and rows are aligned for vector access
  __device__ __forceinline__ void load(const float* st, int D, int rg, int col) {
#pragma unroll
    for (int q = 0; q < kQ; ++q)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        float x[2][CPT];
#pragma unroll
        for (int k = 0; k < 2; ++k) {
          const int i = q * 32 + rg * 4 + e * 2 + k;
          const float* p = st + static_cast<long long>(i) * D + col;
          if (i < D && col + CPT <= D && D % CPT == 0) {
            if constexpr (CPT == 4) {
              const float4 v = *reinterpret_cast<const float4*>(p);
              x[k][0] = v.x; x[k][1] = v.y; x[k][2] = v.z; x[k][3] = v.w;
            } else if constexpr (CPT == 2) {
              const float2 v = *reinterpret_cast<const float2*>(p);
              x[k][0] = v.x; x[k][1] = v.y;
            } else {
              x[k][0] = *p;
            }
          } else {
#pragma unroll
            for (int c = 0; c < CPT; ++c) x[k][c] = (i < D && col + c < D) ? p[c] : 0.f;
          }
        }
#pragma unroll
        for (int c = 0; c < CPT; ++c)
          s[c][q * 2 + e] = pack_f32x2(__float_as_uint(x[0][c]), __float_as_uint(x[1][c]));
      }
  }
  __device__ __forceinline__ void store(float* st, int D, int rg, int col) const {
#pragma unroll
    for (int q = 0; q < kQ; ++q)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        float x[2][CPT];
#pragma unroll
        for (int c = 0; c < CPT; ++c) unpack_f32x2(s[c][q * 2 + e], x[0][c], x[1][c]);
#pragma unroll
        for (int k = 0; k < 2; ++k) {
          const int i = q * 32 + rg * 4 + e * 2 + k;
          float* p = st + static_cast<long long>(i) * D + col;
          if (i < D && col + CPT <= D && D % CPT == 0) {
            if constexpr (CPT == 4) *reinterpret_cast<float4*>(p) = make_float4(x[k][0], x[k][1], x[k][2], x[k][3]);
            else if constexpr (CPT == 2) *reinterpret_cast<float2*>(p) = make_float2(x[k][0], x[k][1]);
            else *p = x[k][0];
          } else {
#pragma unroll
            for (int c = 0; c < CPT; ++c)
              if (i < D && col + c < D) p[c] = x[k][c];
          }
        }
      }
  }
  // One token: op = its operands k, r*w, w, a*u, v [DP each, `pitch` floats apart]; sc = 1/|k|, r.(a*u),
  // r.k.  (u^T S is formed as (k^T S)/|k|: four vectors per token instead of five - a lane's share of them, read
  // from shared memory, is what the loop is bound by when CPT is small.)  o[c] is complete in every lane of a column's row groups.
  __device__ __forceinline__ void token(const float* op, int pitch, const float* sc, int rg, int col,
                                        float (&o)[CPT]) {
    uint64_t d2[CPT], o2[CPT];
#pragma unroll
    for (int c = 0; c < CPT; ++c) d2[c] = o2[c] = 0ull;
#pragma unroll
    for (int q = 0; q < kQ; ++q) {
      const ulonglong2 k = *reinterpret_cast<const ulonglong2*>(op + q * 32 + rg * 4);
      const ulonglong2 rw = *reinterpret_cast<const ulonglong2*>(op + pitch + q * 32 + rg * 4);
#pragma unroll
      for (int c = 0; c < CPT; ++c) {
        d2[c] = fma_f32x2(k.x, s[c][q * 2], d2[c]);
        o2[c] = fma_f32x2(rw.x, s[c][q * 2], o2[c]);
        d2[c] = fma_f32x2(k.y, s[c][q * 2 + 1], d2[c]);
        o2[c] = fma_f32x2(rw.y, s[c][q * 2 + 1], o2[c]);
      }
    }
    float d[CPT];
#pragma unroll
    for (int c = 0; c < CPT; ++c) {
      float x, y;
      unpack_f32x2(d2[c], x, y);
      d[c] = x + y;
      unpack_f32x2(o2[c], x, y);
      o[c] = x + y;
    }
#pragma unroll
    for (int m = 4; m < 32; m <<= 1)
#pragma unroll
      for (int c = 0; c < CPT; ++c) {
        d[c] += __shfl_xor_sync(0xffffffffu, d[c], m);
        o[c] += __shfl_xor_sync(0xffffffffu, o[c], m);
      }
    uint64_t v2[CPT], nd2[CPT];
#pragma unroll
    for (int c = 0; c < CPT; ++c) {
      const float v = op[4 * pitch + col + c];
      d[c] *= sc[0];
      o[c] = fmaf(sc[2], v, fmaf(-sc[1], d[c], o[c]));
      v2[c] = pack_f32x2(__float_as_uint(v), __float_as_uint(v));
      nd2[c] = pack_f32x2(__float_as_uint(-d[c]), __float_as_uint(-d[c]));
    }
#pragma unroll
    for (int q = 0; q < kQ; ++q) {
      const ulonglong2 w = *reinterpret_cast<const ulonglong2*>(op + 2 * pitch + q * 32 + rg * 4);
      const ulonglong2 au = *reinterpret_cast<const ulonglong2*>(op + 3 * pitch + q * 32 + rg * 4);
      const ulonglong2 k = *reinterpret_cast<const ulonglong2*>(op + q * 32 + rg * 4);
#pragma unroll
      for (int c = 0; c < CPT; ++c) {
        s[c][q * 2] = fma_f32x2(w.x, s[c][q * 2], fma_f32x2(au.x, nd2[c], mul_f32x2(k.x, v2[c])));
        s[c][q * 2 + 1] = fma_f32x2(w.y, s[c][q * 2 + 1], fma_f32x2(au.y, nd2[c], mul_f32x2(k.y, v2[c])));
      }
    }
  }
};

// One token's operands from its raw projections (x: r, k, v, g, rate, decay, DP floats each, in shared
// memory), by one warp: op = k, r*w, w, a*u, v, sigmoid(g), `pitch` apart; scalars = 1/|k|, r.(a*u), r.k.
template <int DP>
__device__ __forceinline__ void prepare_token(const DeltaArgs& a, int h, const float* x, float* op, int pitch,
                                              float* scalars) {
  constexpr int kQ = DP / 32;
  const int lane = threadIdx.x & 31, D = a.dim;
  float kk[kQ], ss = 0.f;
#pragma unroll
  for (int q = 0; q < kQ; ++q) {
    const int i = q * 32 + lane;
    kk[q] = i < D ? x[DP + i] : 0.f;
    ss += kk[q] * kk[q];
  }
  const float inv = rsqrtf(warp_sum(ss) + 1e-6f);
  float ra = 0.f, rk = 0.f;
#pragma unroll
  for (int q = 0; q < kQ; ++q) {
    const int i = q * 32 + lane;
    float r = 0.f, w = 0.f, rate = 0.f, v = 0.f, g = 0.f;
    if (i < D) {
      // 1 + expm1: rounded once near 1, where channels that remember for long live (an error of one
      // unit there, repeated at every token, is a drift of the whole memory)
      w = 1.0f + expm1f(-kDecayGain * sigmoid_f32(x[5 * DP + i] + a.decay_bias[h * D + i]));
      rate = sigmoid_f32(x[4 * DP + i] + a.rate_bias[h * D + i]);
      r = x[i];
      v = x[2 * DP + i];
      g = sigmoid_f32(x[3 * DP + i]);
    }
    const float au = rate * (kk[q] * inv);
    ra = fmaf(r, au, ra);
    rk = fmaf(r, kk[q], rk);
    op[i] = kk[q];
    op[pitch + i] = r * w;
    op[2 * pitch + i] = w;
    op[3 * pitch + i] = au;
    op[4 * pitch + i] = v;
    op[5 * pitch + i] = g;
  }
  ra = warp_sum(ra);
  rk = warp_sum(rk);
  if (lane == 0) {
    scalars[0] = inv;
    scalars[1] = ra;
    scalars[2] = rk;
  }
}

// element `i` of raw projection `kind` (r, k, v, g, rate, decay) of token t, head h
__device__ __forceinline__ const float* raw_ptr(const DeltaArgs& a, long long t, int h, int kind, int i) {
  const int HD = a.heads * a.dim;
  return kind < 5 ? a.proj + t * a.ld + static_cast<long long>(kind) * HD + h * a.dim + i : a.decay + t * HD + h * a.dim + i;
}

// ------------------------------------------------------------------------------------------- one token each
constexpr int kTokThreads = 256;

template <typename T, int DP, int CPT>
__global__ void __launch_bounds__(kTokThreads)
delta_token_kernel(const DeltaArgs a, T* __restrict__ out) {
  constexpr int kCols = kTokThreads / 32 * 4 * CPT, CL = DP / kCols;
  __shared__ __align__(16) float raw[6 * DP];
  __shared__ __align__(16) float op[6 * DP];
  __shared__ float so[kCols], sc[3];
  __shared__ RowSum<kTokThreads, CL, 1> sh;
  __shared__ RowSum<kTokThreads, 1, 3> sums;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, rg = lane >> 2, D = a.dim, HD = a.heads * a.dim;
  const int cta = CL > 1 ? static_cast<int>(blockIdx.x) : 0;
  const int h = blockIdx.y, t = blockIdx.z;
  pdl_launch_dependents();
  // Positions, slots and the state were written by earlier steps, which are complete before any kernel of
  // this step starts (a step's first launch follows the sampler's bookkeeping kernel or a copy, neither of
  // which lets its successor start early), so the state is on its way while the projections are finished.
  const bool idle = a.slot_map[t] < 0;
  const bool fresh = a.positions[t] == 0;
  const int lcol = warp * 4 * CPT + (lane & 3) * CPT, col = cta * kCols + lcol;
  float* st = a.state + (static_cast<long long>(a.state_slots[t]) * a.heads + h) * D * D;
  StateTile<DP, CPT> S;
  if (idle || fresh) S.zero();
  else S.load(st, D, rg, col);
  pdl_wait();
  if (idle) return;                                     // the same for the whole cluster
  {   // raw projections: a thread's elements and up to four slabs of each in flight together
    constexpr int kE = (6 * DP + kTokThreads - 1) / kTokThreads;
    const float* src[kE];
    long long stride[kE];
    float acc[kE];
    const int n = max(a.n_partials, a.d_partials);
#pragma unroll
    for (int k = 0; k < kE; ++k) {
      const int e = threadIdx.x + k * kTokThreads, kind = min(e / DP, 5), i = min(e % DP, D - 1);
      src[k] = raw_ptr(a, t, h, kind, i);
      stride[k] = kind < 5 ? a.pstride : a.dstride;
      acc[k] = 0.f;
    }
    for (int s0 = 0; s0 < n; s0 += 4) {
      float v[kE][4];
#pragma unroll
      for (int k = 0; k < kE; ++k)
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          const int np = threadIdx.x + k * kTokThreads < 5 * DP ? a.n_partials : a.d_partials;
          v[k][q] = s0 + q < np ? src[k][(s0 + q) * stride[k]] : 0.f;
        }
#pragma unroll
      for (int k = 0; k < kE; ++k)
#pragma unroll
        for (int q = 0; q < 4; ++q) acc[k] += v[k][q];
    }
#pragma unroll
    for (int k = 0; k < kE; ++k)
      if (threadIdx.x + k * kTokThreads < 6 * DP) raw[threadIdx.x + k * kTokThreads] = acc[k];
  }
  __syncthreads();
  {   // prepare_token with a thread per channel: a single token's latency is on the critical path
    const int i = threadIdx.x;
    float r = 0.f, kx = 0.f, w = 0.f, rate = 0.f, v = 0.f, g = 0.f;
    if (i < D) {
      r = raw[i];
      kx = raw[DP + i];
      v = raw[2 * DP + i];
      g = sigmoid_f32(raw[3 * DP + i]);
      rate = sigmoid_f32(raw[4 * DP + i] + a.rate_bias[h * D + i]);
      w = 1.0f + expm1f(-kDecayGain * sigmoid_f32(raw[5 * DP + i] + a.decay_bias[h * D + i]));
    }
    // sums of k^2, r.(a*k), r.k; the unit key's factor is applied to the sums
    float part[3] = {kx * kx, r * (rate * kx), r * kx};
    row_sum<kTokThreads, 1, 3>(sums, part, 0);
    const float inv = rsqrtf(part[0] + 1e-6f);
    if (i < DP) {
      op[i] = kx;
      op[DP + i] = r * w;
      op[2 * DP + i] = w;
      op[3 * DP + i] = rate * (kx * inv);
      op[4 * DP + i] = v;
      op[5 * DP + i] = g;
    }
    if (i == 0) {
      sc[0] = inv;
      sc[1] = part[1] * inv;
      sc[2] = part[2];
    }
  }
  __syncthreads();
  float o[CPT];
  S.token(op, DP, sc, rg, col, o);
  S.store(st, D, rg, col);
  float ss[1] = {0.f};
#pragma unroll
  for (int c = 0; c < CPT; ++c)
    if (rg == 0) {
      so[lcol + c] = o[c];
      if (col + c < D) ss[0] += o[c] * o[c];
    }
  row_sum<kTokThreads, CL, 1>(sh, ss, 0);               // also orders `so`
  const float inv = rsqrtf(ss[0] / static_cast<float>(D) + a.eps);
  for (int i = threadIdx.x; i < kCols; i += kTokThreads) {
    const int ch = cta * kCols + i;
    if (ch < D)
      out[static_cast<long long>(t) * HD + h * D + ch] = from_f32<T>(so[i] * inv * a.out_norm[h * D + ch] * op[5 * DP + ch]);
  }
  row_sum_exit<CL>();
}

template <typename T, int DP, int CPT>
static int launch_token(const DeltaArgs& a, void* out, int n, cudaStream_t st) {
  constexpr int CL = DP / (kTokThreads / 32 * 4 * CPT);
  BCG_CUDA_CHECK(launch_cluster(delta_token_kernel<T, DP, CPT>, dim3(CL, a.heads, n), dim3(kTokThreads), CL, 0, st, a,
                                static_cast<T*>(out)));
  return BCG_OK;
}
template <typename T>
static int dispatch_token(const DeltaArgs& a, void* out, int n, cudaStream_t st) {
  if (a.dim <= 32) return launch_token<T, 32, 1>(a, out, n, st);
  if (a.dim <= 64) return launch_token<T, 64, 2>(a, out, n, st);
  if (a.dim <= 128) return launch_token<T, 128, 4>(a, out, n, st);
  return launch_token<T, 256, 2>(a, out, n, st);
}

// ------------------------------------------------------------------------------------------- portions
// SW scan warps, PW preparation warps; a chunk is PW tokens, one per preparation warp.
template <int DP, int CPT, int SW, int PW>
struct DsCfg {
  static constexpr int kCols = SW * 4 * CPT, CL = DP / kCols, kThreads = (SW + PW) * 32, kChunk = PW;
  static constexpr int kOps = 6 * DP;                    // operands of one token
  static constexpr int kFloats = 2 * kChunk * kOps + 2 * kChunk * kCols + kChunk * 6 * DP;
};

// wait for a cluster-wide phase; a phase that never comes traps instead of hanging
__device__ __forceinline__ void mbar_wait_cluster(uint64_t* bar, uint32_t parity) {
  uint32_t ok = 0, spins = 0;
  while (!ok) {
    asm volatile(
        "{\n"
        ".reg .pred p;\n"
        "mbarrier.try_wait.parity.acquire.cluster.shared::cta.b64 p, [%1], %2;\n"
        "selp.b32 %0, 1, 0, p;\n"
        "}\n"
        : "=r"(ok)
        : "r"(smem_u32(bar)), "r"(parity)
        : "memory");
    if (++spins > (1u << 26)) __trap();
  }
}
__device__ __forceinline__ uint32_t peer_smem(const void* p, int rank) {
  uint32_t r;
  asm("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(smem_u32(p)), "r"(rank));
  return r;
}

template <typename T, int DP, int CPT, int SW, int PW>
__global__ void __launch_bounds__((SW + PW) * 32, 1)
delta_scan_kernel(const DeltaArgs a, T* __restrict__ out) {
  using C = DsCfg<DP, CPT, SW, PW>;
  constexpr int CL = C::CL;
  extern __shared__ float4 ds_raw[];
  float* ops = reinterpret_cast<float*>(ds_raw);          // [2][chunk][6][DP]
  float* so = ops + 2 * C::kChunk * C::kOps;              // [2][chunk][kCols]
  float* raw = so + 2 * C::kChunk * C::kCols;             // [chunk][6][DP]
  __shared__ float sc[2][C::kChunk][4];
  __shared__ float part[2][C::kChunk][CL];                // sums of squares of the cluster's column blocks
  __shared__ uint64_t part_bar[2];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, D = a.dim, HD = a.heads * a.dim;
  const int cta = CL > 1 ? static_cast<int>(blockIdx.x) : 0;
  const int h = blockIdx.y, s = blockIdx.z;
  pdl_launch_dependents();
  if (CL > 1 && threadIdx.x == 0) {
    mbar_init(&part_bar[0], CL * C::kChunk);
    mbar_init(&part_bar[1], CL * C::kChunk);
    fence_barrier_init();
  }
  pdl_wait();
  if constexpr (CL > 1) cooperative_groups::this_cluster().sync();   // barriers ready before any peer arrives
  const int t0 = a.seq_start ? a.seq_start[s] : s;
  const int t1 = a.seq_start ? a.seq_start[s + 1] : s + 1;
  if (t1 <= t0 || a.slot_map[t0] < 0) return;             // nothing to do (the same for the whole cluster)
  const bool fresh = a.positions[t0] == 0;
  float* st = a.state + (static_cast<long long>(a.state_slots[s]) * a.heads + h) * D * D;
  const int n_chunks = (t1 - t0 + C::kChunk - 1) / C::kChunk;
  const bool copies = a.n_partials == 1 && a.d_partials == 1;
  const bool wide = copies && (D & 3) == 0 && (a.ld & 3) == 0;

  // the raw projections of one token into raw[j], by one warp: asynchronous copies, or sums of slabs
  auto fetch = [&](int j, long long t) {
    float* dst = raw + j * 6 * DP;
#pragma unroll
    for (int kind = 0; kind < 6; ++kind) {
      const float* src = raw_ptr(a, t, h, kind, 0);
      if (wide) {
        for (int i = lane * 4; i < D; i += 128)
          asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst + kind * DP + i)), "l"(src + i) : "memory");
      } else if (copies) {
        for (int i = lane; i < D; i += 32)
          asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst + kind * DP + i)), "l"(src + i) : "memory");
      } else {
        for (int i = lane; i < D; i += 32)
          dst[kind * DP + i] = kind < 5 ? slab_sum(src + i, a.n_partials, a.pstride) : slab_sum(src + i, a.d_partials, a.dstride);
      }
    }
  };
  auto prepare = [&](int c, int j) {      // token j of chunk c, by its warp; then the copy of its next token
    const int t = t0 + c * C::kChunk + j;
    if (t < t1) {
      asm volatile("cp.async.wait_all;" ::: "memory");
      __syncwarp();
      prepare_token<DP>(a, h, raw + j * 6 * DP, ops + ((c & 1) * C::kChunk + j) * C::kOps, DP, sc[c & 1][j]);
      __syncwarp();
      if (t + C::kChunk < t1) fetch(j, t + C::kChunk);
    }
  };
  auto finish = [&](int c, int j) {       // output of token j of chunk c, by its warp
    const int t = t0 + c * C::kChunk + j, b = c & 1;
    const float* o = so + (b * C::kChunk + j) * C::kCols;
    float ss = 0.f;
    if (t < t1)
      for (int i = lane; i < C::kCols; i += 32) ss += cta * C::kCols + i < D ? o[i] * o[i] : 0.f;
    ss = warp_sum(ss);
    if constexpr (CL > 1) {
      // every CTA of the cluster gets every block's sum; tokens past the end arrive too, so that a phase is
      // always CL * chunk arrivals
      if (lane < CL) {
        asm volatile("st.relaxed.cluster.shared::cluster.f32 [%0], %1;" ::"r"(peer_smem(&part[b][j][cta], lane)), "f"(ss) : "memory");
        asm volatile("mbarrier.arrive.release.cluster.shared::cluster.b64 _, [%0];" ::"r"(peer_smem(&part_bar[b], lane)) : "memory");
      }
      __syncwarp();
      mbar_wait_cluster(&part_bar[b], (c >> 1) & 1);
      ss = 0.f;
#pragma unroll
      for (int k = 0; k < CL; ++k) ss += part[b][j][k];
    }
    if (t < t1) {
      const float inv = rsqrtf(ss / static_cast<float>(D) + a.eps);
      const float* g = ops + (b * C::kChunk + j) * C::kOps + 5 * DP;
      for (int i = lane; i < C::kCols; i += 32) {
        const int ch = cta * C::kCols + i;
        if (ch < D)
          out[static_cast<long long>(t) * HD + h * D + ch] = from_f32<T>(o[i] * inv * a.out_norm[h * D + ch] * g[ch]);
      }
    }
    __syncwarp();
  };

  if (warp < SW) {
    // ------------------------------ scan warps ------------------------------
    const int rg = lane >> 2;
    const int lcol = warp * 4 * CPT + (lane & 3) * CPT, col = cta * C::kCols + lcol;
    StateTile<DP, CPT> S;
    if (fresh) S.zero();
    else S.load(st, D, rg, col);
    __syncthreads();
    for (int c = 0; c < n_chunks; ++c) {
      const int n = min(C::kChunk, t1 - t0 - c * C::kChunk), b = c & 1;
      const float* op = ops + b * C::kChunk * C::kOps;
      float* o_row = so + b * C::kChunk * C::kCols;
      for (int j = 0; j < n; ++j, op += C::kOps, o_row += C::kCols) {
        float o[CPT];
        S.token(op, DP, sc[b][j], rg, col, o);
        if (rg == 0) {
#pragma unroll
          for (int k = 0; k < CPT; ++k) o_row[lcol + k] = o[k];
        }
      }
      __syncthreads();
    }
    S.store(st, D, rg, col);
  } else {
    // ------------------------------ preparation warps ------------------------
    const int j = warp - SW;
    if (t0 + j < t1) fetch(j, t0 + j);
    prepare(0, j);
    __syncthreads();
    for (int c = 0; c < n_chunks; ++c) {
      if (c > 0) finish(c - 1, j);        // before its operands (the gate) are overwritten
      if (c + 1 < n_chunks) prepare(c + 1, j);
      __syncthreads();
    }
    finish(n_chunks - 1, j);
  }
  if constexpr (CL > 1) cooperative_groups::this_cluster().sync();   // no peer writes into a CTA that has left
}

template <typename T, int DP, int CPT, int SW, int PW>
static int launch_scan(const DeltaArgs& a, void* out, int n_seqs, cudaStream_t st) {
  using C = DsCfg<DP, CPT, SW, PW>;
  BCG_TRY(ensure_dynamic_smem(reinterpret_cast<const void*>(delta_scan_kernel<T, DP, CPT, SW, PW>), C::kFloats * 4));
  BCG_CUDA_CHECK(launch_cluster(delta_scan_kernel<T, DP, CPT, SW, PW>, dim3(C::CL, a.heads, n_seqs), dim3(C::kThreads),
                                C::CL, C::kFloats * 4, st, a, static_cast<T*>(out)));
  return BCG_OK;
}

template <typename T>
static int dispatch_scan(const DeltaArgs& a, void* out, int n_seqs, cudaStream_t st) {
  const bool many = static_cast<long long>(n_seqs) * a.heads >= 96;   // heads enough for most SMs, one CTA each
  if (a.dim <= 32) return launch_scan<T, 32, 2, 4, 8>(a, out, n_seqs, st);
  if (a.dim <= 64) return launch_scan<T, 64, 2, 8, 8>(a, out, n_seqs, st);
  if (a.dim <= 128)
    return many ? launch_scan<T, 128, 4, 8, 8>(a, out, n_seqs, st) : launch_scan<T, 128, 2, 4, 16>(a, out, n_seqs, st);
  return launch_scan<T, 256, 2, 8, 8>(a, out, n_seqs, st);
}

int delta_low(const bcg_layer* l, const float* proj, int n_partials, long long pstride, void* low, int act_dtype,
              int T, cudaStream_t st) {
  const long long n = static_cast<long long>(T) * l->decay_rank, col0 = 5ll * l->heads * l->dim;
  const dim3 grid(static_cast<unsigned>((n + 255) / 256));
  if (act_dtype == BCG_DT_F32)
    BCG_CUDA_CHECK(launch_k(delta_low_kernel<float>, grid, dim3(256), 0, st, proj, n_partials, pstride,
                            static_cast<long long>(l->n_in), col0, static_cast<float*>(low), T, l->decay_rank));
  else
    BCG_CUDA_CHECK(launch_k(delta_low_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, proj, n_partials, pstride,
                            static_cast<long long>(l->n_in), col0, static_cast<__nv_bfloat16*>(low), T, l->decay_rank));
  return BCG_OK;
}

int delta_scan(const bcg_layer* l, const float* proj, int n_partials, long long pstride, long long ld,
               const float* decay, int d_partials, long long dstride, const int* positions, const int* slot_map,
               const int* seq_start, const int* state_slots, int n_seqs, int one_token, void* out, int act_dtype,
               float eps, cudaStream_t st) {
  if (!l || !proj || !decay || !positions || !slot_map || !state_slots || !out || !l->cache || n_seqs <= 0 ||
      n_seqs > 65535 || l->heads <= 0 || l->dim <= 0 || l->dim > 256 || n_partials < 1 || d_partials < 1) {
    set_last_error("bcg_delta_scan", "bad argument (1..256 channels per head, at most 65535 sequences)");
    return BCG_ERR_ARG;
  }
  DeltaArgs a = {proj, n_partials, pstride, ld, decay, d_partials, dstride, l->decay_bias, l->rate_bias, l->out_norm,
                 positions, slot_map, seq_start, state_slots, static_cast<float*>(l->cache), l->heads, l->dim, eps};
  if (one_token)
    return act_dtype == BCG_DT_F32 ? dispatch_token<float>(a, out, n_seqs, st)
                                   : dispatch_token<__nv_bfloat16>(a, out, n_seqs, st);
  return act_dtype == BCG_DT_F32 ? dispatch_scan<float>(a, out, n_seqs, st)
                                 : dispatch_scan<__nv_bfloat16>(a, out, n_seqs, st);
}

}  // namespace bcg
