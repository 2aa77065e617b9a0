// Generalized delta rule over ragged sequences, state in fp32:
//     S <- diag(w) S - (a * u)(u^T S) + k v^T,     o = S^T r,      u = k / sqrt(|k|^2 + 1e-6),
//     w = exp(-exp(-1/2) sigmoid(decay + decay_bias)),  a = sigmoid(rate + rate_bias)   per key channel,
// followed per head by  o / rms(o) * out_norm * sigmoid(g).
//
// Columns of S evolve independently given (r, k, w, a, u), so a head is spread over threads by columns: a
// lane holds DIM/8 rows of CPT columns in registers (rows interleaved by fours over the warp's eight row
// groups), a warp 4*CPT columns, a CTA 32*CPT columns and a cluster of CL CTAs the whole head.  Few (sequence,
// head) pairs take the many-CTA shape, many take the one-CTA shape.  Tokens are worked off in chunks: all
// gates, unit keys and the two scalars below are prepared for a chunk in parallel, then the recurrence runs
// over the chunk without a barrier.  Both products of a step read the old state,
//     o = (r*w)^T S - (r . (a*u)) (u^T S) + (r . k) v,
// so their reductions overlap and the state update is off the critical path.  Everything is fp32 FMA.
#include "attn_tcgen05.cuh"
#include "stack_common.cuh"
#include "kernels.h"

namespace bcg {

constexpr int kDsThreads = 256;
constexpr int kDsChunk = 16;
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
  int heads, dim, chunk;
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

template <typename T, int DP, int CPT>
__global__ void __launch_bounds__(kDsThreads)
delta_scan_kernel(const DeltaArgs a, T* __restrict__ out) {
  constexpr int kCols = kDsThreads / 32 * 4 * CPT;     // columns per CTA
  constexpr int CL = DP / kCols;
  constexpr int kQ = DP / 32;                           // float4 groups of rows per lane
  extern __shared__ float4 ds_raw[];
  __shared__ float ra_s[kDsChunk], rk_s[kDsChunk], part_s[2][kDsChunk];
  float* su = reinterpret_cast<float*>(ds_raw);         // [chunk][DP] each
  const int C = a.chunk, D = a.dim, HD = a.heads * a.dim;
  float* srw = su + C * DP;
  float* sw = srw + C * DP;
  float* sau = sw + C * DP;
  float* sk = sau + C * DP;
  float* sv = sk + C * DP;
  float* so = sv + C * DP;                              // [chunk][kCols]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int rg = lane >> 2;
  const int cta = CL > 1 ? static_cast<int>(blockIdx.x) : 0;
  const int h = blockIdx.y, s = blockIdx.z;
  pdl_launch_dependents();
  pdl_wait();
  const int t0 = a.seq_start ? a.seq_start[s] : s;
  const int t1 = a.seq_start ? a.seq_start[s + 1] : s + 1;
  if (t1 <= t0 || a.slot_map[t0] < 0) return;           // nothing to do (the same for the whole cluster)
  const bool fresh = a.positions[t0] == 0;
  const int lcol = warp * 4 * CPT + (lane & 3) * CPT;   // first column within the CTA
  const int col = cta * kCols + lcol;
  float* st = a.state + (static_cast<long long>(a.state_slots[s]) * a.heads + h) * D * D;
  uint64_t S[CPT][kQ * 2];
#pragma unroll
  for (int q = 0; q < kQ; ++q)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int i = q * 32 + rg * 4 + e * 2;
#pragma unroll
      for (int c = 0; c < CPT; ++c) {
        float x = 0.f, y = 0.f;
        if (!fresh && col + c < D) {
          if (i < D) x = st[static_cast<long long>(i) * D + col + c];
          if (i + 1 < D) y = st[static_cast<long long>(i + 1) * D + col + c];
        }
        S[c][q * 2 + e] = pack_f32x2(__float_as_uint(x), __float_as_uint(y));
      }
    }

  auto prepare = [&](int tb, int n) {
    for (int j = warp; j < n; j += kDsThreads / 32) {
      const long long t = tb + j;
      const float* p = a.proj + t * a.ld + static_cast<long long>(h) * D;
      const float* pd = a.decay + t * HD + static_cast<long long>(h) * D;
      float kk[kQ], ss = 0.f, r[kQ], au[kQ];
#pragma unroll
      for (int q = 0; q < kQ; ++q) {
        const int i = q * 32 + lane;
        kk[q] = i < D ? slab_sum(p + HD + i, a.n_partials, a.pstride) : 0.f;
        r[q] = i < D ? slab_sum(p + i, a.n_partials, a.pstride) : 0.f;
        ss += kk[q] * kk[q];
      }
      const float inv = rsqrtf(warp_sum(ss) + 1e-6f);
      float ra = 0.f, rk = 0.f;
#pragma unroll
      for (int q = 0; q < kQ; ++q) {
        const int i = q * 32 + lane;
        float w = 0.f, rate = 0.f, v = 0.f;
        if (i < D) {
          // 1 + expm1: rounded once near 1, where channels that remember for long live (an error of one
          // unit there, repeated at every token, is a drift of the whole memory)
          w = 1.0f + expm1f(-kDecayGain * sigmoid_f32(slab_sum(pd + i, a.d_partials, a.dstride) + a.decay_bias[h * D + i]));
          rate = sigmoid_f32(slab_sum(p + 4ll * HD + i, a.n_partials, a.pstride) + a.rate_bias[h * D + i]);
          v = slab_sum(p + 2ll * HD + i, a.n_partials, a.pstride);
        }
        const float u = kk[q] * inv;
        au[q] = rate * u;
        ra = fmaf(r[q], au[q], ra);
        rk = fmaf(r[q], kk[q], rk);
        su[j * DP + i] = u;
        srw[j * DP + i] = r[q] * w;
        sw[j * DP + i] = w;
        sau[j * DP + i] = au[q];
        sk[j * DP + i] = kk[q];
        sv[j * DP + i] = v;
      }
      ra = warp_sum(ra);
      rk = warp_sum(rk);
      if (lane == 0) {
        ra_s[j] = ra;
        rk_s[j] = rk;
      }
    }
  };

  prepare(t0, min(C, t1 - t0));
  __syncthreads();
  for (int tb = t0, par = 0; tb < t1; tb += C, par ^= 1) {
    const int n = min(C, t1 - tb);
    for (int j = 0; j < n; ++j) {
      uint64_t d2[CPT], o2[CPT];
#pragma unroll
      for (int c = 0; c < CPT; ++c) d2[c] = o2[c] = 0ull;
#pragma unroll
      for (int q = 0; q < kQ; ++q) {
        const ulonglong2 u = *reinterpret_cast<const ulonglong2*>(su + j * DP + q * 32 + rg * 4);
        const ulonglong2 rw = *reinterpret_cast<const ulonglong2*>(srw + j * DP + q * 32 + rg * 4);
#pragma unroll
        for (int c = 0; c < CPT; ++c) {
          d2[c] = fma_f32x2(u.x, S[c][q * 2], d2[c]);
          o2[c] = fma_f32x2(rw.x, S[c][q * 2], o2[c]);
          d2[c] = fma_f32x2(u.y, S[c][q * 2 + 1], d2[c]);
          o2[c] = fma_f32x2(rw.y, S[c][q * 2 + 1], o2[c]);
        }
      }
      float d[CPT], o[CPT];
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
        const float v = sv[j * DP + col + c];
        if (rg == 0) so[j * kCols + lcol + c] = fmaf(rk_s[j], v, fmaf(-ra_s[j], d[c], o[c]));
        v2[c] = pack_f32x2(__float_as_uint(v), __float_as_uint(v));
        nd2[c] = pack_f32x2(__float_as_uint(-d[c]), __float_as_uint(-d[c]));
      }
#pragma unroll
      for (int q = 0; q < kQ; ++q) {
        const ulonglong2 w = *reinterpret_cast<const ulonglong2*>(sw + j * DP + q * 32 + rg * 4);
        const ulonglong2 au = *reinterpret_cast<const ulonglong2*>(sau + j * DP + q * 32 + rg * 4);
        const ulonglong2 k = *reinterpret_cast<const ulonglong2*>(sk + j * DP + q * 32 + rg * 4);
#pragma unroll
        for (int c = 0; c < CPT; ++c) {
          S[c][q * 2] = fma_f32x2(w.x, S[c][q * 2], fma_f32x2(au.x, nd2[c], mul_f32x2(k.x, v2[c])));
          S[c][q * 2 + 1] = fma_f32x2(w.y, S[c][q * 2 + 1], fma_f32x2(au.y, nd2[c], mul_f32x2(k.y, v2[c])));
        }
      }
    }
    __syncthreads();
    // this chunk's outputs, and the next chunk's operands, between the same two barriers
    if constexpr (CL > 1) {
      for (int j = warp; j < n; j += kDsThreads / 32) {
        float ss = 0.f;
        for (int i = lane; i < kCols; i += 32) ss += cta * kCols + i < D ? so[j * kCols + i] * so[j * kCols + i] : 0.f;
        ss = warp_sum(ss);
        if (lane == 0) part_s[par][j] = ss;
      }
      cooperative_groups::this_cluster().sync();
    }
    for (int j = warp; j < n; j += kDsThreads / 32) {
      float ss = 0.f;
      if constexpr (CL > 1) {
        auto cluster = cooperative_groups::this_cluster();
#pragma unroll
        for (int k = 0; k < CL; ++k) ss += *cluster.map_shared_rank(&part_s[par][j], k);
      } else {
        for (int i = lane; i < kCols; i += 32) ss += i < D ? so[j * kCols + i] * so[j * kCols + i] : 0.f;
        ss = warp_sum(ss);
      }
      const float inv = rsqrtf(ss / static_cast<float>(D) + a.eps);
      const long long t = tb + j;
      for (int i = lane; i < kCols; i += 32) {
        const int ch = cta * kCols + i;
        if (ch < D) {
          const float g = slab_sum(a.proj + t * a.ld + 3ll * HD + static_cast<long long>(h) * D + ch, a.n_partials, a.pstride);
          out[t * HD + static_cast<long long>(h) * D + ch] =
              from_f32<T>(so[j * kCols + i] * inv * a.out_norm[h * D + ch] * sigmoid_f32(g));
        }
      }
    }
    if (tb + C < t1) prepare(tb + C, min(C, t1 - tb - C));
    __syncthreads();
  }
#pragma unroll
  for (int q = 0; q < kQ; ++q)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int i = q * 32 + rg * 4 + e * 2;
#pragma unroll
      for (int c = 0; c < CPT; ++c) {
        float x, y;
        unpack_f32x2(S[c][q * 2 + e], x, y);
        if (col + c < D) {
          if (i < D) st[static_cast<long long>(i) * D + col + c] = x;
          if (i + 1 < D) st[static_cast<long long>(i + 1) * D + col + c] = y;
        }
      }
    }
  if constexpr (CL > 1) cooperative_groups::this_cluster().sync();
}

template <typename T, int DP, int CPT>
static int launch_scan(const DeltaArgs& a, void* out, int n_seqs, cudaStream_t st) {
  constexpr int kCols = kDsThreads / 32 * 4 * CPT, CL = DP / kCols;
  const size_t sm = static_cast<size_t>(a.chunk) * (6 * DP + kCols) * 4;
  BCG_TRY(ensure_dynamic_smem(reinterpret_cast<const void*>(delta_scan_kernel<T, DP, CPT>),
                              kDsChunk * (6 * DP + kCols) * 4));
  BCG_CUDA_CHECK(launch_cluster(delta_scan_kernel<T, DP, CPT>, dim3(CL, a.heads, n_seqs), dim3(kDsThreads), CL, sm, st, a,
                                static_cast<T*>(out)));
  return BCG_OK;
}

template <typename T>
static int dispatch_scan(const DeltaArgs& a, void* out, int n_seqs, cudaStream_t st) {
  const bool many = static_cast<long long>(n_seqs) * a.heads >= 148;   // enough heads to fill the GPU one CTA each
  if (a.dim <= 32) return launch_scan<T, 32, 1>(a, out, n_seqs, st);
  if (a.dim <= 64) return many ? launch_scan<T, 64, 2>(a, out, n_seqs, st) : launch_scan<T, 64, 1>(a, out, n_seqs, st);
  if (a.dim <= 128)
    return many ? launch_scan<T, 128, 4>(a, out, n_seqs, st) : launch_scan<T, 128, 1>(a, out, n_seqs, st);
  return launch_scan<T, 256, 2>(a, out, n_seqs, st);
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
                 positions, slot_map, seq_start, state_slots, static_cast<float*>(l->cache), l->heads, l->dim,
                 one_token ? 1 : kDsChunk, eps};
  return act_dtype == BCG_DT_F32 ? dispatch_scan<float>(a, out, n_seqs, st)
                                 : dispatch_scan<__nv_bfloat16>(a, out, n_seqs, st);
}

}  // namespace bcg
