// Latent (compressed-KV) attention over paged latents, sliding window and softmax sink.
//
// A cache row holds one token's latent c [kv_rank] and the rotated key part shared by all heads [rot_dim].
// A head's key is (W_uk c, k_rot) and its value W_uv c, so with q~ = W_uk^T q the score is q~ . c + q_rot . k_rot
// and the output W_uv (sum_j p_j c_j): attention can run in latent space, where all heads share the keys.
//   latent_qkv        projection slabs -> rotated queries; latent norm + rotation -> cache row
//   latent_plain      one CTA per (token, head), latent space, any sizes, fp32 or bf16: the fp32 engine's
//                     kernel, and the bf16 one's for sizes the kernels below do not take
//   latent_absorb     q~ for single tokens (decode), W_uk tile staged ahead of the dependency wait
//   latent_decode     split-KV: one CTA per (span of keys, token), mma.sync over 32-head groups
//   latent_combine    spans -> latent-space output;  latent_up: W_uv
//   latent_gather     cache rows -> contiguous rows for the expanded (prefill) form, latent_prefill.cu
#include "mma_sync.cuh"
#include "stack_common.cuh"
#include "kernels.h"

namespace bcg {

// ------------------------------------------------------------------------------------------- q, k, v
constexpr int kQkvThreads = 256;

// grid (T, head groups of 8 [+ 1 for the cache row]); a warp per head.
template <typename T>
__global__ void __launch_bounds__(kQkvThreads)
latent_qkv_kernel(const float* __restrict__ proj, int n_partials, long long pstride, long long ld,
                  const int* __restrict__ positions, const int* __restrict__ slot_map,
                  const float* __restrict__ cos_sin, const float* __restrict__ latent_norm, T* __restrict__ q,
                  T* __restrict__ cache, int heads, int dim, int rot_dim, int rot_dims, int q_row, int kv_rank,
                  int q_groups, float eps) {
  extern __shared__ float stage[];    // latent
  __shared__ RowSum<kQkvThreads, 1, 1> sh;
  pdl_launch_dependents();
  pdl_wait();
  const long long t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const float* row = proj + t * ld;
  const float* cs = cos_sin + static_cast<long long>(positions[t]) * rot_dims;
  const int half = rot_dims >> 1;
  auto rotated = [&](const float* x, int i) {   // element i of the rotated part whose first element is x
    const float a = slab_sum(x + i, n_partials, pstride);
    if (i >= rot_dims) return a;
    const int f = i < half ? i : i - half;
    const float b = slab_sum(x + (i < half ? i + half : i - half), n_partials, pstride);
    const float c = cs[f], s = cs[half + f];
    return i < half ? a * c - b * s : a * c + b * s;
  };
  if (static_cast<int>(blockIdx.y) < q_groups) {
    const int h = blockIdx.y * (kQkvThreads / 32) + warp;
    if (h >= heads) return;
    const float* x = row + static_cast<long long>(h) * (dim + rot_dim);
    T* dst = q + (t * heads + h) * q_row;
    for (int i = lane; i < q_row; i += 32) {
      float v = 0.f;
      if (i < dim) v = slab_sum(x + i, n_partials, pstride);
      else if (i < dim + rot_dim) v = rotated(x + dim, i - dim);
      dst[i] = from_f32<T>(v);
    }
    return;
  }
  const int slot = slot_map[t];
  if (slot < 0) return;
  const float* x = row + static_cast<long long>(heads) * (dim + rot_dim);
  float ss[1] = {0.f};
  for (int i = threadIdx.x; i < kv_rank; i += kQkvThreads) {
    const float v = slab_sum(x + i, n_partials, pstride);
    stage[i] = v;
    ss[0] += v * v;
  }
  row_sum<kQkvThreads, 1, 1>(sh, ss, 0);
  const float inv = rsqrtf(ss[0] / static_cast<float>(kv_rank) + eps);
  T* dst = cache + static_cast<long long>(slot) * (kv_rank + rot_dim);
  for (int i = threadIdx.x; i < kv_rank; i += kQkvThreads) dst[i] = from_f32<T>(stage[i] * inv * latent_norm[i]);
  for (int i = threadIdx.x; i < rot_dim; i += kQkvThreads) dst[kv_rank + i] = from_f32<T>(rotated(x + kv_rank, i));
}

int latent_qkv(const bcg_layer* l, const float* proj, int n_partials, long long pstride, const int* positions,
               const int* slot_map, void* q, int act_dtype, int T, float eps, cudaStream_t st) {
  const int groups = (l->heads + kQkvThreads / 32 - 1) / (kQkvThreads / 32);
  const int q_row = l->q_ld > 0 ? l->q_ld : l->dim + l->rot_dim;
  const dim3 grid(T, groups + (l->owns_cache ? 1 : 0));
  const size_t sm = static_cast<size_t>(l->kv_rank) * 4;
  if (act_dtype == BCG_DT_F32)
    BCG_CUDA_CHECK(launch_k(latent_qkv_kernel<float>, grid, dim3(kQkvThreads), sm, st, proj, n_partials, pstride,
                            static_cast<long long>(l->n_in), positions, slot_map, l->cos_sin, l->latent_norm,
                            static_cast<float*>(q), static_cast<float*>(l->cache), l->heads, l->dim, l->rot_dim,
                            l->rot_dims, q_row, l->kv_rank, groups, eps));
  else
    BCG_CUDA_CHECK(launch_k(latent_qkv_kernel<__nv_bfloat16>, grid, dim3(kQkvThreads), sm, st, proj, n_partials,
                            pstride, static_cast<long long>(l->n_in), positions, slot_map, l->cos_sin,
                            l->latent_norm, static_cast<__nv_bfloat16*>(q), static_cast<__nv_bfloat16*>(l->cache),
                            l->heads, l->dim, l->rot_dim, l->rot_dims, q_row, l->kv_rank, groups, eps));
  return BCG_OK;
}

// ------------------------------------------------------------------------------------------- plain
constexpr int kPlainThreads = 128;
constexpr int kPlainKeys = 256;

template <typename T>
__global__ void __launch_bounds__(kPlainThreads)
latent_plain_kernel(const T* __restrict__ q, const T* __restrict__ cache, const __nv_bfloat16* __restrict__ w_uk,
                    const __nv_bfloat16* __restrict__ w_uv, const float* __restrict__ sink,
                    const int* __restrict__ rows, const int* __restrict__ positions, const int* __restrict__ row_seq,
                    const int* __restrict__ block_table, int max_blocks, int page_size, T* __restrict__ out,
                    int heads, int dim, int rot_dim, int vdim, int kv_rank, int q_row, int window, float scale) {
  extern __shared__ float sm[];
  __shared__ float red[kPlainThreads / 32];
  const int crow = kv_rank + rot_dim;
  float* qa = sm;                 // [kv_rank | rot_dim] query in latent space
  float* oc = qa + crow;          // [kv_rank]
  float* qs = oc + kv_rank;       // [dim]
  float* p = qs + dim;            // [kPlainKeys]
  pdl_launch_dependents();
  pdl_wait();
  const long long t = rows ? rows[blockIdx.x] : blockIdx.x;
  const int h = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pos = positions[t];
  const int* bt = block_table + static_cast<long long>(row_seq ? row_seq[t] : t) * max_blocks;
  const T* qh = q + (t * heads + h) * q_row;
  for (int i = threadIdx.x; i < dim; i += kPlainThreads) qs[i] = to_f32<T>(qh[i]);
  for (int i = threadIdx.x; i < rot_dim; i += kPlainThreads) qa[kv_rank + i] = to_f32<T>(qh[dim + i]);
  __syncthreads();
  for (int r = threadIdx.x; r < kv_rank; r += kPlainThreads) {
    float acc = 0.f;
    const __nv_bfloat16* w = w_uk + static_cast<long long>(h) * dim * kv_rank + r;
    for (int i = 0; i < dim; ++i) acc = fmaf(qs[i], __bfloat162float(w[static_cast<long long>(i) * kv_rank]), acc);
    qa[r] = acc;
    oc[r] = 0.f;
  }
  float m = sink ? sink[h] : -INFINITY, l = sink ? 1.0f : 0.0f;
  const int lo = window > 0 ? max(0, pos - window + 1) : 0;
  for (int j0 = lo; j0 <= pos; j0 += kPlainKeys) {
    const int n = min(kPlainKeys, pos + 1 - j0);
    __syncthreads();
    float mx = -INFINITY;
    for (int j = warp; j < n; j += kPlainThreads / 32) {
      const int key = j0 + j;
      const T* c = cache + (static_cast<long long>(bt[key / page_size]) * page_size + key % page_size) * crow;
      float s = 0.f;
      for (int i = lane; i < crow; i += 32) s = fmaf(qa[i], to_f32<T>(c[i]), s);
      s = warp_sum(s) * scale;
      if (lane == 0) p[j] = s;
      mx = fmaxf(mx, s);
    }
    if (lane == 0) red[warp] = mx;
    __syncthreads();
#pragma unroll
    for (int i = 0; i < kPlainThreads / 32; ++i) mx = fmaxf(mx, red[i]);
    const float m_new = fmaxf(m, mx);
    const float corr = expf(m - m_new);
    float sum = 0.f;
    for (int j = threadIdx.x; j < n; j += kPlainThreads) {
      const float e = expf(p[j] - m_new);
      p[j] = e;
      sum += e;
    }
    sum = warp_sum(sum);
    __syncthreads();
    if (lane == 0) red[warp] = sum;
    __syncthreads();
    sum = 0.f;
#pragma unroll
    for (int i = 0; i < kPlainThreads / 32; ++i) sum += red[i];
    l = l * corr + sum;
    m = m_new;
    for (int r = threadIdx.x; r < kv_rank; r += kPlainThreads) {
      float acc = oc[r] * corr;
      for (int j = 0; j < n; ++j) {
        const int key = j0 + j;
        acc = fmaf(p[j], to_f32<T>(cache[(static_cast<long long>(bt[key / page_size]) * page_size + key % page_size) * crow + r]), acc);
      }
      oc[r] = acc;
    }
  }
  __syncthreads();
  const float inv = 1.0f / l;
  for (int v = warp; v < vdim; v += kPlainThreads / 32) {
    const __nv_bfloat16* w = w_uv + (static_cast<long long>(h) * vdim + v) * kv_rank;
    float acc = 0.f;
    for (int r = lane; r < kv_rank; r += 32) acc = fmaf(__bfloat162float(w[r]), oc[r], acc);
    acc = warp_sum(acc);
    if (lane == 0) out[(t * heads + h) * vdim + v] = from_f32<T>(acc * inv);
  }
}

int latent_plain(const bcg_layer* l, const void* q, void* out, const bcg_step_batch* b, const int* rows, int n,
                 int page_size, int act_dtype, cudaStream_t st) {
  const int q_row = l->q_ld > 0 ? l->q_ld : l->dim + l->rot_dim;
  const int sm = (2 * l->kv_rank + l->rot_dim + l->dim + kPlainKeys) * 4;
  const auto* uk = static_cast<const __nv_bfloat16*>(l->w_uk);
  const auto* uv = static_cast<const __nv_bfloat16*>(l->w_uv);
  const dim3 grid(n, l->heads);
  if (act_dtype == BCG_DT_F32) {
    BCG_TRY(ensure_dynamic_smem(reinterpret_cast<const void*>(latent_plain_kernel<float>), 64 * 1024));
    BCG_CUDA_CHECK(launch_k(latent_plain_kernel<float>, grid, dim3(kPlainThreads), sm, st, static_cast<const float*>(q),
                            static_cast<const float*>(l->cache), uk, uv, l->sink, rows, b->positions, b->row_seq,
                            b->block_table, b->max_blocks, page_size, static_cast<float*>(out), l->heads, l->dim,
                            l->rot_dim, l->vdim, l->kv_rank, q_row, l->window, l->scale));
  } else {
    BCG_TRY(ensure_dynamic_smem(reinterpret_cast<const void*>(latent_plain_kernel<__nv_bfloat16>), 64 * 1024));
    BCG_CUDA_CHECK(launch_k(latent_plain_kernel<__nv_bfloat16>, grid, dim3(kPlainThreads), sm, st,
                            static_cast<const __nv_bfloat16*>(q), static_cast<const __nv_bfloat16*>(l->cache), uk, uv,
                            l->sink, rows, b->positions, b->row_seq, b->block_table, b->max_blocks, page_size,
                            static_cast<__nv_bfloat16*>(out), l->heads, l->dim, l->rot_dim, l->vdim, l->kv_rank,
                            q_row, l->window, l->scale));
  }
  return BCG_OK;
}

// ------------------------------------------------------------------------------------------- absorb
// q_latent[i, h] = (W_uk^T q_unrotated, q_rotated) for single token i = rows[i].  grid (heads, 128-column
// tiles of the latent, groups of 16 tokens); the weight tile is staged ahead of the dependency wait.
constexpr int kAbCols = 128, kAbThreads = 128;

__host__ __device__ constexpr int up16(int n) { return (n + 15) / 16 * 16; }
__host__ __device__ constexpr int absorb_smem(int dim) {
  return (up16(dim) * (kAbCols + 8) + 16 * (up16(dim) + 8)) * 2;
}

__global__ void __launch_bounds__(kAbThreads)
latent_absorb_kernel(const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ w_uk,
                     const int* __restrict__ rows, int n, __nv_bfloat16* __restrict__ q_latent, int heads, int dim,
                     int rot_dim, int kv_rank, int q_row) {
  extern __shared__ __align__(16) uint8_t ab_raw[];
  const int kd = up16(dim), srow = kd + 8;
  constexpr int wrow = kAbCols + 8;
  __nv_bfloat16* wt = reinterpret_cast<__nv_bfloat16*>(ab_raw);   // [kd][wrow]
  __nv_bfloat16* qs = wt + kd * wrow;                             // [16][srow]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.x, c0 = blockIdx.y * kAbCols, crow = kv_rank + rot_dim;
  pdl_launch_dependents();
  for (int i = threadIdx.x; i < kd * (kAbCols / 8); i += kAbThreads) {
    const int d = i / (kAbCols / 8), c = (i % (kAbCols / 8)) * 8;
    if (d < dim && c0 + c < kv_rank)
      cp_async16(wt + d * wrow + c, w_uk + (static_cast<long long>(h) * dim + d) * kv_rank + c0 + c);
    else
      *reinterpret_cast<uint4*>(wt + d * wrow + c) = make_uint4(0, 0, 0, 0);
  }
  cp_async_commit();
  pdl_wait();
  const int r0 = blockIdx.z * 16;
  const bool wide = (dim & 7) == 0 && (q_row & 7) == 0;
  for (int r = warp; r < 16; r += kAbThreads / 32) {
    const long long t = r0 + r < n ? (rows ? rows[r0 + r] : r0 + r) : -1;
    const __nv_bfloat16* src = q + (t * heads + h) * q_row;
    if (wide && t >= 0) {
      for (int d = lane * 8; d < kd; d += 256) {
        if (d < dim) cp_async16(qs + r * srow + d, src + d);
        else *reinterpret_cast<uint4*>(qs + r * srow + d) = make_uint4(0, 0, 0, 0);
      }
    } else {
      for (int d = lane; d < kd; d += 32) qs[r * srow + d] = (t >= 0 && d < dim) ? src[d] : __float2bfloat16(0.f);
    }
    if (blockIdx.y == 0 && t >= 0)
      for (int d = lane; d < rot_dim; d += 32)
        q_latent[(static_cast<long long>(r0 + r) * heads + h) * crow + kv_rank + d] = src[dim + d];
  }
  cp_async_commit();
  cp_async_wait<0>();
  __syncthreads();
  float acc[4][4] = {};
#pragma unroll 4
  for (int k = 0; k < kd; k += 16) {
    uint32_t a[4], b[4];
    ldsm_x4(a, qs + (lane & 15) * srow + k + (lane >> 4) * 8);
#pragma unroll
    for (int g = 0; g < 2; ++g) {
      ldsm_x4_trans(b, wt + (k + (lane & 15)) * wrow + warp * 32 + g * 16 + (lane >> 4) * 8);
      mma_bf16_16816(acc[g * 2], a, b[0], b[1]);
      mma_bf16_16816(acc[g * 2 + 1], a, b[2], b[3]);
    }
  }
#pragma unroll
  for (int g = 0; g < 4; ++g)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = r0 + (lane >> 2) + e * 8, c = c0 + warp * 32 + g * 8 + (lane & 3) * 2;
      if (r < n && c < kv_rank)
        *reinterpret_cast<uint32_t*>(q_latent + (static_cast<long long>(r) * heads + h) * crow + c) =
            pack_bf16(acc[g][2 * e], acc[g][2 * e + 1]);
    }
}

// ------------------------------------------------------------------------------------------- decode
// grid (spans, tokens, head groups of 32).  A token's visible keys, from the 64-aligned start of its window,
// are cut into spans of `tiles` 64-key tiles; a CTA works one span off with a running softmax (two tiles in
// shared memory, the next one in flight) and leaves an unnormalised partial.
constexpr int kLdKeys = 64, kLdHeads = 32, kLdThreads = 512, kLdMaxRank = 512;

__host__ __device__ constexpr int latent_decode_smem(int crow) {
  return (2 * kLdKeys + kLdHeads) * (crow + 8) * 2 + 2 * kLdHeads * (kLdKeys + 4) * 4 + kLdHeads * (kLdKeys + 8) * 2 +
         3 * kLdHeads * 4;
}

__global__ void __launch_bounds__(kLdThreads, 1)
latent_decode_kernel(const __nv_bfloat16* __restrict__ q_latent, const __nv_bfloat16* __restrict__ cache,
                     const int* __restrict__ rows, const int* __restrict__ positions,
                     const int* __restrict__ row_seq, const int* __restrict__ block_table, int max_blocks,
                     int page_size, float* __restrict__ part_o, float* __restrict__ part_ml, int heads, int kv_rank,
                     int rot_dim, int window, int tiles, float scale) {
  extern __shared__ __align__(16) uint8_t ld_raw[];
  constexpr int kSs = kLdKeys + 4, kPs = kLdKeys + 8, kWarps = kLdThreads / 32;
  const int crow = kv_rank + rot_dim, srow = crow + 8;     // +16 bytes: ldmatrix rows on different banks
  __nv_bfloat16* ks = reinterpret_cast<__nv_bfloat16*>(ld_raw);   // [2][64][srow]
  __nv_bfloat16* qs = ks + 2 * kLdKeys * srow;                    // [32][srow]
  float* ss = reinterpret_cast<float*>(qs + kLdHeads * srow);     // [2][32][kSs]: halves of the dot product
  __nv_bfloat16* ps = reinterpret_cast<__nv_bfloat16*>(ss + 2 * kLdHeads * kSs);   // [32][kPs]
  float* m_run = reinterpret_cast<float*>(ps + kLdHeads * kPs);
  float* l_run = m_run + kLdHeads;
  float* corr = l_run + kLdHeads;
  pdl_launch_dependents();
  pdl_wait();
  const int i_tok = blockIdx.y, h0 = blockIdx.z * kLdHeads;
  const int t = rows ? rows[i_tok] : i_tok;
  const int pos = positions[t];
  const int lo = window > 0 ? max(0, pos - window + 1) : 0;
  const int base0 = (lo / kLdKeys + blockIdx.x * tiles) * kLdKeys;
  if (base0 > pos) return;
  const int n_tiles = min(tiles, (pos - base0) / kLdKeys + 1);
  const int nh = min(kLdHeads, heads - h0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int* bt = block_table + static_cast<long long>(row_seq ? row_seq[t] : t) * max_blocks;
  const int vec = crow >> 3;
  auto load_tile = [&](int i) {
    // a warp loads four keys; their cache rows are looked up by four lanes at once
    constexpr int kPer = kLdKeys / kWarps;
    const int mine = base0 + i * kLdKeys + warp * kPer + (lane & (kPer - 1));
    long long at = -1;
    if (mine >= lo && mine <= pos) at = (static_cast<long long>(bt[mine / page_size]) * page_size + mine % page_size) * crow;
#pragma unroll
    for (int k = 0; k < kPer; ++k) {
      __nv_bfloat16* dst = ks + ((i & 1) * kLdKeys + warp * kPer + k) * srow;
      const long long row = __shfl_sync(0xffffffffu, at, k);
      if (row >= 0) {
        const __nv_bfloat16* src = cache + row;
        for (int v = lane; v < vec; v += 32) cp_async16(dst + v * 8, src + v * 8);
      } else {   // outside the window or not written: finite zeros, masked below
        for (int v = lane; v < vec; v += 32) *reinterpret_cast<uint4*>(dst + v * 8) = make_uint4(0, 0, 0, 0);
      }
    }
    cp_async_commit();
  };
  const __nv_bfloat16* qsrc = q_latent + (static_cast<long long>(i_tok) * heads + h0) * crow;
  for (int r = warp; r < kLdHeads; r += kWarps)
    for (int v = lane; v < vec; v += 32) {
      if (r < nh) cp_async16(qs + r * srow + v * 8, qsrc + static_cast<long long>(r) * crow + v * 8);
      else *reinterpret_cast<uint4*>(qs + r * srow + v * 8) = make_uint4(0, 0, 0, 0);
    }
  load_tile(0);
  if (threadIdx.x < kLdHeads) {
    m_run[threadIdx.x] = -INFINITY;
    l_run[threadIdx.x] = 0.f;
  }
  constexpr int kJ = kLdMaxRank / 16 / kWarps;
  float o[kJ][2][2][4] = {};     // 16-column tiles of the latent x (2 x 16 heads) x (2 x 8 columns)
  for (int i = 0; i < n_tiles; ++i) {
    if (i + 1 < n_tiles) {
      load_tile(i + 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const __nv_bfloat16* kt = ks + (i & 1) * kLdKeys * srow;
    {   // scores: warp = 16 heads x 16 keys x half of the dot product
      const int m0 = (warp & 1) * 16, n0 = ((warp >> 1) & 3) * 16, half = warp >> 3;
      const int steps = crow / 16, kb = half ? (steps / 2) * 16 : 0, ke = half ? crow : (steps / 2) * 16;
      float acc[2][4] = {};
      const __nv_bfloat16* kp = kt + (n0 + (lane & 7) + ((lane >> 4) << 3)) * srow + ((lane >> 3) & 1) * 8;
      const __nv_bfloat16* qp = qs + (m0 + (lane & 15)) * srow + (lane >> 4) * 8;
#pragma unroll 6
      for (int k = kb; k < ke; k += 16) {
        uint32_t b[4], a[4];
        ldsm_x4(b, kp + k);
        ldsm_x4(a, qp + k);
        mma_bf16_16816(acc[0], a, b[0], b[1]);
        mma_bf16_16816(acc[1], a, b[2], b[3]);
      }
#pragma unroll
      for (int g = 0; g < 2; ++g)
#pragma unroll
        for (int e = 0; e < 2; ++e)
          *reinterpret_cast<float2*>(ss + (half * kLdHeads + m0 + (lane >> 2) + e * 8) * kSs + n0 + g * 8 + (lane & 3) * 2) =
              make_float2(acc[g][2 * e], acc[g][2 * e + 1]);
    }
    __syncthreads();
    const int k0 = base0 + i * kLdKeys + lane, k1 = k0 + 32;
    const bool ok0 = k0 >= lo && k0 <= pos, ok1 = k1 >= lo && k1 <= pos;
    constexpr int kR = kLdHeads / kWarps;             // softmax of the tile: a warp's heads side by side
    float p0[kR], p1[kR], m[kR], l[kR], m_old[kR];
#pragma unroll
    for (int x = 0; x < kR; ++x) {
      const int r = warp + x * kWarps;
      const float* s0 = ss + r * kSs + lane;
      const float* s1 = s0 + kLdHeads * kSs;
      p0[x] = ok0 ? (s0[0] + s1[0]) * scale : -INFINITY;
      p1[x] = ok1 ? (s0[32] + s1[32]) * scale : -INFINITY;
      m_old[x] = m_run[r];
      m[x] = fmaxf(p0[x], p1[x]);
    }
#pragma unroll
    for (int off = 16; off > 0; off >>= 1)
#pragma unroll
      for (int x = 0; x < kR; ++x) m[x] = fmaxf(m[x], __shfl_xor_sync(0xffffffffu, m[x], off));
#pragma unroll
    for (int x = 0; x < kR; ++x) {                    // every tile has a visible key: m is finite
      const int r = warp + x * kWarps;
      m[x] = fmaxf(m[x], m_old[x]);
      p0[x] = ok0 ? __expf(p0[x] - m[x]) : 0.f;
      p1[x] = ok1 ? __expf(p1[x] - m[x]) : 0.f;
      ps[r * kPs + lane] = __float2bfloat16(p0[x]);
      ps[r * kPs + lane + 32] = __float2bfloat16(p1[x]);
      l[x] = p0[x] + p1[x];
    }
#pragma unroll
    for (int off = 16; off > 0; off >>= 1)
#pragma unroll
      for (int x = 0; x < kR; ++x) l[x] += __shfl_xor_sync(0xffffffffu, l[x], off);
    if (lane == 0) {
#pragma unroll
      for (int x = 0; x < kR; ++x) {
        const int r = warp + x * kWarps;
        const float c = __expf(m_old[x] - m[x]);
        corr[r] = c;
        m_run[r] = m[x];
        l_run[r] = fmaf(l_run[r], c, l[x]);
      }
    }
    __syncthreads();
    uint32_t pa[2][4][4];
#pragma unroll
    for (int m = 0; m < 2; ++m)
#pragma unroll
      for (int k = 0; k < 4; ++k)
        ldsm_x4(pa[m][k], ps + (m * 16 + (lane & 15)) * kPs + k * 16 + (lane >> 4) * 8);
#pragma unroll
    for (int j = 0; j < kJ; ++j) {
      const int n0 = (warp + j * kWarps) * 16;
      if (n0 < kv_rank) {
        if (i > 0) {
#pragma unroll
          for (int m = 0; m < 2; ++m)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
              const float c = corr[m * 16 + (lane >> 2) + e * 8];
#pragma unroll
              for (int g = 0; g < 2; ++g) {
                o[j][m][g][2 * e] *= c;
                o[j][m][g][2 * e + 1] *= c;
              }
            }
        }
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          uint32_t bv[4];
          ldsm_x4_trans(bv, kt + (k * 16 + (lane & 15)) * srow + n0 + (lane >> 4) * 8);
#pragma unroll
          for (int m = 0; m < 2; ++m) {
            mma_bf16_16816(o[j][m][0], pa[m][k], bv[0], bv[1]);
            mma_bf16_16816(o[j][m][1], pa[m][k], bv[2], bv[3]);
          }
        }
      }
    }
    __syncthreads();     // the tile and the probabilities may be overwritten
  }
  const long long span = static_cast<long long>(i_tok) * gridDim.x + blockIdx.x;
#pragma unroll
  for (int j = 0; j < kJ; ++j) {
    const int n0 = (warp + j * kWarps) * 16;
    if (n0 < kv_rank) {
#pragma unroll
      for (int m = 0; m < 2; ++m)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int r = m * 16 + (lane >> 2) + e * 8;
          if (r < nh)
#pragma unroll
            for (int g = 0; g < 2; ++g)
              *reinterpret_cast<float2*>(part_o + (span * heads + h0 + r) * kv_rank + n0 + g * 8 + (lane & 3) * 2) =
                  make_float2(o[j][m][g][2 * e], o[j][m][g][2 * e + 1]);
        }
    }
  }
  if (threadIdx.x < nh) {
    part_ml[(span * heads + h0 + threadIdx.x) * 2] = m_run[threadIdx.x];
    part_ml[(span * heads + h0 + threadIdx.x) * 2 + 1] = l_run[threadIdx.x];
  }
}

// o_latent[i, h] = sum over spans (and the sink's share of the denominator), bf16.  grid (tokens, heads), a
// warp per 128 columns.
__global__ void __launch_bounds__(128)
latent_combine_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml,
                      const float* __restrict__ sink, const int* __restrict__ rows,
                      const int* __restrict__ positions, __nv_bfloat16* __restrict__ o_latent, int spans, int tiles,
                      int heads, int kv_rank, int window) {
  pdl_launch_dependents();
  pdl_wait();
  const int i_tok = blockIdx.x, h = blockIdx.y, lane = threadIdx.x & 31;
  const int pos = positions[rows ? rows[i_tok] : i_tok];
  const int lo = window > 0 ? max(0, pos - window + 1) : 0;
  const int n = min(spans, (pos / kLdKeys - lo / kLdKeys) / tiles + 1);
  const float2* ml = reinterpret_cast<const float2*>(part_ml) + static_cast<long long>(i_tok) * spans * heads + h;
  const float s0 = sink ? sink[h] : -INFINITY;
  float m = -INFINITY, l = 0.f;
  for (int c = lane; c < n; c += 32) {       // a lane's spans, then across lanes
    const float2 v = ml[static_cast<long long>(c) * heads];
    const float mn = fmaxf(m, v.x);
    l = l * __expf(m - mn) + v.y * __expf(v.x - mn);
    m = mn;
  }
  const float top = fmaxf(warp_max(m), s0);
  l = warp_sum(m == -INFINITY ? 0.f : l * __expf(m - top)) + (sink ? __expf(s0 - top) : 0.f);
  const float inv = 1.0f / l;
  const float* src = part_o + (static_cast<long long>(i_tok) * spans * heads + h) * kv_rank;
  const long long pitch = static_cast<long long>(heads) * kv_rank;
  for (int r = threadIdx.x * 4; r < kv_rank; r += 512) {
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int c0 = 0; c0 < n; c0 += 8) {
      float4 v[8];
      float w[8];
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const int c = min(c0 + k, n - 1);
        v[k] = *reinterpret_cast<const float4*>(src + c * pitch + r);
        w[k] = ml[static_cast<long long>(c) * heads].x;
      }
#pragma unroll
      for (int k = 0; k < 8; ++k)
        if (c0 + k < n) {
          const float e = __expf(w[k] - top);
          acc.x = fmaf(e, v[k].x, acc.x);
          acc.y = fmaf(e, v[k].y, acc.y);
          acc.z = fmaf(e, v[k].z, acc.z);
          acc.w = fmaf(e, v[k].w, acc.w);
        }
    }
    store4(o_latent + (static_cast<long long>(i_tok) * heads + h) * kv_rank + r, acc.x * inv, acc.y * inv, acc.z * inv,
           acc.w * inv);
  }
}

// out[t, h, v] = W_uv o_latent.  grid (heads, v tiles of 32, groups of 16 tokens); the weight tile is staged
// ahead of the wait, a warp per 8 values.
constexpr int kUpV = 32, kUpThreads = 128;
__host__ __device__ constexpr int up_row(int kv_rank) { return (kv_rank + 31) / 32 * 32 + 8; }
__host__ __device__ constexpr int up_smem(int kv_rank) { return (kUpV + 16) * up_row(kv_rank) * 2; }

__global__ void __launch_bounds__(kUpThreads)
latent_up_kernel(const __nv_bfloat16* __restrict__ o_latent, const __nv_bfloat16* __restrict__ w_uv,
                 const int* __restrict__ rows, int n, __nv_bfloat16* __restrict__ out, int heads, int vdim,
                 int kv_rank) {
  extern __shared__ __align__(16) uint8_t up_raw[];
  const int srow = up_row(kv_rank), kd = srow - 8;
  __nv_bfloat16* wt = reinterpret_cast<__nv_bfloat16*>(up_raw);   // [32][srow]
  __nv_bfloat16* os = wt + kUpV * srow;                           // [16][srow]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.x, v0 = blockIdx.y * kUpV;
  pdl_launch_dependents();
  auto stage = [&](__nv_bfloat16* dst, const __nv_bfloat16* src, bool there) {   // one row, by a warp
    for (int c = lane * 8; c < kd; c += 256) {
      if (there && c < kv_rank) cp_async16(dst + c, src + c);
      else *reinterpret_cast<uint4*>(dst + c) = make_uint4(0, 0, 0, 0);
    }
  };
  for (int r = warp; r < kUpV; r += kUpThreads / 32)
    stage(wt + r * srow, w_uv + (static_cast<long long>(h) * vdim + v0 + r) * kv_rank, v0 + r < vdim);
  pdl_wait();
  const int r0 = blockIdx.z * 16;
  for (int r = warp; r < 16; r += kUpThreads / 32)
    stage(os + r * srow, o_latent + (static_cast<long long>(r0 + r) * heads + h) * kv_rank, r0 + r < n);
  cp_async_commit();
  cp_async_wait<0>();
  __syncthreads();
  float acc[2][4] = {};
  const __nv_bfloat16* wp = wt + (warp * 8 + (lane & 7)) * srow + (lane >> 3) * 8;
  const __nv_bfloat16* op = os + (lane & 15) * srow + (lane >> 4) * 8;
#pragma unroll 4
  for (int k = 0; k < kd; k += 32) {
    uint32_t b[4], a0[4], a1[4];
    ldsm_x4(b, wp + k);
    ldsm_x4(a0, op + k);
    ldsm_x4(a1, op + k + 16);
    mma_bf16_16816(acc[0], a0, b[0], b[1]);
    mma_bf16_16816(acc[1], a1, b[2], b[3]);
  }
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const int r = r0 + (lane >> 2) + (e >> 1) * 8, v = v0 + warp * 8 + (lane & 3) * 2 + (e & 1);
    if (r < n && v < vdim) {
      const long long t = rows ? rows[r] : r;
      out[(t * heads + h) * vdim + v] = __float2bfloat16(acc[0][e] + acc[1][e]);
    }
  }
}

// Sizes the latent-space tensor-core path takes.
bool latent_decode_ok(const bcg_layer* l) {
  const int crow = l->kv_rank + l->rot_dim;
  return l->kv_rank % 16 == 0 && l->kv_rank <= kLdMaxRank && crow % 16 == 0 &&
         latent_decode_smem(crow) <= 220 * 1024 && absorb_smem(l->dim) <= 200 * 1024 && up_smem(l->kv_rank) <= 200 * 1024;
}

// Key tiles per span, for `rows` (token, head group) pairs of up to `total` tiles each: the choice that needs
// the fewest tile times on 148 SMs (a span costs about two tiles of start-up).
static int span_tiles(int rows, int total) {
  int best = 1;
  long long best_cost = -1;
  for (int t = 1; t <= total; ++t) {
    const long long ctas = static_cast<long long>(rows) * ((total + t - 1) / t);
    const long long cost = ((ctas + 147) / 148) * (t + 2);
    if (best_cost < 0 || cost < best_cost) {
      best_cost = cost;
      best = t;
    }
  }
  return best;
}

int latent_decode(const bcg_layer* l, const bcg_stack_ws* ws, const bcg_step_batch* b, int page_size,
                  cudaStream_t st) {
  const int n = b->single_rows ? b->n_single : b->T;
  const int crow = l->kv_rank + l->rot_dim;
  const int q_row = l->q_ld > 0 ? l->q_ld : l->dim + l->rot_dim;
  const int reach = l->window > 0 && l->window < b->max_context ? l->window + kLdKeys : b->max_context;
  const int total = (reach + kLdKeys - 1) / kLdKeys, groups = (l->heads + kLdHeads - 1) / kLdHeads;
  const int tiles = span_tiles(n * groups, total), spans = (total + tiles - 1) / tiles;
  if (n > ws->D_max || n > 65535 || static_cast<long long>(n) * spans * l->heads * l->kv_rank > ws->part_floats) {
    set_last_error("bcg_latent_attention", "single tokens x key spans exceed the decode scratch");
    return BCG_ERR_TOO_LARGE;
  }
  auto* ql = static_cast<__nv_bfloat16*>(ws->q_latent);
  auto* ol = static_cast<__nv_bfloat16*>(ws->o_latent);
  BCG_TRY(ensure_dynamic_smem(reinterpret_cast<const void*>(latent_absorb_kernel), 200 * 1024));
  BCG_TRY(ensure_dynamic_smem(reinterpret_cast<const void*>(latent_decode_kernel), 220 * 1024));
  BCG_TRY(ensure_dynamic_smem(reinterpret_cast<const void*>(latent_up_kernel), 200 * 1024));
  BCG_CUDA_CHECK(launch_k(latent_absorb_kernel, dim3(l->heads, (l->kv_rank + kAbCols - 1) / kAbCols, (n + 15) / 16), dim3(kAbThreads),
                          absorb_smem(l->dim), st, static_cast<const __nv_bfloat16*>(ws->q),
                          static_cast<const __nv_bfloat16*>(l->w_uk), b->single_rows, n, ql, l->heads, l->dim,
                          l->rot_dim, l->kv_rank, q_row));
  BCG_CUDA_CHECK(launch_k(latent_decode_kernel, dim3(spans, n, groups), dim3(kLdThreads),
                          latent_decode_smem(crow), st, ql, static_cast<const __nv_bfloat16*>(l->cache),
                          b->single_rows, b->positions, b->row_seq, b->block_table, b->max_blocks, page_size,
                          ws->part_o, ws->part_ml, l->heads, l->kv_rank, l->rot_dim, l->window, tiles, l->scale));
  BCG_CUDA_CHECK(launch_k(latent_combine_kernel, dim3(n, l->heads), dim3(128), 0, st, ws->part_o, ws->part_ml, l->sink,
                          b->single_rows, b->positions, ol, spans, tiles, l->heads, l->kv_rank, l->window));
  BCG_CUDA_CHECK(launch_k(latent_up_kernel, dim3(l->heads, (l->vdim + kUpV - 1) / kUpV, (n + 15) / 16), dim3(kUpThreads),
                          up_smem(l->kv_rank), st, ol, static_cast<const __nv_bfloat16*>(l->w_uv), b->single_rows, n,
                          static_cast<__nv_bfloat16*>(ws->mix), l->heads, l->vdim, l->kv_rank));
  return BCG_OK;
}

// ------------------------------------------------------------------------------------------- gather
__global__ void __launch_bounds__(128)
latent_gather_kernel(const __nv_bfloat16* __restrict__ cache, const int* __restrict__ slots,
                     __nv_bfloat16* __restrict__ out, int n, int crow) {
  pdl_launch_dependents();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long r = static_cast<long long>(blockIdx.x) * 4 + warp;
  if (r >= n) return;
  const uint4* src = reinterpret_cast<const uint4*>(cache + static_cast<long long>(slots[r]) * crow);
  uint4* dst = reinterpret_cast<uint4*>(out + r * crow);
  for (int i = lane; i < crow / 8; i += 32) dst[i] = src[i];
}

int latent_gather(const void* cache, const int* slots, void* out, int n, int crow, cudaStream_t st) {
  BCG_CUDA_CHECK(launch_k(latent_gather_kernel, dim3((n + 3) / 4), dim3(128), 0, st,
                          static_cast<const __nv_bfloat16*>(cache), slots, static_cast<__nv_bfloat16*>(out), n, crow));
  return BCG_OK;
}

}  // namespace bcg
