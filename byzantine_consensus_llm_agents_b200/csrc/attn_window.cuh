// Prompt attention on tcgen05: 128 query rows of one head against keys in blocks of 64, causal with an optional
// sliding window.  Options: a softmax sink, a linear distance bias per head (SLOPES), keys and values read from
// contiguous rows or through a block table of 16-token pages (PAGED); with pages and without a bias, blocks of means
// of the tokens in front of the window, which have pages of their own, and outputs turned back by the query's position.
//
//   grid (heads, tiles), 192 threads; keys from the first one any row of the tile sees.
//     warp 0      TMA producer: Q tile once, then K and V blocks (64-column boxes of 64 rows, or of the 16 rows
//                 of a page; 128B swizzle)
//     warp 1      MMA issuer: S_j = Q K_j^T into one of two TMEM accumulators; O += P_j V_j in TMEM
//     warps 2-5   softmax, thread = query row = TMEM lane; the running maximum starts at the sink with
//                 denominator 1 (exp(sink - sink)), which is the sink's whole effect; rescaling of O is
//                 lazy (only when a block's maximum exceeds the running one by more than 8 in log2 units).
//                 The distance bias slope * (j - i) is formed relative to the row's own key, so that it is
//                 exact where weights are not negligible.
// tiles[tile] = {first token, its position, tokens (<= 128), row of key position k0, k0, sequence, 0, 0}; PAGED
// uses the sequence's block-table row, otherwise rows follow one another from k0's.
#pragma once
#include "attn_tcgen05.cuh"
#include "stack_common.cuh"
#include "kernels.h"

namespace bcg {

constexpr int kWaBM = 128, kWaBN = 64, kWaThreads = 192, kWaPage = 16;
constexpr int kWaQHalf = kWaBM * 64 * 2;     // [128 rows][64 bf16]
constexpr int kWaKvHalf = kWaBN * 64 * 2;    // [64 keys][64 bf16]
constexpr float kWaRescaleGap = 8.0f;
constexpr float kWaNoSink = -1e30f;          // finite "minus infinity" for the running maximum

template <int QD, int VD>
struct WaCfg {
  static constexpr int kQ = QD / 64 * kWaQHalf, kK = QD / 64 * kWaKvHalf, kV = VD / 64 * kWaKvHalf, kP = kWaQHalf;
  static constexpr int kFixed = kQ + kP + 256 + 768;
  // two CTAs per SM (one hides the other's bubbles) where one-stage rings make that fit, else two stages
  static constexpr int kStages = (kFixed + 2 * (kK + kV) > 113 * 1024 && kFixed + kK + kV <= 113 * 1024) ? 1 : 2;
  static constexpr int kOffK = kQ, kOffV = kOffK + kStages * kK, kOffP = kOffV + kStages * kV, kOffBar = kOffP + kP;
  static constexpr int kSlack = 768;
  static constexpr int kSmem = kOffBar + 256 + kSlack;
  static constexpr uint32_t kTmemCols = 2 * kWaBN + VD <= 256 ? 256 : 512;
  static constexpr int kCtasPerSm = (kSmem <= 113 * 1024 && kTmemCols == 256) ? 2 : 1;
};

// One block of keys or values: D / 64 column boxes of 64 rows, or of four pages of 16.
template <int D, bool PAGED>
__device__ __forceinline__ void load_block(uint8_t* dst, const CUtensorMap* map, uint64_t* bar, int col, int row,
                                           const int (&prow)[kWaBN / kWaPage]) {
#pragma unroll
  for (int c = 0; c < D / 64; ++c) {
    if constexpr (PAGED) {
#pragma unroll
      for (int pg = 0; pg < kWaBN / kWaPage; ++pg)
        tma_load_2d(dst + c * kWaKvHalf + pg * kWaPage * 128, map, bar, c * 64, prow[pg], kEvictNormal);
    } else {
      tma_load_2d(dst + c * kWaKvHalf, map, bar, col + c * 64, row, kEvictNormal);
    }
  }
}

// Means of blocks of `pool` tokens that a query sees beside its window: block b from position b * pool + pool - 1 + window on.
struct PooledKeys {
  int pool, col;            // col: first column of their pages in the block table; pool = 0: none
  __device__ __forceinline__ int visible(int pos, int window) const {
    const int gone = pos - window + 1;             // tokens in front of the window
    return pool > 0 && gone >= pool ? gone / pool : 0;
  }
};

struct WindowAttn {
  const int* tiles;
  int n_tiles;
  const float* sink;        // [heads] or NULL
  const float* slopes;      // [heads], SLOPES only
  const int* block_table;   // PAGED only
  int max_blocks, page_heads;   // page_heads: key/value heads of a page
  int k_col, v_col;         // contiguous rows: columns per head of a key / first column of the values
  int group;                // query heads per key/value head
  const float* gates;       // [tokens][heads] factors of the outputs, or NULL
  PooledKeys pooled;        // PAGED without SLOPES only
  const float* v_cos_sin;   // outputs turn back in pairs of neighbours, or NULL
  int v_rot_dims;
  __nv_bfloat16* out;
  long long out_ld;         // row pitch
  int heads, vdim, window;
  float scale_log2e;
};

// Columns c0 .. c0 + 31 of an output row turned back: pairs (2m, 2m + 1), cosines at m of the table's row, sines at dims / 2 + m.
__device__ __forceinline__ void turn_back(uint32_t (&o)[32], const float* row, int dims, int c0) {
  const int half = dims / 2;
#pragma unroll
  for (int i = 0; i < 16; i += 4) {
    const int m = c0 / 2 + i;
    float cs[4], sn[4];
    if (m + 4 <= half && dims % 8 == 0) {
      const float4 c = __ldg(reinterpret_cast<const float4*>(row + m)), s = __ldg(reinterpret_cast<const float4*>(row + half + m));
      cs[0] = c.x; cs[1] = c.y; cs[2] = c.z; cs[3] = c.w;
      sn[0] = s.x; sn[1] = s.y; sn[2] = s.z; sn[3] = s.w;
    } else {
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        cs[k] = m + k < half ? row[m + k] : 1.f;
        sn[k] = m + k < half ? row[half + m + k] : 0.f;
      }
    }
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const float u = __uint_as_float(o[2 * (i + k)]), v = __uint_as_float(o[2 * (i + k) + 1]);
      o[2 * (i + k)] = __float_as_uint(u * cs[k] + v * sn[k]);
      o[2 * (i + k) + 1] = __float_as_uint(v * cs[k] - u * sn[k]);
    }
  }
}

template <int QD, int VD, bool PAGED, bool SLOPES>
__global__ void __launch_bounds__(kWaThreads, WaCfg<QD, VD>::kCtasPerSm)
window_attn_kernel(const __grid_constant__ CUtensorMap q_map, const __grid_constant__ CUtensorMap k_map,
                   const __grid_constant__ CUtensorMap v_map, const WindowAttn a) {
  using C = WaCfg<QD, VD>;
  constexpr int ST = C::kStages;
  constexpr uint32_t kIdescQK = make_idesc_bf16_m128(kWaBN);
  constexpr uint32_t kIdescPV = make_idesc_bf16_m128(VD) | (1u << 16);   // B (values) is MN-major
  extern __shared__ __align__(1024) uint8_t wa_raw[];
  const uint32_t pad = (1024u - (smem_u32(wa_raw) & 1023u)) & 1023u;
  if (pad > static_cast<uint32_t>(C::kSlack)) __trap();
  uint8_t* smem = wa_raw + pad;
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + C::kOffBar);
  uint64_t* q_full = bars + 0;
  uint64_t* k_full = bars + 1;    // [ST]
  uint64_t* k_empty = bars + 3;
  uint64_t* v_full = bars + 5;
  uint64_t* v_empty = bars + 7;
  uint64_t* s_full = bars + 9;    // [2]
  uint64_t* s_free = bars + 11;   // [2]
  uint64_t* p_full = bars + 13;
  uint64_t* pv_done = bars + 14;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 15);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_launch_dependents();

  const int head = blockIdx.x;
  const int kvh = head / a.group;
  const int* ti = a.tiles + (a.n_tiles - 1 - static_cast<int>(blockIdx.y)) * 8;
  if (threadIdx.x == 0) {
    tma_prefetch_desc(&q_map);
    tma_prefetch_desc(&k_map);
    tma_prefetch_desc(&v_map);
    mbar_init(q_full, 1);
    for (int i = 0; i < ST; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&k_empty[i], 1);
      mbar_init(&v_full[i], 1);
      mbar_init(&v_empty[i], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&s_full[i], 1);
      mbar_init(&s_free[i], 128);
    }
    mbar_init(p_full, 128);
    mbar_init(pv_done, 1);
    fence_barrier_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, C::kTmemCols);
    tmem_relinquish();
  }
  pdl_wait();
  const int row0 = ti[0], pos0 = ti[1], n_rows = ti[2];
  const int window = a.window;
  // first key of block 0: the first one a row sees (gathered rows start no later), or its page's first
  const int first = max(window > 0 ? pos0 - window + 1 : 0, PAGED ? 0 : ti[4]);
  const int kb = PAGED ? first & ~(kWaPage - 1) : first;
  const int kv_row = ti[3] + kb - ti[4];
  const int nb_tok = (pos0 + n_rows - kb + kWaBN - 1) / kWaBN;
  constexpr bool kPools = PAGED && !SLOPES;
  const int n_pooled = kPools ? a.pooled.visible(pos0 + n_rows - 1, window) : 0;    // pooled blocks come behind the tokens
  const int nb = nb_tok + (n_pooled + kWaBN - 1) / kWaBN;
  // With a distance bias the newest keys usually hold the maximum: they come first, so that O is rarely rescaled.
  auto block_at = [&](int j) { return SLOPES ? nb - 1 - j : j; };
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t tmem_o = tmem_base + 2 * kWaBN;

  if (warp == 0) {
    if (lane == 0) {
      mbar_arrive_expect_tx(q_full, C::kQ);
#pragma unroll
      for (int c = 0; c < QD / 64; ++c)
        tma_load_2d(smem + c * kWaQHalf, &q_map, q_full, head * QD + c * 64, row0, kEvictFirst);
      const int* bt = PAGED ? a.block_table + static_cast<long long>(ti[5]) * a.max_blocks : nullptr;
      const int last_page = (pos0 + n_rows - 1) / kWaPage;   // pages past it are never read (clamped)
      for (int j = 0; j < nb; ++j) {
        const int st = j % ST;
        const uint32_t par = (j / ST) & 1;
        const int jb = block_at(j);
        int prow[kWaBN / kWaPage];      // PAGED: first row of every page of the block
        if constexpr (PAGED) {
#pragma unroll
          for (int pg = 0; pg < kWaBN / kWaPage; ++pg) {
            int at = min((kb + jb * kWaBN) / kWaPage + pg, last_page);
            if (kPools && jb >= nb_tok)
              at = a.pooled.col + min((jb - nb_tok) * (kWaBN / kWaPage) + pg, (n_pooled - 1) / kWaPage);
            prow[pg] = (bt[at] * a.page_heads + kvh) * kWaPage;
          }
        }
        uint8_t* dk = smem + C::kOffK + st * C::kK;
        mbar_wait(&k_empty[st], par ^ 1);
        mbar_arrive_expect_tx(&k_full[st], C::kK);
        load_block<QD, PAGED>(dk, &k_map, &k_full[st], kvh * a.k_col, kv_row + jb * kWaBN, prow);
        uint8_t* dv = smem + C::kOffV + st * C::kV;
        mbar_wait(&v_empty[st], par ^ 1);
        mbar_arrive_expect_tx(&v_full[st], C::kV);
        load_block<VD, PAGED>(dv, &v_map, &v_full[st], a.v_col + kvh * VD, kv_row + jb * kWaBN, prow);
      }
    }
  } else if (warp == 1) {
    const uint32_t sq = smem_u32(smem);
    const uint32_t sp = smem_u32(smem + C::kOffP);
    auto issue_s = [&](int j) {
      const int st = j % ST;
      mbar_wait(&k_full[st], (j / ST) & 1);
      mbar_wait(&s_free[j & 1], ((j >> 1) & 1) ^ 1);
      tc_fence_after();
      if (lane == 0) {
        const uint32_t sk = smem_u32(smem + C::kOffK + st * C::kK);
        const uint32_t d = tmem_base + static_cast<uint32_t>((j & 1) * kWaBN);
#pragma unroll
        for (int ks = 0; ks < QD / 16; ++ks)
          umma_bf16(d, make_kmajor_sw128_desc(sq + (ks >> 2) * kWaQHalf + (ks & 3) * 32),
                    make_kmajor_sw128_desc(sk + (ks >> 2) * kWaKvHalf + (ks & 3) * 32), kIdescQK, ks > 0 ? 1u : 0u);
        umma_commit(&k_empty[st]);
        umma_commit(&s_full[j & 1]);
      }
      __syncwarp();
    };
    auto issue_pv = [&](int j) {
      const int st = j % ST;
      mbar_wait(p_full, j & 1);
      mbar_wait(&v_full[st], (j / ST) & 1);
      tc_fence_after();
      if (lane == 0) {
        const uint32_t sv = smem_u32(smem + C::kOffV + st * C::kV);
#pragma unroll
        for (int kk = 0; kk < kWaBN / 16; ++kk)
          umma_bf16(tmem_o, make_kmajor_sw128_desc(sp + kk * 32), make_mnmajor_sw128_desc(sv + kk * 16 * 128, kWaKvHalf),
                    kIdescPV, (j > 0 || kk > 0) ? 1u : 0u);
        umma_commit(&v_empty[st]);
        umma_commit(pv_done);
      }
      __syncwarp();
    };
    mbar_wait(q_full, 0);
    issue_s(0);
    for (int j = 0; j < nb; ++j) {
      if (j + 1 < nb) issue_s(j + 1);
      issue_pv(j);
    }
  } else {
    const int q4 = warp & 3;
    const int r = q4 * 32 + lane;
    const uint32_t lane_addr = static_cast<uint32_t>(q4 * 32) << 16;
    const int tok_limit = pos0 + r - kb;                                   // last visible key, counted from kb
    const int tok_low = window > 0 ? max(0, pos0 + r - window + 1 - kb) : 0;   // first visible key
    uint8_t* p_row = smem + C::kOffP + r * 128;
    const int sw = r & 7;
    float m_run = a.sink ? a.sink[head] * 1.4426950408889634f : kWaNoSink;
    float l_run = a.sink ? 1.0f : 0.0f;
    const float slope = SLOPES ? a.slopes[head] * 1.4426950408889634f : 0.f;
    const uint64_t scale2 = pack_f32x2(__float_as_uint(a.scale_log2e), __float_as_uint(a.scale_log2e));
    for (int j = 0; j < nb; ++j) {
      const bool pooled = kPools && j >= nb_tok;
      const int col0 = pooled ? (j - nb_tok) * kWaBN : block_at(j) * kWaBN;
      const int limit = pooled ? a.pooled.visible(pos0 + r, window) - 1 : tok_limit, low = pooled ? 0 : tok_low;
      const bool need_mask = col0 + kWaBN - 1 > limit || col0 < low;
      mbar_wait(&s_full[j & 1], (j >> 1) & 1);
      tc_fence_after();
      uint32_t s[kWaBN];
#pragma unroll
      for (int c = 0; c < kWaBN / 32; ++c)
        tmem_ld_x32(tmem_base + lane_addr + (j & 1) * kWaBN + c * 32, s + c * 32);
      tmem_ld_wait();
      tc_fence_before();
      mbar_arrive(&s_free[j & 1]);
      if constexpr (SLOPES) {       // biased scores, log2 units
        const float off = slope * static_cast<float>(col0 - limit);
        const uint64_t slope2 = pack_f32x2(__float_as_uint(slope), __float_as_uint(slope));
        const uint64_t off2 = pack_f32x2(__float_as_uint(off), __float_as_uint(off));
#pragma unroll
        for (int i = 0; i < kWaBN; i += 2) {
          const uint64_t at = pack_f32x2(__float_as_uint(static_cast<float>(i)), __float_as_uint(static_cast<float>(i + 1)));
          float x0, x1;
          unpack_f32x2(fma_f32x2(pack_f32x2(s[i], s[i + 1]), scale2, fma_f32x2(at, slope2, off2)), x0, x1);
          s[i] = __float_as_uint(x0);
          s[i + 1] = __float_as_uint(x1);
        }
      }
      float mx = -INFINITY;
      if (need_mask) {
#pragma unroll
        for (int i = 0; i < kWaBN; ++i) {
          if (col0 + i > limit || col0 + i < low) s[i] = 0xff800000u;   // -inf
          mx = fmaxf(mx, __uint_as_float(s[i]));
        }
      } else {
#pragma unroll
        for (int i = 0; i < kWaBN; ++i) mx = fmaxf(mx, __uint_as_float(s[i]));
      }
      const float m_blk = SLOPES ? mx : mx * a.scale_log2e;
      const bool grow = m_blk > m_run + kWaRescaleGap;
      const float m_new = grow ? m_blk : m_run;
      mbar_wait(pv_done, (j & 1) ^ 1);   // PV_{j-1} complete: P may be overwritten, O rescaled
      if (__any_sync(0xffffffffu, grow)) {
        const float corr = grow ? ex2_approx(m_run - m_new) : 1.0f;
        if (j > 0) {
          tc_fence_after();
#pragma unroll
          for (int c = 0; c < VD / 32; ++c) {
            uint32_t o[32];
            tmem_ld_x32(tmem_o + lane_addr + c * 32, o);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * corr);
            tmem_st_x32(tmem_o + lane_addr + c * 32, o);
          }
          tmem_st_wait();
        }
        l_run *= corr;
      }
      m_run = m_new;
      const uint64_t negm2 = pack_f32x2(__float_as_uint(-m_run), __float_as_uint(-m_run));
      uint64_t l2 = pack_f32x2(0u, 0u);
#pragma unroll
      for (int c = 0; c < kWaBN / 8; ++c) {
        uint32_t pk[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          float x0, x1;
          const uint64_t raw = pack_f32x2(s[c * 8 + 2 * i], s[c * 8 + 2 * i + 1]);
          unpack_f32x2(SLOPES ? add_f32x2(raw, negm2) : fma_f32x2(raw, scale2, negm2), x0, x1);
          const float p0 = ex2_approx(x0), p1 = ex2_approx(x1);
          l2 = add_f32x2(l2, pack_f32x2(__float_as_uint(p0), __float_as_uint(p1)));
          pk[i] = pack_bf16(p0, p1);
        }
        *reinterpret_cast<uint4*>(p_row + ((c ^ sw) << 4)) = make_uint4(pk[0], pk[1], pk[2], pk[3]);
      }
      float l_lo, l_hi;
      unpack_f32x2(l2, l_lo, l_hi);
      l_run += l_lo + l_hi;
      tc_fence_before();
      fence_proxy_async();
      mbar_arrive(p_full);
    }
    mbar_wait(pv_done, (nb - 1) & 1);
    tc_fence_after();
    float inv = l_run > 0.f ? 1.0f / l_run : 0.f;
    if (a.gates && r < n_rows) inv *= a.gates[(static_cast<long long>(row0) + r) * a.heads + head];
    __nv_bfloat16* dst = a.out + (static_cast<long long>(row0) + r) * a.out_ld + static_cast<long long>(head) * a.vdim;
#pragma unroll
    for (int c = 0; c < VD / 32; ++c) {
      uint32_t o[32];
      tmem_ld_x32(tmem_o + lane_addr + c * 32, o);
      tmem_ld_wait();
      if (r < n_rows) {
        if constexpr (kPools) {
          if (a.v_cos_sin) turn_back(o, a.v_cos_sin + static_cast<long long>(pos0 + r) * a.v_rot_dims, a.v_rot_dims, c * 32);
        }
#pragma unroll
        for (int g = 0; g < 4; ++g)
          if (c * 32 + g * 8 < a.vdim) {
            uint4 w;
            w.x = pack_bf16(__uint_as_float(o[8 * g + 0]) * inv, __uint_as_float(o[8 * g + 1]) * inv);
            w.y = pack_bf16(__uint_as_float(o[8 * g + 2]) * inv, __uint_as_float(o[8 * g + 3]) * inv);
            w.z = pack_bf16(__uint_as_float(o[8 * g + 4]) * inv, __uint_as_float(o[8 * g + 5]) * inv);
            w.w = pack_bf16(__uint_as_float(o[8 * g + 6]) * inv, __uint_as_float(o[8 * g + 7]) * inv);
            reinterpret_cast<uint4*>(dst)[c * 4 + g] = w;
          }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem_base, C::kTmemCols);
}

template <int QD, int VD, bool PAGED, bool SLOPES>
static int launch_window_attn(const CUtensorMap& qm, const CUtensorMap& km, const CUtensorMap& vm, const WindowAttn& a,
                              cudaStream_t st) {
  using C = WaCfg<QD, VD>;
  BCG_TRY(ensure_dynamic_smem(reinterpret_cast<const void*>(window_attn_kernel<QD, VD, PAGED, SLOPES>), C::kSmem));
  BCG_CUDA_CHECK(launch_k(window_attn_kernel<QD, VD, PAGED, SLOPES>, dim3(a.heads, a.n_tiles), dim3(kWaThreads), C::kSmem,
                          st, qm, km, vm, a));
  return BCG_OK;
}

// The instance for padded head sizes qd (64 .. 256) and vd (64, 128, 256).
template <bool PAGED, bool SLOPES>
static int window_attn(int qd, int vd, const CUtensorMap& qm, const CUtensorMap& km, const CUtensorMap& vm,
                       const WindowAttn& a, cudaStream_t st) {
#define BCG_WA(Q, V) \
  if (qd == Q && vd == V) return launch_window_attn<Q, V, PAGED, SLOPES>(qm, km, vm, a, st)
  BCG_WA(64, 64);
  BCG_WA(64, 128);
  BCG_WA(64, 256);
  BCG_WA(128, 64);
  BCG_WA(128, 128);
  BCG_WA(128, 256);
  BCG_WA(192, 64);
  BCG_WA(192, 128);
  BCG_WA(192, 256);
  BCG_WA(256, 64);
  BCG_WA(256, 128);
  BCG_WA(256, 256);
#undef BCG_WA
  set_last_error("bcg window attention", "no kernel for this head size");
  return BCG_ERR_UNSUPPORTED;
}

}  // namespace bcg
