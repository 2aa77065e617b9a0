// Prompt attention of latent layers in expanded form: the step's cache rows (gathered, history inside the
// window included) are multiplied once into every head's keys and values, and a tcgen05 flash kernel runs
// over them with a causal sliding window and a softmax sink.
//
// The expanded row of head h is  K: [W_uk c | k_rot | 0] (QD columns),  V: [W_uv c | 0] (VD columns): the
// expansion matrix holds the identity on the rotated part, so one GEMM over cache rows produces keys with
// the shared rotated part already in place (exactly: bf16 times one).
//
//   grid (heads, tiles), 192 threads.  One CTA = 128 query rows of one head, keys in blocks of 64 from the
//   first one any row of the tile sees.
//     warp 0      TMA producer: Q tile once, then K and V blocks (64 x 64 boxes, 128B swizzle)
//     warp 1      MMA issuer: S_j = Q K_j^T into one of two TMEM accumulators; O += P_j V_j in TMEM
//     warps 2-5   softmax, thread = query row = TMEM lane; the running maximum starts at the sink with
//                 denominator 1 (exp(sink - sink)), which is the sink's whole effect; rescaling of O is
//                 lazy (only when a block's maximum exceeds the running one by more than 8 in log2 units)
#include "attn_tcgen05.cuh"
#include "stack_common.cuh"
#include "kernels.h"

namespace bcg {

constexpr int kLpBM = 128, kLpBN = 64, kLpThreads = 192;
constexpr int kLpQHalf = kLpBM * 64 * 2;     // [128 rows][64 bf16]
constexpr int kLpKvHalf = kLpBN * 64 * 2;    // [64 keys][64 bf16]
constexpr float kLpRescaleGap = 8.0f;
constexpr float kLpNoSink = -1e30f;          // finite "minus infinity" for the running maximum

template <int QD, int VD>
struct LpCfg {
  static constexpr int kQ = QD / 64 * kLpQHalf, kK = QD / 64 * kLpKvHalf, kV = VD / 64 * kLpKvHalf, kP = kLpQHalf;
  static constexpr int kFixed = kQ + kP + 256 + 768;
  // two CTAs per SM (one hides the other's bubbles) where one-stage rings make that fit, else two stages
  static constexpr int kStages = (kFixed + 2 * (kK + kV) > 113 * 1024 && kFixed + kK + kV <= 113 * 1024) ? 1 : 2;
  static constexpr int kOffK = kQ, kOffV = kOffK + kStages * kK, kOffP = kOffV + kStages * kV, kOffBar = kOffP + kP;
  static constexpr int kSlack = 768;
  static constexpr int kSmem = kOffBar + 256 + kSlack;
  static constexpr uint32_t kTmemCols = 2 * kLpBN + VD <= 256 ? 256 : 512;
  static constexpr int kCtasPerSm = (kSmem <= 113 * 1024 && kTmemCols == 256) ? 2 : 1;
};

template <int QD, int VD>
__global__ void __launch_bounds__(kLpThreads, LpCfg<QD, VD>::kCtasPerSm)
latent_prefill_kernel(const __grid_constant__ CUtensorMap q_map, const __grid_constant__ CUtensorMap kv_map,
                      const int* __restrict__ tiles, int n_tiles, const float* __restrict__ sink,
                      __nv_bfloat16* __restrict__ out, int n_heads, int vdim, int window, float scale_log2e) {
  using C = LpCfg<QD, VD>;
  constexpr int ST = C::kStages;
  constexpr uint32_t kIdescQK = make_idesc_bf16_m128(kLpBN);
  constexpr uint32_t kIdescPV = make_idesc_bf16_m128(VD) | (1u << 16);   // B (values) is MN-major
  extern __shared__ __align__(1024) uint8_t lp_raw[];
  const uint32_t pad = (1024u - (smem_u32(lp_raw) & 1023u)) & 1023u;
  if (pad > static_cast<uint32_t>(C::kSlack)) __trap();
  uint8_t* smem = lp_raw + pad;
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
  const int* ti = tiles + (n_tiles - 1 - static_cast<int>(blockIdx.y)) * 8;
  if (threadIdx.x == 0) {
    tma_prefetch_desc(&q_map);
    tma_prefetch_desc(&kv_map);
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
  const int kb = max(window > 0 ? pos0 - window + 1 : 0, ti[4]);   // first key of block 0 (ti[4] <= it, or 0)
  const int kv_row = ti[3] + kb - ti[4];
  const int nb = (pos0 + n_rows - kb + kLpBN - 1) / kLpBN;
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t tmem_o = tmem_base + 2 * kLpBN;

  if (warp == 0) {
    if (lane == 0) {
      mbar_arrive_expect_tx(q_full, C::kQ);
#pragma unroll
      for (int c = 0; c < QD / 64; ++c)
        tma_load_2d(smem + c * kLpQHalf, &q_map, q_full, head * QD + c * 64, row0, kEvictFirst);
      for (int j = 0; j < nb; ++j) {
        const int st = j % ST;
        const uint32_t par = (j / ST) & 1;
        uint8_t* dk = smem + C::kOffK + st * C::kK;
        mbar_wait(&k_empty[st], par ^ 1);
        mbar_arrive_expect_tx(&k_full[st], C::kK);
#pragma unroll
        for (int c = 0; c < QD / 64; ++c)
          tma_load_2d(dk + c * kLpKvHalf, &kv_map, &k_full[st], head * QD + c * 64, kv_row + j * kLpBN, kEvictNormal);
        uint8_t* dv = smem + C::kOffV + st * C::kV;
        mbar_wait(&v_empty[st], par ^ 1);
        mbar_arrive_expect_tx(&v_full[st], C::kV);
#pragma unroll
        for (int c = 0; c < VD / 64; ++c)
          tma_load_2d(dv + c * kLpKvHalf, &kv_map, &v_full[st], n_heads * QD + head * VD + c * 64,
                      kv_row + j * kLpBN, kEvictNormal);
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
        const uint32_t d = tmem_base + static_cast<uint32_t>((j & 1) * kLpBN);
#pragma unroll
        for (int ks = 0; ks < QD / 16; ++ks)
          umma_bf16(d, make_kmajor_sw128_desc(sq + (ks >> 2) * kLpQHalf + (ks & 3) * 32),
                    make_kmajor_sw128_desc(sk + (ks >> 2) * kLpKvHalf + (ks & 3) * 32), kIdescQK, ks > 0 ? 1u : 0u);
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
        for (int kk = 0; kk < kLpBN / 16; ++kk)
          umma_bf16(tmem_o, make_kmajor_sw128_desc(sp + kk * 32), make_mnmajor_sw128_desc(sv + kk * 16 * 128, kLpKvHalf),
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
    const int limit = pos0 + r - kb;                                   // last visible key, counted from kb
    const int low = window > 0 ? max(0, pos0 + r - window + 1 - kb) : 0;   // first visible key
    uint8_t* p_row = smem + C::kOffP + r * 128;
    const int sw = r & 7;
    float m_run = sink ? sink[head] * 1.4426950408889634f : kLpNoSink;
    float l_run = sink ? 1.0f : 0.0f;
    for (int j = 0; j < nb; ++j) {
      const int col0 = j * kLpBN;
      const bool need_mask = col0 + kLpBN - 1 > limit || col0 < low;
      mbar_wait(&s_full[j & 1], (j >> 1) & 1);
      tc_fence_after();
      uint32_t s[kLpBN];
#pragma unroll
      for (int c = 0; c < kLpBN / 32; ++c)
        tmem_ld_x32(tmem_base + lane_addr + (j & 1) * kLpBN + c * 32, s + c * 32);
      tmem_ld_wait();
      tc_fence_before();
      mbar_arrive(&s_free[j & 1]);
      float mx = -INFINITY;
      if (need_mask) {
#pragma unroll
        for (int i = 0; i < kLpBN; ++i) {
          if (col0 + i > limit || col0 + i < low) s[i] = 0xff800000u;   // -inf
          mx = fmaxf(mx, __uint_as_float(s[i]));
        }
      } else {
#pragma unroll
        for (int i = 0; i < kLpBN; ++i) mx = fmaxf(mx, __uint_as_float(s[i]));
      }
      const float m_blk = mx * scale_log2e;
      const bool grow = m_blk > m_run + kLpRescaleGap;
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
      const uint64_t scale2 = pack_f32x2(__float_as_uint(scale_log2e), __float_as_uint(scale_log2e));
      const uint64_t negm2 = pack_f32x2(__float_as_uint(-m_run), __float_as_uint(-m_run));
      uint64_t l2 = pack_f32x2(0u, 0u);
#pragma unroll
      for (int c = 0; c < kLpBN / 8; ++c) {
        uint32_t pk[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          float x0, x1;
          unpack_f32x2(fma_f32x2(pack_f32x2(s[c * 8 + 2 * i], s[c * 8 + 2 * i + 1]), scale2, negm2), x0, x1);
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
    const float inv = l_run > 0.f ? 1.0f / l_run : 0.f;
    __nv_bfloat16* dst = out + ((static_cast<long long>(row0) + r) * n_heads + head) * vdim;
#pragma unroll
    for (int c = 0; c < VD / 32; ++c) {
      uint32_t o[32];
      tmem_ld_x32(tmem_o + lane_addr + c * 32, o);
      tmem_ld_wait();
      if (r < n_rows) {
#pragma unroll
        for (int g = 0; g < 4; ++g)
          if (c * 32 + g * 8 < vdim) {
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

template <int QD, int VD>
static int launch_prefill(const CUtensorMap& qm, const CUtensorMap& km, const bcg_layer* l, const int* tiles,
                          int n_tiles, void* out, cudaStream_t st) {
  using C = LpCfg<QD, VD>;
  BCG_TRY(ensure_dynamic_smem(reinterpret_cast<const void*>(latent_prefill_kernel<QD, VD>), C::kSmem));
  BCG_CUDA_CHECK(launch_k(latent_prefill_kernel<QD, VD>, dim3(l->heads, n_tiles), dim3(kLpThreads), C::kSmem, st, qm, km,
                          tiles, n_tiles, l->sink, static_cast<__nv_bfloat16*>(out), l->heads, l->vdim, l->window,
                          l->scale * 1.4426950408889634f));
  return BCG_OK;
}

bool latent_prefill_ok(const bcg_layer* l) {
  return l->w_expand && (l->kv_rank + l->rot_dim) % 8 == 0 && l->vdim % 8 == 0 && l->q_ld % 64 == 0 && l->q_ld <= 256 &&
         l->dim + l->rot_dim <= l->q_ld && (l->v_ld == 64 || l->v_ld == 128 || l->v_ld == 256) && l->vdim <= l->v_ld &&
         l->q_ld > 0 && l->scale > 0.f;
}

// latents: gathered cache rows [n_gather, kv_rank + rot_dim]; tiles as in bcg_step_batch.
int latent_prefill(const bcg_layer* l, const bcg_stack_ws* ws, const bcg_step_batch* b, cudaStream_t st) {
  const int crow = l->kv_rank + l->rot_dim, n_exp = l->heads * (l->q_ld + l->v_ld);
  BCG_TRY(gemm_bf16_tn(ws->latents, l->w_expand, ws->expanded, b->n_gather, n_exp, crow, crow, crow, n_exp,
                       BCG_EPI_BF16, 1, 0, st));
  CUtensorMap qm, km;
  BCG_TRY(make_tmap_bf16_sw128(&qm, ws->q, b->T, static_cast<long long>(l->heads) * l->q_ld,
                               static_cast<long long>(l->heads) * l->q_ld, kLpBM));
  BCG_TRY(make_tmap_bf16_sw128(&km, ws->expanded, b->n_gather, n_exp, n_exp, kLpBN));
#define BCG_LP(Q, V) \
  if (l->q_ld == Q && l->v_ld == V) return launch_prefill<Q, V>(qm, km, l, b->tiles, b->n_tiles, ws->mix, st)
  BCG_LP(64, 64);
  BCG_LP(64, 128);
  BCG_LP(64, 256);
  BCG_LP(128, 64);
  BCG_LP(128, 128);
  BCG_LP(128, 256);
  BCG_LP(192, 64);
  BCG_LP(192, 128);
  BCG_LP(192, 256);
  BCG_LP(256, 64);
  BCG_LP(256, 128);
  BCG_LP(256, 256);
#undef BCG_LP
  set_last_error("bcg_latent_attention", "no expanded kernel for this head size");
  return BCG_ERR_UNSUPPORTED;
}

}  // namespace bcg
