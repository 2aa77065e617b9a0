// Linear recurrences with scalar decays per head, chunks of 64 tokens on tensor cores:
//     S <- keep S + x b^T,   y = S c,   weights in front of x, b and c as a RULE says.
// Inside a chunk the recurrence is a product, y_i = e_i S c_i + sum_{j <= i} weight_ij (b_j . c_i) x_j, and the state moves once per
// chunk, S <- keep S + sum_j w_j x_j b_j^T.  Everything is held transposed (rows = entries of a head's output), so that the state
// stays in fp32 accumulators and becomes an operand without leaving the registers.  What is added to the state enters its product
// as two bf16 halves (hi + lo); what is only read out is rounded like any activation.
//
// RULE: Args (x, x_ld(), in_col / out_col / row_col(head): columns of b, c and x, entries(), state_of(slot, head), y, inner(), ...);
// scalars of a chunk in shared memory, the last 64 of them w (scalars(), by one warp, from what request() asked for); weights(),
// readout() and keep() of them; skip(): factor of x in y; finish() behind the last chunk.  kNormalized: a normalizer follows the
// state's rows, n <- keep n + sum_j w_j b_j, the CTAs of a head's first block carry it and hand n . c to denominator().
#pragma once
#include <type_traits>

#include "state_rows.cuh"

namespace bcg {

constexpr int kChTok = 64, kChWarps = 4, kChThreads = kChWarps * 32;

// Tiles in shared memory are rows of 16-byte pieces, piece p of row r at place p ^ (r & 7).  B and x are there for two chunks.
template <int NP, class RULE>
struct ChCfg {
  static constexpr int kBC = kChTok * NP * 2, kX = kChTok * kSsRows * 2, kM = kChTok * kChTok * 2;     // bytes
  static constexpr int kOffC = 2 * kBC, kOffX = kOffC + kBC, kOffM = kOffX + 2 * kX, kOffS = kOffM + kM;
  static constexpr int kOffN = kOffS + 2 * RULE::kScalars * 4;                                         // normalizer as hi | lo
  static constexpr int kSmem = kOffN + (RULE::kNormalized ? 2 * NP * 2 : 0) + 128;
  static constexpr int kCtasPerSm = NP <= 128 ? 3 : 2;
};

// matrix loads from shared-memory addresses: offsets that are constants cost no instruction
__device__ __forceinline__ void ldsm_at(uint32_t (&r)[4], uint32_t p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(p));
}
__device__ __forceinline__ void ldsm_trans_at(uint32_t (&r)[4], uint32_t p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(p));
}
// hi + lo = v to about 2^-17
__device__ __forceinline__ void split_bf16(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16(a, b);
  lo = pack_bf16(a - bf16lo(hi), b - bf16hi(hi));
}
__device__ __forceinline__ void scale2(float& a, float& b, float fa, float fb) {
  unpack_f32x2(mul_f32x2(pack_f32x2(__float_as_uint(a), __float_as_uint(b)), pack_f32x2(__float_as_uint(fa), __float_as_uint(fb))), a, b);
}
__device__ __forceinline__ uint32_t transpose_8x8(uint32_t v) {
  uint32_t r;
  asm volatile("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;" : "=r"(r) : "r"(v));
  return r;
}

// M[i][j] = weight_ij (C_i . B_j) for j <= i, tokens i = 16 RT .. 16 RT + 15.  sB, sC, sM, sN: addresses.  normalizer: also the
// denominators of these tokens, from the sums of M's rows and the normalizer at the chunk's start.
template <int NP, int RT, class RULE>
__device__ __forceinline__ void chunk_matrix(const RULE& rule, uint32_t sB, uint32_t sC, const float* sc, uint32_t sM, uint32_t sN,
                                             bool normalizer, int first) {
  const int lane = threadIdx.x & 31, q2 = (lane & 3) * 2;
  float acc[2 * RT + 2][4] = {}, nq[4] = {};
  const uint32_t pc = sC + (RT * 16 + (lane & 15)) * NP * 2, xc = ((lane >> 4) ^ (lane & 7)) << 4;
  const uint32_t pb = sB + ((lane & 7) + ((lane >> 4) << 3)) * NP * 2, xb = (((lane >> 3) & 1) ^ (lane & 7)) << 4;
#pragma unroll
  for (int k = 0; k < NP / 16; ++k) {
    uint32_t ca[4];
    ldsm_at(ca, pc + (xc ^ (k << 5)));
    const uint32_t at = pb + (xb ^ (k << 5));
    if constexpr (RULE::kNormalized) {
      if (normalizer) {         // even columns: the high halves, odd ones: the low halves
        uint32_t nb[4];
        ldsm_at(nb, sN + (lane & 1) * NP * 2 + k * 32 + ((lane >> 3) & 1) * 16);
        mma_bf16_16816(nq, ca, nb[0], nb[1]);
      }
    }
#pragma unroll
    for (int jp = 0; jp <= RT; ++jp) {
      uint32_t bb[4];
      ldsm_at(bb, at + jp * 16 * NP * 2);
      mma_bf16_16816(acc[2 * jp], ca, bb[0], bb[1]);
      mma_bf16_16816(acc[2 * jp + 1], ca, bb[2], bb[3]);
    }
  }
  const int i0 = RT * 16 + (lane >> 2);
  const float ci[2] = {sc[i0], sc[i0 + 8]};
  float sum[2] = {0.f, 0.f};
#pragma unroll
  for (int jt = 0; jt < 2 * RT + 2; ++jt) {
    const int j = jt * 8 + q2;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int i = i0 + e * 8;
      const float2 w = rule.weights(sc, ci[e], j);
      float m0 = acc[jt][2 * e] * w.x;
      float m1 = acc[jt][2 * e + 1] * w.y;
      if (jt >= 2 * RT) {                       // the diagonal block
        if (j > i) m0 = 0.f;
        if (j + 1 > i) m1 = 0.f;
      }
      if constexpr (RULE::kNormalized) sum[e] += m0 + m1;
      asm volatile("st.shared.b32 [%0], %1;" ::"r"(sM + i * kChTok * 2 + ((jt ^ (lane >> 2)) << 4) + q2 * 2), "r"(pack_bf16(m0, m1))
                   : "memory");
    }
  }
  if constexpr (RULE::kNormalized) {
    if (normalizer) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        sum[e] += __shfl_xor_sync(0xffffffffu, sum[e], 1);
        sum[e] += __shfl_xor_sync(0xffffffffu, sum[e], 2);
        if ((lane & 3) == 0) rule.denominator(sc, i0 + e * 8, first, sum[e], nq[2 * e] + nq[2 * e + 1]);
      }
    }
  }
}

// grid (heads, blocks of 64 head entries, sequences); warp w has entries 16 w .. 16 w + 15 of the block.
template <int NP, class RULE>
__global__ void __launch_bounds__(kChThreads, ChCfg<NP, RULE>::kCtasPerSm)
chunk_kernel(const typename RULE::Args a) {
  using C = ChCfg<NP, RULE>;
  extern __shared__ __align__(128) uint8_t ch_raw[];
  const uint32_t base = (smem_u32(ch_raw) + 127u) & ~127u;
  float* scalars = reinterpret_cast<float*>(ch_raw + (base - smem_u32(ch_raw)) + C::kOffS);     // [2][kScalars]
  const uint32_t sC = base + C::kOffC, sM = base + C::kOffM, sN = base + C::kOffN;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.x, p0 = blockIdx.y * kSsRows, sq = blockIdx.z;
  const int rows = min(kSsRows, a.vdim - p0), N = a.entries(), inner = a.inner();
  const bool normalizer = RULE::kNormalized && blockIdx.y == 0;
  pdl_launch_dependents();
  pdl_wait();
  const int t0 = a.first_of(sq), t1 = a.end_of(sq);
  if (t1 <= t0 || a.slot_map[t0] < 0) return;
  const __nv_bfloat16* xbc = static_cast<const __nv_bfloat16*>(a.x);
  const int x_ld = a.x_ld(), b_col = a.in_col(h), c_col = a.out_col(h), x_col = a.row_col(h) + p0;

  // 64 tokens from `first` on, up to 8 `units` columns from `col` on, `valid` of them; the rest and tokens past the end are
  // zero
  auto copy_rows = [&](auto units, uint32_t dst, int col, int valid, int first) {
    constexpr int kUnits = decltype(units)::value, kPass = kChThreads / kUnits;
    const int u = threadIdx.x % kUnits, r = threadIdx.x / kUnits, wide = max(0, min(16, (valid - u * 8) * 2));
    const __nv_bfloat16* src = xbc + static_cast<long long>(first + r) * x_ld + col + u * 8;
#pragma unroll
    for (int i = 0; i < kChTok / kPass; ++i) {
      const int row = r + i * kPass, bytes = first + row < t1 ? wide : 0;
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst + row * kUnits * 16 + ((u ^ (row & 7)) << 4)),
                   "l"(bytes ? src : xbc), "r"(bytes)
                   : "memory");
      src += static_cast<long long>(kPass) * x_ld;
    }
  };
  using BCUnits = std::integral_constant<int, NP / 8>;
  using XUnits = std::integral_constant<int, kSsRows / 8>;

  const int n_chunks = (t1 - t0 + kChTok - 1) / kChTok;
  const int pr = warp * 16 + (lane >> 2);       // this lane's rows of the state: pr, pr + 8; entries nt * 8 + 2 (lane & 3) ..
  const int q2 = (lane & 3) * 2;
  float* head = a.state_of(a.state_slots[sq], h);
  float* st = head + static_cast<long long>(p0) * N;
  copy_rows(BCUnits{}, base, b_col, N, t0);
  copy_rows(BCUnits{}, sC, c_col, N, t0);
  copy_rows(XUnits{}, base + C::kOffX, x_col, rows, t0);
  cp_async_commit();
  float S[NP / 8][4];
  const bool fresh = a.positions[t0] == 0;
#pragma unroll
  for (int nt = 0; nt < NP / 8; ++nt)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int p = pr + (i >> 1) * 8, n = nt * 8 + q2 + (i & 1);
      S[nt][i] = !fresh && p < rows && n < N ? st[static_cast<long long>(p) * N + n] : 0.f;
    }
  // warp 0: the scalars of chunk c, then what those of the chunk behind it are made of
  RULE rule(a, h, t0, t1, static_cast<int>(blockIdx.y), fresh);
  const float skip = rule.skip();
  auto scalars_of = [&](int c) {
    rule.scalars(scalars + (c & 1) * RULE::kScalars, c, lane);
    rule.request(c + 1, lane);
  };
  if (warp == 0) {
    rule.request(0, lane);
    scalars_of(0);
  }
  // normalizer: a thread has entries e0 .. of it, and writes them as two halves for the products
  constexpr int kPer = NP / kChThreads > 0 ? NP / kChThreads : 1;
  const int e0 = static_cast<int>(threadIdx.x) * kPer;
  float norm[kPer];
  auto halves = [&]() {
#pragma unroll
    for (int i = 0; i < kPer; ++i) {
      const __nv_bfloat16 hi = __float2bfloat16(norm[i]), lo = __float2bfloat16(norm[i] - __bfloat162float(hi));
      const uint32_t at = sN + (e0 + i) * 2;
      asm volatile("st.shared.u16 [%0], %1;" ::"r"(at), "h"(__bfloat16_as_ushort(hi)) : "memory");
      asm volatile("st.shared.u16 [%0], %1;" ::"r"(at + NP * 2), "h"(__bfloat16_as_ushort(lo)) : "memory");
    }
  };
  if constexpr (RULE::kNormalized) {
    if (normalizer && e0 < NP) {
#pragma unroll
      for (int i = 0; i < kPer; ++i) norm[i] = !fresh && e0 + i < N ? head[static_cast<long long>(a.vdim) * N + e0 + i] : 0.f;
      halves();
    }
  }

  for (int c = 0; c < n_chunks; ++c) {
    const int first = t0 + c * kChTok, nt_tok = min(kChTok, t1 - first);
    const float* sc = scalars + (c & 1) * RULE::kScalars;
    const float* w_s = sc + 3 * kChTok;
    cp_async_wait<0>();
    __syncthreads();                            // the chunk is there, everybody is done with the previous one
    const uint32_t sB = base + (c & 1) * C::kBC, sX = base + C::kOffX + (c & 1) * C::kX;
    if (c + 1 < n_chunks) {
      copy_rows(BCUnits{}, base + ((c + 1) & 1) * C::kBC, b_col, N, first + kChTok);
      copy_rows(XUnits{}, base + C::kOffX + ((c + 1) & 1) * C::kX, x_col, rows, first + kChTok);
    }

    if (warp * 16 < nt_tok) {
      if (warp == 0) chunk_matrix<NP, 0>(rule, sB, sC, sc, sM, sN, normalizer, first);
      else if (warp == 1) chunk_matrix<NP, 1>(rule, sB, sC, sc, sM, sN, normalizer, first);
      else if (warp == 2) chunk_matrix<NP, 2>(rule, sB, sC, sc, sM, sN, normalizer, first);
      else chunk_matrix<NP, 3>(rule, sB, sC, sc, sM, sN, normalizer, first);
    }
    if (warp == 0) scalars_of(c + 1);           // the warp with the smallest share of M

    // ---- Y^T = S^T C^T, columns (tokens) scaled by exp(c_i)
    float Y[kChTok / 8][4] = {};
    const uint32_t r8 = (lane & 7) + ((lane >> 4) << 3), x8 = (((lane >> 3) & 1) ^ (lane & 7)) << 4;
    const uint32_t pc = sC + r8 * NP * 2;
#pragma unroll
    for (int k = 0; k < NP / 16; ++k) {
      const uint32_t sa[4] = {pack_bf16(S[2 * k][0], S[2 * k][1]), pack_bf16(S[2 * k][2], S[2 * k][3]),
                              pack_bf16(S[2 * k + 1][0], S[2 * k + 1][1]), pack_bf16(S[2 * k + 1][2], S[2 * k + 1][3])};
#pragma unroll
      for (int ip = 0; ip < kChTok / 16; ++ip) {
        uint32_t cb[4];
        ldsm_at(cb, pc + (x8 ^ (k << 5)) + ip * 16 * NP * 2);
        mma_bf16_16816(Y[2 * ip], sa, cb[0], cb[1]);
        mma_bf16_16816(Y[2 * ip + 1], sa, cb[2], cb[3]);
      }
    }
#pragma unroll
    for (int it = 0; it < kChTok / 8; ++it) {
      const float2 e = rule.readout(sc, it * 8 + q2);
      scale2(Y[it][0], Y[it][1], e.x, e.y);
      scale2(Y[it][2], Y[it][3], e.x, e.y);
    }
    const float keep = rule.keep(sc);
#pragma unroll
    for (int nt = 0; nt < NP / 8; ++nt) {
      scale2(S[nt][0], S[nt][1], keep, keep);
      scale2(S[nt][2], S[nt][3], keep, keep);
    }
    __syncthreads();                            // M is complete, C has been read
    if (c + 1 < n_chunks) copy_rows(BCUnits{}, sC, c_col, N, first + kChTok);
    cp_async_commit();
    if constexpr (RULE::kNormalized) {
      if (normalizer && e0 < NP) {
        float add[kPer] = {};
#pragma unroll 8
        for (int j = 0; j < kChTok; ++j) {
          const uint32_t at = sB + j * NP * 2 + (((e0 >> 3) ^ (j & 7)) << 4) + (e0 & 7) * 2;
          const float w = w_s[j];
          if constexpr (kPer == 2) {
            uint32_t v;
            asm volatile("ld.shared.u32 %0, [%1];" : "=r"(v) : "r"(at));
            add[0] = fmaf(w, bf16lo(v), add[0]);
            add[1] = fmaf(w, bf16hi(v), add[1]);
          } else {
            unsigned short v;
            asm volatile("ld.shared.u16 %0, [%1];" : "=h"(v) : "r"(at));
            add[0] = fmaf(w, __bfloat162float(__ushort_as_bfloat16(v)), add[0]);
          }
        }
#pragma unroll
        for (int i = 0; i < kPer; ++i) norm[i] = fmaf(keep, norm[i], add[i]);
        halves();
      }
    }

    // ---- Y^T += x^T M^T + skip x^T;   S^T += (w x)^T B
    const uint32_t px = sX + r8 * kSsRows * 2 + (x8 ^ (warp << 5));
    const uint32_t pb = sB + (lane & 15) * NP * 2, xb = ((lane >> 4) ^ (lane & 7)) << 4;
    const uint32_t pm = sM + r8 * kChTok * 2;
#pragma unroll
    for (int jp = 0; jp < kChTok / 16; ++jp) {
      uint32_t xa[4];
      ldsm_trans_at(xa, px + jp * 16 * kSsRows * 2);
#pragma unroll
      for (int ip = jp; ip < kChTok / 16; ++ip)
        if (ip * 16 < nt_tok) {
          uint32_t mb[4];
          ldsm_at(mb, pm + (x8 ^ (jp << 5)) + ip * 16 * kChTok * 2);
          mma_bf16_16816(Y[2 * ip], xa, mb[0], mb[1]);
          mma_bf16_16816(Y[2 * ip + 1], xa, mb[2], mb[3]);
        }
      float xf[4][2];                           // rows pr, pr + 8 of tokens j, j + 1; the same of tokens j + 8, j + 9
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        xf[i][0] = bf16lo(xa[i]);
        xf[i][1] = bf16hi(xa[i]);
      }
      if constexpr (!RULE::kNormalized) {
#pragma unroll
        for (int e = 0; e < 2; ++e)
#pragma unroll
          for (int k = 0; k < 2; ++k) {
            Y[2 * jp + e][k] = fmaf(skip, xf[2 * e][k], Y[2 * jp + e][k]);
            Y[2 * jp + e][2 + k] = fmaf(skip, xf[2 * e + 1][k], Y[2 * jp + e][2 + k]);
          }
      }
      const float2 w0 = *reinterpret_cast<const float2*>(w_s + jp * 16 + q2), w1 = *reinterpret_cast<const float2*>(w_s + jp * 16 + 8 + q2);
      uint32_t hi[4], lo[4];
      split_bf16(w0.x * xf[0][0], w0.y * xf[0][1], hi[0], lo[0]);
      split_bf16(w0.x * xf[1][0], w0.y * xf[1][1], hi[1], lo[1]);
      split_bf16(w1.x * xf[2][0], w1.y * xf[2][1], hi[2], lo[2]);
      split_bf16(w1.x * xf[3][0], w1.y * xf[3][1], hi[3], lo[3]);
#pragma unroll
      for (int np = 0; np < NP / 16; np += 2) {
        uint32_t b0[4], b1[4];
        ldsm_trans_at(b0, pb + (xb ^ (np << 5)) + jp * 16 * NP * 2);
        ldsm_trans_at(b1, pb + (xb ^ ((np + 1) << 5)) + jp * 16 * NP * 2);
        mma_bf16_16816(S[2 * np], hi, b0[0], b0[1]);
        mma_bf16_16816(S[2 * np + 1], hi, b0[2], b0[3]);
        mma_bf16_16816(S[2 * np + 2], hi, b1[0], b1[1]);
        mma_bf16_16816(S[2 * np + 3], hi, b1[2], b1[3]);
        mma_bf16_16816(S[2 * np], lo, b0[0], b0[1]);
        mma_bf16_16816(S[2 * np + 1], lo, b0[2], b0[3]);
        mma_bf16_16816(S[2 * np + 2], lo, b1[0], b1[1]);
        mma_bf16_16816(S[2 * np + 3], lo, b1[2], b1[3]);
      }
    }

    // ---- store: pairs are transposed on the way out (token lane >> 2, entries q2, q2 + 1)
    __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.y) + static_cast<long long>(first + (lane >> 2)) * inner + h * a.vdim + p0 +
                         warp * 16 + q2;
    const bool whole = nt_tok == kChTok && warp * 16 + 16 <= rows && (a.vdim & 1) == 0;
#pragma unroll
    for (int it = 0; it < kChTok / 8; ++it) {
      if (it * 8 >= nt_tok) break;
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const uint32_t v = transpose_8x8(pack_bf16(Y[it][2 * e], Y[it][2 * e + 1]));
        __nv_bfloat16* dst = out + e * 8;
        const int p = warp * 16 + e * 8 + q2;
        if (whole) {
          *reinterpret_cast<uint32_t*>(dst) = v;
        } else if (it * 8 + (lane >> 2) < nt_tok) {
          if (p < rows) dst[0] = __ushort_as_bfloat16(static_cast<unsigned short>(v & 0xffffu));
          if (p + 1 < rows) dst[1] = __ushort_as_bfloat16(static_cast<unsigned short>(v >> 16));
        }
        __syncwarp();
      }
      out += 8ll * inner;
    }
  }
#pragma unroll
  for (int nt = 0; nt < NP / 8; ++nt)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int p = pr + (i >> 1) * 8, n = nt * 8 + q2 + (i & 1);
      if (p < rows && n < N) st[static_cast<long long>(p) * N + n] = S[nt][i];
    }
  if constexpr (RULE::kNormalized) {
    if (normalizer && e0 < NP) {
#pragma unroll
      for (int i = 0; i < kPer; ++i)
        if (e0 + i < N) head[static_cast<long long>(a.vdim) * N + e0 + i] = norm[i];
    }
  }
  rule.finish(sq, p0, rows, fresh);
}

template <int NP, class RULE>
static int launch_chunks(const typename RULE::Args& a, dim3 grid, cudaStream_t st) {
  constexpr int kSmem = ChCfg<NP, RULE>::kSmem;
  BCG_TRY(ensure_dynamic_smem(reinterpret_cast<const void*>(chunk_kernel<NP, RULE>), kSmem));
  BCG_CUDA_CHECK(launch_k(chunk_kernel<NP, RULE>, grid, dim3(kChThreads), kSmem, st, a));
  return BCG_OK;
}


}  // namespace bcg
