// Grouped-query attention over paged keys and values, with what a layer has of: a linear distance bias, a sliding
// window, a query temperature, query and key norms over all heads at once or head by head, rotated queries, keys and
// values, means of blocks of tokens in front of the window, an output gate per head.
//
// A layer's cache is two pools of 16-token pages, keys [page][kv head][16][q_ld] and values [page][kv head][16][v_ld];
// heads are padded to q_ld / v_ld columns, the padding is zero and stays so.
//   grouped_in      projection slabs -> queries (bias, temperature), keys and values (bias, value mixing) into the
//                   pages, squared-relu activations of a parallel feed-forward, routing of a parallel mixture;
//                   where there are norms or gates, a CTA or a cluster has a whole token (grouped_norm_in); where
//                   heads are normed or rotated one by one, a warp has a head (head_in)
//   pool_blocks     means of the blocks of tokens that a ragged step completes, into their own pages (single tokens:
//                   head_in makes them)
//   grouped_plain   one CTA per (token, head), any sizes, fp32 or bf16: the fp32 engine's kernel, and the bf16
//                   one's for head sizes the kernels below do not take
//   grouped_decode  single tokens: a cluster per (token, kv head) shares the key pages, a ring of TMA loads and a
//                   running softmax per warp, partial results merged through distributed shared memory
//   prompts run on the tcgen05 window attention kernel (attn_window.cuh), reading pages directly
#include "attn_window.cuh"
#include "mma_sync.cuh"
#include "moe.cuh"

namespace bcg {

constexpr float kLog2e = 1.4426950408889634f;

// ------------------------------------------------------------------------------------------- inputs
constexpr int kInThreads = 256;

struct GroupedIn {
  const float* proj;          // [n_partials][T][ld]
  int n_partials;
  long long pstride, ld;
  const int *positions, *slot_map;
  const float* bias;          // [q + k + v columns]
  void *q, *k_cache, *v_cache, *act;
  float* v_first;             // [T][kv_heads * vdim]
  int heads, kv_heads, dim, vdim, q_ld, v_ld, page_size;
  float temp_coef, temp_every;
  int v_role;
  float v_mix;
  int ff, act_from;           // squared-relu columns of proj (ff = 0: none)
  long long act_ld;
  int n_tokens, blocks;       // blocks: CTAs per token that share the columns
  MoeRoute route;             // experts = 0: none
  int route_tokens;           // tokens per routing CTA
  const float *q_norm, *k_norm;   // [heads * dim], [kv_heads * dim] or NULL
  float* gates;               // [T][heads] or NULL; logits are columns gate_col.. of proj
  int gate_col;
  float gate_scale, eps;
  // heads one by one (head_in): q_norm and k_norm are [dim]
  const float *cos_sin, *v_cos_sin;   // [positions][dims]: cosines of the dims / 2 angles, then sines
  int rot_dims, rot_pairs, v_rot_dims;
  int pool, pool_col;         // pool > 0: single tokens that complete a block write its means
  const int* block_table;
  int max_blocks;
};

// Where a token's columns go.
struct InToken {
  long long t, page;
  int slot, in_page;
  float temp;
  __device__ __forceinline__ InToken(const GroupedIn& a, long long t_) : t(t_) {
    const int pos = a.positions[t];
    slot = a.slot_map[t];
    temp = 1.0f + a.temp_coef * logf(floorf(static_cast<float>(pos + 1) / a.temp_every) + 1.0f);
    page = slot >= 0 ? slot / a.page_size : 0;
    in_page = slot >= 0 ? slot % a.page_size : 0;
  }
};

// Biased (and normed) columns c.. of q | k | v to the query buffer or the token's place in the pages.
template <typename T, int V>
__device__ __forceinline__ void store_columns(const GroupedIn& a, const InToken& tok, int c, Vec<V>& x) {
  const int nq = a.heads * a.dim, nk = nq + a.kv_heads * a.dim;
  const long long t = tok.t;
  if (c < nq) {
    const int h = c / a.dim, i = c - h * a.dim;
#pragma unroll
    for (int k = 0; k < V; ++k) x.x[k] *= tok.temp;
    store_vec<V>(static_cast<T*>(a.q) + (t * a.heads + h) * a.q_ld + i, x);
  } else if (c < nk) {
    const int g = (c - nq) / a.dim, i = c - nq - g * a.dim;
    if (tok.slot >= 0)
      store_vec<V>(static_cast<T*>(a.k_cache) + ((tok.page * a.kv_heads + g) * a.page_size + tok.in_page) * a.q_ld + i, x);
  } else {
    const int o = c - nk, g = o / a.vdim, i = o - g * a.vdim;
    float* first = a.v_first + t * (a.kv_heads * a.vdim) + o;
    if (a.v_role == BCG_VALUES_FIRST) {
      store_vec<V>(first, x);
    } else if (a.v_role == BCG_VALUES_MIX) {
      const Vec<V> f = load_vec<V>(first);
#pragma unroll
      for (int k = 0; k < V; ++k) x.x[k] = (1.0f - a.v_mix) * x.x[k] + a.v_mix * f.x[k];
    }
    if (tok.slot >= 0)
      store_vec<V>(static_cast<T*>(a.v_cache) + ((tok.page * a.kv_heads + g) * a.page_size + tok.in_page) * a.v_ld + i, x);
  }
}

// grid: `blocks` CTAs per token, then the routing CTAs (`route_tokens` tokens each).  Columns go to their destination four at a
// time (V = 4) or one by one.
template <typename T, int V>
__global__ void __launch_bounds__(kInThreads)
grouped_in_kernel(const GroupedIn a) {
  extern __shared__ uint32_t route_mem[];   // route_words(experts)
  pdl_launch_dependents();
  pdl_wait();
  const int split = blockIdx.x - a.n_tokens * a.blocks;
  if (split >= 0) {
    const int t0 = split * a.route_tokens;
    route_tokens<kInThreads>(a.route, a.proj, a.n_partials, a.pstride, a.ld, t0, min(t0 + a.route_tokens, a.n_tokens),
                             route_mem);
    return;
  }
  const long long t = blockIdx.x / a.blocks;
  const int part = blockIdx.x % a.blocks;
  const float* row = a.proj + t * a.ld;
  const InToken tok(a, t);
  const int nv = a.heads * a.dim + a.kv_heads * (a.dim + a.vdim);
  const int step = a.blocks * kInThreads * V;
  for (int c = (part * kInThreads + threadIdx.x) * V; c < nv; c += step) {
    Vec<V> x = slab_sum_vec<V>(row + c, a.n_partials, a.pstride);
    x.add(load_vec<V>(a.bias + c));
    store_columns<T, V>(a, tok, c, x);
  }
  for (int c = (part * kInThreads + threadIdx.x) * V; c < a.ff; c += step) {
    Vec<V> x = slab_sum_vec<V>(row + a.act_from + c, a.n_partials, a.pstride);
#pragma unroll
    for (int k = 0; k < V; ++k) {
      const float r = fmaxf(x.x[k], 0.f);
      x.x[k] = r * r;
    }
    store_vec<V>(static_cast<T*>(a.act) + t * a.act_ld + c, x);
  }
}

// One token per CTA, or per cluster of CL CTAs that have a range of its columns each: query and key norms span all
// heads.
template <typename T, int V, int CL>
__global__ void __launch_bounds__(kInThreads)
grouped_norm_in_kernel(const GroupedIn a) {
  extern __shared__ float4 stage_raw[];
  float* stage = reinterpret_cast<float*>(stage_raw);
  __shared__ RowSum<kInThreads, CL, 2> sh;
  pdl_launch_dependents();
  pdl_wait();
  const int cta = CL > 1 ? static_cast<int>(blockIdx.x) : 0;
  const InToken tok(a, CL > 1 ? blockIdx.y : blockIdx.x);
  const float* row = a.proj + tok.t * a.ld;
  const int nq = a.heads * a.dim, nk = nq + a.kv_heads * a.dim, nv = nk + a.kv_heads * a.vdim;
  const int per = (nv / V + CL - 1) / CL * V;
  const int c0 = cta * per, c1 = min(nv, c0 + per);
  float ss[2] = {0.f, 0.f};     // queries, keys
  for (int c = c0 + threadIdx.x * V; c < c1; c += kInThreads * V) {
    Vec<V> x = slab_sum_vec<V>(row + c, a.n_partials, a.pstride);
    x.add(load_vec<V>(a.bias + c));
    store_vec<V>(stage + c - c0, x);
    if (c < nq) ss[0] += x.sumsq();
    else if (c < nk) ss[1] += x.sumsq();
  }
  if (a.gates)
    for (int h = cta * kInThreads + threadIdx.x; h < a.heads; h += CL * kInThreads)
      a.gates[tok.t * a.heads + h] = a.gate_scale * sigmoid_f32(slab_sum(row + a.gate_col + h, a.n_partials, a.pstride));
  row_sum<kInThreads, CL, 2>(sh, ss, 0);
  const float inv_q = rsqrtf(ss[0] / static_cast<float>(nq) + a.eps);
  const float inv_k = rsqrtf(ss[1] / static_cast<float>(nk - nq) + a.eps);
  for (int c = c0 + threadIdx.x * V; c < c1; c += kInThreads * V) {
    Vec<V> x = load_vec<V>(stage + c - c0);
    const float* w = c < nq ? (a.q_norm ? a.q_norm + c : nullptr) : c < nk ? (a.k_norm ? a.k_norm + c - nq : nullptr) : nullptr;
    if (w) {
      const Vec<V> ww = load_vec<V>(w);
      const float inv = c < nq ? inv_q : inv_k;
#pragma unroll
      for (int k = 0; k < V; ++k) x.x[k] = x.x[k] * inv * ww.x[k];
    }
    store_columns<T, V>(a, tok, c, x);
  }
  row_sum_exit<CL>();
}

template <typename T, int V>
static int norm_in_t(const GroupedIn& a, cudaStream_t st) {
  const int cols = a.heads * a.dim + a.kv_heads * (a.dim + a.vdim);
  if (a.n_tokens <= 128 && cols >= 1024) {
    const size_t sm = static_cast<size_t>((cols / V + 7) / 8 * V) * 4;
    BCG_TRY(ensure_dynamic_smem(reinterpret_cast<const void*>(grouped_norm_in_kernel<T, V, 8>), 48 * 1024));
    BCG_CUDA_CHECK(launch_cluster(grouped_norm_in_kernel<T, V, 8>, dim3(8, a.n_tokens), dim3(kInThreads), 8, sm, st, a));
  } else {
    BCG_TRY(ensure_dynamic_smem(reinterpret_cast<const void*>(grouped_norm_in_kernel<T, V, 1>), 200 * 1024));
    BCG_CUDA_CHECK(launch_k(grouped_norm_in_kernel<T, V, 1>, dim3(a.n_tokens), dim3(kInThreads), static_cast<size_t>(cols) * 4,
                            st, a));
  }
  return BCG_OK;
}

// Row of a key/value head in the pages: entry i of logical page j0 + i / page_size of a sequence's row of the block table.
__device__ __forceinline__ long long page_row(const int* bt, int j0, int i, int kv_heads, int g, int page_size) {
  return (static_cast<long long>(bt[j0 + i / page_size]) * kv_heads + g) * page_size + i % page_size;
}

// Sum of n rows of a cache from position p0 on, in their order: NV vectors of V columns per lane, the first at column c, for the lanes
// that want it.  Groups of L lanes share the look-ups; n is the warp's.
template <typename T, int V, int NV, int L>
__device__ __forceinline__ void rows_sum(Vec<V> (&sum)[NV], const T* cache, const int* bt, int kv_heads, int g, int page_size, int ld, int c,
                                         bool want, int p0, int n) {
  const int lane = threadIdx.x % L;
#pragma unroll
  for (int i = 0; i < NV; ++i) sum[i] = Vec<V>{};
  for (int j0 = 0; j0 < n; j0 += L) {
    const int mine = static_cast<int>(page_row(bt, 0, p0 + min(j0 + lane, n - 1), kv_heads, g, page_size));
    const int m = min(L, n - j0);
    for (int j1 = 0; j1 < m; j1 += 8) {
      Vec<V> v[8][NV];
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const T* row = cache + static_cast<long long>(__shfl_sync(0xffffffffu, mine, min(j1 + j, m - 1), L)) * ld + c;
#pragma unroll
        for (int i = 0; i < NV; ++i)
          if (want) v[j][i] = load_vec<V>(row + i * V);
      }
#pragma unroll
      for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int i = 0; i < NV; ++i)
          if (j1 + j < m && want) sum[i].add(v[j][i]);
    }
  }
}
template <int V>
__device__ __forceinline__ Vec<V> divided(Vec<V> sum, int n) {
#pragma unroll
  for (int k = 0; k < V; ++k) sum.x[k] /= static_cast<float>(n);
  return sum;
}

// A token whose heads (queries, then keys, then values) warps take one by one.
struct HeadToken {
  int t, pos, slot, n_heads;
  bool ends_block;             // of pooled keys
  __device__ __forceinline__ HeadToken(const GroupedIn& a, int t_) : t(t_), pos(a.positions[t_]), slot(a.slot_map[t_]), n_heads(a.heads + 2 * a.kv_heads) {
    ends_block = a.pool > 0 && slot >= 0 && (pos + 1) % a.pool == 0;
  }
};
struct HeadUnit {
  int g, width, dims, col, ld;
  bool is_q, is_v;
  __device__ __forceinline__ HeadUnit(const GroupedIn& a, int s) {
    is_q = s < a.heads;
    is_v = s >= a.heads + a.kv_heads;
    g = is_q ? s : s - a.heads - (is_v ? a.kv_heads : 0);
    width = is_v ? a.vdim : a.dim;
    dims = is_v ? a.v_rot_dims : a.rot_dims;
    col = is_v ? (a.heads + a.kv_heads) * a.dim + g * a.vdim : s * a.dim;
    ld = is_v ? a.v_ld : a.q_ld;
  }
  template <typename T>
  __device__ __forceinline__ T* cache(const GroupedIn& a) const { return static_cast<T*>(is_v ? a.v_cache : a.k_cache); }
  // row of the queries or of the cache, NULL: the token is not stored
  template <typename T>
  __device__ __forceinline__ T* destination(const GroupedIn& a, const HeadToken& at) const {
    if (is_q) return static_cast<T*>(a.q) + (static_cast<long long>(at.t) * a.heads + g) * ld;
    if (at.slot < 0) return nullptr;
    const int page = at.slot / a.page_size;
    return cache<T>(a) + ((static_cast<long long>(page) * a.kv_heads + g) * a.page_size + at.slot - page * a.page_size) * ld;
  }
  __device__ __forceinline__ const float* norm(const GroupedIn& a) const { return is_q ? a.q_norm : is_v ? nullptr : a.k_norm; }
  // cosines, sines dims / 2 behind them
  __device__ __forceinline__ const float* angles(const GroupedIn& a, int pos) const {
    return (is_v ? a.v_cos_sin : a.cos_sin) + static_cast<long long>(pos) * dims;
  }
  template <typename T>
  __device__ __forceinline__ T* block_row(const GroupedIn& a, const HeadToken& at) const {
    return cache<T>(a) +
           page_row(a.block_table + static_cast<long long>(at.t) * a.max_blocks, a.pool_col, at.pos / a.pool, a.kv_heads, g, a.page_size) * ld;
  }
};

// Cosines and sines of the four pairs from column c (a multiple of eight) on; pairs behind `dims` do not turn.
struct PairAngles {
  float cs[4], sn[4];
  __device__ __forceinline__ void load(const float* row, int dims, int c) {
    const int m = c / 2, half = dims / 2;
    if (c + 8 <= dims && dims % 8 == 0) {
      const float4 a = __ldg(reinterpret_cast<const float4*>(row + m)), b = __ldg(reinterpret_cast<const float4*>(row + half + m));
      cs[0] = a.x; cs[1] = a.y; cs[2] = a.z; cs[3] = a.w;
      sn[0] = b.x; sn[1] = b.y; sn[2] = b.z; sn[3] = b.w;
    } else {
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        cs[k] = m + k < half ? row[m + k] : 1.f;
        sn[k] = m + k < half ? row[half + m + k] : 0.f;
      }
    }
  }
  __device__ __forceinline__ void turn(Vec<4>& v, int first) const {
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      const float p = v.x[2 * k], q = v.x[2 * k + 1];
      v.x[2 * k] = p * cs[first + k] - q * sn[first + k];
      v.x[2 * k + 1] = q * cs[first + k] + p * sn[first + k];
    }
  }
};

// Heads in registers: rotation in pairs of neighbours, multiples of eight entries up to 8 * L.  L lanes have a head, a warp has 32 / L
// at a time and U times that; `groups` CTAs per token.  blocks: the step has one token per sequence, so whoever writes the last row
// of a block also writes its mean.
template <typename T, int L, int U>
__global__ void __launch_bounds__(kInThreads)
head_pairs_kernel(const GroupedIn a, int groups, bool blocks) {
  constexpr int kAtOnce = 32 / L, kPerCta = kInThreads / 32 * kAtOnce * U;
  const int t = blockIdx.x / groups, c = threadIdx.x % L * 8;
  const int warp_first = (blockIdx.x - t * groups) * kPerCta + static_cast<int>(threadIdx.x >> 5) * kAtOnce * U;
  const int first = warp_first + static_cast<int>(threadIdx.x & 31) / L;
  pdl_launch_dependents();
  const HeadToken at(a, t);
  if (warp_first >= at.n_heads) return;
  auto unit = [&](int i) { return HeadUnit(a, min(first + i * kAtOnce, at.n_heads - 1)); };
  Vec<4> x[U][2], sum[2];
  const bool whole = U == 1 && blocks && at.ends_block;
  if constexpr (U == 1) {         // the block's other rows and the positions were there before this step
    if (whole && warp_first + kAtOnce > a.heads) {
      const HeadUnit u = unit(0);
      rows_sum<T, 4, 2, L>(sum, u.cache<T>(a), a.block_table + static_cast<long long>(t) * a.max_blocks, a.kv_heads, u.is_q ? 0 : u.g, a.page_size,
                           u.ld, c, !u.is_q && c < u.width, at.pos + 1 - a.pool, a.pool - 1);
    }
  }
  pdl_wait();
  const float* row = a.proj + t * a.ld;
#pragma unroll
  for (int i = 0; i < U; ++i) {
    const HeadUnit u = unit(i);
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      x[i][n] = Vec<4>{};
      if (c < u.width) {
        const float* src = row + u.col + c + n * 4;
        x[i][n] = U > 1 && a.n_partials == 1 ? load_vec<4>(src) : slab_sum_vec<4>(src, a.n_partials, a.pstride);
        if (a.bias) x[i][n].add(load_vec<4>(a.bias + u.col + c + n * 4));
      }
    }
  }
  PairAngles of_qk = {}, of_v = {};
  if (a.rot_dims > 0 && warp_first < a.heads + a.kv_heads) of_qk.load(a.cos_sin + static_cast<long long>(at.pos) * a.rot_dims, a.rot_dims, c);
  if (a.v_rot_dims > 0 && warp_first + kAtOnce * U > a.heads + a.kv_heads)
    of_v.load(a.v_cos_sin + static_cast<long long>(at.pos) * a.v_rot_dims, a.v_rot_dims, c);
  const float inv_dim = 1.0f / static_cast<float>(a.dim);
#pragma unroll
  for (int i = 0; i < U; ++i) {
    const HeadUnit u = unit(i);
    float ss = x[i][0].sumsq() + x[i][1].sumsq();
#pragma unroll
    for (int o = L / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (first + i * kAtOnce >= at.n_heads || c >= u.width) continue;
    if (const float* w = u.norm(a)) {
      const float inv = rsqrtf(ss * inv_dim + a.eps);
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        const Vec<4> ww = load_vec<4>(w + c + n * 4);
#pragma unroll
        for (int k = 0; k < 4; ++k) x[i][n].x[k] *= inv * ww.x[k];
      }
    }
    if (u.dims > 0) {
      PairAngles an;
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        an.cs[k] = u.is_v ? of_v.cs[k] : of_qk.cs[k];
        an.sn[k] = u.is_v ? of_v.sn[k] : of_qk.sn[k];
      }
      an.turn(x[i][0], 0);
      an.turn(x[i][1], 2);
    }
    if (T* dst = u.destination<T>(a, at)) {
      store_vec<4>(dst + c, x[i][0]);
      store_vec<4>(dst + c + 4, x[i][1]);
    }
    if (whole && !u.is_q) {
#pragma unroll
      for (int n = 0; n < 2; ++n) {
#pragma unroll
        for (int k = 0; k < 4; ++k) sum[n].x[k] += sizeof(T) == 2 ? to_f32<T>(from_f32<T>(x[i][n].x[k])) : x[i][n].x[k];   // as the cache holds it
        store_vec<4>(u.block_row<T>(a, at) + c + n * 4, divided(sum[n], a.pool));
      }
    }
  }
}

// Any head: a warp has one, through shared memory.
template <typename T, int V>
__global__ void __launch_bounds__(kInThreads)
head_in_kernel(const GroupedIn a, int groups, int pitch, bool blocks) {
  extern __shared__ float4 stage_raw[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* x = reinterpret_cast<float*>(stage_raw) + warp * pitch;
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x / groups, s = (blockIdx.x - t * groups) * (kInThreads / 32) + warp;
  const HeadToken at(a, t);
  if (s >= at.n_heads) return;
  const HeadUnit u(a, s);
  const int half = u.dims / 2;
  const bool pairs = u.is_v || a.rot_pairs;
  const float* row = a.proj + t * a.ld + u.col;
  float ss = 0.f;
  for (int c = lane * V; c < u.width; c += 32 * V) {
    Vec<V> v = slab_sum_vec<V>(row + c, a.n_partials, a.pstride);
    if (a.bias) v.add(load_vec<V>(a.bias + u.col + c));
    store_vec<V>(x + c, v);
    ss += v.sumsq();
  }
  const float* w = u.norm(a);
  const float inv = w ? rsqrtf(warp_sum(ss) / static_cast<float>(u.width) + a.eps) : 1.0f;
  __syncwarp();
  const float* angle = u.angles(a, at.pos);
  T* dst = u.destination<T>(a, at);
  const bool whole = blocks && at.ends_block && !u.is_q;
  for (int c0 = 0; c0 < u.width; c0 += 32 * V) {
    const int c = c0 + lane * V;
    Vec<V> y;
#pragma unroll
    for (int k = 0; k < V; ++k) {
      const int e = c + k;
      if (e >= u.width) continue;
      const float own = x[e] * (w ? inv * w[e] : 1.0f);
      y.x[k] = own;
      if (e < u.dims) {
        const bool first = pairs ? !(e & 1) : e < half;
        const int p = pairs ? e ^ 1 : first ? e + half : e - half, i = pairs ? e >> 1 : first ? e : e - half;
        const float other = x[p] * (w ? inv * w[p] : 1.0f), cs = angle[i], sn = angle[half + i];
        y.x[k] = first ? own * cs - other * sn : own * cs + other * sn;
      }
      if (sizeof(T) == 2) y.x[k] = to_f32<T>(from_f32<T>(y.x[k]));      // as the cache holds it
    }
    if (dst && c < u.width) store_vec<V>(dst + c, y);
    if (whole) {
      Vec<V> sum[1];
      rows_sum<T, V, 1, 32>(sum, u.cache<T>(a), a.block_table + static_cast<long long>(t) * a.max_blocks, a.kv_heads, u.g, a.page_size, u.ld, c,
                            c < u.width, at.pos + 1 - a.pool, a.pool - 1);
      if (c < u.width) {
        sum[0].add(y);
        store_vec<V>(u.block_row<T>(a, at) + c, divided(sum[0], a.pool));
      }
    }
  }
}

// A warp has a run of `run` tokens (up to 32) and a key or value head: the means of the blocks that end there.
template <typename T, int V>
__global__ void __launch_bounds__(kInThreads, 3)
pool_blocks_kernel(const GroupedIn a, const int* __restrict__ row_seq, int run) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int unit = blockIdx.x * (kInThreads / 32) + (threadIdx.x >> 5), r = unit / (2 * a.kv_heads), s = unit - r * 2 * a.kv_heads;
  const long long t0 = static_cast<long long>(r) * run;
  if (t0 >= a.n_tokens) return;
  const bool is_v = s >= a.kv_heads, mine = lane < run && t0 + lane < a.n_tokens;
  const int g = is_v ? s - a.kv_heads : s, width = is_v ? a.vdim : a.dim, ld = is_v ? a.v_ld : a.q_ld;
  T* cache = static_cast<T*>(is_v ? a.v_cache : a.k_cache);
  const int pos = mine ? a.positions[t0 + lane] : 0;
  unsigned ends = __ballot_sync(0xffffffffu, mine && a.slot_map[t0 + lane] >= 0 && (pos + 1) % a.pool == 0);
  for (; ends; ends &= ends - 1) {
    const int i = __ffs(ends) - 1, b = __shfl_sync(0xffffffffu, pos, i) / a.pool;
    const int* bt = a.block_table + static_cast<long long>(row_seq ? row_seq[t0 + i] : t0 + i) * a.max_blocks;
    T* dst = cache + page_row(bt, a.pool_col, b, a.kv_heads, g, a.page_size) * ld;
    for (int c0 = 0; c0 < width; c0 += 32 * V) {
      const int c = c0 + lane * V;
      Vec<V> sum[1];
      rows_sum<T, V, 1, 32>(sum, cache, bt, a.kv_heads, g, a.page_size, ld, c, c < width, b * a.pool, a.pool);
      if (c < width) store_vec<V>(dst + c, divided(sum[0], a.pool));
    }
  }
}

template <typename T, int L>
static int head_pairs_t(const GroupedIn& a, bool one_token, cudaStream_t st) {
  const bool few = one_token || a.n_tokens <= 128;
  const int per = (few ? 1 : 2) * (kInThreads / L), groups = (a.heads + 2 * a.kv_heads + per - 1) / per;
  const dim3 grid(static_cast<unsigned>(a.n_tokens * groups));
  if (few) BCG_CUDA_CHECK(launch_k(head_pairs_kernel<T, L, 1>, grid, dim3(kInThreads), 0, st, a, groups, one_token));
  else BCG_CUDA_CHECK(launch_k(head_pairs_kernel<T, L, 2>, grid, dim3(kInThreads), 0, st, a, groups, false));
  return BCG_OK;
}

template <typename T, int V>
static int head_in_t(const GroupedIn& a, const int* row_seq, bool one_token, cudaStream_t st) {
  const int wide = max(a.dim, a.vdim);
  if (V == 4 && a.rot_pairs && wide <= 256 && a.dim % 8 == 0 && a.vdim % 8 == 0) {
    BCG_TRY(wide <= 128 ? (head_pairs_t<T, 16>(a, one_token, st)) : (head_pairs_t<T, 32>(a, one_token, st)));
  } else {
    const int pitch = (wide + 3) / 4 * 4;
    const size_t sm = static_cast<size_t>(kInThreads / 32) * pitch * 4;
    if (sm > 200 * 1024) {
      set_last_error("bcg_grouped_in", "heads are too large");
      return BCG_ERR_UNSUPPORTED;
    }
    if (sm > 48 * 1024) BCG_TRY(ensure_dynamic_smem(reinterpret_cast<const void*>(head_in_kernel<T, V>), 200 * 1024));
    const int groups = (a.heads + 2 * a.kv_heads + kInThreads / 32 - 1) / (kInThreads / 32);
    BCG_CUDA_CHECK(launch_k(head_in_kernel<T, V>, dim3(static_cast<unsigned>(a.n_tokens * groups)), dim3(kInThreads), sm, st, a, groups, pitch,
                            one_token));
  }
  if (a.pool > 0 && !one_token) {
    const int run = min(max(a.pool, 4), 32);
    const long long runs = static_cast<long long>((a.n_tokens + run - 1) / run) * 2 * a.kv_heads;
    BCG_CUDA_CHECK(launch_k(pool_blocks_kernel<T, V>, dim3(static_cast<unsigned>((runs + 7) / 8)), dim3(kInThreads), 0, st, a, row_seq, run));
  }
  return BCG_OK;
}

template <typename T>
static int grouped_in_t(const GroupedIn& a, cudaStream_t st) {
  const bool wide = ((a.dim | a.vdim | a.ff | a.act_from) & 3) == 0 && a.ld % 4 == 0 && a.pstride % 4 == 0;
  if (a.q_norm || a.k_norm || a.gates) {
    if (a.ff > 0 || a.route.experts > 0 || a.heads * a.dim + a.kv_heads * (a.dim + a.vdim) > 51200) {
      set_last_error("bcg_grouped_in", "norms and gates: no parallel feed-forward, at most 51,200 columns");
      return BCG_ERR_UNSUPPORTED;
    }
    return wide ? norm_in_t<T, 4>(a, st) : norm_in_t<T, 1>(a, st);
  }
  const dim3 grid(a.n_tokens * a.blocks + (a.route.experts > 0 ? (a.n_tokens + a.route_tokens - 1) / a.route_tokens : 0));
  const size_t sm = static_cast<size_t>(route_words(a.route.experts, kInThreads)) * 4;
  if (sm > 48 * 1024) {
    set_last_error("bcg_grouped_in", "too many experts");
    return BCG_ERR_UNSUPPORTED;
  }
  if (wide) BCG_CUDA_CHECK(launch_k(grouped_in_kernel<T, 4>, grid, dim3(kInThreads), sm, st, a));
  else BCG_CUDA_CHECK(launch_k(grouped_in_kernel<T, 1>, grid, dim3(kInThreads), sm, st, a));
  return BCG_OK;
}

// with_act: the activations of the feed-forward are columns l->n_qkv.. of proj (else the GEMM made them)
int grouped_in(const bcg_stack* m, const bcg_layer* l, const bcg_stack_ws* ws, const bcg_step_batch* b, int n_partials,
               long long pstride, long long ld, bool with_act, cudaStream_t st) {
  const size_t act_bytes = m->act_dtype == BCG_DT_F32 ? 4 : 2;
  GroupedIn a = {};
  a.proj = ws->proj;
  a.n_partials = n_partials;
  a.pstride = pstride;
  a.ld = ld;
  a.positions = b->positions;
  a.slot_map = b->slot_map;
  a.bias = l->in_bias;
  a.q = ws->q;
  a.k_cache = l->cache;
  a.v_cache = l->cache_v;
  a.v_first = ws->v_first;
  a.heads = l->heads;
  a.kv_heads = l->kv_heads;
  a.dim = l->dim;
  a.vdim = l->vdim;
  a.q_ld = l->q_ld;
  a.v_ld = l->v_ld;
  a.page_size = m->page_size;
  a.temp_coef = l->temp_coef;
  a.temp_every = l->temp_every;
  a.v_role = l->v_role;
  a.v_mix = l->v_mix;
  a.ff = with_act ? l->ff : 0;
  a.act_from = with_act ? l->n_qkv : 0;
  a.act = static_cast<char*>(ws->mix) + l->act_col * act_bytes;
  a.act_ld = l->mix_ld;
  a.q_norm = l->q_norm;
  a.k_norm = l->k_norm;
  a.gates = l->gated ? ws->gates : nullptr;
  a.gate_col = l->gate_col;
  a.gate_scale = l->gate_scale;
  a.eps = m->eps;
  if (l->by_head) {
    if ((l->rot_dims && !l->cos_sin) || (l->v_rot_dims && !l->v_cos_sin) || l->rot_dims % 2 || l->rot_dims > l->dim || l->v_rot_dims % 2 ||
        l->v_rot_dims > l->vdim || l->gated || l->v_role || l->slopes || l->temp_coef != 0.f || with_act || l->pool < 0) {
      set_last_error("bcg_grouped_in", "heads one by one: even rotary sizes with tables; no gates, mixed values, bias or temperature");
      return BCG_ERR_ARG;
    }
    a.cos_sin = l->cos_sin;
    a.v_cos_sin = l->v_cos_sin;
    a.rot_dims = l->rot_dims;
    a.rot_pairs = l->rot_pairs;
    a.v_rot_dims = l->v_rot_dims;
    a.pool = l->pool;
    a.pool_col = l->pool_col;
    a.block_table = b->block_table;
    a.max_blocks = b->max_blocks;
    a.n_tokens = b->T;
    const bool wide = ((a.dim | a.vdim) & 3) == 0 && a.ld % 4 == 0 && a.pstride % 4 == 0, one = b->T == b->n_seqs;
    if (m->act_dtype == BCG_DT_F32)
      return wide ? head_in_t<float, 4>(a, b->row_seq, one, st) : head_in_t<float, 1>(a, b->row_seq, one, st);
    return wide ? head_in_t<__nv_bfloat16, 4>(a, b->row_seq, one, st) : head_in_t<__nv_bfloat16, 1>(a, b->row_seq, one, st);
  }
  if (!l->in_bias) {
    set_last_error("bcg_grouped_in", "projections without bias: heads one by one");
    return BCG_ERR_UNSUPPORTED;
  }
  if (l->experts > 0) a.route = moe_route(l, ws);
  const int cols = l->heads * l->dim + l->kv_heads * (l->dim + l->vdim);
  a.blocks = b->T <= 128 ? max(1, ((cols > a.ff ? cols : a.ff) + kInThreads * 4 - 1) / (kInThreads * 4)) : 1;
  a.n_tokens = b->T;
  a.route_tokens = b->T <= 128 ? kInThreads / 32 : kInThreads / 4;
  return m->act_dtype == BCG_DT_F32 ? grouped_in_t<float>(a, st) : grouped_in_t<__nv_bfloat16>(a, st);
}

// ------------------------------------------------------------------------------------------- plain
constexpr int kGpThreads = 128, kGpKeys = 256;

struct GroupedAttn {
  const void *q, *k_cache, *v_cache;
  const float *slopes, *gates;
  const int *rows, *positions, *row_seq, *block_table;
  int max_blocks, page_size;
  void* out;
  long long out_ld;
  int heads, kv_heads, dim, vdim, q_ld, v_ld, window;
  float scale;
  PooledKeys pooled;
  const float* v_cos_sin;     // outputs turn back in pairs of neighbours, or NULL
  int v_rot_dims;
  // Output columns c (even) and c + 1 of a token at position pos.
  __device__ __forceinline__ void turn_back(int pos, int c, float& u, float& v) const {
    if (!v_cos_sin || c >= v_rot_dims) return;
    const float* row = v_cos_sin + static_cast<long long>(pos) * v_rot_dims + c / 2;
    const float cs = row[0], sn = row[v_rot_dims / 2], x = u;
    u = x * cs + v * sn;
    v = v * cs - x * sn;
  }
};

template <typename T>
__global__ void __launch_bounds__(kGpThreads)
grouped_plain_kernel(const GroupedAttn a) {
  extern __shared__ float sm[];
  __shared__ float red[kGpThreads / 32];
  float* qs = sm;             // [dim]
  float* oc = qs + a.dim;     // [vdim]
  float* p = oc + a.vdim;     // [kGpKeys]
  pdl_launch_dependents();
  pdl_wait();
  const long long t = a.rows ? a.rows[blockIdx.x] : blockIdx.x;
  const int h = blockIdx.y, g = h / (a.heads / a.kv_heads);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pos = a.positions[t];
  const int* bt = a.block_table + static_cast<long long>(a.row_seq ? a.row_seq[t] : t) * a.max_blocks;
  const T* qh = static_cast<const T*>(a.q) + (t * a.heads + h) * a.q_ld;
  const float slope = a.slopes ? a.slopes[h] : 0.f;
  for (int i = threadIdx.x; i < a.dim; i += kGpThreads) qs[i] = to_f32<T>(qh[i]);
  for (int i = threadIdx.x; i < a.vdim; i += kGpThreads) oc[i] = 0.f;
  float m = -INFINITY, l = 0.f;
  const int lo = a.window > 0 ? max(0, pos - a.window + 1) : 0;
  // tokens lo .. pos, then the pooled blocks that are seen
  const int n_tok = pos + 1 - lo, n_all = n_tok + a.pooled.visible(pos, a.window);
  auto row_of = [&](int u) {
    return u < n_tok ? page_row(bt, 0, lo + u, a.kv_heads, g, a.page_size) : page_row(bt, a.pooled.col, u - n_tok, a.kv_heads, g, a.page_size);
  };
  for (int j0 = 0; j0 < n_all; j0 += kGpKeys) {
    const int n = min(kGpKeys, n_all - j0);
    __syncthreads();
    float mx = -INFINITY;
    for (int j = warp; j < n; j += kGpThreads / 32) {
      const T* k = static_cast<const T*>(a.k_cache) + row_of(j0 + j) * a.q_ld;
      float s = 0.f;
      for (int i = lane; i < a.dim; i += 32) s = fmaf(qs[i], to_f32<T>(k[i]), s);
      s = warp_sum(s) * a.scale - slope * static_cast<float>(pos - lo - (j0 + j));
      if (lane == 0) p[j] = s;
      mx = fmaxf(mx, s);
    }
    if (lane == 0) red[warp] = mx;
    __syncthreads();
#pragma unroll
    for (int i = 0; i < kGpThreads / 32; ++i) mx = fmaxf(mx, red[i]);
    const float m_new = fmaxf(m, mx);
    const float corr = expf(m - m_new);
    float sum = 0.f;
    for (int j = threadIdx.x; j < n; j += kGpThreads) {
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
    for (int i = 0; i < kGpThreads / 32; ++i) sum += red[i];
    l = l * corr + sum;
    m = m_new;
    for (int r = threadIdx.x; r < a.vdim; r += kGpThreads) {
      float acc = oc[r] * corr;
      for (int j = 0; j < n; ++j)
        acc = fmaf(p[j], to_f32<T>(static_cast<const T*>(a.v_cache)[row_of(j0 + j) * a.v_ld + r]), acc);
      oc[r] = acc;
    }
  }
  __syncthreads();
  const float inv = (a.gates ? a.gates[t * a.heads + h] : 1.0f) / l;
  T* dst = static_cast<T*>(a.out) + t * a.out_ld + static_cast<long long>(h) * a.vdim;
  for (int r = threadIdx.x * 2; r < a.vdim; r += kGpThreads * 2) {
    float u = oc[r] * inv, v = r + 1 < a.vdim ? oc[r + 1] * inv : 0.f;
    a.turn_back(pos, r, u, v);
    dst[r] = from_f32<T>(u);
    if (r + 1 < a.vdim) dst[r + 1] = from_f32<T>(v);
  }
}

static GroupedAttn attn_args(const bcg_stack* m, const bcg_layer* l, const bcg_stack_ws* ws, const bcg_step_batch* b,
                             const int* rows) {
  GroupedAttn a = {};
  a.q = ws->q;
  a.k_cache = l->cache;
  a.v_cache = l->cache_v;
  a.slopes = l->slopes;
  a.gates = l->gated ? ws->gates : nullptr;
  a.rows = rows;
  a.positions = b->positions;
  a.row_seq = b->row_seq;
  a.block_table = b->block_table;
  a.max_blocks = b->max_blocks;
  a.page_size = m->page_size;
  a.out = ws->mix;
  a.out_ld = l->mix_ld;
  a.heads = l->heads;
  a.kv_heads = l->kv_heads;
  a.dim = l->dim;
  a.vdim = l->vdim;
  a.q_ld = l->q_ld;
  a.v_ld = l->v_ld;
  a.window = l->window;
  a.scale = l->scale;
  a.pooled = {l->pool, l->pool_col};
  a.v_cos_sin = l->v_rot_dims > 0 ? l->v_cos_sin : nullptr;
  a.v_rot_dims = l->v_rot_dims;
  return a;
}

static int grouped_plain(const bcg_stack* m, const bcg_layer* l, const bcg_stack_ws* ws, const bcg_step_batch* b,
                         const int* rows, int n, cudaStream_t st) {
  const GroupedAttn a = attn_args(m, l, ws, b, rows);
  const int sm = (l->dim + l->vdim + kGpKeys) * 4;
  const dim3 grid(n, l->heads);
  if (m->act_dtype == BCG_DT_F32) {
    BCG_TRY(ensure_dynamic_smem(reinterpret_cast<const void*>(grouped_plain_kernel<float>), 64 * 1024));
    BCG_CUDA_CHECK(launch_k(grouped_plain_kernel<float>, grid, dim3(kGpThreads), sm, st, a));
  } else {
    BCG_TRY(ensure_dynamic_smem(reinterpret_cast<const void*>(grouped_plain_kernel<__nv_bfloat16>), 64 * 1024));
    BCG_CUDA_CHECK(launch_k(grouped_plain_kernel<__nv_bfloat16>, grid, dim3(kGpThreads), sm, st, a));
  }
  return BCG_OK;
}

// ------------------------------------------------------------------------------------------- decode
// grid (cluster, tokens, kv heads x groups of 16 query heads), 4 warps.  The visible pages of a token are dealt
// round-robin to the cluster's warps; a warp keeps `stages` pages in flight, each a stage of its own ring.
constexpr int kGdWarps = 4, kGdThreads = kGdWarps * 32, kGdHeads = 16, kGdPage = 16, kGdMaxCluster = 8;

template <int QD, int VD>
struct GdCfg {
  static constexpr int kK = kGdPage * QD * 2, kV = kGdPage * VD * 2, kStage = kK + kV;
  static constexpr int kFit = 96 * 1024 / (kGdWarps * kStage);
  static constexpr int kStages = kFit < 2 ? 2 : kFit > 6 ? 6 : kFit;
  static constexpr int kRing = kStages * kStage;                      // a warp's ring; later its partial output
  static constexpr int kQRow = QD + 8;
  static constexpr int kOffQ = kGdWarps * kRing;
  static constexpr int kOffMl = kOffQ + kGdHeads * kQRow * 2;         // [5][16] (maximum, denominator)
  static constexpr int kOffBar = kOffMl + (kGdWarps + 1) * kGdHeads * 8;
  static constexpr int kSmem = kOffBar + kGdWarps * kStages * 8 + 1024;
  static_assert(kGdHeads * VD * 4 <= kRing, "a warp's partial output fits its ring");
};

// 16 x D tile of D / 64 boxes of [16 rows][128 bytes], 128B-swizzled: address of 16-byte chunk `chunk` of a row
__device__ __forceinline__ const void* swizzled(const uint8_t* tile, int row, int chunk) {
  return tile + (chunk >> 3) * (kGdPage * 128) + row * 128 + (((chunk & 7) ^ (row & 7)) << 4);
}

template <int QD, int VD>
__global__ void __launch_bounds__(kGdThreads)
grouped_decode_kernel(const __grid_constant__ CUtensorMap k_map, const __grid_constant__ CUtensorMap v_map,
                      const GroupedAttn a) {
  using C = GdCfg<QD, VD>;
  namespace cg = cooperative_groups;
  extern __shared__ __align__(16) uint8_t gd_raw[];
  uint8_t* smem = gd_raw + ((1024u - (smem_u32(gd_raw) & 1023u)) & 1023u);
  __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(smem + C::kOffQ);
  float2* ml = reinterpret_cast<float2*>(smem + C::kOffMl);   // [warp][16], then the CTA's
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + C::kOffBar) + warp * C::kStages;
  uint8_t* ring = smem + warp * C::kRing;
  pdl_launch_dependents();
  if (lane == 0) {
    tma_prefetch_desc(&k_map);
    tma_prefetch_desc(&v_map);
    for (int s = 0; s < C::kStages; ++s) mbar_init(&full[s], 1);
    fence_barrier_init();
  }
  __syncwarp();
  pdl_wait();
  cg::cluster_group cluster = cg::this_cluster();
  const int rank = blockIdx.x, n_cta = gridDim.x;
  const int i_tok = blockIdx.y, g = blockIdx.z % a.kv_heads, group = a.heads / a.kv_heads;
  const int h0 = g * group + blockIdx.z / a.kv_heads * kGdHeads;
  const int nh = min(kGdHeads, (g + 1) * group - h0);
  const int t = a.rows ? a.rows[i_tok] : i_tok;
  const int pos = a.positions[t];
  const int lo = a.window > 0 ? max(0, pos - a.window + 1) : 0;
  const int* bt = a.block_table + static_cast<long long>(a.row_seq ? a.row_seq[t] : t) * a.max_blocks;
  // the token's pages, then those of the pooled blocks it sees: the warp has first, first + stride, ...
  const int n_pooled = a.pooled.visible(pos, a.window), tok_pages = pos / kGdPage - lo / kGdPage + 1;
  const int n_pages = tok_pages + (n_pooled + kGdPage - 1) / kGdPage;
  const int first = rank * kGdWarps + warp, stride = n_cta * kGdWarps;
  const int n = n_pages > first ? (n_pages - 1 - first) / stride + 1 : 0;
  auto load = [&](int i) {    // lane 0
    const int st = i % C::kStages;
    const int u = first + i * stride;
    const int row = (bt[u < tok_pages ? lo / kGdPage + u : a.pooled.col + u - tok_pages] * a.kv_heads + g) * kGdPage;
    uint8_t* dst = ring + st * C::kStage;
    mbar_arrive_expect_tx(&full[st], C::kStage);
#pragma unroll
    for (int c = 0; c < QD / 64; ++c)
      tma_load_2d(dst + c * kGdPage * 128, &k_map, &full[st], c * 64, row, kEvictNormal);
#pragma unroll
    for (int c = 0; c < VD / 64; ++c)
      tma_load_2d(dst + C::kK + c * kGdPage * 128, &v_map, &full[st], c * 64, row, kEvictNormal);
  };
  if (lane == 0)
    for (int i = 0; i < C::kStages && i < n; ++i) load(i);
  const __nv_bfloat16* qsrc = static_cast<const __nv_bfloat16*>(a.q) + (static_cast<long long>(t) * a.heads + h0) * a.q_ld;
  for (int i = threadIdx.x; i < kGdHeads * (QD / 8); i += kGdThreads) {
    const int r = i / (QD / 8), c = i % (QD / 8) * 8;
    *reinterpret_cast<uint4*>(qs + r * C::kQRow + c) =
        r < nh ? *reinterpret_cast<const uint4*>(qsrc + static_cast<long long>(r) * a.q_ld + c) : make_uint4(0, 0, 0, 0);
  }
  __syncthreads();
  const float scale2 = a.scale * kLog2e;
  float slope[2], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int r = (lane >> 2) + e * 8;
    slope[e] = (a.slopes && r < nh) ? a.slopes[h0 + r] * kLog2e : 0.f;
  }
  float o[VD / 8][4] = {};
  for (int i = 0; i < n; ++i) {
    const int st = i % C::kStages;
    const uint8_t* kt = ring + st * C::kStage;
    const uint8_t* vt = kt + C::kK;
    mbar_wait(&full[st], (i / C::kStages) & 1);
    float s[2][4] = {};
#pragma unroll
    for (int k = 0; k < QD / 16; ++k) {
      uint32_t qa[4], kb[4];
      ldsm_x4(qa, qs + (lane & 15) * C::kQRow + k * 16 + (lane >> 4) * 8);
      ldsm_x4(kb, swizzled(kt, (lane & 7) + ((lane >> 4) << 3), k * 2 + ((lane >> 3) & 1)));
      mma_bf16_16816(s[0], qa, kb[0], kb[1]);
      mma_bf16_16816(s[1], qa, kb[2], kb[3]);
    }
    const int page = first + i * stride;
    const bool pooled = page >= tok_pages;
    const int key0 = (pooled ? page - tok_pages : lo / kGdPage + page) * kGdPage + (lane & 3) * 2;
    const int key_lo = pooled ? 0 : lo, key_hi = pooled ? n_pooled - 1 : pos;
    float corr[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      float mx = -INFINITY;
#pragma unroll
      for (int c = 0; c < 4; ++c) {      // keys key0, key0 + 1, key0 + 8, key0 + 9
        const int key = key0 + (c >> 1) * 8 + (c & 1);
        float& x = s[c >> 1][2 * e + (c & 1)];
        x = key >= key_lo && key <= key_hi ? fmaf(x, scale2, slope[e] * static_cast<float>(key - pos)) : -INFINITY;
        mx = fmaxf(mx, x);
      }
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
      const float m_new = fmaxf(m[e], mx);       // every page has a visible key: finite
      corr[e] = ex2_approx(m[e] - m_new);
      m[e] = m_new;
      float sum = 0.f;
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        float& x = s[c >> 1][2 * e + (c & 1)];
        x = ex2_approx(x - m_new);
        sum += x;
      }
      l[e] = l[e] * corr[e] + sum;
    }
    const uint32_t pa[4] = {pack_bf16(s[0][0], s[0][1]), pack_bf16(s[0][2], s[0][3]), pack_bf16(s[1][0], s[1][1]),
                            pack_bf16(s[1][2], s[1][3])};
    if (__any_sync(0xffffffffu, corr[0] != 1.0f || corr[1] != 1.0f)) {
#pragma unroll
      for (int j = 0; j < VD / 8; ++j) {
        o[j][0] *= corr[0];
        o[j][1] *= corr[0];
        o[j][2] *= corr[1];
        o[j][3] *= corr[1];
      }
    }
#pragma unroll
    for (int j = 0; j < VD / 16; ++j) {
      uint32_t vb[4];
      ldsm_x4_trans(vb, swizzled(vt, lane & 15, j * 2 + (lane >> 4)));
      mma_bf16_16816(o[2 * j], pa, vb[0], vb[1]);
      mma_bf16_16816(o[2 * j + 1], pa, vb[2], vb[3]);
    }
    __syncwarp();                        // everybody has read the page: its stage may be filled again
    if (lane == 0 && i + C::kStages < n) load(i + C::kStages);
  }
  // ---- merge: the warps of a CTA, then the CTAs of the cluster
  float* part = reinterpret_cast<float*>(ring);      // [16][VD]
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    l[e] += __shfl_xor_sync(0xffffffffu, l[e], 1);
    l[e] += __shfl_xor_sync(0xffffffffu, l[e], 2);
    const int r = (lane >> 2) + e * 8;
    if ((lane & 3) == 0) ml[warp * kGdHeads + r] = make_float2(m[e], l[e]);
#pragma unroll
    for (int j = 0; j < VD / 8; ++j)
      *reinterpret_cast<float2*>(part + r * VD + j * 8 + (lane & 3) * 2) = make_float2(o[j][2 * e], o[j][2 * e + 1]);
  }
  __syncthreads();
  auto weight = [](float mine, float top) { return mine == -INFINITY ? 0.f : ex2_approx(mine - top); };
  float* mine = reinterpret_cast<float*>(smem);      // the CTA's result takes warp 0's place
  for (int i = threadIdx.x; i < nh * VD; i += kGdThreads) {
    const int r = i / VD;
    float top = -INFINITY, x = 0.f, den = 0.f;
#pragma unroll
    for (int w = 0; w < kGdWarps; ++w) top = fmaxf(top, ml[w * kGdHeads + r].x);
#pragma unroll
    for (int w = 0; w < kGdWarps; ++w) {
      const float f = weight(ml[w * kGdHeads + r].x, top);
      x = fmaf(f, reinterpret_cast<const float*>(smem + w * C::kRing)[i], x);
      den = fmaf(f, ml[w * kGdHeads + r].y, den);
    }
    mine[i] = x;                                     // element i is read and written by this thread only
    if (i % VD == 0) ml[kGdWarps * kGdHeads + r] = make_float2(top, den);
  }
  if (n_cta > 1) cluster.sync();
  else __syncthreads();
  auto* dst = static_cast<__nv_bfloat16*>(a.out) + static_cast<long long>(t) * a.out_ld + static_cast<long long>(h0) * a.vdim;
  for (int i = (rank * kGdThreads + threadIdx.x) * 2; i < nh * VD; i += n_cta * kGdThreads * 2) {
    const int r = i / VD, c = i % VD;
    if (c >= a.vdim) continue;
    float top = -INFINITY, x0 = 0.f, x1 = 0.f, den = 0.f;
    for (int q = 0; q < n_cta; ++q) {
      const float2 other = *cluster.map_shared_rank(ml + kGdWarps * kGdHeads + r, q);
      const float2 val = *reinterpret_cast<const float2*>(cluster.map_shared_rank(mine, q) + i);
      const float up = fmaxf(top, other.x);
      const float f0 = weight(top, up), f1 = weight(other.x, up);
      x0 = x0 * f0 + val.x * f1;
      x1 = x1 * f0 + val.y * f1;
      den = den * f0 + other.y * f1;
      top = up;
    }
    if (a.gates) {
      const float gate = a.gates[static_cast<long long>(t) * a.heads + h0 + r];
      x0 *= gate;
      x1 *= gate;
    }
    x0 /= den;
    x1 /= den;
    a.turn_back(pos, c, x0, x1);
    dst[static_cast<long long>(r) * a.vdim + c] = __float2bfloat16(x0);
    if (c + 1 < a.vdim) dst[static_cast<long long>(r) * a.vdim + c + 1] = __float2bfloat16(x1);
  }
  if (n_cta > 1) cluster.sync();                     // nobody leaves while its shared memory is being read
}

template <int QD, int VD>
static int launch_decode(const CUtensorMap& km, const CUtensorMap& vm, const GroupedAttn& a, dim3 grid, cudaStream_t st) {
  using C = GdCfg<QD, VD>;
  BCG_TRY(ensure_dynamic_smem(reinterpret_cast<const void*>(grouped_decode_kernel<QD, VD>), C::kSmem));
  BCG_CUDA_CHECK(launch_cluster(grouped_decode_kernel<QD, VD>, grid, dim3(kGdThreads), static_cast<int>(grid.x), C::kSmem,
                                st, km, vm, a));
  return BCG_OK;
}

static bool padded_head(int q_ld, int v_ld) {
  return q_ld % 64 == 0 && q_ld >= 64 && q_ld <= 256 && (v_ld == 64 || v_ld == 128 || v_ld == 256);
}

// CTAs per (token, kv head): the choice with the fewest page times on 148 SMs with two CTAs each (a CTA costs
// about four pages of start-up).
static int decode_cluster(int rows, int pages) {
  int best = 1;
  long long best_cost = -1;
  for (int c = 1; c <= kGdMaxCluster; c *= 2) {
    if (c > 1 && pages < c * kGdWarps) break;
    const long long waves = (static_cast<long long>(rows) * c + 295) / 296;
    const long long cost = waves * ((pages + c * kGdWarps - 1) / (c * kGdWarps) + 4);
    if (best_cost < 0 || cost < best_cost) {
      best_cost = cost;
      best = c;
    }
  }
  return best;
}

static int grouped_decode(const bcg_stack* m, const bcg_layer* l, const bcg_stack_ws* ws, const bcg_step_batch* b,
                          cudaStream_t st) {
  const int n = b->single_rows ? b->n_single : b->T;
  const int reach = l->window > 0 && l->window < b->max_context ? l->window + kGdPage - 1 : b->max_context;
  const int blocks = l->pool > 0 && b->max_context > l->window ? (b->max_context - l->window) / l->pool : 0;
  const int pages = (reach + kGdPage - 1) / kGdPage + (blocks + kGdPage - 1) / kGdPage;
  const int groups = l->kv_heads * ((l->heads / l->kv_heads + kGdHeads - 1) / kGdHeads);
  if (n > 65535 || groups > 65535) {
    set_last_error("bcg_grouped_attention", "too many single tokens or heads");
    return BCG_ERR_TOO_LARGE;
  }
  const dim3 grid(decode_cluster(n * groups, pages), n, groups);
  CUtensorMap km, vm;
  BCG_TRY(make_tmap_bf16_sw128(&km, l->cache, 1ll << 30, l->q_ld, l->q_ld, kGdPage));
  BCG_TRY(make_tmap_bf16_sw128(&vm, l->cache_v, 1ll << 30, l->v_ld, l->v_ld, kGdPage));
  const GroupedAttn a = attn_args(m, l, ws, b, b->single_rows);
#define BCG_GD(Q, V) \
  if (l->q_ld == Q && l->v_ld == V) return launch_decode<Q, V>(km, vm, a, grid, st)
  BCG_GD(64, 64);
  BCG_GD(64, 128);
  BCG_GD(64, 256);
  BCG_GD(128, 64);
  BCG_GD(128, 128);
  BCG_GD(128, 256);
  BCG_GD(192, 64);
  BCG_GD(192, 128);
  BCG_GD(192, 256);
  BCG_GD(256, 64);
  BCG_GD(256, 128);
  BCG_GD(256, 256);
#undef BCG_GD
  set_last_error("bcg_grouped_attention", "no decode kernel for this head size");
  return BCG_ERR_UNSUPPORTED;
}

// ------------------------------------------------------------------------------------------- prompts
static int grouped_prefill(const bcg_layer* l, const bcg_stack_ws* ws, const bcg_step_batch* b, cudaStream_t st) {
  CUtensorMap qm, km, vm;
  const long long q_cols = static_cast<long long>(l->heads) * l->q_ld;
  BCG_TRY(make_tmap_bf16_sw128(&qm, ws->q, b->T, q_cols, q_cols, kWaBM));
  BCG_TRY(make_tmap_bf16_sw128(&km, l->cache, 1ll << 30, l->q_ld, l->q_ld, kWaPage));
  BCG_TRY(make_tmap_bf16_sw128(&vm, l->cache_v, 1ll << 30, l->v_ld, l->v_ld, kWaPage));
  WindowAttn a = {};
  a.tiles = b->tiles;
  a.n_tiles = b->n_tiles;
  a.slopes = l->slopes;
  a.gates = l->gated ? ws->gates : nullptr;
  a.block_table = b->block_table;
  a.max_blocks = b->max_blocks;
  a.page_heads = l->kv_heads;
  a.group = l->heads / l->kv_heads;
  a.out = static_cast<__nv_bfloat16*>(ws->mix);
  a.out_ld = l->mix_ld;
  a.heads = l->heads;
  a.vdim = l->vdim;
  a.window = l->window;
  a.pooled = {l->pool, l->pool_col};
  a.v_cos_sin = l->v_rot_dims > 0 ? l->v_cos_sin : nullptr;
  a.v_rot_dims = l->v_rot_dims;
  a.scale_log2e = l->scale * kLog2e;
  return l->slopes ? window_attn<true, true>(l->q_ld, l->v_ld, qm, km, vm, a, st)
                   : window_attn_paged(l->q_ld, l->v_ld, qm, km, vm, a, st);
}

int grouped_attention(const bcg_stack* m, const bcg_stack_ws* ws, const bcg_step_batch* b, const bcg_layer* l, int mode,
                      cudaStream_t st) {
  if (l->slopes && (l->pool > 0 || l->v_rot_dims > 0)) {
    set_last_error("bcg_grouped_attention", "a distance bias does not come with pooled blocks or rotated values");
    return BCG_ERR_UNSUPPORTED;
  }
  const int n_single = b->single_rows ? b->n_single : (b->n_tiles > 0 ? 0 : b->T);
  const bool tensor = m->act_dtype == BCG_DT_BF16 && mode == 0 && m->page_size == kGdPage && padded_head(l->q_ld, l->v_ld);
  if (!tensor) return grouped_plain(m, l, ws, b, nullptr, b->T, st);
  if (b->n_tiles > 0) {
    // the prompt kernel stores 16 bytes at a time; without slopes it takes maxima in front of the scale
    if ((l->slopes || l->scale > 0.f) && l->vdim % 8 == 0 && l->mix_ld % 8 == 0) BCG_TRY(grouped_prefill(l, ws, b, st));
    else BCG_TRY(grouped_plain(m, l, ws, b, nullptr, b->T, st));   // single tokens are recomputed below: harmless
  }
  if (n_single > 0) BCG_TRY(grouped_decode(m, l, ws, b, st));
  return BCG_OK;
}

}  // namespace bcg
