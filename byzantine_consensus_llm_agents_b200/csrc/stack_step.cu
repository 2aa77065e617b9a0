// One step of a layer stack: whatever tokens the batch brings (whole prompts, portions, single decoded
// tokens, mixed), launched from C++ on one stream.  Generation, trace replay and the captured decode graph
// all go through stack_step; only the work lists differ.
#include "stack_common.cuh"
#include "kernels.h"

namespace bcg {

static int check_stack(const bcg_stack* m, const bcg_stack_ws* ws) {
  if (!m || !ws || m->n_layers <= 0 || m->d_model <= 0 || !m->embed || !m->lm_head ||
      !m->final_norm || !m->layers || !ws->residual || !ws->xn || !ws->proj || !ws->logits ||
      (m->act_dtype != BCG_DT_BF16 && m->act_dtype != BCG_DT_F32) || m->page_size <= 0) {
    set_last_error("bcg_stack", "incomplete model / workspace description");
    return BCG_ERR_ARG;
  }
  return BCG_OK;
}

// The tensor-core GEMM where TMA can address the operands, the CUDA-core one otherwise (and for fp32).
static bool tensor_gemm(int act_dtype, int M, int N, int K) {
  return act_dtype == BCG_DT_BF16 && K % 8 == 0 && (M <= 128 || N % 16 == 0);
}
// Rows of up to 128 tokens split K into slabs (a function of N and K only); larger launches do not.
int stack_splits(int act_dtype, int M, int N, int K) {
  return tensor_gemm(act_dtype, M, N, K) && M <= 128 ? gemm_splits_for(M, N, K) : 1;
}
static int project(const bcg_stack* m, const void* x, const void* w, float* out, long long cap, int M, int N, int K,
                   int* splits, cudaStream_t st) {
  *splits = stack_splits(m->act_dtype, M, N, K);
  if (static_cast<long long>(*splits) * M * N > cap) {
    set_last_error("bcg_stack_step", "projection scratch too small");
    return BCG_ERR_TOO_LARGE;
  }
  if (tensor_gemm(m->act_dtype, M, N, K))
    return gemm_bf16_tn(x, w, out, M, N, K, K, K, N, BCG_EPI_F32, *splits, launch_flags() & BCG_GEMM_PDL, st);
  return gemm_any(x, m->act_dtype, w, out, M, N, K, K, K, N, st);
}

struct FlagScope {
  int saved;
  explicit FlagScope(int f) : saved(launch_flags()) { launch_flags() = f; }
  ~FlagScope() { launch_flags() = saved; }
};

// Latent attention of one layer over the step's queries; `gathered` remembers whose cache rows ws->latents holds.
static int latent_mix(const bcg_stack* m, const bcg_stack_ws* ws, const bcg_step_batch* b, const bcg_layer* l,
                     int mode, const void** gathered, cudaStream_t st) {
  const int n_single = b->single_rows ? b->n_single : (b->n_tiles > 0 ? 0 : b->T);
  const bool bf16 = m->act_dtype == BCG_DT_BF16 && mode == 0;
  const bool fast_single = bf16 && latent_decode_ok(l), fast_tiles = bf16 && latent_prefill_ok(l);
  if (!fast_single && !fast_tiles) return latent_plain(l, ws->q, ws->mix, b, nullptr, b->T, m->page_size, m->act_dtype, st);
  if (b->n_tiles > 0) {
    if (fast_tiles) {
      if (b->n_gather > ws->K_max || !ws->latents || !ws->expanded) {
        set_last_error("bcg_latent_attention", "gathered keys exceed the workspace");
        return BCG_ERR_TOO_LARGE;
      }
      if (*gathered != l->cache) {
        BCG_TRY(latent_gather(l->cache, b->gather, ws->latents, b->n_gather, l->kv_rank + l->rot_dim, st));
        *gathered = l->cache;
      }
      BCG_TRY(latent_prefill(l, ws, b, st));
    } else {   // single tokens are recomputed here too, which is harmless
      BCG_TRY(latent_plain(l, ws->q, ws->mix, b, nullptr, b->T, m->page_size, m->act_dtype, st));
    }
  }
  if (n_single > 0) {
    if (fast_single) BCG_TRY(latent_decode(l, ws, b, m->page_size, st));
    else BCG_TRY(latent_plain(l, ws->q, ws->mix, b, b->single_rows, n_single, m->page_size, m->act_dtype, st));
  }
  return BCG_OK;
}

int latent_attention(const bcg_stack* m, const bcg_stack_ws* ws, const bcg_step_batch* b, int layer, int mode,
                     cudaStream_t st) {
  BCG_TRY(check_stack(m, ws));
  if (!b || layer < 0 || layer >= m->n_layers || m->layers[layer].mixer != BCG_MIXER_LATENT_ATTN) {
    set_last_error("bcg_latent_attention", "not a latent attention layer");
    return BCG_ERR_ARG;
  }
  const void* gathered = nullptr;
  return latent_mix(m, ws, b, &m->layers[layer], mode, &gathered, st);
}

static const bcg_layer* layer_of(const bcg_stack* m, int layer, bool fits, const char* what) {
  if (!fits || layer < 0 || layer >= m->n_layers || m->layers[layer].mixer != BCG_MIXER_GROUPED_ATTN) {
    set_last_error(what, "not a grouped attention layer");
    return nullptr;
  }
  return &m->layers[layer];
}

int grouped_in_step(const bcg_stack* m, const bcg_stack_ws* ws, const bcg_step_batch* b, int layer, int n_partials,
                    long long pstride, long long ld, int with_act, cudaStream_t st) {
  BCG_TRY(check_stack(m, ws));
  const bcg_layer* l = layer_of(m, layer, b && b->T > 0 && b->T <= ws->T_max && n_partials > 0, "bcg_grouped_in");
  return l ? grouped_in(m, l, ws, b, n_partials, pstride, ld, with_act != 0, st) : static_cast<int>(BCG_ERR_ARG);
}

int grouped_attention_step(const bcg_stack* m, const bcg_stack_ws* ws, const bcg_step_batch* b, int layer, int mode,
                           cudaStream_t st) {
  BCG_TRY(check_stack(m, ws));
  const bcg_layer* l = layer_of(m, layer, b && b->T > 0 && b->T <= ws->T_max, "bcg_grouped_attention");
  return l ? grouped_attention(m, ws, b, l, mode, st) : static_cast<int>(BCG_ERR_ARG);
}

static const bcg_layer* expert_layer(const bcg_stack* m, int layer, bool fits) {
  if (!fits || layer < 0 || layer >= m->n_layers || m->layers[layer].experts <= 0) {
    set_last_error("bcg_experts", "the layer has no experts, or a bad batch");
    return nullptr;
  }
  return &m->layers[layer];
}

int experts_step(const bcg_stack* m, const bcg_stack_ws* ws, int layer, int T, int* splits, cudaStream_t st) {
  BCG_TRY(check_stack(m, ws));
  const bcg_layer* l = expert_layer(m, layer, T > 0 && T <= ws->T_max && splits);
  return l ? experts(m, l, ws, T, splits, st) : static_cast<int>(BCG_ERR_ARG);
}

int expert_in_step(const bcg_stack* m, const bcg_stack_ws* ws, int layer, int T, int n_partials, long long pstride, long long ld,
                   int with_act, cudaStream_t st) {
  BCG_TRY(check_stack(m, ws));
  const bcg_layer* l = expert_layer(m, layer, T > 0 && T <= ws->T_max && n_partials > 0);
  return l ? expert_in(m, l, ws, T, n_partials, pstride, ld, with_act != 0, st) : static_cast<int>(BCG_ERR_ARG);
}

// A parallel layer: attention and feed-forward read one norm, their outputs meet in one residual addition.  The
// input projection holds q | k | v (| router) and, behind them, a dense feed-forward's up rows; attention output and
// activations lie side by side in ws->mix, so that one product applies both output matrices.
static int parallel_layer(const bcg_stack* m, const bcg_stack_ws* ws, const bcg_step_batch* b, const bcg_layer* l,
                          const float* next, cudaStream_t st) {
  const int T = b->T, d = m->d_model, dt = m->act_dtype;
  const size_t size = dt == BCG_DT_F32 ? 4 : 2;
  int s = 1;
  // long launches: the squared relu is the up product's epilogue
  const int n_up = l->n_in - l->n_qkv;
  const bool apart = l->ff > 0 && T > 128 && tensor_gemm(dt, T, n_up, d) && tensor_gemm(dt, T, l->n_qkv, d);
  const int n_in = apart ? l->n_qkv : l->n_in;
  BCG_TRY(project(m, ws->xn, l->w_in, ws->proj, ws->proj_floats, T, n_in, d, &s, st));
  if (apart)
    BCG_TRY(gemm_bf16_tn(ws->xn, static_cast<const char*>(l->w_in) + static_cast<size_t>(l->n_qkv) * d * 2,
                         static_cast<char*>(ws->mix) + l->act_col * size, T, n_up, d, d, d, l->mix_ld, BCG_EPI_RELU2, 1,
                         launch_flags() & BCG_GEMM_PDL, st));
  BCG_TRY(grouped_in(m, l, ws, b, s, static_cast<long long>(T) * n_in, n_in, !apart, st));
  NormExtra extra;
  extra.bias = l->out_bias;
  if (l->experts > 0) {
    BCG_TRY(experts(m, l, ws, T, &extra.n_partials, st));
    extra.rows = ws->moe_out;
    extra.index = ws->moe_row;
    extra.per_row = l->top;
    extra.partial_stride = static_cast<long long>(T) * l->top * d;
  }
  BCG_TRY(grouped_attention(m, ws, b, l, 0, st));
  BCG_TRY(project(m, ws->mix, l->w_out, ws->proj, ws->proj_floats, T, d, l->mix_ld, &s, st));
  return sandwich_norm(ws->residual, ws->proj, s, static_cast<long long>(T) * d, nullptr, next, ws->xn, dt, T, d, m->eps,
                       extra, st);
}

// Gate and up products with their unit: in the GEMM's epilogue where K is not split, else behind the slabs.
static int glu_up(const bcg_stack* m, const bcg_stack_ws* ws, const bcg_layer* l, int T, cudaStream_t st) {
  const int n = 2 * l->ff, d = m->d_model, unit = l->ff_kind == BCG_FF_GELU_GLU ? BCG_EPI_GELU_GLU : BCG_EPI_GLU;
  int s = stack_splits(m->act_dtype, T, n, d);
  if (s == 1 && tensor_gemm(m->act_dtype, T, n, d))
    return gemm_bf16_glu(ws->xn, l->w_up, ws->act, T, n, d, unit, l->glu_limit, l->glu_alpha, launch_flags() & BCG_GEMM_PDL, st);
  BCG_TRY(project(m, ws->xn, l->w_up, ws->proj, ws->proj_floats, T, n, d, &s, st));
  return unit_rows(ws->proj, s, static_cast<long long>(T) * n, nullptr, ws->act, m->act_dtype, T, l->ff, unit, l->glu_limit,
                   l->glu_alpha, st);
}

// Router, experts and the shared expert of a layer that is not parallel, up to their sum with the stream: the router's rows and
// the shared expert's first matrix are one product; *splits slabs of the shared expert's output are left in ws->proj (0: none).
static int expert_ff(const bcg_stack* m, const bcg_stack_ws* ws, const bcg_layer* l, int T, NormExtra* extra, int* splits,
                     cudaStream_t st) {
  const int d = m->d_model, dt = m->act_dtype, n_all = l->n_router + l->ff;
  // long launches: the gelu is the shared product's epilogue
  const bool apart = l->ff > 0 && T > 128 && tensor_gemm(dt, T, l->ff, d) && tensor_gemm(dt, T, l->n_router, d);
  const int n = apart ? l->n_router : n_all;
  int s = 1;
  BCG_TRY(project(m, ws->xn, l->w_up, ws->proj, ws->proj_floats, T, n, d, &s, st));
  BCG_TRY(expert_in(m, l, ws, T, s, static_cast<long long>(T) * n, n, !apart, st));
  if (apart)
    BCG_TRY(gemm_bf16_gelu(ws->xn, static_cast<const char*>(l->w_up) + static_cast<size_t>(l->n_router) * d * 2, ws->act, T, l->ff, d,
                           launch_flags() & BCG_GEMM_PDL, st));
  BCG_TRY(experts(m, l, ws, T, &extra->n_partials, st));
  extra->rows = ws->moe_out;
  extra->index = ws->moe_row;
  extra->weight = ws->moe_weight;
  extra->per_row = l->top;
  extra->partial_stride = static_cast<long long>(T) * l->top * d;
  *splits = 0;
  return l->ff > 0 ? project(m, ws->act, l->w_down, ws->proj, ws->proj_floats, T, d, l->ff, splits, st) : static_cast<int>(BCG_OK);
}

// Long launches: queries, keys, values and output gates leave their product as the activations that the matrix memory reads; the
// input and forget gates, a product of their own, stay fp32.
static bool memory_splits(const bcg_stack* m, const bcg_layer* l, int T) {
  return m->act_dtype == BCG_DT_BF16 && T > 128 && l->dim % 8 == 0 && l->vdim % 8 == 0 && tensor_gemm(m->act_dtype, T, l->gate_col, m->d_model) &&
         tensor_gemm(m->act_dtype, T, l->n_in - l->gate_col, m->d_model);
}
static int memory_products(const bcg_stack* m, const bcg_stack_ws* ws, const bcg_layer* l, int T, cudaStream_t st) {
  const int d = m->d_model, n = l->gate_col;
  int s;
  if (!ws->ssm_x) {
    set_last_error("bcg_stack_step", "incomplete workspace");
    return BCG_ERR_ARG;
  }
  BCG_TRY(gemm_bf16_tn(ws->xn, l->w_in, ws->ssm_x, T, n, d, d, d, n, BCG_EPI_BF16, 1, launch_flags() & BCG_GEMM_PDL, st));
  return project(m, ws->xn, static_cast<const char*>(l->w_in) + static_cast<size_t>(n) * d * 2, ws->proj, ws->proj_floats, T, l->n_in - n, d,
                 &s, st);
}

int matrix_memory_step(const bcg_stack* m, const bcg_stack_ws* ws, const bcg_step_batch* b, int layer, int n_partials,
                       long long pstride, long long ld, int mode, cudaStream_t st) {
  BCG_TRY(check_stack(m, ws));
  if (!b || b->T <= 0 || b->T > ws->T_max || n_partials < 1 || layer < 0 || layer >= m->n_layers ||
      m->layers[layer].mixer != BCG_MIXER_MATRIX_MEMORY) {
    set_last_error("bcg_matrix_memory", "not a matrix memory layer, or a bad batch");
    return BCG_ERR_ARG;
  }
  const bcg_layer* l = &m->layers[layer];
  if (mode == 2 && (l->dim % 8 || l->vdim % 8 || n_partials != 1)) {
    set_last_error("bcg_matrix_memory", "operands that are activations already: heads in multiples of 8 columns, one slab of gates");
    return BCG_ERR_ARG;
  }
  return matrix_memory(m, l, ws, b, n_partials, pstride, ld, mode == 2 ? 0 : mode, mode == 2, st);
}

int state_space_step(const bcg_stack* m, const bcg_stack_ws* ws, const bcg_step_batch* b, int layer, int n_partials,
                     long long pstride, long long ld, int mode, cudaStream_t st) {
  BCG_TRY(check_stack(m, ws));
  if (!b || b->T <= 0 || b->T > ws->T_max || n_partials < 1 || layer < 0 || layer >= m->n_layers ||
      m->layers[layer].ssm_heads <= 0) {
    set_last_error("bcg_state_space", "not a state-space layer, or a bad batch");
    return BCG_ERR_ARG;
  }
  return state_space(m, &m->layers[layer], ws, b, n_partials, pstride, ld, mode, st);
}

int stack_step(const bcg_stack* m, const bcg_stack_ws* ws, const bcg_step_batch* b, cudaStream_t st) {
  BCG_TRY(check_stack(m, ws));
  if (!b || b->T <= 0 || b->T > ws->T_max || b->n_seqs <= 0 || !b->ids || !b->positions || !b->slot_map ||
      !b->block_table || (!b->row_seq != !b->seq_start)) {
    set_last_error("bcg_stack_step", "bad batch (T within the workspace, row_seq and seq_start together)");
    return BCG_ERR_ARG;
  }
  FlagScope scope(b->flags & BCG_GEMM_PDL);
  const int T = b->T, d = m->d_model, dt = m->act_dtype;
  const void* gathered = nullptr;
  const EmbedArgs embed = {b->ids, b->positions, static_cast<const __nv_bfloat16*>(m->embed), m->embed_scale,
                           static_cast<const __nv_bfloat16*>(m->pos_embed), m->n_pos, m->pos_turns, ws->moe_counts,
                           ws->moe_counts_n, m->embed_norm};
  BCG_TRY(embed_norm(embed, m->layers[0].norm1, ws->residual, ws->xn, dt, T, d, m->eps, st));
  for (int i = 0; i < m->n_layers; ++i) {
    const bcg_layer* l = &m->layers[i];
    const float* next = i + 1 < m->n_layers ? m->layers[i + 1].norm1 : m->final_norm;
    if (l->parallel) {
      if (l->mixer != BCG_MIXER_GROUPED_ATTN) {
        set_last_error("bcg_stack_step", "parallel layers have grouped attention");
        return BCG_ERR_UNSUPPORTED;
      }
      BCG_TRY(parallel_layer(m, ws, b, l, next, st));
      continue;
    }
    int s = 1, mix_out = 0;
    const bool split = l->mixer == BCG_MIXER_MATRIX_MEMORY && T != b->n_seqs && memory_splits(m, l, T);
    if (split) BCG_TRY(memory_products(m, ws, l, T, st));
    else BCG_TRY(project(m, ws->xn, l->w_in, ws->proj, ws->proj_floats, T, l->n_in, d, &s, st));
    const long long in_stride = static_cast<long long>(T) * l->n_in;
    if (l->mixer == BCG_MIXER_LATENT_ATTN) {
      mix_out = l->heads * l->vdim;
      BCG_TRY(latent_qkv(l, ws->proj, s, in_stride, b->positions, b->slot_map, ws->q, dt, T, m->eps, st));
      if (gathered == l->cache && l->owns_cache) gathered = nullptr;
      BCG_TRY(latent_mix(m, ws, b, l, 0, &gathered, st));
    } else if (l->mixer == BCG_MIXER_GENERAL_DELTA) {
      mix_out = l->heads * l->dim;
      int sd = 1;
      BCG_TRY(delta_low(l, ws->proj, s, in_stride, ws->low, dt, T, st));
      BCG_TRY(project(m, ws->low, l->w_decay, ws->decay, ws->decay_floats, T, mix_out, l->decay_rank, &sd, st));
      BCG_TRY(delta_scan(l, ws->proj, s, in_stride, l->n_in, ws->decay, sd, static_cast<long long>(T) * mix_out,
                         b->positions, b->slot_map, b->seq_start, b->state_slots, b->n_seqs, T == b->n_seqs, ws->mix,
                         dt, m->eps, st));
    } else if (l->mixer == BCG_MIXER_GROUPED_ATTN || (l->mixer == BCG_MIXER_STATE_SPACE && l->ssm_heads > 0)) {
      // attention and a state-space mixer, or one of them, behind one input projection; their outputs lie side by side
      mix_out = l->mix_ld;
      if (l->mixer == BCG_MIXER_GROUPED_ATTN) {
        BCG_TRY(grouped_in(m, l, ws, b, s, in_stride, l->n_in, false, st));
        BCG_TRY(grouped_attention(m, ws, b, l, 0, st));
      }
      if (l->ssm_heads > 0) BCG_TRY(state_space(m, l, ws, b, s, in_stride, l->n_in, 0, st));
    } else if (l->mixer == BCG_MIXER_MATRIX_MEMORY) {
      mix_out = l->mix_ld;
      BCG_TRY(matrix_memory(m, l, ws, b, s, in_stride, split ? l->n_in - l->gate_col : l->n_in, 0, split, st));
    } else {
      set_last_error("bcg_stack_step", "unknown mixer");
      return BCG_ERR_UNSUPPORTED;
    }
    BCG_TRY(project(m, ws->mix, l->w_out, ws->proj, ws->proj_floats, T, d, mix_out, &s, st));
    NormExtra extra;
    extra.bias = l->out_bias;
    const bool has_ff = l->ff > 0 || l->ff_kind == BCG_FF_EXPERTS;
    BCG_TRY(sandwich_norm(ws->residual, ws->proj, s, static_cast<long long>(T) * d, l->norm1b, has_ff ? l->norm2 : next,
                          ws->xn, dt, T, d, m->eps, extra, st));
    if (l->ff_kind == BCG_FF_EXPERTS) {
      NormExtra rows;
      BCG_TRY(expert_ff(m, ws, l, T, &rows, &s, st));
      BCG_TRY(sandwich_norm(ws->residual, s ? ws->proj : nullptr, s ? s : 1, static_cast<long long>(T) * d, l->norm2b, next, ws->xn, dt,
                            T, d, m->eps, rows, st));
    } else if (l->ff) {
      if (l->ff_kind == BCG_FF_CLAMPED_GLU || l->ff_kind == BCG_FF_GELU_GLU) {
        BCG_TRY(glu_up(m, ws, l, T, st));
      } else {
        BCG_TRY(project(m, ws->xn, l->w_up, ws->proj, ws->proj_floats, T, l->ff, d, &s, st));
        BCG_TRY(poly_norm(ws->proj, s, static_cast<long long>(T) * l->ff, l->act_coef, ws->act, dt, T, l->ff, m->eps, st));
      }
      BCG_TRY(project(m, ws->act, l->w_down, ws->proj, ws->proj_floats, T, d, l->ff, &s, st));
      BCG_TRY(sandwich_norm(ws->residual, ws->proj, s, static_cast<long long>(T) * d, l->norm2b, next, ws->xn, dt, T, d,
                            m->eps, {}, st));
    }
  }
  return BCG_OK;
}

int stack_head(const bcg_stack* m, const bcg_stack_ws* ws, const int* rows, int n, int row0, int flags,
               cudaStream_t st) {
  BCG_TRY(check_stack(m, ws));
  if (n <= 0 || row0 < 0 || row0 + n > ws->B_max || (rows && !ws->xn_rows)) {
    set_last_error("bcg_stack_head", "rows exceed the logits buffer");
    return BCG_ERR_TOO_LARGE;
  }
  FlagScope scope(flags & BCG_GEMM_PDL);
  const void* x = ws->xn;
  if (rows) {
    BCG_TRY(rows_norm(ws->residual, rows, m->final_norm, ws->xn_rows, m->act_dtype, n, m->d_model, m->eps, st));
    x = ws->xn_rows;
  }
  float* out = ws->logits + static_cast<long long>(row0) * m->vocab_ld;
  const int d = m->d_model, V = m->vocab_ld;
  if (tensor_gemm(m->act_dtype, n, V, d))
    return gemm_bf16_tn(x, m->lm_head, out, n, V, d, d, d, V, BCG_EPI_F32, 1, launch_flags() & BCG_GEMM_PDL, st);
  return gemm_any(x, m->act_dtype, m->lm_head, out, n, V, d, d, d, V, st);
}

}  // namespace bcg
