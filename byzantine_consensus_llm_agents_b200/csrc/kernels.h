// Internal C++ declarations shared by the .cu files; the public C ABI is include/bcg_b200.h.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include <cuda.h>

#include "../../include/bcg_b200.h"

namespace bcg {

int gemm_bf16_tn(const void* X, const void* W, void* out, int M, int N, int K, long long ldx,
                 long long ldw, long long ld_out, int epi, int splits, int flags,
                 cudaStream_t stream);
int gemm_bf16_tn_fused(const void* X, const void* W, void* out, int M, int N, int K, long long ldx,
                       long long ldw, long long ld_out, int epi, int splits, int flags,
                       const bcg_gemm_fusion* fusion, cudaStream_t stream);
// epilogue BCG_EPI_GLU or BCG_EPI_GELU_GLU: W rows interleaved [16 gate | 16 up], out bf16 [M, N / 2]
int gemm_bf16_glu(const void* X, const void* W, void* out, int M, int N, int K, int epi, float limit, float alpha, int flags,
                  cudaStream_t stream);
// epilogue BCG_EPI_GELU: out bf16 [M, N], M > 128, N % 16 == 0
int gemm_bf16_gelu(const void* X, const void* W, void* out, int M, int N, int K, int flags, cudaStream_t stream);
int gemm_splits_for(int M, int N, int K);
// Rows sorted by group (mixture of experts).  Internal epilogues: BCG_EPI_GLU, columns interleaved [16 gate | 16 up], each
// row's accumulators times its weight (groups only), clamped gated unit, bf16 [rows, N / 2]; BCG_EPI_GELU_GLU, the same columns,
// gelu(gate) * up with gelu's tanh form (no groups); BCG_EPI_GELU, gelu's erf form, bf16 [rows, N]
constexpr int BCG_EPI_GLU = 16, BCG_EPI_GELU_GLU = 17, BCG_EPI_GELU = 18;
constexpr int kMaxGroups = 512;
struct GemmGroups {
  const int* counts;         // device [n_groups]: rows of every group
  int n_groups, max_rows;    // max_rows: host-side bound on the rows of one group
  const float* row_weight;   // [rows]
  float glu_limit, glu_alpha;
};
int gemm_grouped(const void* X, const void* W, void* out, int rows, int N, int K, int epi, int splits, const GemmGroups& g,
                 cudaStream_t stream);
int gemm_any_grouped(const void* X, int x_dtype, const void* W, float* out, int N, int K, const GemmGroups& g,
                     cudaStream_t stream);
// Prefill shapes on CTA pairs (tcgen05.mma.cta_group::2); BCG_ERR_UNSUPPORTED = not a shape for it
int gemm2sm_bf16_tn(const void* X, const void* W, void* out, int M, int N, int K, long long ldx, long long ldw,
                    long long ld_out, int epi, float glu_limit, float glu_alpha, cudaStream_t stream);
// TMA descriptor of a row-major bf16 matrix (rows x K, pitch ld elements): boxes of box_rows x 64
// elements land in shared memory 128B-swizzled, out-of-bounds elements read as zero.
int make_tmap_bf16_sw128(CUtensorMap* m, const void* ptr, long long rows, long long K, long long ld,
                         int box_rows);

int embed_rmsnorm(const int* ids, const void* embed, const float* w, float* residual, void* xn,
                  int T, int d, float eps, cudaStream_t stream);
int add_norm_stats(float* residual, const void* delta, int delta_is_f32, int n_partials,
                   long long partial_stride, const float* w, void* xn, float* sumsq, int T, int d,
                   cudaStream_t stream);
int add_rmsnorm(float* residual, const void* delta, int delta_is_f32, int n_partials,
                long long partial_stride, const float* w, void* xn, const int* src_rows, int T,
                int d, float eps, cudaStream_t stream);
int qknorm_rope_kvwrite(const void* qkv, int qkv_is_f32, int n_partials, long long partial_stride,
                        long long ld_qkv, const float* q_norm_w, const float* k_norm_w,
                        const float* cos_sin, const int* positions, const int* slot_map,
                        void* q_out, void* kv_cache, int T, int n_heads, int n_kv_heads,
                        int page_size, float eps, cudaStream_t stream);
int swiglu_reduce(const float* partials, int n_partials, long long partial_stride, void* act,
                  int T, int two_f, cudaStream_t stream);

int decode_attn_paged(const void* q, const void* kv_cache, const int* block_table,
                      int max_blocks_per_seq, const int* seq_lens, void* out, float* scratch_o,
                      float* scratch_ml, int* counters, int B, int n_heads, int n_kv_heads,
                      int page_size, int max_splits, float scale, cudaStream_t stream);
int decode_attn_paged_qkv(const float* qkv, int n_partials, long long partial_stride, long long ld_qkv,
                          const float* q_norm_w, const float* k_norm_w, const float* cos_sin,
                          const int* positions, const int* slot_map, float eps, void* kv_cache,
                          const int* block_table, int max_blocks_per_seq, const int* seq_lens, void* out,
                          float* scratch_o, float* scratch_ml, int* counters, int B, int n_heads,
                          int n_kv_heads, int page_size, int max_splits, float scale,
                          cudaStream_t stream);
int decode_attn_paged_static(const void* q, const void* kv_cache, const int* block_table,
                             int max_blocks_per_seq, const int* seq_lens, void* out, int B,
                             int n_heads, int n_kv_heads, int page_size, int max_splits, float scale,
                             cudaStream_t stream);
int prefill_attn_paged(const void* q, const void* kv_cache, const int* block_table,
                       int max_blocks_per_seq, const int* tile_info, int n_tiles, void* out,
                       int n_q_rows, int n_heads, int n_kv_heads, int page_size, float scale,
                       cudaStream_t stream);

int mask_sample(const bcg_sampler_args* a, cudaStream_t stream);

// Further summands of sandwich_norm's delta: a bias, and `per_row` rows of a second set of slabs.
struct NormExtra {
  const float* bias = nullptr;      // [d]
  const float* rows = nullptr;      // [n_partials][any][d]
  const int* index = nullptr;       // [T][per_row] rows of it
  const float* weight = nullptr;    // [T][per_row] their factors, or NULL
  int per_row = 0, n_partials = 1;
  long long partial_stride = 0;
};
// layer stacks (stack_*.cu, latent_*.cu, grouped_*.cu, delta_scan.cu, state_space.cu, moe.cu, gemm_simt.cu); act_dtype = BCG_DT_*
// What the embedding kernel adds and multiplies; zero[0..n_zero) is set to zero on the way.
struct EmbedArgs {
  const int *ids, *positions;
  const __nv_bfloat16* embed;
  float scale;
  const __nv_bfloat16* pos_embed;   // [n_pos, d] or NULL
  int n_pos;
  const double* pos_turns;          // [(d + 1) / 2] turns per position, or NULL: sin, cos in turn
  int* zero;
  int n_zero;
  const float* norm;                // [d] weight of a norm of the embedding, or NULL
};
int embed_norm(const EmbedArgs& a, const float* w, float* residual, void* xn, int act_dtype, int T, int d, float eps,
               cudaStream_t stream);
int rows_norm(const float* residual, const int* rows, const float* w, void* xn, int act_dtype, int n, int d,
              float eps, cudaStream_t stream);
int sandwich_norm(float* residual, const float* delta, int n_partials, long long partial_stride,
                  const float* w_post, const float* w_next, void* xn, int act_dtype, int T, int d, float eps,
                  const NormExtra& extra, cudaStream_t stream);
int poly_norm(const float* z, int n_partials, long long partial_stride, const float* coef, void* out, int act_dtype,
              int T, int ff, float eps, cudaStream_t stream);
int gemm_any(const void* X, int x_dtype, const void* W, float* out, int M, int N, int K, long long ldx,
             long long ldw, long long ldo, cudaStream_t stream);
int latent_qkv(const bcg_layer* l, const float* proj, int n_partials, long long pstride, const int* positions,
               const int* slot_map, void* q, int act_dtype, int T, float eps, cudaStream_t stream);
int latent_plain(const bcg_layer* l, const void* q, void* out, const bcg_step_batch* b, const int* rows, int n,
                 int page_size, int act_dtype, cudaStream_t stream);
bool latent_decode_ok(const bcg_layer* l);
int latent_decode(const bcg_layer* l, const bcg_stack_ws* ws, const bcg_step_batch* b, int page_size,
                  cudaStream_t stream);
int latent_gather(const void* cache, const int* slots, void* out, int n, int crow, cudaStream_t stream);
bool latent_prefill_ok(const bcg_layer* l);
int latent_prefill(const bcg_layer* l, const bcg_stack_ws* ws, const bcg_step_batch* b, cudaStream_t stream);
int delta_low(const bcg_layer* l, const float* proj, int n_partials, long long pstride, void* low, int act_dtype,
              int T, cudaStream_t stream);
int delta_scan(const bcg_layer* l, const float* proj, int n_partials, long long pstride, long long ld,
               const float* decay, int d_partials, long long dstride, const int* positions, const int* slot_map,
               const int* seq_start, const int* state_slots, int n_seqs, int one_token, void* out, int act_dtype,
               float eps, cudaStream_t stream);
int latent_attention(const bcg_stack* m, const bcg_stack_ws* ws, const bcg_step_batch* b, int layer, int mode,
                     cudaStream_t stream);
int grouped_in(const bcg_stack* m, const bcg_layer* l, const bcg_stack_ws* ws, const bcg_step_batch* b, int n_partials,
               long long pstride, long long ld, bool with_act, cudaStream_t stream);
int grouped_attention(const bcg_stack* m, const bcg_stack_ws* ws, const bcg_step_batch* b, const bcg_layer* l, int mode,
                      cudaStream_t stream);
// ws->xn through the layer's experts into ws->moe_out (*splits slabs), rows ws->moe_row
int experts(const bcg_stack* m, const bcg_layer* l, const bcg_stack_ws* ws, int T, int* splits, cudaStream_t stream);
int moe_splits(int T, int top, int N, int K);
// A feed-forward's unit (BCG_EPI_GLU, BCG_EPI_GELU_GLU or BCG_EPI_GELU) of slabs [rows][2 * ff_ld] (16 gate | 16 up) or
// [rows][ff_ld]; row_weight (NULL: 1) scales its input
int unit_rows(const float* z, int n_partials, long long pstride, const float* row_weight, void* out, int act_dtype, int rows,
              int ff_ld, int unit, float limit, float alpha, cudaStream_t stream);
// Routing of a layer with experts that is not parallel (logits are the first columns of ws->proj) and, with_act, gelu of the
// columns behind them into ws->act
int expert_in(const bcg_stack* m, const bcg_layer* l, const bcg_stack_ws* ws, int T, int n_partials, long long pstride, long long ld,
              bool with_act, cudaStream_t stream);
int expert_in_step(const bcg_stack* m, const bcg_stack_ws* ws, int layer, int T, int n_partials, long long pstride, long long ld,
                   int with_act, cudaStream_t stream);
// split: the operands are activations in ws->ssm_x already, ws->proj has just the gates
int matrix_memory(const bcg_stack* m, const bcg_layer* l, const bcg_stack_ws* ws, const bcg_step_batch* b, int n_partials,
                  long long pstride, long long ld, int mode, bool split, cudaStream_t stream);
int matrix_memory_step(const bcg_stack* m, const bcg_stack_ws* ws, const bcg_step_batch* b, int layer, int n_partials,
                       long long pstride, long long ld, int mode, cudaStream_t stream);
struct WindowAttn;
// paged prompt attention without a distance bias (grouped_prefill.cu)
int window_attn_paged(int q_ld, int v_ld, const CUtensorMap& qm, const CUtensorMap& km, const CUtensorMap& vm,
                      const WindowAttn& a, cudaStream_t stream);
int state_space(const bcg_stack* m, const bcg_layer* l, const bcg_stack_ws* ws, const bcg_step_batch* b, int n_partials,
                long long pstride, long long ld, int mode, cudaStream_t stream);
int state_space_step(const bcg_stack* m, const bcg_stack_ws* ws, const bcg_step_batch* b, int layer, int n_partials,
                     long long pstride, long long ld, int mode, cudaStream_t stream);
int grouped_in_step(const bcg_stack* m, const bcg_stack_ws* ws, const bcg_step_batch* b, int layer, int n_partials,
                    long long pstride, long long ld, int with_act, cudaStream_t stream);
int grouped_attention_step(const bcg_stack* m, const bcg_stack_ws* ws, const bcg_step_batch* b, int layer, int mode,
                           cudaStream_t stream);
int experts_step(const bcg_stack* m, const bcg_stack_ws* ws, int layer, int T, int* splits, cudaStream_t stream);
int stack_step(const bcg_stack* m, const bcg_stack_ws* ws, const bcg_step_batch* b, cudaStream_t stream);
int stack_head(const bcg_stack* m, const bcg_stack_ws* ws, const int* rows, int n, int row0, int flags,
               cudaStream_t stream);

// tensor parallelism (tp_comm.cu)
int tp_unique_id(void* out128);
int tp_init(const void* id128, int rank, int size);
int tp_shutdown();
int tp_size();
int tp_rank();
int tp_all_reduce_f32(float* buf, long long count, cudaStream_t stream);
int tp_all_gather_f32(const float* send, float* recv, long long count, cudaStream_t stream);
int tp_symm_create(long long bytes, void* handle_out64, void** local_ptr);
int tp_symm_open(const void* handles, int rank, int size);
void* tp_symm_local();
void* const* tp_symm_peers_device();
long long tp_symm_bytes();
// fused cross-GPU reduction + residual add + RMSNorm statistics over peer memory (tp_reduce_norm.cu)
int tp_add_norm_stats(float* residual, const float* partials, int n_partials, long long partial_stride,
                      const float* w, void* xn, float* sumsq, int slot, long long region_floats, int T,
                      int d, cudaStream_t stream);
long long tp_symm_flag_floats();

}  // namespace bcg
