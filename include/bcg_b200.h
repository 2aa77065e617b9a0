/* bcg_b200.h — C ABI of the B200-native agent-step engine kernels.
 *
 * The reference (leorugli/byzantine-consensus-llm-agents) has no FFI of its own: its hot
 * path is `VLLMAgent.generate_json / batch_generate_json`
 * (byzantine_consensus_game/vllm_agent.py:294-455), which hands everything to
 * `vllm.LLM.generate` (vllm_agent.py:195,331,430,502).  The Python class in
 * byzantine_consensus_llm_agents_b200/vllm_agent.py replaces that module one-for-one; the
 * functions below are what that class binds (ctypes) in place of the third-party engine's
 * CUDA ops.  Each entry cites the engine op it stands in for.
 *
 * Conventions: plain pointers and sizes only; every pointer is DEVICE memory owned by the
 * caller unless the comment says host; `stream` is a cudaStream_t passed as void*; no entry
 * point allocates or frees device memory; return value 0 = ok, otherwise a BCG_ERR_* code
 * and bcg_last_error() holds a message.  Re-entrant per stream.  sm_100a only.
 */
#ifndef BCG_B200_H_
#define BCG_B200_H_

#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

#define BCG_ABI_VERSION 5

/* status codes */
#define BCG_STATUS_OK 0
#define BCG_STATUS_ARG 1
#define BCG_STATUS_CUDA 2
#define BCG_STATUS_UNSUPPORTED 3
#define BCG_STATUS_TOO_LARGE 4

/* GEMM epilogues */
#define BCG_EPI_BF16 0   /* out bf16 [M, ld_out]                                         */
#define BCG_EPI_F32 1    /* out fp32 [splits][M, ld_out] (split-K partials, or logits)   */
#define BCG_EPI_SWIGLU 2 /* W rows interleaved [16 gate | 16 up]; out bf16 [M, N/2]      */
#define BCG_EPI_RELU2 3  /* out bf16 [M, ld_out] = max(y, 0)^2 (M > 128, N % 16 == 0)    */
/* GEMM flags */
#define BCG_GEMM_PDL 1   /* programmatic dependent launch: weights prefetch before the wait */

int bcg_abi_version(void);
/* Last error message of the calling thread's most recent failing call (host string). */
const char* bcg_last_error(void);

/* Y[M,N] = X[M,K] · W[N,K]^T, bf16 inputs, fp32 accumulation on tcgen05 tensor cores with
 * TMEM accumulators and TMA-fed operands.  Stands in for the cuBLAS `F.linear` calls of
 * qkv_proj / o_proj / gate_up_proj (+ `_C.silu_and_mul`) / down_proj / lm_head
 * (vLLM model_executor/models/qwen3.py:145-162,216-236).
 * M <= 128 selects the weight-streaming (swap-AB, optional split-K) decode path.
 * ldx, ldw, ld_out are row pitches in elements.  splits > 1 requires BCG_EPI_F32 and an
 * `out` buffer of splits*M*ld_out floats; the consumer sums the partials in index order. */
int bcg_gemm_bf16_tn(const void* X, const void* W, void* out, int M, int N, int K, long long ldx,
                     long long ldw, long long ld_out, int epilogue, int splits, int flags,
                     void* stream);
/* Decode-only fusion of the `fused_add_rms_norm` that vLLM runs between two projections
 * (vLLM model_executor/layers/layernorm.py RMSNorm.forward_cuda with a residual;
 * models/qwen3.py:216-236 decoder layer) into the projections on either side of it, so that the
 * norm costs no kernel of its own.  M <= 128, N % 128 == 0, ld_out == N for the producer side.
 *   producer (red_counters != NULL; BCG_EPI_F32, splits <= 16): the work item that completes a
 *     128-column tile adds the split-K partials (index order) to red_residual, writes it back,
 *     writes red_xn = bf16(residual * red_w) — NOT yet divided by the row's RMS — and the tile's
 *     per-row sum of squares to red_sumsq[tile][128].  red_counters: N/128 ints, zero on entry,
 *     zero again on exit.
 *   consumer (scale_sumsq != NULL): X is such a red_xn; every output row m is multiplied by
 *     rsqrt(sum_t scale_sumsq[t][m] / scale_d + scale_eps) in the epilogue (tiles added in order).
 * Either half may be unused (NULL). */
typedef struct bcg_gemm_fusion {
  const float* scale_sumsq;
  int scale_tiles;
  int scale_d;
  float scale_eps;
  float* red_residual;
  const float* red_w;
  void* red_xn;
  float* red_sumsq;
  int* red_counters;
} bcg_gemm_fusion;
int bcg_gemm_bf16_tn_fused(const void* X, const void* W, void* out, int M, int N, int K,
                           long long ldx, long long ldw, long long ld_out, int epilogue, int splits,
                           int flags, const bcg_gemm_fusion* fusion, void* stream);
/* Split-K factor the engine uses for a decode GEMM of this shape (host helper, no GPU work). */
int bcg_gemm_splits_for(int M, int N, int K);

/* residual[t,:] = embed[ids[t],:] (fp32); xn[t,:] = rmsnorm(residual[t,:]) * w  (bf16).
 * Stands in for `F.embedding` + `_C.rms_norm`. */
int bcg_embed_rmsnorm(const int* ids, const void* embed, const float* w, float* residual, void* xn,
                      int T, int d, float eps, void* stream);

/* residual += delta; xn = rmsnorm(residual) * w.  delta is bf16 [T,d] (delta_is_f32 = 0) or
 * n_partials fp32 slabs [T,d] spaced partial_stride floats apart, summed in index order;
 * delta may be NULL.  If src_rows != NULL, output row i is computed from row src_rows[i] and
 * residual is not written (last-token gather in front of lm_head).
 * Stands in for `_C.fused_add_rms_norm`. */
int bcg_add_rmsnorm(float* residual, const void* delta, int delta_is_f32, int n_partials,
                    long long partial_stride, const float* w, void* xn, const int* src_rows, int T,
                    int d, float eps, void* stream);

/* Decode-only variant of bcg_add_rmsnorm with the 1/RMS factor deferred to the consuming GEMM:
 * residual += delta (same operand rules), xn = bf16(residual * w) — NOT divided by the RMS — and
 * sumsq[s * 128 + t] = sum of squares of segment s (of 8) of row t.  Pass `sumsq` as
 * bcg_gemm_fusion.scale_sumsq with scale_tiles = 8, scale_d = d to the projection that reads xn.
 * T <= 128.  Takes the row-wide reduction (a cluster barrier and a DSMEM exchange in
 * bcg_add_rmsnorm) off the critical path between two GEMMs.  Stands in for the same vllm op,
 * `_C.fused_add_rms_norm`, with its last multiply moved into the next projection. */
int bcg_add_norm_stats(float* residual, const void* delta, int delta_is_f32, int n_partials,
                       long long partial_stride, const float* w, void* xn, float* sumsq, int T, int d,
                       void* stream);

/* Per-head q/k RMSNorm (weights may be NULL: Mistral), rotate-half RoPE from a
 * [max_pos][128] fp32 table (cos[0..63] | sin[0..63]), q -> bf16 [T, n_heads*128], k/v ->
 * paged cache at slot_map[t] (slot = page*page_size + offset; negative = skip).
 * qkv is bf16 [T, ld_qkv] or fp32 split-K partials.  head_dim is 128.
 * KV cache layout (one layer): [page][2][n_kv_heads][page_size][128] bf16.
 * Stands in for `_C.rms_norm` on heads + `_C.rotary_embedding` + `reshape_and_cache_flash`
 * (SURVEY.md K4-K6). */
int bcg_qknorm_rope_kvwrite(const void* qkv, int qkv_is_f32, int n_partials,
                            long long partial_stride, long long ld_qkv, const float* q_norm_w,
                            const float* k_norm_w, const float* cos_sin, const int* positions,
                            const int* slot_map, void* q_out, void* kv_cache, int T, int n_heads,
                            int n_kv_heads, int page_size, float eps, void* stream);

/* act[t, j] = silu(gate) * up summed over fp32 split-K partials of the interleaved gate_up
 * GEMM (only needed when that GEMM ran with splits > 1).  Stands in for `_C.silu_and_mul`. */
int bcg_swiglu_reduce(const float* partials, int n_partials, long long partial_stride, void* act,
                      int T, int two_f, void* stream);

/* One query token per row over the paged KV cache (GQA, head_dim 128, page_size 16).
 * seq_lens[b] counts the current token.  scratch_o: B*n_heads*max_splits*128 floats;
 * scratch_ml: B*n_heads*max_splits*2 floats; chunk_counters: B*n_kv_heads int32 that must be
 * ZERO before the first call and that every call leaves zero again (keep them in a buffer of
 * their own: partial results written by a call of another shape must never land on them);
 * max_splits >= ceil(max seq_len / 256) — a longer row makes the kernel trap (the launch fails with
 * a CUDA error) rather than leave its output unwritten.
 * Stands in for the FlashInfer paged decode kernel vLLM dispatches on sm_100. */
int bcg_decode_attn_paged(const void* q, const void* kv_cache, const int* block_table,
                          int max_blocks_per_seq, const int* seq_lens, void* out, float* scratch_o,
                          float* scratch_ml, int* chunk_counters, int B, int n_heads, int n_kv_heads,
                          int page_size, int max_splits, float scale, void* stream);

/* bcg_qknorm_rope_kvwrite + bcg_decode_attn_paged in ONE launch (decode only): takes the qkv
 * projection's fp32 split-K slabs [n_partials][B, ld_qkv] (q heads | k heads | v heads) and the
 * RoPE / norm / slot arguments of bcg_qknorm_rope_kvwrite.  Every chunk CTA rebuilds its queries
 * itself; the CTA of a row's last chunk also builds the new token's K/V row, writes it to
 * kv_cache (slot_map[b], negative = skip) and patches it into the page it streamed in.  Stands in
 * for the same vLLM ops as the two entry points it replaces (`_C.rotary_embedding`,
 * `reshape_and_cache_flash`, FlashInfer paged decode).  Other arguments as
 * for bcg_decode_attn_paged. */
int bcg_decode_attn_paged_qkv(const float* qkv, int n_partials, long long partial_stride,
                              long long ld_qkv, const float* q_norm_w, const float* k_norm_w,
                              const float* cos_sin, const int* positions, const int* slot_map,
                              float eps, void* kv_cache, const int* block_table,
                              int max_blocks_per_seq, const int* seq_lens, void* out, float* scratch_o,
                              float* scratch_ml, int* chunk_counters, int B, int n_heads,
                              int n_kv_heads, int page_size, int max_splits, float scale,
                              void* stream);

/* Same computation as bcg_decode_attn_paged, for callers that cannot allocate device memory.
 * No counterpart in the reference (the reference never manages device memory itself); it exists
 * for hosts of this library that have no memory left to give, or no safe moment to ask for it:
 * a server whose whole device budget already went to weights and KV pages, or a decode loop that
 * must avoid cudaMalloc/cudaFree because they synchronise the device.  The scratch is a 16 MiB
 * array inside the library (held by every GPU that loads it, until exit), so the problem must
 * satisfy B * n_heads * max_splits * 130 <= 4 * 1024 * 1024 floats and B * n_kv_heads <= 4096;
 * larger calls return BCG_STATUS_TOO_LARGE, and every seq_lens[b] must be <= 256 * max_splits (a longer
 * row traps, as above).  The first call on a device resolves the array's address — make it
 * before any stream capture.  Calls share the array: keep them on one stream (overlapping calls
 * race); the caller never has to clear anything (the chunk counters inside start at zero and every
 * call returns them to zero).  Allocates nothing, frees nothing. */
int bcg_decode_attn_paged_static(const void* q, const void* kv_cache, const int* block_table,
                                 int max_blocks_per_seq, const int* seq_lens, void* out, int B,
                                 int n_heads, int n_kv_heads, int page_size, int max_splits,
                                 float scale, void* stream);

/* Causal attention of ragged new-token rows against cached prefix + new tokens, both read
 * through the block table.  q and out are bf16 [n_q_rows, n_heads*128]; tile_info: int32
 * [n_tiles][4] = {sequence, first q row, position of that row in its sequence, rows (<= 128)}.
 * Both contractions run on tcgen05 tensor cores (accumulators in TMEM); q tiles and KV pages are
 * fetched by TMA through tensor maps over the caller's q buffer and KV cache.  Every KV page a tile
 * reads (pages 0 .. ceil((position + rows) / 16) - 1 of its sequence's block-table row) must hold
 * finite values, including the unwritten tail of the last page (zero-initialise the cache).
 * Stands in for the FlashInfer paged prefill kernel. */
int bcg_prefill_attn_paged(const void* q, const void* kv_cache, const int* block_table,
                           int max_blocks_per_seq, const int* tile_info, int n_tiles, void* out,
                           int n_q_rows, int n_heads, int n_kv_heads, int page_size, float scale,
                           void* stream);

/* Grammar-constrained sampler + per-row decode bookkeeping, one thread-block cluster per row.
 * Applies the JSON-schema token bitmask of the row's DFA state, then greedy argmax
 * (temperature < 1e-5) or temperature sampling as an exponential race
 * argmax_i(logit_i / T - log(q_i)), q_i = -log(u_i), u_i from Philox4x32-10(seed[b]; i, step),
 * with a reproducible fp32 log (see oracle/sampler.py); advances the DFA over the token's
 * bytes; appends the token; updates next_ids / positions / seq_lens / slot_map so the next
 * decode step needs no host round-trip.
 * Stands in for xgrammar `apply_token_bitmask_inplace` + vLLM `Sampler` + the scheduler's
 * accept_token/stop bookkeeping (vllm v1/sample/sampler.py:91,223-297,
 * v1/sample/ops/topk_topp_sampler.py:395-416, v1/structured_output/backend_xgrammar.py:148-192). */
typedef struct bcg_sampler_args {
  const float* logits;     /* [B, ld_logits]; or vocab-sharded, see shard_v */
  long long ld_logits;
  int B;
  int V;                   /* multiple of 4 */
  int mask_words;          /* int32 words per mask row = ceil(V/32) */
  int max_steps;           /* row pitch of out_tokens / chosen / forced */
  int eos_id0, eos_id1;    /* stop ids (-1 = unused) */
  int page_size;
  int max_blocks_per_seq;
  /* grammar tables */
  const int* grammar_id;              /* [B], -1 = unconstrained */
  const int32_t* const* mask_tables;  /* [n_grammars] -> int32 [n_states][mask_words], bit=1 allowed, LSB first */
  const int16_t* const* trans_tables; /* [n_grammars] -> int16 [n_states][256], -1 = reject */
  const uint8_t* tok_bytes;           /* concatenated token byte strings */
  const int* tok_offsets;             /* [V+1] */
  /* per-row sampling state */
  const float* temperature;  /* [B] */
  const uint32_t* seed;      /* [B][2] */
  const int* max_tokens;     /* [B] */
  const int* forced;         /* [B, max_steps] teacher-forced ids (<0 = none) or NULL */
  int* state;                /* [B] DFA state, in/out */
  int* n_out;                /* [B] tokens emitted so far, in/out */
  int* finished;             /* [B] in/out: 0 running, 1 eos, 2 length, 3 grammar dead end */
  int* out_tokens;           /* [B, max_steps] accepted tokens */
  int* chosen;               /* [B, max_steps] the sampler's own pick (== out_tokens unless forced) or NULL */
  /* decode bookkeeping */
  int* next_ids;             /* [B] */
  int* positions;            /* [B] */
  int* seq_lens;             /* [B] */
  int* slot_map;             /* [B] */
  const int* block_table;    /* [B, max_blocks_per_seq] */
  int* n_active;             /* [1] number of unfinished rows after this call, or NULL */
  /* vocab-parallel logits as NCCL all-gather leaves them: shard_v > 0 means token i of row b is at
   * logits[(i / shard_v) * shard_stride + b * shard_v + i % shard_v]; 0 = plain [B, ld_logits] */
  int shard_v;
  long long shard_stride;
  /* vocab-parallel sampling without moving logits (tensor parallelism): tp_size > 1
   * means `logits` holds only this rank's shard — V tokens starting at token id vocab_base (a
   * multiple of 4; mask rows still span the whole vocabulary) — and the ranks trade one
   * (score, token id) candidate per row through the symmetric buffer (bcg_tp_symm_create / _open)
   * inside the kernel; every rank ends with the same token and does the same bookkeeping.
   * B <= 128.  0 or 1 = single GPU. */
  int tp_rank, tp_size;
  int vocab_base;
} bcg_sampler_args;

/* Launches the sampler described above on `stream` (stands in for xgrammar's mask apply + vLLM's
 * Sampler + accept_token bookkeeping).  `args` is a HOST struct of device pointers. */
int bcg_mask_sample(const bcg_sampler_args* args, void* stream);

/* Tensor parallelism (Qwen3-32B TP=8, Mistral-22B TP=2 in the reference's presets): one process per
 * GPU, one NCCL communicator per process.  Rank 0 obtains an id with bcg_tp_unique_id, ships the
 * 128 bytes to the other ranks by any means, everyone calls bcg_tp_init (collective).  The model
 * steps then all-reduce the outputs of the row-parallel o / down projections (2 per layer); the
 * vocab-parallel logits stay sharded and the sampler exchanges one candidate per row, standing in
 * for vLLM's TP collectives
 * (vllm_agent.py:131,141-142).  libnccl.so.2 is resolved at run time. */
int bcg_tp_unique_id(void* out_128_bytes /* host */);
int bcg_tp_init(const void* id_128_bytes /* host */, int rank, int size);
int bcg_tp_shutdown(void);
/* The symmetric buffer every rank of the replica maps (cudaIpc over NVLink).  It carries the
 * sampler's per-row candidate exchange (bcg_sampler_args.tp_size > 1) and, when
 * bcg_workspace.tp_region_floats > 0, the decode step's two per-layer all-reduces, fused into the
 * norm-statistics kernel that follows each row-parallel projection (bcg_tp_add_norm_stats: {value,
 * epoch} pushes over NVLink, no flag, no fence, no NCCL launch); with tp_region_floats == 0 the decode step all-reduces with
 * NCCL.  create: cudaMalloc's `bytes` (the only allocation this library ever makes; freed by
 * bcg_tp_shutdown) and returns the 64-byte IPC handle; open: takes all ranks' handles in rank
 * order.  bytes = bcg_tp_symm_bytes_for(region, size) = 4 * (32768 + 4 * size * region) with
 * region = tp_region_floats >= B_max * d_model (0 if only the sampler uses the buffer): two slots,
 * one inbox per source rank, every value stored beside the launch's epoch. */
long long bcg_tp_symm_bytes_for(long long region_floats, int size);
int bcg_tp_symm_create(long long bytes, void* handle_out_64_bytes /* host */);
int bcg_tp_symm_open(const void* handles_size_x_64_bytes /* host */, int rank, int size);
/* Tensor-parallel counterpart of bcg_add_norm_stats (decode, T <= 128): `partials` are THIS rank's
 * n_partials fp32 split-K slabs [T, d] of a row-parallel projection (o_proj / down_proj); the kernel
 * adds them, exchanges the reduced [T, d] message with the other ranks through the symmetric buffer
 * (slot 0 or 1, alternate between consecutive calls), adds the ranks' contributions in rank order
 * (bit-identical on every rank), then residual += sum, xn = bf16(residual * w) and
 * sumsq[s * 128 + t] as bcg_add_norm_stats.  Collective: every rank of the replica must make the same
 * sequence of calls.  Stands in for vLLM's tensor_model_parallel_all_reduce after RowParallelLinear
 * + `_C.fused_add_rms_norm`. */
int bcg_tp_add_norm_stats(float* residual, const float* partials, int n_partials, long long partial_stride,
                          const float* w, void* xn, float* sumsq, int slot, long long region_floats, int T,
                          int d, void* stream);

/* Whole-model steps: the layer stack launched from C++ on one stream so a decode step is one
 * host call (captured into a CUDA graph by the engine). */
typedef struct bcg_model {
  /* With tensor parallelism n_heads, n_kv_heads, d_ff and vocab are THIS RANK's shard sizes
   * (column-parallel qkv / gate_up, row-parallel o / down, vocab-parallel lm_head). */
  int n_layers, d_model, n_heads, n_kv_heads, head_dim, d_ff, vocab;
  float rms_eps;
  int page_size;
  const void* embed;             /* bf16 [vocab, d_model] */
  const void* lm_head;           /* bf16 [vocab, d_model] */
  const float* final_norm;       /* [d_model] */
  const float* const* ln1;       /* host array [n_layers] of device [d_model] */
  const float* const* ln2;
  const void* const* w_qkv;      /* bf16 [(n_heads+2*n_kv_heads)*128, d_model] */
  const void* const* w_o;        /* bf16 [d_model, n_heads*128] */
  const void* const* w_gate_up;  /* bf16 [2*d_ff, d_model], rows interleaved 16 gate / 16 up */
  const void* const* w_down;     /* bf16 [d_model, d_ff] */
  const float* const* q_norm;    /* [128] per layer or NULL array (Mistral) */
  const float* const* k_norm;
  void* const* kv_cache;         /* per-layer cache base */
  const float* cos_sin;          /* [max_pos][128] */
  int tp_size;                   /* 1, or the size given to bcg_tp_init */
} bcg_model;

typedef struct bcg_workspace {
  float* residual;    /* [T_max, d_model] */
  void* xn;           /* bf16 [T_max, d_model] */
  float* qkv;         /* fp32 [T_max, qkv_dim]   (prefill)  */
  void* q;            /* bf16 [T_max, n_heads*128] */
  void* attn;         /* bf16 [T_max, n_heads*128] */
  void* act;          /* bf16 [T_max, d_ff] */
  float* delta;       /* fp32 [T_max, d_model]   (prefill)  */
  float* partials;    /* fp32 split-K scratch, partials_floats long (decode) */
  long long partials_floats;
  float* attn_scratch_o;
  float* attn_scratch_ml;
  int* attn_counters;  /* int32 [B_max * n_kv_heads], zero-initialised once */
  int max_splits;
  float* logits;      /* fp32 [B_max, vocab] (with TP: this rank's vocabulary shard, vocab = shard size) */
  float* logits_local; /* unused (kept for layout compatibility) */
  long long tp_region_floats; /* > 0: fused peer-memory all-reduce in decode; floats per (slot, source
                                 rank) region of the symmetric buffer, >= B_max * d_model */
  void* xn_last;      /* bf16 [B_max, d_model] */
  int T_max, B_max;
  /* decode norm fusion (bcg_gemm_bf16_tn_fused); both NULL = separate add_rmsnorm kernels */
  float* row_sumsq;   /* fp32 [2][max(d_model/128, 8)][128]: row sums of squares per tile / segment, one table per norm */
  int* tile_counters; /* int32 [d_model/128], zero-initialised once */
} bcg_workspace;

/* T new tokens (ragged over sequences) -> KV cache filled, logits of each sequence's last
 * token in ws->logits[0..n_seqs).  last_rows: device int32 [n_seqs].  Stands in for one prefill
 * pass of vLLM's Qwen3Model.forward + LogitsProcessor (models/qwen3.py:216-236, 328-333). */
int bcg_model_prefill(const bcg_model* m, const bcg_workspace* ws, const int* ids,
                      const int* positions, const int* slot_map, const int* block_table,
                      int max_blocks_per_seq, const int* tile_info, int n_tiles,
                      const int* last_rows, int n_seqs, int T, void* stream);
/* Logits of `n` more tokens (device list `rows`) of the prefill step just run, into ws->logits rows
 * row0.. (stands in for vLLM's LogitsProcessor over chosen positions). */
int bcg_model_head(const bcg_model* m, const bcg_workspace* ws, const int* rows, int n, int row0, void* stream);
/* One decode step for B rows: ids/positions/slot_map/seq_lens are the arrays bcg_mask_sample
 * maintains; logits land in ws->logits[0..B).  Stands in for one decode step of the same vLLM
 * forward.  flags: BCG_GEMM_PDL, plus how the residual add + RMSNorm between two
 * projections is executed on a single GPU (both variants need ws->row_sumsq / ws->tile_counters):
 *   default                   bcg_add_rmsnorm kernels (complete norm, then the projection)
 *   BCG_STEP_DEFERRED_NORM    bcg_add_norm_stats + 1/RMS applied in the next projection's epilogue
 *   BCG_STEP_FUSED_NORM       the producing projection finishes the residual itself
 *                             (bcg_gemm_bf16_tn_fused producer half; measured slower) */
#define BCG_STEP_FUSED_NORM 0x20000
#define BCG_STEP_DEFERRED_NORM 0x40000
#define BCG_STEP_FUSED_ROPE 0x80000 /* bcg_decode_attn_paged_qkv instead of rope kernel + attention */
int bcg_model_decode(const bcg_model* m, const bcg_workspace* ws, const int* ids,
                     const int* positions, const int* slot_map, const int* seq_lens,
                     const int* block_table, int max_blocks_per_seq, int B, int flags,
                     void* stream);

/* ---------------------------------------------------------------------------------------------
 * Layer stacks: models whose layers differ in kind (the reference has no counterpart; its engine
 * only meets uniform dense decoders).  Every layer is a mixer and, optionally, a feed-forward, each
 * with a norm before and (norm1b / norm2b not NULL) a norm after it:  x += norm1b(mixer(norm1(x))),
 * x += norm2b(ff(norm2(x))), or, `parallel`, both behind one norm:  h = norm1(x),  x += mixer(h) + ff(h).
 * norm1 / norm2 NULL: the sublayers read x itself.  A mixer may be two side by side, grouped attention and a state-space
 * mixer, that read the same h.
 * `act_dtype` selects the activations that feed matrix products, the latent cache and the attention
 * operands: BCG_DT_BF16 (tensor-core kernels, fp32 accumulation) or BCG_DT_F32 (true fp32
 * throughout, CUDA-core kernels).  Weights are bf16 in both; the residual, norms, scores, gates and
 * recurrent states are fp32 in both. */
#define BCG_DT_BF16 0
#define BCG_DT_F32 1
#define BCG_MIXER_LATENT_ATTN 1
#define BCG_MIXER_GENERAL_DELTA 2
#define BCG_MIXER_GROUPED_ATTN 3
#define BCG_MIXER_STATE_SPACE 4   /* alone; beside grouped attention: ssm_heads > 0 */
#define BCG_MIXER_MATRIX_MEMORY 5
#define BCG_FF_POLY_NORM 0   /* bcg_layer.ff_kind of layers that are not parallel */
#define BCG_FF_CLAMPED_GLU 1 /* w_up rows interleaved [16 gate | 16 up], glu_limit, glu_alpha */
#define BCG_FF_GELU_GLU 2    /* the same rows; gelu(gate) * up, gelu in its tanh form */
#define BCG_FF_EXPERTS 3     /* experts without gates, gelu in its erf form; w_up: n_router router rows, then the ff rows of a
                                shared expert (ff = 0: none), whose output matrix is w_down */
#define BCG_VALUES_FIRST 1   /* bcg_layer.v_role: the layer's values are what later layers mix in */
#define BCG_VALUES_MIX 2     /* values are (1 - v_mix) of its own and v_mix of those */

typedef struct bcg_layer {
  int mixer;               /* BCG_MIXER_* */
  int heads, dim;          /* latent attention: unrotated q/k dims per head; delta: channels per head */
  int rot_dim, rot_dims;   /* rotated q/k dims per head, and how many of them rotate (rotate-half) */
  int vdim, kv_rank;
  int window;              /* keys a query sees, itself included; 0 = all earlier ones */
  float scale;
  int q_ld, v_ld;          /* padded q/k and v head sizes of the expanded form (multiples of 64), 0 = none */
  int owns_cache;          /* 0: the layer reads `cache`, which an earlier layer writes */
  int n_in;                /* rows of w_in */
  int decay_rank;          /* columns of w_decay */
  int ff;                  /* 0 = no feed-forward */
  const float* norm1;      /* [d] */
  const float* norm1b;
  const float* norm2;
  const float* norm2b;
  const void* w_in;        /* bf16 [n_in, d]: latent attention q | down-projection (owners only);
                              delta r | k | v | g | rate | decay-in; zero rows after */
  const void* w_out;       /* bf16 [d, heads * (vdim or dim)] */
  const float* latent_norm; /* [kv_rank] */
  const float* sink;       /* [heads] or NULL */
  const float* cos_sin;    /* [max_pos][rot_dims]: cos of the rot_dims/2 angles, then sin */
  const void* w_uk;        /* bf16 [heads * dim, kv_rank] */
  const void* w_uv;        /* bf16 [heads * vdim, kv_rank] */
  const void* w_expand;    /* bf16 [heads * (q_ld + v_ld), kv_rank + rot_dim]: cache row -> all heads' keys
                              (w_uk rows, then the identity on the rotated part, then zero rows), then
                              all heads' values; NULL = no expanded form */
  const float* decay_bias; /* [heads * dim] */
  const float* rate_bias;  /* [heads * dim] */
  const float* out_norm;   /* [heads * dim] */
  const void* w_decay;     /* bf16 [heads * dim, decay_rank] */
  const void* w_up;        /* bf16 [ff, d] */
  const void* w_down;      /* bf16 [d, ff] */
  const float* act_coef;   /* PolyNorm's four numbers (device) */
  void* cache;             /* latent pages [pages][page_size][kv_rank + rot_dim], or state
                              fp32 [slots][heads][dim][dim]; grouped attention: keys
                              [pages][kv_heads][page_size][q_ld], columns past dim zero */
  /* grouped attention (parallel layers) and their feed-forward */
  int parallel;
  int kv_heads;            /* query head h reads key/value head h / (heads / kv_heads) */
  float temp_coef, temp_every; /* queries times 1 + temp_coef * ln(floor((position + 1) / temp_every) + 1) */
  int v_role;              /* 0 or BCG_VALUES_* */
  float v_mix;
  int n_qkv;               /* rows of w_in in front of the up rows: q | k | v | router; zero rows after */
  int act_col, mix_ld;     /* rows of ws->mix: heads * vdim attention columns, ff activations (squared relu) from act_col
                              on; mix_ld columns of w_out */
  int router_col;          /* first router row of w_in */
  int experts, top;        /* mixture of experts; experts = 0: none */
  int expert_ld;           /* an expert's inner size, padded to a multiple of 16 */
  float glu_limit, glu_alpha;
  int moe_counts_at;       /* the layer's place in ws->moe_counts */
  const float* slopes;     /* [heads] slope * (query position - key position) is taken off the score; NULL = none */
  const float* in_bias;    /* [q + k + v rows] */
  const float* out_bias;   /* [d] */
  const void* w_experts_in;  /* bf16 [experts][2 * expert_ld][d], rows interleaved [16 gate | 16 up] */
  const void* w_experts_out; /* bf16 [experts][d][expert_ld] */
  void* cache_v;           /* values [pages][kv_heads][page_size][v_ld], columns past vdim zero */
  /* grouped attention: RMS norms over all heads of a token's queries / keys at once, and an output gate per head */
  const float* q_norm;     /* [heads * dim] or NULL */
  const float* k_norm;     /* [kv_heads * dim] or NULL */
  int gated, gate_col;     /* head outputs times gate_scale * sigmoid(column gate_col + head of the projection) */
  float gate_scale;
  int ff_kind;             /* BCG_FF_* */
  /* state-space mixer: rows z | x | B | C | step of w_in from ssm_col on (ssm_heads * ssm_vdim, the same,
     ssm_groups * ssm_n twice, ssm_heads rows); x, B and C pass a causal convolution of ssm_taps taps and silu */
  int ssm_heads, ssm_vdim, ssm_n, ssm_groups;
  int ssm_norm_parts;      /* equal parts of the output that are normed each by its own root mean square */
  int ssm_taps, ssm_col;
  int ssm_mix_col;         /* first column of ws->mix */
  const float* conv_w;     /* [taps][channels], last row = current token */
  const float* conv_b;     /* [channels] */
  const float* step_bias;  /* [heads] */
  const float* decay_rate; /* [heads] state decays by exp(-decay_rate * step) */
  const float* skip;       /* [heads] */
  const float* ssm_norm;   /* [heads * vdim] */
  float* ssm_state;        /* fp32 [slots][heads][vdim][n] */
  float* conv_state;       /* fp32 [slots][taps - 1][channels]: the last inputs of the convolution, oldest first */
  /* grouped attention whose heads are normed (q_norm, k_norm: [dim], or NULL) and rotated one by one */
  int by_head;
  int rot_pairs;           /* entries 2i and 2i + 1 turn together, else i and rot_dims / 2 + i */
  int v_rot_dims;          /* entries of the values that turn, in pairs 2i, 2i + 1; outputs are turned back; 0 = none */
  const float* v_cos_sin;  /* [max_pos][v_rot_dims] as cos_sin */
  int pool;                /* tokens of a pooled block; 0 = none.  Block b's key and value are the means of the cached ones of
                              tokens b * pool .. + pool - 1; query i sees it if b * pool + pool - 1 <= i - window */
  int pool_col;            /* column of the block table with the page of pooled blocks 0 .. page_size - 1, and so on */
  /* matrix memory: rows q | k (heads * dim each) | v | output gate (heads * vdim each) of w_in, from gate_col on input and
     forget gates (heads each); log gates cap * tanh((z + bias) / cap), the forget gate's logsigmoid of that */
  float gate_cap;
  const float* mem_bias;   /* [2 * heads] */
  const float* mem_norm;   /* [heads * vdim] */
  float* mem_state;        /* fp32 [slots][heads][vdim + 1][dim], last row = normalizer */
  float* mem_max;          /* fp32 [slots][heads][(vdim + 63) / 64]: running maximum of the log gates, one copy per 64 rows */
  /* BCG_FF_EXPERTS */
  int n_router;
  const float* router_bias; /* [experts] */
} bcg_layer;

typedef struct bcg_stack {
  int n_layers, d_model, vocab_ld; /* vocab_ld: rows of lm_head (vocabulary, padded to a multiple of 4) */
  int act_dtype, page_size;
  float eps;
  const void* embed;        /* bf16 [vocab, d] */
  const void* lm_head;      /* bf16 [vocab_ld, d] */
  const float* final_norm;
  const bcg_layer* layers;  /* host array */
  const void* pos_embed;    /* bf16 [n_pos, d] added to the embedding, or NULL */
  int n_pos;
  float embed_scale;        /* factor of the embedding */
  const double* pos_turns;  /* [(d + 1) / 2] turns per position: sin at entry 2i, cos at 2i + 1 are added; or NULL */
  const float* embed_norm;  /* [d] weight of a norm of the embedding, or NULL */
} bcg_stack;

typedef struct bcg_stack_ws {
  float* residual;  /* [T_max, d] */
  void* xn;         /* act [T_max, d]; after a step: the final norm of every row */
  float* proj;      /* fp32 projection outputs / split-K slabs */
  long long proj_floats;
  float* decay;     /* fp32 [T_max, heads * dim] slabs of w_decay */
  long long decay_floats;
  void* q;          /* act [T_max, heads * q_row] */
  void* mix;        /* act [T_max, columns of w_out] */
  void* act;        /* act [T_max, ff] */
  void* low;        /* act [T_max, decay_rank] */
  void* latents;    /* bf16 [K_max, kv_rank + rot_dim] gathered cache rows */
  void* expanded;   /* bf16 [K_max, heads * (q_ld + v_ld)] */
  void* q_latent;   /* bf16 [D_max, heads, kv_rank + rot_dim]: queries in latent space */
  void* o_latent;   /* bf16 [D_max, heads, kv_rank] */
  float* part_o;    /* fp32 decode partials [D_max, chunks, heads, kv_rank], part_floats long */
  long long part_floats;
  float* part_ml;   /* fp32 [D_max, chunks, heads, 2] */
  void* xn_rows;    /* act [B_max, d] */
  float* logits;    /* fp32 [B_max, vocab_ld] */
  int T_max, K_max, D_max, B_max;
  float* v_first;   /* fp32 [T_max, kv_heads * vdim]: the step's values of the BCG_VALUES_FIRST layer */
  /* mixture of experts; rows = (token, choice) pairs */
  void* moe_x;      /* act [moe_rows_max, d] rows sorted by expert */
  void* moe_h;      /* act [moe_rows_max, expert_ld] */
  float* moe_proj;  /* fp32 slabs of [rows, 2 * expert_ld] */
  long long moe_proj_floats;
  float* moe_out;   /* fp32 slabs of [rows, d] */
  long long moe_out_floats;
  int* moe_expert;  /* [T][top] */
  int* moe_rank;    /* [T][top] */
  float* moe_weight;     /* [T][top] */
  int* moe_row;          /* [T][top] sorted row of each choice */
  float* moe_row_weight; /* [rows] */
  int* moe_counts;       /* rows per expert, all layers' one after another; cleared at the start of a step */
  int moe_counts_n, moe_rows_max;
  float* gates;     /* fp32 [T_max, heads]: factors of the head outputs */
  void* ssm_x;      /* act [T_max, ssm_x_ld(layer)]: convolved x | B | C, heads and groups padded to multiples of 8 */
  float* ssm_step;  /* fp32 [T_max, ssm_heads] */
  void* ssm_y;      /* act [T_max, ssm_heads * ssm_vdim]: outputs in front of gate and norm */
  float* mem_den;   /* fp32 [T_max, heads]: denominators of a matrix memory's outputs (ssm_x and ssm_y are its other buffers) */
} bcg_stack_ws;

/* A step: T new tokens of n_seqs sequences, portions of prompts beside single decoded tokens.  All
 * pointers are device int32. */
typedef struct bcg_step_batch {
  int T, n_seqs;
  const int* ids;          /* [T] */
  const int* positions;    /* [T] */
  const int* slot_map;     /* [T] cache row of each token (< 0: writes nothing, keeps the state) */
  const int* row_seq;      /* [T] sequence of each token, NULL = token t belongs to sequence t */
  const int* seq_start;    /* [n_seqs + 1] first token of each sequence, NULL = one token each */
  const int* block_table;  /* [n_seqs, max_blocks]: pages of the tokens, then, from bcg_layer.pool_col on, of pooled blocks */
  int max_blocks;
  const int* state_slots;  /* [n_seqs] */
  int max_context;         /* upper bound on positions + 1 of the single tokens (sizes the grid) */
  /* attention work lists of the bf16 kernels */
  const int* single_rows;  /* [n_single] tokens attended one by one in latent space, NULL = all T */
  int n_single;
  const int* tiles;        /* [n_tiles][8] {first token, its position, tokens (<= 128), expanded row of
                              key position k0, k0, sequence, 0, 0} */
  int n_tiles;
  const int* gather;       /* [n_gather] cache row behind every expanded row */
  int n_gather;
  int flags;               /* BCG_GEMM_PDL */
} bcg_step_batch;

/* Runs the layers over a step's tokens: caches and states advanced, ws->residual and ws->xn (final norm)
 * filled.  One call = prefill, decode or a mixture; the reference has no counterpart (vLLM's
 * GPUModelRunner.execute_model is the nearest relative). */
int bcg_stack_step(const bcg_stack* m, const bcg_stack_ws* ws, const bcg_step_batch* b, void* stream);
/* Logits of `n` tokens of the step just run, in ws->logits rows row0..: rows = device list of token
 * indices, or NULL = tokens 0..n-1.  The reference has no counterpart of its own (vLLM LogitsProcessor). */
int bcg_stack_head(const bcg_stack* m, const bcg_stack_ws* ws, const int* rows, int n, int row0, int flags,
                   void* stream);

/* The mechanisms one by one (what bcg_stack_step launches; the reference has no counterpart).
 * `in` arguments with n_partials slabs are fp32 split-K outputs added in index order. */
/* out fp32 [M, ldo] = X [M, ldx] (act_dtype) * W bf16 [N, ldw]^T on CUDA cores, any shape. */
int bcg_gemm_any(const void* X, int x_dtype, const void* W, float* out, int M, int N, int K, long long ldx,
                 long long ldw, long long ldo, void* stream);
/* No counterpart in the reference: residual += w_post ? rmsnorm(delta) * w_post : delta, then
 * xn = rmsnorm(residual) * w_next (w_next NULL: xn = residual; xn NULL: skipped). */
int bcg_sandwich_norm(float* residual, const float* delta, int n_partials, long long partial_stride,
                      const float* w_post, const float* w_next, void* xn, int act_dtype, int T, int d, float eps,
                      void* stream);
/* No counterpart in the reference: the same with further summands: delta (may be NULL when per_row > 0) + bias (may be NULL) +
 * sum over k < per_row of rows[index[t * per_row + k]] (fp32 slabs too) times weight[t * per_row + k] (NULL: 1). */
int bcg_residual_norm(float* residual, const float* delta, int n_partials, long long partial_stride, const float* bias,
                      const float* rows, const int* index, const float* weight, int per_row, int row_partials,
                      long long row_stride, const float* w_post, const float* w_next, void* xn, int act_dtype, int T, int d,
                      float eps, void* stream);
/* No counterpart in the reference: a N(z) + b N(z^2) + c N(z^3) + e with N = division by the row's RMS. */
int bcg_poly_norm(const float* z, int n_partials, long long partial_stride, const float* coef, void* out,
                  int act_dtype, int T, int ff, float eps, void* stream);
/* No counterpart in the reference: generalized delta rule over ragged sequences; proj rows are
 * r | k | v | g | rate (heads * dim each, row pitch ld), decay the fp32 pre-activation without its bias. */
int bcg_delta_scan(const bcg_layer* l, const float* proj, int n_partials, long long partial_stride, long long ld,
                   const float* decay, int decay_partials, long long decay_stride, const int* positions,
                   const int* slot_map, const int* seq_start, const int* state_slots, int n_seqs, void* out,
                   int act_dtype, float eps, void* stream);
/* No counterpart in the reference: attention of a step's queries (ws->q) over the latent pages.
 * mode 0: what bcg_stack_step picks; 1: the plain kernel; ws->mix receives the heads' values. */
int bcg_latent_attention(const bcg_stack* m, const bcg_stack_ws* ws, const bcg_step_batch* b, int layer, int mode,
                         void* stream);
/* No counterpart in the reference: a grouped attention layer's input projection (ws->proj, row pitch ld) to queries, key
 * and value pages, activations (with_act: columns n_qkv.. are up rows), and the routing of its experts
 * (ws->moe_counts must be zero). */
int bcg_grouped_in(const bcg_stack* m, const bcg_stack_ws* ws, const bcg_step_batch* b, int layer, int n_partials,
                   long long partial_stride, long long ld, int with_act, void* stream);
/* No counterpart in the reference: attention of a step's queries (ws->q) over the key and value pages.
 * mode 0: what bcg_stack_step picks; 1: the plain kernel; columns 0.. of ws->mix receive the heads' values. */
int bcg_grouped_attention(const bcg_stack* m, const bcg_stack_ws* ws, const bcg_step_batch* b, int layer, int mode,
                          void* stream);
/* No counterpart in the reference (vLLM's fused_moe is the nearest relative): rows sorted by group, X bf16 [rows, K]
 * times the groups' matrices W bf16 [n_groups * N, K]; counts: device, rows per group, at most max_rows each.  K % 8 == 0,
 * N % 16 == 0 where max_rows > 128, n_groups <= 512.  row_weight NULL: out fp32 [splits][rows, N] (splits > 1 only where
 * max_rows <= 128).  Otherwise max_rows > 128, W rows interleaved [16 gate | 16 up], out bf16 [rows, N / 2] =
 * g * sigmoid(alpha * g) * (u + 1) of the weighted accumulators, g = min(., limit), u clamped to +-limit. */
int bcg_gemm_grouped(const void* X, const void* W, void* out, int rows, int N, int K, const int* counts, int n_groups,
                     int max_rows, int splits, const float* row_weight, float limit, float alpha, int flags, void* stream);
/* No counterpart in the reference: ws->xn through the experts that bcg_grouped_in chose; ws->moe_out receives *splits
 * slabs of [T * top, d], row ws->moe_row[t * top + k] for choice k of token t. */
int bcg_experts(const bcg_stack* m, const bcg_stack_ws* ws, int layer, int T, int* splits, void* stream);

/* No counterpart in the reference: a state-space mixer behind its input projection (ws->proj, row pitch ld): convolution,
 * recurrence, gate and norm; states advanced, ws->mix columns ssm_mix_col.. filled.  mode 0: what bcg_stack_step picks
 * (tensor-core chunks or, one token each, the decode kernel); 1: token by token on CUDA cores. */
int bcg_state_space(const bcg_stack* m, const bcg_stack_ws* ws, const bcg_step_batch* b, int layer, int n_partials,
                    long long partial_stride, long long ld, int mode, void* stream);
/* No counterpart in the reference: clamped gated unit of split-K slabs z [T, 2 * ff], columns interleaved [16 gate | 16 up],
 * ff % 16 == 0:  out = g * sigmoid(alpha * g) * (u + 1), g = min(gate, limit), u clamped to +-limit. */
int bcg_clamped_glu(const float* z, int n_partials, long long partial_stride, void* out, int act_dtype, int T, int ff,
                    float limit, float alpha, void* stream);
/* No counterpart in the reference: bcg_gemm_bf16_tn with that unit as its epilogue; out bf16 [M, N / 2], N % 32 == 0. */
int bcg_gemm_bf16_glu(const void* X, const void* W, void* out, int M, int N, int K, float limit, float alpha, int flags,
                      void* stream);

/* No counterpart in the reference: gelu of split-K slabs; gated: z [T, 2 * ff], columns interleaved [16 gate | 16 up], out =
 * gelu(gate) * up with the tanh form; else z [T, ff], the erf form.  ff % 16 == 0. */
int bcg_gelu_unit(const float* z, int n_partials, long long partial_stride, void* out, int act_dtype, int T, int ff, int gated,
                  void* stream);
/* No counterpart in the reference: bcg_gemm_bf16_tn with that unit as its epilogue: gated, out bf16 [M, N / 2], N % 32 == 0; else
 * out bf16 [M, N], N % 16 == 0, M > 128. */
int bcg_gemm_bf16_gelu(const void* X, const void* W, void* out, int M, int N, int K, int gated, int flags, void* stream);
/* No counterpart in the reference: bcg_gemm_grouped with gelu (erf form) as its epilogue, out bf16 [rows, N], max_rows > 128. */
int bcg_gemm_grouped_gelu(const void* X, const void* W, void* out, int rows, int N, int K, const int* counts, int n_groups, int max_rows,
                          int flags, void* stream);
/* No counterpart in the reference: routing of a BCG_FF_EXPERTS layer whose logits are the first columns of ws->proj (row pitch ld;
 * ws->moe_counts must be zero) and, with_act, gelu of the columns behind n_router into ws->act. */
int bcg_expert_in(const bcg_stack* m, const bcg_stack_ws* ws, int layer, int T, int n_partials, long long partial_stride, long long ld,
                  int with_act, void* stream);
/* No counterpart in the reference: a matrix memory behind its input projection (ws->proj, row pitch ld): recurrence, norm and output
 * gate; states advanced, ws->mix filled.  mode 0: tensor-core chunks or, one token each, the decode kernel; 1: token by token on CUDA
 * cores; 2: as 0 with queries, keys, values and output gates in ws->ssm_x as activations already (heads in multiples of 8 columns),
 * ws->proj just the input and forget gates: what bcg_stack_step does in launches of more than 128 tokens. */
int bcg_matrix_memory(const bcg_stack* m, const bcg_stack_ws* ws, const bcg_step_batch* b, int layer, int n_partials,
                      long long partial_stride, long long ld, int mode, void* stream);

#ifdef __cplusplus
}
#endif
#endif /* BCG_B200_H_ */
