// Prompt attention of latent layers in expanded form: the step's cache rows (gathered, history inside the
// window included) are multiplied once into every head's keys and values, and the window attention kernel
// (attn_window.cuh) runs over them.
//
// The expanded row of head h is  K: [W_uk c | k_rot | 0] (QD columns),  V: [W_uv c | 0] (VD columns): the
// expansion matrix holds the identity on the rotated part, so one GEMM over cache rows produces keys with
// the shared rotated part already in place (exactly: bf16 times one).
#include "attn_window.cuh"

namespace bcg {

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
                               static_cast<long long>(l->heads) * l->q_ld, kWaBM));
  BCG_TRY(make_tmap_bf16_sw128(&km, ws->expanded, b->n_gather, n_exp, n_exp, kWaBN));
  WindowAttn a = {};
  a.tiles = b->tiles;
  a.n_tiles = b->n_tiles;
  a.sink = l->sink;
  a.k_col = l->q_ld;
  a.v_col = l->heads * l->q_ld;
  a.group = 1;
  a.out = static_cast<__nv_bfloat16*>(ws->mix);
  a.out_ld = static_cast<long long>(l->heads) * l->vdim;
  a.heads = l->heads;
  a.vdim = l->vdim;
  a.window = l->window;
  a.scale_log2e = l->scale * 1.4426950408889634f;
  return window_attn<false, false>(l->q_ld, l->v_ld, qm, km, km, a, st);
}

}  // namespace bcg
