"""ctypes binding of libbcg_b200.so (include/bcg_b200.h).

There is no CPU or PyTorch fallback: if the library is missing, or a call fails, this module
raises.  PyTorch only owns device memory and streams; all arithmetic on the product path
happens inside the library's sm_100a kernels.
"""
from __future__ import annotations

import ctypes as C
from pathlib import Path

PKG = Path(__file__).resolve().parent
LIB_PATH = PKG / "_lib" / "libbcg_b200.so"

EPI_BF16, EPI_F32, EPI_SWIGLU, EPI_RELU2 = 0, 1, 2, 3
GEMM_PDL = 1
STEP_FUSED_NORM = 0x20000   # bcg_model_decode: fold add+RMSNorm into the GEMMs (opt-in, slower)
STEP_FUSED_ROPE = 0x80000     # bcg_model_decode: qk-norm/RoPE/KV-write folded into decode attention
STEP_DEFERRED_NORM = 0x40000  # bcg_model_decode: norm statistics kernel + 1/RMS in the next GEMM's epilogue

DT_BF16, DT_F32 = 0, 1                          # activation dtype of a layer stack
MIXER_LATENT_ATTN, MIXER_GENERAL_DELTA, MIXER_GROUPED_ATTN, MIXER_STATE_SPACE, MIXER_MATRIX_MEMORY = 1, 2, 3, 4, 5
FF_POLY_NORM, FF_CLAMPED_GLU, FF_GELU_GLU, FF_EXPERTS = 0, 1, 2, 3      # Layer.ff_kind
MAX_GROUPS = 512                                # experts the grouped tensor-core GEMM takes
VALUES_FIRST, VALUES_MIX = 1, 2                 # Layer.v_role

c_int_p = C.POINTER(C.c_int)
c_float_p = C.POINTER(C.c_float)
vp = C.c_void_p


class BcgError(RuntimeError):
    pass


class SamplerArgs(C.Structure):
    _fields_ = [
        ("logits", vp), ("ld_logits", C.c_longlong),
        ("B", C.c_int), ("V", C.c_int), ("mask_words", C.c_int), ("max_steps", C.c_int),
        ("eos_id0", C.c_int), ("eos_id1", C.c_int), ("page_size", C.c_int),
        ("max_blocks_per_seq", C.c_int),
        ("grammar_id", vp), ("mask_tables", vp), ("trans_tables", vp),
        ("tok_bytes", vp), ("tok_offsets", vp),
        ("temperature", vp), ("seed", vp), ("max_tokens", vp), ("forced", vp),
        ("state", vp), ("n_out", vp), ("finished", vp), ("out_tokens", vp), ("chosen", vp),
        ("next_ids", vp), ("positions", vp), ("seq_lens", vp), ("slot_map", vp),
        ("block_table", vp), ("n_active", vp),
        ("shard_v", C.c_int), ("shard_stride", C.c_longlong),
        ("tp_rank", C.c_int), ("tp_size", C.c_int), ("vocab_base", C.c_int),
    ]


class GemmFusion(C.Structure):
    _fields_ = [
        ("scale_sumsq", vp), ("scale_tiles", C.c_int), ("scale_d", C.c_int), ("scale_eps", C.c_float),
        ("red_residual", vp), ("red_w", vp), ("red_xn", vp), ("red_sumsq", vp), ("red_counters", vp),
    ]


class Model(C.Structure):
    _fields_ = [
        ("n_layers", C.c_int), ("d_model", C.c_int), ("n_heads", C.c_int), ("n_kv_heads", C.c_int),
        ("head_dim", C.c_int), ("d_ff", C.c_int), ("vocab", C.c_int),
        ("rms_eps", C.c_float), ("page_size", C.c_int),
        ("embed", vp), ("lm_head", vp), ("final_norm", vp),
        ("ln1", C.POINTER(vp)), ("ln2", C.POINTER(vp)),
        ("w_qkv", C.POINTER(vp)), ("w_o", C.POINTER(vp)),
        ("w_gate_up", C.POINTER(vp)), ("w_down", C.POINTER(vp)),
        ("q_norm", C.POINTER(vp)), ("k_norm", C.POINTER(vp)),
        ("kv_cache", C.POINTER(vp)), ("cos_sin", vp), ("tp_size", C.c_int),
    ]


class Workspace(C.Structure):
    _fields_ = [
        ("residual", vp), ("xn", vp), ("qkv", vp), ("q", vp), ("attn", vp), ("act", vp),
        ("delta", vp), ("partials", vp), ("partials_floats", C.c_longlong),
        ("attn_scratch_o", vp), ("attn_scratch_ml", vp), ("attn_counters", vp),
        ("max_splits", C.c_int),
        ("logits", vp), ("logits_local", vp), ("tp_region_floats", C.c_longlong), ("xn_last", vp),
        ("T_max", C.c_int), ("B_max", C.c_int),
        ("row_sumsq", vp), ("tile_counters", vp),
    ]


class Layer(C.Structure):
    _fields_ = [
        ("mixer", C.c_int), ("heads", C.c_int), ("dim", C.c_int), ("rot_dim", C.c_int),
        ("rot_dims", C.c_int), ("vdim", C.c_int), ("kv_rank", C.c_int), ("window", C.c_int),
        ("scale", C.c_float), ("q_ld", C.c_int), ("v_ld", C.c_int), ("owns_cache", C.c_int),
        ("n_in", C.c_int), ("decay_rank", C.c_int), ("ff", C.c_int), ("norm1", vp), ("norm1b", vp),
        ("norm2", vp), ("norm2b", vp), ("w_in", vp), ("w_out", vp), ("latent_norm", vp), ("sink", vp),
        ("cos_sin", vp), ("w_uk", vp), ("w_uv", vp), ("w_expand", vp), ("decay_bias", vp), ("rate_bias", vp),
        ("out_norm", vp), ("w_decay", vp), ("w_up", vp), ("w_down", vp), ("act_coef", vp), ("cache", vp),
        ("parallel", C.c_int), ("kv_heads", C.c_int), ("temp_coef", C.c_float), ("temp_every", C.c_float),
        ("v_role", C.c_int), ("v_mix", C.c_float), ("n_qkv", C.c_int), ("act_col", C.c_int), ("mix_ld", C.c_int),
        ("router_col", C.c_int), ("experts", C.c_int), ("top", C.c_int), ("expert_ld", C.c_int),
        ("glu_limit", C.c_float), ("glu_alpha", C.c_float), ("moe_counts_at", C.c_int), ("slopes", vp),
        ("in_bias", vp), ("out_bias", vp), ("w_experts_in", vp), ("w_experts_out", vp), ("cache_v", vp),
        ("q_norm", vp), ("k_norm", vp), ("gated", C.c_int), ("gate_col", C.c_int), ("gate_scale", C.c_float),
        ("ff_kind", C.c_int), ("ssm_heads", C.c_int), ("ssm_vdim", C.c_int), ("ssm_n", C.c_int), ("ssm_groups", C.c_int),
        ("ssm_norm_parts", C.c_int), ("ssm_taps", C.c_int), ("ssm_col", C.c_int), ("ssm_mix_col", C.c_int),
        ("conv_w", vp), ("conv_b", vp), ("step_bias", vp), ("decay_rate", vp), ("skip", vp), ("ssm_norm", vp),
        ("ssm_state", vp), ("conv_state", vp),
        ("by_head", C.c_int), ("rot_pairs", C.c_int), ("v_rot_dims", C.c_int), ("v_cos_sin", vp), ("pool", C.c_int),
        ("pool_col", C.c_int), ("gate_cap", C.c_float), ("mem_bias", vp), ("mem_norm", vp), ("mem_state", vp), ("mem_max", vp),
        ("n_router", C.c_int), ("router_bias", vp),
    ]


class Stack(C.Structure):
    _fields_ = [
        ("n_layers", C.c_int), ("d_model", C.c_int), ("vocab_ld", C.c_int), ("act_dtype", C.c_int),
        ("page_size", C.c_int), ("eps", C.c_float), ("embed", vp), ("lm_head", vp), ("final_norm", vp),
        ("layers", C.POINTER(Layer)), ("pos_embed", vp), ("n_pos", C.c_int),
        ("embed_scale", C.c_float), ("pos_turns", vp), ("embed_norm", vp),
    ]


class StackWs(C.Structure):
    _fields_ = [
        ("residual", vp), ("xn", vp), ("proj", vp), ("proj_floats", C.c_longlong), ("decay", vp),
        ("decay_floats", C.c_longlong), ("q", vp), ("mix", vp), ("act", vp), ("low", vp), ("latents", vp),
        ("expanded", vp), ("q_latent", vp), ("o_latent", vp), ("part_o", vp), ("part_floats", C.c_longlong),
        ("part_ml", vp), ("xn_rows", vp), ("logits", vp), ("T_max", C.c_int), ("K_max", C.c_int),
        ("D_max", C.c_int), ("B_max", C.c_int), ("v_first", vp), ("moe_x", vp), ("moe_h", vp), ("moe_proj", vp),
        ("moe_proj_floats", C.c_longlong), ("moe_out", vp), ("moe_out_floats", C.c_longlong), ("moe_expert", vp),
        ("moe_rank", vp), ("moe_weight", vp), ("moe_row", vp), ("moe_row_weight", vp), ("moe_counts", vp),
        ("moe_counts_n", C.c_int), ("moe_rows_max", C.c_int), ("gates", vp), ("ssm_x", vp), ("ssm_step", vp), ("ssm_y", vp),
        ("mem_den", vp),
    ]


class StepBatch(C.Structure):
    _fields_ = [
        ("T", C.c_int), ("n_seqs", C.c_int), ("ids", vp), ("positions", vp), ("slot_map", vp),
        ("row_seq", vp), ("seq_start", vp), ("block_table", vp), ("max_blocks", C.c_int),
        ("state_slots", vp), ("max_context", C.c_int), ("single_rows", vp), ("n_single", C.c_int),
        ("tiles", vp), ("n_tiles", C.c_int), ("gather", vp), ("n_gather", C.c_int), ("flags", C.c_int),
    ]


_SIGS = {
    "bcg_abi_version": (C.c_int, []),
    "bcg_last_error": (C.c_char_p, []),
    "bcg_gemm_bf16_tn": (C.c_int, [vp, vp, vp, C.c_int, C.c_int, C.c_int, C.c_longlong,
                                   C.c_longlong, C.c_longlong, C.c_int, C.c_int, C.c_int, vp]),
    "bcg_gemm_bf16_tn_fused": (C.c_int, [vp, vp, vp, C.c_int, C.c_int, C.c_int, C.c_longlong,
                                         C.c_longlong, C.c_longlong, C.c_int, C.c_int, C.c_int,
                                         C.POINTER(GemmFusion), vp]),
    "bcg_gemm_splits_for": (C.c_int, [C.c_int, C.c_int, C.c_int]),
    "bcg_embed_rmsnorm": (C.c_int, [vp, vp, vp, vp, vp, C.c_int, C.c_int, C.c_float, vp]),
    "bcg_add_rmsnorm": (C.c_int, [vp, vp, C.c_int, C.c_int, C.c_longlong, vp, vp, vp, C.c_int,
                                  C.c_int, C.c_float, vp]),
    "bcg_add_norm_stats": (C.c_int, [vp, vp, C.c_int, C.c_int, C.c_longlong, vp, vp, vp, C.c_int, C.c_int, vp]),
    "bcg_qknorm_rope_kvwrite": (C.c_int, [vp, C.c_int, C.c_int, C.c_longlong, C.c_longlong, vp, vp,
                                          vp, vp, vp, vp, vp, C.c_int, C.c_int, C.c_int, C.c_int,
                                          C.c_float, vp]),
    "bcg_swiglu_reduce": (C.c_int, [vp, C.c_int, C.c_longlong, vp, C.c_int, C.c_int, vp]),
    "bcg_decode_attn_paged": (C.c_int, [vp, vp, vp, C.c_int, vp, vp, vp, vp, vp, C.c_int, C.c_int,
                                        C.c_int, C.c_int, C.c_int, C.c_float, vp]),
    "bcg_decode_attn_paged_qkv": (C.c_int, [vp, C.c_int, C.c_longlong, C.c_longlong, vp, vp, vp, vp, vp, C.c_float,
                                            vp, vp, C.c_int, vp, vp, vp, vp, vp, C.c_int, C.c_int, C.c_int,
                                            C.c_int, C.c_int, C.c_float, vp]),
    "bcg_decode_attn_paged_static": (C.c_int, [vp, vp, vp, C.c_int, vp, vp, C.c_int, C.c_int, C.c_int,
                                               C.c_int, C.c_int, C.c_float, vp]),
    "bcg_prefill_attn_paged": (C.c_int, [vp, vp, vp, C.c_int, vp, C.c_int, vp, C.c_int, C.c_int, C.c_int,
                                         C.c_int, C.c_float, vp]),
    "bcg_mask_sample": (C.c_int, [C.POINTER(SamplerArgs), vp]),
    "bcg_tp_unique_id": (C.c_int, [vp]),
    "bcg_tp_init": (C.c_int, [vp, C.c_int, C.c_int]),
    "bcg_tp_shutdown": (C.c_int, []),
    "bcg_tp_symm_bytes_for": (C.c_longlong, [C.c_longlong, C.c_int]),
    "bcg_tp_symm_create": (C.c_int, [C.c_longlong, vp]),
    "bcg_tp_add_norm_stats": (C.c_int, [vp, vp, C.c_int, C.c_longlong, vp, vp, vp, C.c_int, C.c_longlong,
                                        C.c_int, C.c_int, vp]),
    "bcg_tp_symm_open": (C.c_int, [vp, C.c_int, C.c_int]),
    "bcg_model_prefill": (C.c_int, [C.POINTER(Model), C.POINTER(Workspace), vp, vp, vp, vp, C.c_int,
                                    vp, C.c_int, vp, C.c_int, C.c_int, vp]),
    "bcg_model_head": (C.c_int, [C.POINTER(Model), C.POINTER(Workspace), vp, C.c_int, C.c_int, vp]),
    "bcg_model_decode": (C.c_int, [C.POINTER(Model), C.POINTER(Workspace), vp, vp, vp, vp, vp,
                                   C.c_int, C.c_int, C.c_int, vp]),
    "bcg_stack_step": (C.c_int, [C.POINTER(Stack), C.POINTER(StackWs), C.POINTER(StepBatch), vp]),
    "bcg_stack_head": (C.c_int, [C.POINTER(Stack), C.POINTER(StackWs), vp, C.c_int, C.c_int, C.c_int, vp]),
    "bcg_gemm_any": (C.c_int, [vp, C.c_int, vp, vp, C.c_int, C.c_int, C.c_int, C.c_longlong, C.c_longlong,
                               C.c_longlong, vp]),
    "bcg_sandwich_norm": (C.c_int, [vp, vp, C.c_int, C.c_longlong, vp, vp, vp, C.c_int, C.c_int, C.c_int, C.c_float,
                                    vp]),
    "bcg_residual_norm": (C.c_int, [vp, vp, C.c_int, C.c_longlong, vp, vp, vp, vp, C.c_int, C.c_int, C.c_longlong, vp, vp, vp,
                                    C.c_int, C.c_int, C.c_int, C.c_float, vp]),
    "bcg_poly_norm": (C.c_int, [vp, C.c_int, C.c_longlong, vp, vp, C.c_int, C.c_int, C.c_int, C.c_float, vp]),
    "bcg_delta_scan": (C.c_int, [C.POINTER(Layer), vp, C.c_int, C.c_longlong, C.c_longlong, vp, C.c_int,
                                 C.c_longlong, vp, vp, vp, vp, C.c_int, vp, C.c_int, C.c_float, vp]),
    "bcg_latent_attention": (C.c_int, [C.POINTER(Stack), C.POINTER(StackWs), C.POINTER(StepBatch), C.c_int, C.c_int,
                                       vp]),
    "bcg_grouped_in": (C.c_int, [C.POINTER(Stack), C.POINTER(StackWs), C.POINTER(StepBatch), C.c_int, C.c_int,
                                 C.c_longlong, C.c_longlong, C.c_int, vp]),
    "bcg_grouped_attention": (C.c_int, [C.POINTER(Stack), C.POINTER(StackWs), C.POINTER(StepBatch), C.c_int, C.c_int,
                                        vp]),
    "bcg_gemm_grouped": (C.c_int, [vp, vp, vp, C.c_int, C.c_int, C.c_int, vp, C.c_int, C.c_int, C.c_int, vp, C.c_float,
                                   C.c_float, C.c_int, vp]),
    "bcg_state_space": (C.c_int, [C.POINTER(Stack), C.POINTER(StackWs), C.POINTER(StepBatch), C.c_int, C.c_int,
                                  C.c_longlong, C.c_longlong, C.c_int, vp]),
    "bcg_clamped_glu": (C.c_int, [vp, C.c_int, C.c_longlong, vp, C.c_int, C.c_int, C.c_int, C.c_float, C.c_float, vp]),
    "bcg_gemm_bf16_glu": (C.c_int, [vp, vp, vp, C.c_int, C.c_int, C.c_int, C.c_float, C.c_float, C.c_int, vp]),
    "bcg_gelu_unit": (C.c_int, [vp, C.c_int, C.c_longlong, vp, C.c_int, C.c_int, C.c_int, C.c_int, vp]),
    "bcg_gemm_bf16_gelu": (C.c_int, [vp, vp, vp, C.c_int, C.c_int, C.c_int, C.c_int, C.c_int, vp]),
    "bcg_gemm_grouped_gelu": (C.c_int, [vp, vp, vp, C.c_int, C.c_int, C.c_int, vp, C.c_int, C.c_int, C.c_int, vp]),
    "bcg_expert_in": (C.c_int, [C.POINTER(Stack), C.POINTER(StackWs), C.c_int, C.c_int, C.c_int, C.c_longlong, C.c_longlong, C.c_int,
                                vp]),
    "bcg_matrix_memory": (C.c_int, [C.POINTER(Stack), C.POINTER(StackWs), C.POINTER(StepBatch), C.c_int, C.c_int,
                                    C.c_longlong, C.c_longlong, C.c_int, vp]),
    "bcg_experts": (C.c_int, [C.POINTER(Stack), C.POINTER(StackWs), C.c_int, C.c_int, c_int_p, vp]),
}

EXPORTED = tuple(_SIGS)

_lib = None


def load(build_if_missing: bool = False) -> C.CDLL:
    """dlopen the in-tree library; raise (never fall back) if it is absent."""
    global _lib
    if _lib is not None:
        return _lib
    if not LIB_PATH.exists():
        if build_if_missing:
            from . import build as _build
            _build.build()
        else:
            raise BcgError(
                f"{LIB_PATH} is missing: run `python -m byzantine_consensus_llm_agents_b200.build` "
                "(there is no CPU fallback)")
    lib = C.CDLL(str(LIB_PATH))
    for name, (res, args) in _SIGS.items():
        fn = getattr(lib, name)
        fn.restype = res
        fn.argtypes = args
    _lib = lib
    return lib


def check(rc: int, what: str = "") -> None:
    if rc != 0:
        msg = load().bcg_last_error()
        raise BcgError(f"{what or 'bcg call'} failed (status {rc}): "
                       f"{msg.decode() if msg else ''}")


def ptr(t) -> int:
    """Device pointer of a torch tensor (or None -> NULL)."""
    return None if t is None else t.data_ptr()


def stream_ptr() -> int:
    import torch
    return torch.cuda.current_stream().cuda_stream


# ---- thin per-kernel wrappers (tensors in, status checked) ---------------------------------

def gemm(x, w, out, epilogue=EPI_BF16, splits=1, flags=0, M=None):
    """out = x @ w.T through bcg_gemm_bf16_tn.  x [M,K] bf16, w [N,K] bf16."""
    lib = load()
    M = x.shape[0] if M is None else M
    K = x.shape[1]
    N = w.shape[0]
    ld_out = out.stride(-2)
    check(lib.bcg_gemm_bf16_tn(ptr(x), ptr(w), ptr(out), M, N, K, x.stride(0), w.stride(0), ld_out,
                               epilogue, splits, flags, stream_ptr()), "bcg_gemm_bf16_tn")
    return out


def splits_for(M, N, K) -> int:
    return load().bcg_gemm_splits_for(M, N, K)
