"""Throughput of a layer-stack design beside a uniform dense decoder of equal size (bench.py --design).

For each size: prefill tokens/s (8 prompts of 1,536 tokens in one launch, and a single one), decode tokens/s at
8 and 64 rows with 1,600 tokens of context (the decode step as the engine captures it, without the sampler),
end-to-end generation through Engine.generate, and the kernels that differ between the two, one by one, each with
its roofline (measured HBM bandwidth and bf16 rate; nominal fp32 FMA rate for the recurrence, which runs on CUDA
cores in fp32).  A design with experts is measured twice: with dense feed-forwards of the dense model's size, and with
experts whose active part has that size.  Random-init weights.  Times are CUDA events; weights of a step (over 1 GB) exceed L2, single
kernels are timed with L2 flushed before every launch.  The reference has no counterpart.
"""
from __future__ import annotations

import ctypes as C
import time

import numpy as np
import torch

from . import lib as L
from . import model as M
from . import stack as S
from .engine import Engine, Request
from .executors import PAGE, Entry
from .tokenizer import get_tokenizer

# name -> (width, dense ff, layers): widths and feed-forward sizes of 1-2B / 8B class models.  Fewer layers than a whole
# model (layers repeat; throughput per layer is what is compared), the same vocabulary.
SIZES = {"2k": (2048, 6144, 8), "4k": (4096, 12288, 8)}
# a stack's ff makes its layers (no gate matrix, other mixer projections) the dense layers' size
BEKOPEL_FF = {"2k": 7424, "4k": 14592}
MERULORN_FF = {"2k": 11520, "4k": 23680}       # of one layer in four; the others have none
VOSOLORN_FF, VOSOLORN_EXPERT_FF = {"2k": 5632, "4k": 10752}, {"2k": 960, "4k": 1792}     # one expert in TOP + 1 is the shared one
EXPERTS, TOP = 64, 8
VOCAB, CTX, PROMPT, PROMPTS = 32768, 1600, 1536, 8
FP32_FMA = 148 * 128 * 1.965e9       # nominal
KINDS = {"bekopel": ("qwen3", "bekopel"), "lerazen": ("qwen3", "lerazen", "lerazen-moe"),
         "merulorn": ("qwen3", "bekopel", "merulorn"),
         "vosolorn": ("qwen3", "merulorn", "lerazen-moe", "vosolorn", "vosolorn-moe")}


def _config(kind: str, size: str):
    d, ff, layers = SIZES[size]
    name, heads = f"{kind}-{size}", d // 128
    if kind == "bekopel":
        return S.bekopel_preset(name, layers, d, BEKOPEL_FF[size], VOCAB, heads=heads)
    if kind == "merulorn":
        return S.merulorn_preset(name, layers, d, MERULORN_FF[size], VOCAB, heads=heads)
    if kind.startswith("vosolorn"):
        return S.vosolorn_preset(name, layers, d, VOSOLORN_FF[size], VOCAB, heads=heads, experts=EXPERTS if kind.endswith("moe") else 0,
                                 top=TOP, expert_ff=VOSOLORN_EXPERT_FF[size])
    if kind.startswith("lerazen"):      # two matrices instead of three; experts: three matrices, TOP of them active
        return S.lerazen_preset(name, layers, d, ff * 3 // 2, VOCAB, heads=heads, kv_heads=8,
                                experts=EXPERTS if kind.endswith("moe") else 0, top=TOP, expert_ff=ff // TOP)
    return M.ModelConfig(name, layers, d, heads, 8, ff, VOCAB)


def _engine(kind: str, size: str, tokenizer) -> Engine:
    cfg = _config(kind, size)
    w = M.weights_for(cfg).random_init(cfg, torch.device("cuda:0"))
    return Engine(cfg, w, tokenizer, max_model_len=2048, max_rows=64, prefill_tokens=PROMPTS * PROMPT, kv_pages=64 * 128)


def _events(fn, n: int, warm: int = 3, flush=None) -> float:
    """Milliseconds per call; with `flush`, every call is timed alone after L2 has been overwritten."""
    ev = lambda: torch.cuda.Event(enable_timing=True)
    for _ in range(warm):
        fn()
    torch.cuda.synchronize()
    if flush is None:
        a, b = ev(), ev()
        a.record()
        for _ in range(n):
            fn()
        b.record()
        torch.cuda.synchronize()
        return a.elapsed_time(b) / n
    pairs = []
    for _ in range(n):
        flush.zero_()
        a, b = ev(), ev()
        a.record()
        fn()
        b.record()
        pairs.append((a, b))
    torch.cuda.synchronize()
    return float(np.median([a.elapsed_time(b) for a, b in pairs]))


def _prefill(e: Engine, n: int):
    """A launch of n prompts, staged once."""
    rng = np.random.default_rng(0)
    entries = []
    for i in range(n):
        bt = np.zeros(e.max_blocks, np.int32)
        bt[:128] = np.arange(128) + i * 128
        entries.append(Entry(rng.integers(0, VOCAB, PROMPT).tolist(), 0, bt, i, (PROMPT - 1,)))
    plan, views, _ = e._launch_group(entries, 0)
    return plan, views


def _decode_rows(e: Engine, B: int) -> None:
    r = e.row
    r["positions"][:B], r["seq_lens"][:B] = CTX - 1, CTX
    r["state_slot"][:B] = torch.arange(B, device="cuda").int()
    r["next_ids"][:B] = torch.arange(B, device="cuda").int()
    r["block_table"][:, :128] = torch.arange(64 * 128, device="cuda").int().view(64, 128)
    r["slot_map"][:B] = (torch.arange(B, device="cuda") * 128 * PAGE + CTX - 1).int()


def _graph(fn, times: int = 1):
    fn()
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        for _ in range(times):
            fn()
    return g.replay


class _Bench:
    """Rows {kernel, shape, us, ideal_us, x_ideal} of single kernels of an engine."""

    def __init__(self, e: Engine, hbm: float, tf: float):
        self.e, self.hbm, self.tf, self.rows = e, hbm, tf, []
        self.flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")

    def add(self, name, shape, fn, nbytes=0.0, flops=0.0, fma=0.0):
        L.check(fn())
        us = _events(fn, 20, 3, self.flush) * 1e3
        ideal = max(nbytes / self.hbm * 1e-3, flops / self.tf * 1e-6, fma / FP32_FMA * 1e6)
        self.rows.append({"kernel": name, "shape": shape, "us": round(us, 1), "ideal_us": round(ideal, 1),
                          "x_ideal": round(us / max(ideal, 1e-3), 2)})

    def gemm(self, name, shape, x, w, out, M_, N, K, epi, splits):
        """A plain projection; out holds fp32 slabs, or bf16 columns of an epilogue."""
        size = {L.EPI_F32: 4.0 * splits, L.EPI_SWIGLU: 1.0}.get(epi, 2.0)
        ld = N // 2 if epi == L.EPI_SWIGLU else N
        self.add(name, shape, lambda: self.e.lib.bcg_gemm_bf16_tn(
            x.data_ptr(), w.data_ptr(), out.data_ptr(), M_, N, K, K, K, ld, epi, splits, 0, L.stream_ptr()),
            nbytes=2.0 * N * K + 2.0 * M_ * K + size * M_ * N, flops=2.0 * M_ * N * K)


def _dense_kernels(k: _Bench, what: str, B: int, T: int, shape: str, v, plan) -> None:
    e, b, cfg, lib, st = k.e, k.e.buf, k.e.cfg, k.e.lib, L.stream_ptr
    d, hq, hkv = cfg.d_model, cfg.n_heads, cfg.n_kv_heads
    if what == "prefill":
        keys = PROMPT * (PROMPT + 1) // 2
        k.add("attention", shape, lambda: lib.bcg_prefill_attn_paged(
            b["q"].data_ptr(), e.kv_layers[0].data_ptr(), v["bt"].data_ptr(), e.max_blocks, v["tiles"].data_ptr(),
            plan.extra["n_tiles"], b["attn"].data_ptr(), T, hq, hkv, PAGE, 128 ** -0.5, st()), flops=4.0 * B * keys * hq * 128)
        k.add("norm", shape, lambda: lib.bcg_add_rmsnorm(
            b["residual"].data_ptr(), b["delta"].data_ptr(), 1, 1, 0, e.w.ln1[0].data_ptr(), b["xn"].data_ptr(), None, T, d, 1e-6,
            st()), nbytes=T * d * 14.0)
        k.add("input split", shape, lambda: lib.bcg_qknorm_rope_kvwrite(
            b["qkv"].data_ptr(), 1, 1, 0, cfg.qkv_dim, e.w.q_norm[0].data_ptr(), e.w.k_norm[0].data_ptr(), e.w.cos_sin.data_ptr(),
            v["pos"].data_ptr(), v["slots"].data_ptr(), b["q"].data_ptr(), e.kv_layers[0].data_ptr(), T, hq, hkv, PAGE, 1e-6,
            st()), nbytes=T * cfg.qkv_dim * 6.0)
        k.gemm("up product", shape, b["xn"], e.w.w_gate_up[0], b["act"], T, 2 * cfg.d_ff, d, L.EPI_SWIGLU, 1)
        k.gemm("down product", shape, b["act"], e.w.w_down[0], b["delta"], T, d, cfg.d_ff, L.EPI_F32, 1)
        return
    r, parts = e.row, 4
    k.add("attention", shape, lambda: lib.bcg_decode_attn_paged(
        b["q"].data_ptr(), e.kv_layers[0].data_ptr(), r["block_table"].data_ptr(), e.max_blocks, r["seq_lens"].data_ptr(),
        b["attn"].data_ptr(), b["so"].data_ptr(), b["sml"].data_ptr(), b["attn_counters"].data_ptr(), B, hq, hkv, PAGE,
        (CTX + 255) // 256, 128 ** -0.5, st()), nbytes=B * CTX * hkv * 512.0)
    k.add("norm", shape, lambda: lib.bcg_add_norm_stats(
        b["residual"].data_ptr(), b["partials"].data_ptr(), 1, parts, B * d, e.w.ln1[0].data_ptr(), b["xn"].data_ptr(),
        b["row_sumsq"].data_ptr(), B, d, st()), nbytes=B * d * (10.0 + 4 * parts))
    s = L.splits_for(B, cfg.qkv_dim, d)
    k.add("input split", shape, lambda: lib.bcg_qknorm_rope_kvwrite(
        b["partials"].data_ptr(), 1, s, B * cfg.qkv_dim, cfg.qkv_dim, e.w.q_norm[0].data_ptr(), e.w.k_norm[0].data_ptr(),
        e.w.cos_sin.data_ptr(), r["positions"].data_ptr(), r["slot_map"].data_ptr(), b["q"].data_ptr(), e.kv_layers[0].data_ptr(), B,
        hq, hkv, PAGE, 1e-6, st()), nbytes=B * cfg.qkv_dim * (4.0 * s + 2))
    k.add("activation", shape, lambda: lib.bcg_swiglu_reduce(
        b["partials"].data_ptr(), 2, B * 2 * cfg.d_ff, b["act"].data_ptr(), B, 2 * cfg.d_ff, st()), nbytes=B * cfg.d_ff * (16.0 + 2))
    s = L.splits_for(B, 2 * cfg.d_ff, d)
    k.gemm("up product", shape, b["xn"], e.w.w_gate_up[0], b["partials"], B, 2 * cfg.d_ff, d, L.EPI_F32 if s > 1 else L.EPI_SWIGLU, s)
    k.gemm("down product", shape, b["act"], e.w.w_down[0], b["partials"], B, d, cfg.d_ff, L.EPI_F32, L.splits_for(B, d, cfg.d_ff))


def _step_batch(e: Engine, what: str, T: int, B: int, v, plan) -> L.StepBatch:
    bt = e.exec._batch(T, B)
    if what == "prefill":
        bt.positions, bt.slot_map, bt.row_seq = v["pos"].data_ptr(), v["slots"].data_ptr(), v["row_seq"].data_ptr()
        bt.seq_start, bt.block_table, bt.state_slots = v["seq_start"].data_ptr(), v["bt"].data_ptr(), v["state_slots"].data_ptr()
        bt.tiles, bt.n_tiles = v["tiles"].data_ptr(), plan.extra["n_tiles"]
        bt.gather, bt.n_gather, bt.max_context = v["gather"].data_ptr(), plan.extra["n_gather"], 1
    else:
        r = e.row
        bt.positions, bt.slot_map, bt.block_table = r["positions"].data_ptr(), r["slot_map"].data_ptr(), r["block_table"].data_ptr()
        bt.state_slots, bt.max_context = r["state_slot"].data_ptr(), CTX
    return bt


def _window_keys(window: int) -> int:
    """(query, key) pairs of a prompt."""
    w = min(window, PROMPT)
    return w * (w + 1) // 2 + (PROMPT - w) * w


def _bekopel_kernels(k: _Bench, what: str, B: int, T: int, shape: str, v, plan) -> None:
    e, b, cfg, lib, x, st = k.e, k.e.buf, k.e.cfg, k.e.lib, k.e.exec, L.stream_ptr
    d, parts = cfg.d_model, 1 if what == "prefill" else 4
    i_attn = next(i for i, l in enumerate(cfg.layers) if isinstance(l.mixer, S.LatentAttention))
    i_delta = next(i for i, l in enumerate(cfg.layers) if isinstance(l.mixer, S.GeneralDelta))
    m, dl, ff = cfg.layers[i_attn].mixer, cfg.layers[i_delta].mixer, cfg.layers[0].mlp.ff
    wl, n = e.w.layers[i_delta], dl.out_dim
    bt = _step_batch(e, what, T, B, v, plan)
    if what == "prefill":
        cost = dict(flops=2.0 * T * m.heads * (m.dim + m.vdim) * m.kv_rank
                    + 2.0 * B * _window_keys(m.window) * m.heads * (m.dim + m.rot_dim + m.vdim))
        cost_d = dict(fma=4.5 * T * dl.heads * dl.dim ** 2)
    else:
        cost = dict(nbytes=B * m.window * m.cache_row * 2.0 + 2.0 * m.heads * (m.dim + m.vdim) * m.kv_rank)
        cost_d = dict(nbytes=B * dl.heads * dl.dim ** 2 * 8.0)
    k.add("attention", shape, lambda: lib.bcg_latent_attention(
        C.byref(x.model.struct), C.byref(x.ws), C.byref(bt), i_attn, 0, st()), **cost)
    k.add("delta rule", shape, lambda: lib.bcg_delta_scan(
        C.byref(x.model.struct.layers[i_delta]), b["proj"].data_ptr(), parts, T * cfg.in_rows(i_delta), cfg.in_rows(i_delta),
        b["decay"].data_ptr(), 1, T * n, bt.positions, bt.slot_map, bt.seq_start, bt.state_slots, B, b["mix"].data_ptr(),
        L.DT_BF16, 1e-5, st()), **cost_d)
    k.add("norm", shape, lambda: lib.bcg_sandwich_norm(
        b["residual"].data_ptr(), b["proj"].data_ptr(), parts, T * d, wl["norm1b"].data_ptr(), wl["norm2"].data_ptr(),
        b["xn"].data_ptr(), L.DT_BF16, T, d, 1e-5, st()), nbytes=T * d * (10.0 + 4 * parts))
    k.add("activation", shape, lambda: lib.bcg_poly_norm(
        b["proj"].data_ptr(), min(parts, 2), T * ff, wl["act_coef"].data_ptr(), b["act"].data_ptr(), L.DT_BF16, T, ff, 1e-5,
        st()), nbytes=T * ff * (2.0 + 4 * min(parts, 2)))


def _route_at_random(k: _Bench, layer: int, T: int) -> int:
    """The routing buffers of a layer as T tokens with random experts fill them; returns how many experts are used."""
    b, f = k.e.buf, k.e.cfg.layers[layer].mlp
    rows = T * f.top
    pick = torch.rand(T, f.experts, generator=torch.Generator().manual_seed(0)).topk(f.top).indices.cuda()
    counts = torch.bincount(pick.flatten(), minlength=f.experts)
    order = pick.flatten().argsort(stable=True)
    rank = torch.empty(rows, dtype=torch.int64, device="cuda")
    rank[order] = torch.arange(rows, device="cuda")
    rank -= (counts.cumsum(0) - counts)[pick.flatten()]
    at = k.e.exec.model.struct.layers[layer].moe_counts_at
    b["moe_counts"][at:at + f.experts], b["moe_expert"][:rows], b["moe_rank"][:rows] = counts.int(), pick.flatten().int(), rank.int()
    b["moe_weight"][:rows] = 0.7
    return int((counts > 0).sum())


def _lerazen_kernels(k: _Bench, what: str, B: int, T: int, shape: str, v, plan) -> None:
    e, b, cfg, lib, x, st = k.e, k.e.buf, k.e.cfg, k.e.lib, k.e.exec, L.stream_ptr
    d, layer = cfg.d_model, cfg.n_layers - 1
    m, f, w = cfg.layers[layer].mixer, cfg.layers[layer].mlp, e.w.layers[layer]
    moe, prefill = isinstance(f, S.MoeMlp), what == "prefill"
    bt = _step_batch(e, what, T, B, v, plan)
    model, ws = C.byref(x.model.struct), C.byref(x.ws)
    kv = m.kv_heads * (m.dim + m.vdim)
    k.add("attention", shape, lambda: lib.bcg_grouped_attention(model, ws, C.byref(bt), layer, 0, st()),
          **(dict(flops=2.0 * B * _window_keys(m.window) * m.heads * (m.dim + m.vdim)) if prefill
             else dict(nbytes=B * min(m.window, CTX) * kv * 2.0)))
    # decode: one product makes q | k | v and the up rows, and one kernel takes them apart
    n_in = cfg.qkv_rows(layer) if prefill and not moe else cfg.in_rows(layer)
    s = 1 if prefill else L.splits_for(B, n_in, d)
    k.add("input split", shape, lambda: lib.bcg_grouped_in(model, ws, C.byref(bt), layer, s, T * n_in, n_in, int(not prefill), st()),
          nbytes=T * n_in * (4.0 * s + 2) + T * m.kv_heads * m.vdim * 4.0)
    if moe:
        top, ff, rows = f.top, f.ff_ld, T * f.top
        used, splits = _route_at_random(k, layer, T), C.c_int()
        cp = b["moe_counts"].data_ptr() + 4 * x.model.struct.layers[layer].moe_counts_at
        s1, s2 = (1, 1) if prefill else (L.splits_for(1, top * 2 * ff, d), L.splits_for(1, top * d, ff))
        size = 2.0 if prefill else 8.0 * s1
        k.add("experts, all launches", shape, lambda: lib.bcg_experts(model, ws, layer, T, C.byref(splits), st()),
              nbytes=used * 6.0 * ff * d + rows * d * 4.0, flops=6.0 * rows * ff * d)
        k.add("up product", shape, lambda: lib.bcg_gemm_grouped(
            b["moe_x"].data_ptr(), w["w_experts_in"].data_ptr(), (b["moe_h"] if prefill else b["moe_proj"]).data_ptr(), rows, 2 * ff, d,
            cp, f.experts, T, s1, b["moe_row_weight"].data_ptr() if prefill else None, f.limit, f.alpha, 0, st()),
            nbytes=used * 4.0 * ff * d + rows * (2.0 * d + size * ff), flops=4.0 * rows * ff * d)
        k.add("down product", shape, lambda: lib.bcg_gemm_grouped(
            b["moe_h"].data_ptr(), w["w_experts_out"].data_ptr(), b["moe_out"].data_ptr(), rows, d, ff, cp, f.experts, T, s2, None, 0.0,
            0.0, 0, st()), nbytes=used * 2.0 * ff * d + rows * (2.0 * ff + 4.0 * s2 * d), flops=2.0 * rows * ff * d)
        extra = (b["moe_out"].data_ptr(), b["moe_row"].data_ptr(), None, top, s2, rows * d)
    else:
        act_col, cols = cfg.mix_cols(layer)
        out = b["mix"][act_col:]
        up = w["w_in"][cfg.qkv_rows(layer):]
        if prefill:
            k.gemm("up product", shape, b["xn"], up, out[:T * (cols - act_col)], T, cols - act_col, d, L.EPI_RELU2, 1)
        else:
            k.gemm("up product", shape, b["xn"], w["w_in"], b["proj"], B, n_in, d, L.EPI_F32, s)
        extra = (None, None, None, 0, 1, 0)
    cols = cfg.mix_cols(layer)[1]
    s3 = 1 if prefill else L.splits_for(B, d, cols)
    k.gemm("output product" if moe else "down product", shape, b["mix"], w["w_out"], b["proj"], T, d, cols, L.EPI_F32, s3)
    k.add("norm", shape, lambda: lib.bcg_residual_norm(
        b["residual"].data_ptr(), b["proj"].data_ptr(), s3, T * d, w["out_bias"].data_ptr(), *extra, None, w["norm1"].data_ptr(),
        b["xn"].data_ptr(), L.DT_BF16, T, d, 1e-5, st()), nbytes=T * d * (10.0 + 4 * s3 + 4 * extra[3] * extra[4]))


def _merulorn_kernels(k: _Bench, what: str, B: int, T: int, shape: str, v, plan) -> None:
    e, b, cfg, lib, x, st = k.e, k.e.buf, k.e.cfg, k.e.lib, k.e.exec, L.stream_ptr
    d, layer = cfg.d_model, next(i for i, l in enumerate(cfg.layers) if l.one(S.GroupedAttention))
    spec, w, prefill = cfg.layers[layer], e.w.layers[layer], what == "prefill"
    m, ssm, f = spec.one(S.GroupedAttention), spec.one(S.StateSpace), spec.mlp
    bt = _step_batch(e, what, T, B, v, plan)
    model, ws = C.byref(x.model.struct), C.byref(x.ws)
    n_in, cols = cfg.in_rows(layer), cfg.mix_cols(layer)[1]
    splits = lambda n, kk: 1 if prefill else L.splits_for(B, n, kk)
    s, s3 = splits(n_in, d), splits(d, cols)
    keys = PROMPT * (PROMPT + 1) // 2
    k.add("attention", shape, lambda: lib.bcg_grouped_attention(model, ws, C.byref(bt), layer, 0, st()),
          **(dict(flops=2.0 * B * keys * m.heads * (m.dim + m.vdim)) if prefill
             else dict(nbytes=B * CTX * m.kv_heads * (m.dim + m.vdim) * 2.0)))
    k.add("input split", shape, lambda: lib.bcg_grouped_in(model, ws, C.byref(bt), layer, s, T * n_in, n_in, 0, st()),
          nbytes=T * m.in_dim * (4.0 * s + 2))
    # the projection in, outputs out, states in and out; the products of 64-token chunks
    k.add("state space, all launches", shape, lambda: lib.bcg_state_space(model, ws, C.byref(bt), layer, s, T * n_in, n_in, 0, st()),
          nbytes=T * (ssm.in_dim * 4.0 * s + ssm.out_dim * 2) + B * ssm.state_floats * 8.0,
          flops=2.0 * T * (ssm.heads * ssm.vdim * (32 + 2 * ssm.state) + ssm.groups * 32 * ssm.state) if prefill else 0.0)
    k.add("norm", shape, lambda: lib.bcg_sandwich_norm(
        b["residual"].data_ptr(), b["proj"].data_ptr(), s3, T * d, None, w["norm2"].data_ptr(), b["xn"].data_ptr(), L.DT_BF16, T, d,
        1e-5, st()), nbytes=T * d * (10.0 + 4 * s3))
    k.gemm("input product", shape, b["xn"], w["w_in"], b["proj"], T, n_in, d, L.EPI_F32, s)
    n_up = f.up_rows
    if prefill or splits(n_up, d) == 1:
        k.add("up product", shape, lambda: lib.bcg_gemm_bf16_glu(
            b["xn"].data_ptr(), w["w_up"].data_ptr(), b["act"].data_ptr(), T, n_up, d, f.limit, f.alpha, 0, st()),
            nbytes=2.0 * n_up * d + 2.0 * T * d + T * n_up, flops=2.0 * T * n_up * d)
    else:
        k.gemm("up product", shape, b["xn"], w["w_up"], b["proj"], T, n_up, d, L.EPI_F32, splits(n_up, d))
        k.add("activation", shape, lambda: lib.bcg_clamped_glu(
            b["proj"].data_ptr(), splits(n_up, d), T * n_up, b["act"].data_ptr(), L.DT_BF16, T, f.ff_ld, f.limit, f.alpha, st()),
            nbytes=T * f.ff_ld * (8.0 * splits(n_up, d) + 2))
    k.gemm("down product", shape, b["act"], w["w_down"], b["proj"], T, d, f.ff_ld, L.EPI_F32, splits(d, f.ff_ld))
    k.gemm("output product", shape, b["mix"], w["w_out"], b["proj"], T, d, cols, L.EPI_F32, s3)


def _vosolorn_kernels(k: _Bench, what: str, B: int, T: int, shape: str, v, plan) -> None:
    e, b, cfg, lib, x, st = k.e, k.e.buf, k.e.cfg, k.e.lib, k.e.exec, L.stream_ptr
    d, prefill = cfg.d_model, what == "prefill"
    i_att = max(i for i, l in enumerate(cfg.layers) if l.one(S.GroupedAttention))
    i_mem = max(i for i, l in enumerate(cfg.layers) if l.one(S.MatrixMemory))
    m, mem, f, w = cfg.layers[i_att].mixer, cfg.layers[i_mem].mixer, cfg.layers[i_mem].mlp, e.w.layers[i_mem]
    bt = _step_batch(e, what, T, B, v, plan)
    model, ws = C.byref(x.model.struct), C.byref(x.ws)
    splits = lambda n, kk: 1 if prefill else L.splits_for(B, n, kk)
    blocks = lambda ctx: max(0, ctx - m.window) // m.pool
    n_in, n_mem, s_out = cfg.in_rows(i_att), cfg.in_rows(i_mem), splits(d, mem.out_dim)
    s, s_mem = splits(n_in, d), splits(n_mem, d)
    pairs = _window_keys(m.window) + sum(blocks(p + 1) for p in range(PROMPT))
    k.add("attention", shape, lambda: lib.bcg_grouped_attention(model, ws, C.byref(bt), i_att, 0, st()),
          **(dict(flops=2.0 * B * pairs * m.heads * (m.dim + m.vdim)) if prefill
             else dict(nbytes=B * (min(m.window, CTX) + blocks(CTX)) * m.kv_heads * (m.dim + m.vdim) * 2.0)))
    k.add("input split", shape, lambda: lib.bcg_grouped_in(model, ws, C.byref(bt), i_att, s, T * n_in, n_in, 0, st()),
          nbytes=T * m.in_dim * (4.0 * s + 2))
    # operands in (prompts: activations and fp32 gates), outputs out, states in and out; the products of 64-token chunks
    ld, mode = (n_mem - mem.gate_col, 2) if prefill else (n_mem, 0)
    operands = mem.x_ld * 2.0 + 8.0 * mem.heads if prefill else mem.in_dim * 4.0 * s_mem
    k.add("matrix memory, all launches", shape, lambda: lib.bcg_matrix_memory(model, ws, C.byref(bt), i_mem, s_mem, T * ld, ld, mode, st()),
          nbytes=T * (operands + mem.out_dim * 2) + B * mem.state_floats * 8.0,
          flops=2.0 * T * mem.heads * (mem.vdim * (32 + 2 * mem.dim) + 32 * mem.dim) if prefill else 0.0)
    k.add("norm", shape, lambda: lib.bcg_sandwich_norm(
        b["residual"].data_ptr(), b["proj"].data_ptr(), s_out, T * d, w["norm1b"].data_ptr(), None, b["xn"].data_ptr(), L.DT_BF16, T, d,
        1e-5, st()), nbytes=T * d * (10.0 + 4 * s_out))
    if prefill:
        k.gemm("input product", shape, b["xn"], w["w_in"], b["ssm_x"], T, mem.gate_col, d, L.EPI_BF16, 1)
        k.gemm("gate product", shape, b["xn"], w["w_in"][mem.gate_col:], b["proj"], T, n_mem - mem.gate_col, d, L.EPI_F32, 1)
    else:
        k.gemm("input product", shape, b["xn"], w["w_in"], b["proj"], T, n_mem, d, L.EPI_F32, s_mem)
    k.gemm("output product", shape, b["mix"], w["w_out"], b["proj"], T, d, mem.out_dim, L.EPI_F32, s_out)
    if isinstance(f, S.MoeMlp):
        used, rows, ff = _route_at_random(k, i_mem, T), T * f.top, f.ff_ld
        out = C.c_int()
        k.add("experts, all launches", shape, lambda: lib.bcg_experts(model, ws, i_mem, T, C.byref(out), st()),
              nbytes=used * 4.0 * ff * d + rows * d * 4.0, flops=4.0 * rows * ff * d)
        n = f.router_rows + f.shared_ld
        k.gemm("router and shared product", shape, b["xn"], w["w_up"], b["proj"], T, n, d, L.EPI_F32, splits(n, d))
        s_sh = splits(d, f.shared_ld)
        k.add("norm with experts", shape, lambda: lib.bcg_residual_norm(
            b["residual"].data_ptr(), b["proj"].data_ptr(), s_sh, T * d, None, b["moe_out"].data_ptr(), b["moe_row"].data_ptr(),
            b["moe_weight"].data_ptr(), f.top, out.value, rows * d, w["norm2b"].data_ptr(), None, b["xn"].data_ptr(), L.DT_BF16, T, d, 1e-5,
            st()), nbytes=T * d * (10.0 + 4 * s_sh + 4 * f.top * out.value))
        return
    n_up = f.up_rows
    if splits(n_up, d) == 1:
        k.add("up product", shape, lambda: lib.bcg_gemm_bf16_gelu(
            b["xn"].data_ptr(), w["w_up"].data_ptr(), b["act"].data_ptr(), T, n_up, d, 1, 0, st()),
            nbytes=2.0 * n_up * d + 2.0 * T * d + T * n_up, flops=2.0 * T * n_up * d)
    else:
        k.gemm("up product", shape, b["xn"], w["w_up"], b["proj"], T, n_up, d, L.EPI_F32, splits(n_up, d))
        k.add("activation", shape, lambda: lib.bcg_gelu_unit(
            b["proj"].data_ptr(), splits(n_up, d), T * n_up, b["act"].data_ptr(), L.DT_BF16, T, f.ff_ld, 1, st()),
            nbytes=T * f.ff_ld * (8.0 * splits(n_up, d) + 2))
    k.gemm("down product", shape, b["act"], w["w_down"], b["proj"], T, d, f.ff_ld, L.EPI_F32, splits(d, f.ff_ld))


def _kernels(e: Engine, kind: str, hbm: float, tf: float) -> list:
    k = _Bench(e, hbm, tf)
    run = {"qwen3": _dense_kernels, "bekopel": _bekopel_kernels, "merulorn": _merulorn_kernels, "vosolorn": _vosolorn_kernels,
           "vosolorn-moe": _vosolorn_kernels}.get(kind, _lerazen_kernels)
    for what, B in (("prefill", PROMPTS), ("decode", 8), ("decode", 64)):
        T = B * PROMPT if what == "prefill" else B
        plan, v = _prefill(e, B) if what == "prefill" else (None, None)
        if what == "decode":
            _decode_rows(e, B)
        run(k, what, B, T, f"{what} {T} tokens", v, plan)
    return k.rows


def _run(kind: str, size: str, tokenizer, hbm: float, tf: float, kernels: bool) -> dict:
    e = _engine(kind, size, tokenizer)
    out = {"layers": e.cfg.n_layers, "decode_weight_gb": round(e.cfg.decode_weight_bytes() / 1e9, 3)}
    for n in (PROMPTS, 1):
        plan, views = _prefill(e, n)
        ms = _events(lambda: e.exec.launch(plan, views, 0), 10)
        out[f"prefill_tok_s_{n}x{PROMPT}"] = round(n * PROMPT / ms * 1e3)
    for B in (8, 64):
        _decode_rows(e, B)
        ms = _events(_graph(lambda: e.exec.decode(e.row, B, (CTX + 255) // 256), 4), 20) / 4
        cache = e.cfg.kv_bytes_per_token * (CTX if kind == "qwen3" else min(CTX, e.cfg.max_window or CTX))
        weights = e.cfg.decode_weight_bytes()
        if kind.endswith("-moe"):           # the experts that the step's tokens used
            f = e.cfg.layers[-1].mlp
            used = int((e.buf["moe_counts"][:e.ws.moe_counts_n] > 0).sum())
            weights = e.cfg.decode_weight_bytes(0) + used * (6 if f.glu else 4) * f.ff * e.cfg.d_model
            out[f"experts_used_per_layer_{B}"] = round(used * f.experts / e.ws.moe_counts_n, 1)
        if kind == "bekopel":     # layers that share a cache read it once each; states are read and written
            own = sum(isinstance(l.mixer, S.LatentAttention) for l in e.cfg.layers)
            has = sum(isinstance(l.mixer, S.LatentAttention) and l.mixer.kv_from is None for l in e.cfg.layers)
            cache = cache * own // max(has, 1) + 2 * e.cfg.state_bytes_per_row
        if kind.startswith("vosolorn"):     # the blocks behind the window, too
            cache += sum(e.cfg.pool_bytes_per_block(p) * max(0, CTX - e.cfg.max_window) // p for p in e.cfg.pools)
        if kind == "merulorn" or kind.startswith("vosolorn"):
            cache += 2 * e.cfg.state_bytes_per_row
        out[f"decode_ms_{B}"] = round(ms, 4)
        out[f"decode_tok_s_{B}"] = round(B / ms * 1e3)
        out[f"decode_of_hbm_roofline_{B}"] = round((weights + B * cache) / hbm / ms * 1e-6, 3)
    rng = np.random.default_rng(1)
    reqs = [Request("", prompt_ids=rng.integers(0, 4000, 1024).tolist(), max_tokens=129, forced=[65] * 129) for _ in range(8)]
    e.generate(reqs)
    e.reset_prefix_cache()
    torch.cuda.synchronize()
    t0 = time.perf_counter()
    e.generate(reqs)
    out["generate_tok_s_8x(1024+129)"] = round(8 * 129 / (time.perf_counter() - t0))
    if kernels:
        out["kernels"] = _kernels(e, kind, hbm, tf)
    e.close()
    return out


def run(design: str, hbm_gbs: float, tflops: float, peaks: str, sizes=None, kernels: bool = True) -> dict:
    kinds = KINDS.get(design.lower())
    if kinds is None:
        raise ValueError(f"no layer-stack design {design!r} (there are: {', '.join(KINDS)})")
    tk = get_tokenizer("qwen3", VOCAB)
    res = {}
    for size in sizes or SIZES:
        res[size] = {}
        for kind in kinds:
            res[size][kind] = _run(kind, size, tk, hbm_gbs, tflops, kernels)
            torch.cuda.empty_cache()
    return {"metric": "design_throughput", "design": design, "unit": "tokens/s", "data": "synthetic", "dtype": "bf16",
            "peaks": f"{hbm_gbs} GB/s, {tflops} TFLOP/s ({peaks})",
            "config": {"vocab": VOCAB, "context": CTX, "prompt": PROMPT,
                       "l2": "a step's weights exceed L2; single kernels are timed after an L2 flush"}, "sizes": res}
