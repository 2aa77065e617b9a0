"""Throughput of a layer-stack design beside a uniform dense decoder of equal size (bench.py --design).

For each size: prefill tokens/s (8 prompts of 1,536 tokens in one launch, and a single one), decode tokens/s at
8 and 64 rows with 1,600 tokens of context (the decode step as the engine captures it, without the sampler),
end-to-end generation through Engine.generate, and the kernels that differ between the two, one by one, each with
its roofline (measured HBM bandwidth and bf16 rate; nominal fp32 FMA rate for the recurrence, which runs on CUDA
cores in fp32).  Random-init weights.  Times are CUDA events; weights of a step (over 1 GB) exceed L2, single
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

# name -> (width, dense ff, stack ff, layers): widths and feed-forward sizes of 1-2B / 8B class models; the stack's ff
# makes its layers (no gate matrix, five mixer projections) the dense layers' size.  Fewer layers than a whole
# model (layers repeat; throughput per layer is what is compared), the same vocabulary.
SIZES = {"2k": (2048, 6144, 7424, 8), "4k": (4096, 12288, 14592, 8)}
VOCAB, CTX, PROMPT, PROMPTS = 32768, 1600, 1536, 8
FP32_FMA = 148 * 128 * 1.965e9       # nominal


def _engine(kind: str, size: str, tokenizer) -> Engine:
    d, ff_dense, ff_stack, layers = SIZES[size]
    if kind == "bekopel":
        cfg = S.bekopel_preset(f"bekopel-{size}", layers, d, ff_stack, VOCAB, heads=d // 128)
    else:
        cfg = M.ModelConfig(f"qwen3-{size}", layers, d, d // 128, 8, ff_dense, VOCAB)
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


def _kernels(e: Engine, hbm: float, tf: float) -> list:
    """Rows {kernel, shape, us, ideal_us, x_ideal} of the kernels that are not plain GEMMs."""
    flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
    rows, lib, st, b = [], e.lib, L.stream_ptr, e.buf
    stack = isinstance(e.cfg, S.StackConfig)
    d = e.cfg.d_model

    def add(name, shape, fn, nbytes=0.0, flops=0.0, fma=0.0):
        us = _events(fn, 20, 3, flush) * 1e3
        ideal = max(nbytes / hbm * 1e-3, flops / tf * 1e-6, fma / FP32_FMA * 1e6)
        rows.append({"kernel": name, "shape": shape, "us": round(us, 1), "ideal_us": round(ideal, 1),
                     "x_ideal": round(us / max(ideal, 1e-3), 2)})

    for what, B in (("prefill", PROMPTS), ("decode", 8), ("decode", 64)):
        T = B * PROMPT if what == "prefill" else B
        shape = f"{what} {T} tokens"
        if what == "prefill":
            plan, v = _prefill(e, B)
        else:
            _decode_rows(e, B)
        parts = 1 if what == "prefill" else 4
        if not stack:
            hq, hkv, cfg = e.cfg.n_heads, e.cfg.n_kv_heads, e.cfg
            if what == "prefill":
                keys = PROMPT * (PROMPT + 1) // 2
                add("attention", shape, lambda: L.check(lib.bcg_prefill_attn_paged(
                    b["q"].data_ptr(), e.kv_layers[0].data_ptr(), v["bt"].data_ptr(), e.max_blocks, v["tiles"].data_ptr(),
                    plan.extra["n_tiles"], b["attn"].data_ptr(), T, hq, hkv, PAGE, 128 ** -0.5, st())),
                    flops=4.0 * B * keys * hq * 128)
                add("norm", shape, lambda: L.check(lib.bcg_add_rmsnorm(
                    b["residual"].data_ptr(), b["delta"].data_ptr(), 1, 1, 0, e.w.ln1[0].data_ptr(), b["xn"].data_ptr(), None,
                    T, d, 1e-6, st())), nbytes=T * d * 14.0)
                add("rope + cache write", shape, lambda: L.check(lib.bcg_qknorm_rope_kvwrite(
                    b["qkv"].data_ptr(), 1, 1, 0, cfg.qkv_dim, e.w.q_norm[0].data_ptr(), e.w.k_norm[0].data_ptr(),
                    e.w.cos_sin.data_ptr(), v["pos"].data_ptr(), v["slots"].data_ptr(), b["q"].data_ptr(),
                    e.kv_layers[0].data_ptr(), T, hq, hkv, PAGE, 1e-6, st())), nbytes=T * cfg.qkv_dim * 6.0)
            else:
                r = e.row
                add("attention", shape, lambda: L.check(lib.bcg_decode_attn_paged(
                    b["q"].data_ptr(), e.kv_layers[0].data_ptr(), r["block_table"].data_ptr(), e.max_blocks,
                    r["seq_lens"].data_ptr(), b["attn"].data_ptr(), b["so"].data_ptr(), b["sml"].data_ptr(),
                    b["attn_counters"].data_ptr(), B, hq, hkv, PAGE, (CTX + 255) // 256, 128 ** -0.5, st())),
                    nbytes=B * CTX * hkv * 512.0)
                add("norm", shape, lambda: L.check(lib.bcg_add_norm_stats(
                    b["residual"].data_ptr(), b["partials"].data_ptr(), 1, parts, B * d, e.w.ln1[0].data_ptr(),
                    b["xn"].data_ptr(), b["row_sumsq"].data_ptr(), B, d, st())), nbytes=B * d * (10.0 + 4 * parts))
                add("activation", shape, lambda: L.check(lib.bcg_swiglu_reduce(
                    b["partials"].data_ptr(), 2, B * 2 * cfg.d_ff, b["act"].data_ptr(), B, 2 * cfg.d_ff, st())),
                    nbytes=B * cfg.d_ff * (16.0 + 2))
            continue
        x, cfg = e.exec, e.cfg
        i_attn = next(i for i, l in enumerate(cfg.layers) if isinstance(l.mixer, S.LatentAttention))
        i_delta = next(i for i, l in enumerate(cfg.layers) if isinstance(l.mixer, S.GeneralDelta))
        m, dl, ff = cfg.layers[i_attn].mixer, cfg.layers[i_delta].mixer, cfg.layers[0].mlp.ff
        wl = e.w.layers[i_delta]
        bt = x._batch(T, B)
        if what == "prefill":
            bt.positions, bt.slot_map, bt.row_seq = v["pos"].data_ptr(), v["slots"].data_ptr(), v["row_seq"].data_ptr()
            bt.seq_start, bt.block_table, bt.state_slots = v["seq_start"].data_ptr(), v["bt"].data_ptr(), v["state_slots"].data_ptr()
            bt.tiles, bt.n_tiles = v["tiles"].data_ptr(), plan.extra["n_tiles"]
            bt.gather, bt.n_gather, bt.max_context = v["gather"].data_ptr(), plan.extra["n_gather"], 1
            w = min(m.window, PROMPT)
            keys = w * (w + 1) // 2 + (PROMPT - w) * w
            cost = dict(flops=2.0 * T * m.heads * (m.dim + m.vdim) * m.kv_rank
                        + 2.0 * B * keys * m.heads * (m.dim + m.rot_dim + m.vdim))
            cost_d = dict(fma=4.5 * T * dl.heads * dl.dim ** 2)
        else:
            r = e.row
            bt.positions, bt.slot_map, bt.block_table = r["positions"].data_ptr(), r["slot_map"].data_ptr(), r["block_table"].data_ptr()
            bt.state_slots, bt.max_context = r["state_slot"].data_ptr(), CTX
            cost = dict(nbytes=B * m.window * m.cache_row * 2.0 + 2.0 * m.heads * (m.dim + m.vdim) * m.kv_rank)
            cost_d = dict(nbytes=B * dl.heads * dl.dim ** 2 * 8.0)
        add("attention", shape, lambda: L.check(lib.bcg_latent_attention(
            C.byref(x.model.struct), C.byref(x.ws), C.byref(bt), i_attn, 0, st())), **cost)
        n = dl.out_dim
        add("delta rule", shape, lambda: L.check(lib.bcg_delta_scan(
            C.byref(x.model.struct.layers[i_delta]), b["proj"].data_ptr(), parts, T * cfg.in_rows(i_delta), cfg.in_rows(i_delta),
            b["decay"].data_ptr(), 1, T * n, bt.positions, bt.slot_map, bt.seq_start, bt.state_slots, B, b["mix"].data_ptr(),
            L.DT_BF16, 1e-5, st())), **cost_d)
        add("norm", shape, lambda: L.check(lib.bcg_sandwich_norm(
            b["residual"].data_ptr(), b["proj"].data_ptr(), parts, T * d, wl["norm1b"].data_ptr(), wl["norm2"].data_ptr(),
            b["xn"].data_ptr(), L.DT_BF16, T, d, 1e-5, st())), nbytes=T * d * (10.0 + 4 * parts))
        add("activation", shape, lambda: L.check(lib.bcg_poly_norm(
            b["proj"].data_ptr(), min(parts, 2), T * ff, wl["act_coef"].data_ptr(), b["act"].data_ptr(), L.DT_BF16, T, ff, 1e-5,
            st())), nbytes=T * ff * (2.0 + 4 * min(parts, 2)))
    return rows


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
        cache = e.cfg.kv_bytes_per_token * (min(CTX, e.cfg.max_window or CTX) if kind == "bekopel" else CTX)
        if kind == "bekopel":     # layers that share a cache read it once each; states are read and written
            own = sum(isinstance(l.mixer, S.LatentAttention) for l in e.cfg.layers)
            has = sum(isinstance(l.mixer, S.LatentAttention) and l.mixer.kv_from is None for l in e.cfg.layers)
            cache = cache * own // max(has, 1) + 2 * e.cfg.state_bytes_per_row
        out[f"decode_ms_{B}"] = round(ms, 4)
        out[f"decode_tok_s_{B}"] = round(B / ms * 1e3)
        out[f"decode_of_hbm_roofline_{B}"] = round((e.cfg.decode_weight_bytes() + B * cache) / hbm / ms * 1e-6, 3)
    rng = np.random.default_rng(1)
    reqs = [Request("", prompt_ids=rng.integers(0, 4000, 1024).tolist(), max_tokens=129, forced=[65] * 129) for _ in range(8)]
    e.generate(reqs)
    e.reset_prefix_cache()
    torch.cuda.synchronize()
    t0 = time.perf_counter()
    e.generate(reqs)
    out["generate_tok_s_8x(1024+129)"] = round(8 * 129 / (time.perf_counter() - t0))
    if kernels:
        out["kernels"] = _kernels(e, hbm, tf)
    e.close()
    return out


def run(design: str, hbm_gbs: float, tflops: float, peaks: str, sizes=None, kernels: bool = True) -> dict:
    if design.lower() != "bekopel":
        raise ValueError(f"no layer-stack design {design!r}")
    tk = get_tokenizer("qwen3", VOCAB)
    res = {}
    for size in sizes or SIZES:
        res[size] = {}
        for kind in ("qwen3", "bekopel"):
            res[size][kind] = _run(kind, size, tk, hbm_gbs, tflops, kernels)
            torch.cuda.empty_cache()
    return {"metric": "design_throughput", "design": design, "unit": "tokens/s", "data": "synthetic", "dtype": "bf16",
            "peaks": f"{hbm_gbs} GB/s, {tflops} TFLOP/s ({peaks})",
            "config": {"vocab": VOCAB, "context": CTX, "prompt": PROMPT,
                       "l2": "a step's weights exceed L2; single kernels are timed after an L2 flush"}, "sizes": res}
