"""What the engine runs a model through: one executor per kind of model.

The engine owns scheduling, pages, state slots, row state and sampling; an executor owns the device buffers of
a model's forward pass and knows how to launch it.  Both kinds offer the same interface:

  buf, page_bytes, state_slot_bytes, table_cols (columns of the block table)
  block_pools                   pooled blocks of tokens: [(tokens of a block, first column of the block table)]
  alloc_cache(pages, slots, block_pages)
  plan(entries)                 host arrays (int32) describing one ragged step over `entries`
  launch(plan, views, row0)     the step: every entry's tokens through the model, the wanted logits into rows
                                row0.. of buf["logits"]
  head(views, first, n, row0)   logits of further wanted tokens of the step just launched
  decode(row, B, ...)           one token for every row of the device row state (graph-capturable)

`DenseExecutor` drives bcg_model_prefill / bcg_model_decode (uniform dense decoders), `StackExecutor`
bcg_stack_step (layer stacks, stack.py).
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass, field
from typing import Dict, List, Sequence

import numpy as np
import torch

from . import lib as L
from .model import ModelHandle
from .stack import GeneralDelta, GroupedAttention, LatentAttention, MatrixMemory, MoeMlp, StackHandle, StateSpace

PAGE = 16
SPLIT_TOKENS = 256
PREFILL_TILE = 128      # query rows per prefill-attention CTA
SINGLE_MAX = 4          # portions up to this long are attended token by token (latent attention)


def block_pages_for(tokens: int, pool: int) -> int:
    """Pages that the whole blocks of `pool` tokens of a sequence fill."""
    return -(-(tokens // pool) // PAGE)


@dataclass
class Entry:
    """One sequence's share of a ragged step: tokens at positions start.., logits wanted after `want`."""
    tokens: Sequence[int]
    start: int
    block_row: np.ndarray              # its row of the block table
    slot: int = 0                      # its state slot
    want: Sequence[int] = ()


@dataclass
class Plan:
    arrays: Dict[str, np.ndarray]      # staged to the device in one copy
    T: int
    n_seqs: int
    n_want: int
    extra: dict = field(default_factory=dict)


def _common(entries: List[Entry]):
    """ids, positions, cache rows, first token of each entry, wanted tokens — of a ragged batch."""
    ids, pos, slots, starts, want = [], [], [], [0], []
    for e in entries:
        p = np.arange(e.start, e.start + len(e.tokens))
        ids.append(np.asarray(e.tokens, np.int64))
        pos.append(p)
        slots.append(e.block_row[p // PAGE].astype(np.int64) * PAGE + p % PAGE)
        want += [starts[-1] + w for w in e.want]
        starts.append(starts[-1] + len(p))
    return np.concatenate(ids), np.concatenate(pos), np.concatenate(slots), starts, want


class DenseExecutor:
    """Uniform dense decoders (Qwen3 / Mistral class)."""

    def __init__(self, cfg, lcfg, weights, dev, *, max_rows: int, T_max: int, max_model_len: int, logit_rows: int,
                 flags: int, tp_rank: int, tp_size: int, tp_fused_allreduce: bool, tp_group):
        self.lib, self.cfg, self.lcfg, self.dev, self.flags = L.load(), cfg, lcfg, dev, flags
        self.weights, self.tp_size = weights, tp_size
        self.has_state, self.state_slot_bytes = False, 0
        d, B, T = cfg.d_model, max_rows, T_max
        bf, f32, i32 = torch.bfloat16, torch.float32, torch.int32
        z = lambda *s, dt=bf: torch.zeros(*s, dtype=dt, device=dev)
        self.max_splits_cap = (max_model_len + SPLIT_TOKENS - 1) // SPLIT_TOKENS
        self.max_blocks = self.table_cols = (max_model_len + PAGE - 1) // PAGE
        self.block_pools = []
        self.B_max, self.T_max = max(B, logit_rows), T
        lc = lcfg
        splits = [L.splits_for(1, n, k) for n, k in ((lc.qkv_dim, d), (d, lc.n_heads * 128),
                                                      (2 * lc.d_ff, d), (d, lc.d_ff))]
        pf = max(splits[0] * B * lc.qkv_dim, splits[1] * B * d,
                 (splits[2] * B * 2 * lc.d_ff) if splits[2] > 1 else 0, splits[3] * B * d)
        self.buf = dict(
            residual=z(T, d, dt=f32), xn=z(T, d), qkv=z(T, lc.qkv_dim, dt=f32), q=z(T, lc.n_heads * 128),
            attn=z(T, lc.n_heads * 128), act=z(T, lc.d_ff), delta=z(T, d, dt=f32), partials=z(pf, dt=f32),
            so=z(B * lc.n_heads * self.max_splits_cap * 128, dt=f32),
            sml=z(B * lc.n_heads * self.max_splits_cap * 2, dt=f32),
            attn_counters=z(B * lc.n_kv_heads, dt=i32),
            row_sumsq=z(2 * max((d + 127) // 128, 8) * 128, dt=f32), tile_counters=z((d + 127) // 128, dt=i32),
            # under tensor parallelism the logits stay sharded: [B, vocab / tp] per rank
            logits=z(self.B_max, lc.vocab, dt=f32), xn_last=z(self.B_max, d))
        ws = L.Workspace()
        b = self.buf
        ws.residual, ws.xn, ws.qkv, ws.q = b["residual"].data_ptr(), b["xn"].data_ptr(), b["qkv"].data_ptr(), b["q"].data_ptr()
        ws.attn, ws.act, ws.delta = b["attn"].data_ptr(), b["act"].data_ptr(), b["delta"].data_ptr()
        ws.partials, ws.partials_floats = b["partials"].data_ptr(), pf
        ws.attn_scratch_o, ws.attn_scratch_ml = b["so"].data_ptr(), b["sml"].data_ptr()
        ws.attn_counters = b["attn_counters"].data_ptr()
        ws.max_splits = self.max_splits_cap
        ws.logits, ws.xn_last, ws.T_max, ws.B_max = b["logits"].data_ptr(), b["xn_last"].data_ptr(), T, self.B_max
        ws.logits_local = None
        # tables for the deferred / fused norm (row sums of squares; tile counters for fused_norm=True)
        ws.row_sumsq = b["row_sumsq"].data_ptr()
        ws.tile_counters = b["tile_counters"].data_ptr() if (tp_size == 1 and d % 128 == 0) else None
        ws.tp_region_floats = 0
        if tp_size > 1:
            # The symmetric buffer (cudaIpc over NVLink) carries the sampler's candidate exchange
            # and, with tp_fused_allreduce, the decode step's all-reduces (bcg_tp_add_norm_stats).
            from . import tp as _tp
            region = B * d if tp_fused_allreduce else 0
            _tp.setup_symmetric(int(self.lib.bcg_tp_symm_bytes_for(region, tp_size)), tp_rank, tp_size, tp_group)
            ws.tp_region_floats = region
        self.ws = ws
        self.page_bytes = 2 * lc.n_kv_heads * PAGE * 128 * 2 * cfg.n_layers
        # ids | positions | slots | wanted rows | tiles | block table
        self.staging_words = 4 * T + self.B_max + 4 * (T // PREFILL_TILE + B) + B * self.max_blocks + 32

    def alloc_cache(self, pages: int, slots: int, block_pages: Sequence[int] = ()):
        self.kv_layers = [torch.zeros(pages, 2, self.lcfg.n_kv_heads, PAGE, 128, dtype=torch.bfloat16, device=self.dev)
                          for _ in range(self.cfg.n_layers)]
        self.model = ModelHandle(self.weights, self.kv_layers, PAGE, self.tp_size)

    def max_tokens_of(self, start: int) -> int:
        """Most tokens of one entry at `start` that a single launch takes."""
        return self.T_max

    def cost(self, e: Entry):
        """(tokens, gathered keys) an entry adds to a launch."""
        return len(e.tokens), 0

    K_max = 0

    def plan(self, entries: List[Entry]) -> Plan:
        ids, pos, slots, starts, want = _common(entries)
        tiles = []
        for s, e in enumerate(entries):
            n = len(e.tokens)
            for q0 in range(0, n, PREFILL_TILE):
                tiles.append((s, starts[s] + q0, e.start + q0, min(PREFILL_TILE, n - q0)))
        rows = want if want else [starts[-1] - 1]        # the forward always ends in the head
        return Plan(dict(ids=ids, pos=pos, slots=slots, rows=np.array(rows), tiles=np.array(tiles).reshape(-1),
                         bt=np.concatenate([e.block_row for e in entries])), starts[-1], len(entries), len(want),
                    dict(n_tiles=len(tiles)))

    def launch(self, p: Plan, v: dict, row0: int) -> int:
        """Wanted logits (at most B_max - row0 of them) land in rows row0..; returns how many did."""
        n = min(max(p.n_want, 1), self.B_max - row0)
        base = self.buf["logits"].data_ptr()
        self.ws.logits = base + row0 * self.lcfg.vocab * 4
        try:
            L.check(self.lib.bcg_model_prefill(C.byref(self.model.struct), C.byref(self.ws), v["ids"].data_ptr(),
                                               v["pos"].data_ptr(), v["slots"].data_ptr(), v["bt"].data_ptr(),
                                               self.max_blocks, v["tiles"].data_ptr(), p.extra["n_tiles"],
                                               v["rows"].data_ptr(), n, p.T, L.stream_ptr()), "bcg_model_prefill")
        finally:
            self.ws.logits = base
        return min(n, p.n_want)

    def head(self, v: dict, first: int, n: int, row0: int) -> None:
        L.check(self.lib.bcg_model_head(C.byref(self.model.struct), C.byref(self.ws), v["rows"].data_ptr() + 4 * first,
                                        n, row0, L.stream_ptr()), "bcg_model_head")

    def launches_prefill(self) -> int:
        return self.cfg.n_layers * 8 + 2

    def decode(self, row: dict, B: int, max_splits: int) -> None:
        self.ws.max_splits = max_splits
        L.check(self.lib.bcg_model_decode(C.byref(self.model.struct), C.byref(self.ws), row["next_ids"].data_ptr(),
                                          row["positions"].data_ptr(), row["slot_map"].data_ptr(),
                                          row["seq_lens"].data_ptr(), row["block_table"].data_ptr(), self.max_blocks,
                                          B, self.flags, L.stream_ptr()), "bcg_model_decode")

    def launches_per_decode_step(self, B: int) -> int:
        cfg = self.cfg
        s_gu = L.splits_for(B, 2 * cfg.d_ff, cfg.d_model)
        per_layer = 8 + (1 if s_gu > 1 else 0)   # norm, qkv, rope, attn, o, norm, gate_up(+reduce), down
        return cfg.n_layers * per_layer + 2      # final norm + lm_head


class StackExecutor:
    """Layer stacks: latent or key/value pages for attention layers, fp32 state slots for recurrent ones."""

    def __init__(self, cfg, weights, dev, *, max_rows: int, T_max: int, max_model_len: int, logit_rows: int, flags: int):
        self.lib, self.cfg, self.lcfg, self.dev, self.flags = L.load(), cfg, cfg, dev, flags
        self.weights, self.has_state = weights, cfg.has_state
        self.max_blocks = self.table_cols = (max_model_len + PAGE - 1) // PAGE
        self.block_pools = []
        for pool in cfg.pools:
            self.block_pools.append((pool, self.table_cols))
            self.table_cols += block_pages_for(max_model_len, pool)
        self.max_model_len, self.T_max, self.D_max = max_model_len, T_max, max_rows
        self.B_max = max(max_rows, logit_rows)
        act, f32, bf = cfg.torch_dtype, torch.float32, torch.bfloat16
        T, D, d = T_max, max_rows, cfg.d_model
        attn, grouped, delta, ssm, mem = (cfg.mixers(k) for k in (LatentAttention, GroupedAttention, GeneralDelta, StateSpace,
                                                                  MatrixMemory))
        moes = [l.mlp for l in cfg.layers if isinstance(l.mlp, MoeMlp)]
        # rows of the first and columns of the second matrix of feed-forwards of their own
        mlps = [(l.mlp.router_rows + l.mlp.shared_ld, l.mlp.shared_ld) if isinstance(l.mlp, MoeMlp) else (l.mlp.up_rows, l.mlp.ff_ld)
                for l in cfg.layers if l.mlp and not l.parallel]
        top = lambda xs: max([8, *xs])
        self.history = min(cfg.max_window - 1 if cfg.max_window else max_model_len, max_model_len)
        expanded = [m for m in attn if m.q_ld and cfg.act_dtype == "bfloat16"]
        self.K_max = T + min(T, max_rows * self.history) if expanded else 0
        wide = act == bf
        shapes = [(cfg.in_rows(i), d) for i in range(cfg.n_layers)]
        for i in range(cfg.n_layers):
            shapes.append((d, cfg.mix_cols(i)[1]))
        for up, down in mlps:
            shapes += [(up, d)] + ([(d, down)] if down else [])
        slabs = lambda n, k: min(T, 128) * n * (L.splits_for(1, n, k) if wide else 1)
        proj = max([T * n for n, _ in shapes] + [slabs(n, k) for n, k in shapes])
        dec = max([8] + [max(T * m.out_dim, slabs(m.out_dim, m.rank_ld)) for m in delta])
        chunks = lambda m: min((min(m.window or max_model_len, max_model_len)) // 64 + 2, (max_model_len + 63) // 64)
        part = top(D * chunks(m) * m.heads * m.kv_rank for m in attn) if wide else 8
        # experts: rows are (token, choice) pairs; long bf16 launches keep gate and up in the GEMM's epilogue
        choices = max([m.top for m in moes], default=0)
        cut = lambda m, n, k: min(T, 128) * m.top * n * (L.splits_for(1, m.top * n, k) if wide else 1)
        moe_in = top([cut(m, m.in_rows, d) for m in moes] + [T * m.top * m.in_rows for m in moes
                                                             if not (wide and d % 8 == 0 and m.experts <= L.MAX_GROUPS)])
        moe_out = top([max(T * m.top * d, cut(m, d, m.ff_ld)) for m in moes])
        counts = sum(m.experts for m in moes)
        z = lambda n, dt: torch.zeros(int(n), dtype=dt, device=dev)
        self.buf = b = dict(
            residual=z(T * d, f32), xn=z(T * d, act), proj=z(proj, f32), decay=z(dec, f32),
            q=z(T * top(m.heads * m.q_row for m in attn + grouped), act),
            mix=z(T * top(cfg.mix_cols(i)[1] for i in range(cfg.n_layers)), act),
            v_first=z(T * top(m.kv_heads * m.vdim for m in grouped if m.v_mix), f32),
            moe_x=z(max(8, T * choices * d), act), moe_h=z(max(8, T * top(m.top * m.ff_ld for m in moes)), act),
            moe_proj=z(moe_in, f32), moe_out=z(moe_out, f32), moe_expert=z(T * choices + 8, torch.int32),
            moe_rank=z(T * choices + 8, torch.int32), moe_weight=z(T * choices + 8, f32),
            moe_row=z(T * choices + 8, torch.int32), moe_row_weight=z(T * choices + 8, f32),
            moe_counts=z(counts + 8, torch.int32),
            act=z(T * top(down for _, down in mlps), act), gates=z(T * top(m.heads for m in grouped if m.gate), f32),
            ssm_x=z(T * top(m.x_ld for m in ssm + mem) if ssm or mem else 8, act),
            ssm_step=z(T * top(m.heads for m in ssm) if ssm else 8, f32),
            ssm_y=z(T * top(m.out_dim for m in ssm + mem) if ssm or mem else 8, act),
            mem_den=z(T * top(m.heads for m in mem) if mem else 8, f32), low=z(T * top(m.rank_ld for m in delta), act),
            latents=z(max(8, self.K_max * top(m.cache_row for m in expanded)), bf),
            expanded=z(max(8, self.K_max * top(m.heads * (m.q_ld + m.v_ld) for m in expanded)), bf),
            q_latent=z(D * top(m.heads * m.cache_row for m in attn) if wide else 8, bf),
            o_latent=z(D * top(m.heads * m.kv_rank for m in attn) if wide else 8, bf),
            part_o=z(part, f32), part_ml=z(top(D * chunks(m) * m.heads * 2 for m in attn), f32),
            xn_rows=z(self.B_max * d, act), logits=torch.zeros(self.B_max, cfg.vocab_ld, dtype=f32, device=dev))
        ws = L.StackWs()
        for n in b:
            setattr(ws, n, b[n].data_ptr())
        ws.proj_floats, ws.decay_floats, ws.part_floats = proj, dec, part
        ws.moe_proj_floats, ws.moe_out_floats, ws.moe_counts_n, ws.moe_rows_max = moe_in, moe_out, counts, T * choices
        ws.T_max, ws.K_max, ws.D_max, ws.B_max = T, self.K_max, D, self.B_max
        self.ws = ws
        self.page_bytes = PAGE * cfg.kv_bytes_per_token + sum(-(-PAGE * cfg.pool_bytes_per_block(p) // p) for p in cfg.pools)
        self.state_slot_bytes = cfg.state_bytes_per_row
        # ids | positions | slots | row_seq | wanted rows (<= T) | seq_start, state slots | singles | tiles | gather | bt
        self.staging_words = 5 * T + 4 * (2 * max_rows + 2) + 8 * (T // PREFILL_TILE + max_rows + 1) + T + self.K_max + \
            max_rows * self.table_cols + 64

    def alloc_cache(self, pages: int, slots: int, block_pages: Sequence[int] = ()):
        """block_pages: pages of every entry of block_pools, numbered from `pages` on."""
        self.caches = []
        extra = {pool: n for (pool, _), n in zip(self.block_pools, block_pages)}
        for l in self.cfg.layers:
            m, att, ssm, mem = l.mixer, l.one(GroupedAttention), l.one(StateSpace), l.one(MatrixMemory)
            z = lambda *s, dt=torch.float32: torch.zeros(*s, dtype=dt, device=self.dev)
            if att or ssm or mem:
                t = {}
                if mem:
                    t.update(mem_state=z(slots, mem.heads, mem.vdim + 1, mem.dim), mem_max=z(slots, mem.heads, mem.blocks))
                if att:
                    t.update({n: z(pages + (extra[att.pool] if att.pool else 0), att.kv_heads, PAGE, ld, dt=self.cfg.torch_dtype)
                              for n, ld in (("cache", att.q_ld), ("cache_v", att.v_ld))})
                if ssm:
                    t.update(ssm_state=z(slots, ssm.heads, ssm.vdim, ssm.state), conv_state=z(slots, ssm.conv - 1, ssm.channels))
            elif isinstance(m, GeneralDelta):
                t = torch.zeros(slots, m.heads, m.dim, m.dim, dtype=torch.float32, device=self.dev)
            else:
                t = torch.zeros(pages, PAGE, m.cache_row, dtype=self.cfg.torch_dtype, device=self.dev) \
                    if m.kv_from is None else None
            self.caches.append(t)
        self.kv_layers = [c for c in self.caches if c is not None]
        self.model = StackHandle(self.weights, self.caches, self.max_model_len, PAGE, dict(self.block_pools))

    def max_tokens_of(self, start: int) -> int:
        if not self.K_max:
            return self.T_max
        return min(self.T_max, self.K_max - min(start, self.history))

    def cost(self, e: Entry):
        n = len(e.tokens)
        return n, (n + min(e.start, self.history) if self.K_max else 0)

    def plan(self, entries: List[Entry]) -> Plan:
        ids, pos, slots, starts, want = _common(entries)
        T, n_seqs = starts[-1], len(entries)
        lens = np.diff(starts)
        a = dict(ids=ids, pos=pos, slots=slots, row_seq=np.repeat(np.arange(n_seqs), lens), seq_start=np.array(starts),
                 state_slots=np.array([e.slot for e in entries]), rows=np.array(want, np.int64),
                 bt=np.concatenate([e.block_row for e in entries]))
        singles, tiles, gather, context, n_gather = [], [], [], 1, 0
        room = self.D_max
        for s, e in enumerate(entries):
            n = int(lens[s])
            if n <= SINGLE_MAX and n <= room - (n_seqs - s - 1):     # leave one place to every entry behind
                singles += range(starts[s], starts[s] + n)
                room -= n
                context = max(context, e.start + n)
                continue
            k0 = max(0, e.start - self.history)
            for q0 in range(0, n, PREFILL_TILE):
                tiles.append((starts[s] + q0, e.start + q0, min(PREFILL_TILE, n - q0), n_gather, k0, s, 0, 0))
            keys = np.arange(k0, e.start + n)
            gather.append(e.block_row[keys // PAGE].astype(np.int64) * PAGE + keys % PAGE)
            n_gather += len(keys)
        a["singles"] = np.array(singles, np.int64)
        a["tiles"] = np.array(tiles, np.int64).reshape(-1)
        a["gather"] = np.concatenate(gather) if gather and self.K_max else np.zeros(0, np.int64)
        return Plan(a, T, n_seqs, len(want), dict(n_single=len(singles), n_tiles=len(tiles), n_gather=len(a["gather"]),
                                                  context=context))

    def _batch(self, T, n_seqs) -> L.StepBatch:
        b = L.StepBatch()
        # programmatic dependent launch pays for short kernels; long ones only occupy SMs while they wait
        b.T, b.n_seqs, b.max_blocks, b.flags = T, n_seqs, self.table_cols, self.flags & L.GEMM_PDL if T <= 128 else 0
        return b

    def _run(self, b: L.StepBatch) -> None:
        L.check(self.lib.bcg_stack_step(C.byref(self.model.struct), C.byref(self.ws), C.byref(b), L.stream_ptr()),
                "bcg_stack_step")

    def launch(self, p: Plan, v: dict, row0: int) -> int:
        b = self._batch(p.T, p.n_seqs)
        b.ids, b.positions, b.slot_map = v["ids"].data_ptr(), v["pos"].data_ptr(), v["slots"].data_ptr()
        b.block_table, b.state_slots = v["bt"].data_ptr(), v["state_slots"].data_ptr()
        b.max_context = p.extra["context"]
        if p.T != p.n_seqs or p.extra["n_tiles"]:        # otherwise: exactly the shape of a decode step
            b.row_seq, b.seq_start = v["row_seq"].data_ptr(), v["seq_start"].data_ptr()
            b.single_rows, b.n_single = v["singles"].data_ptr() if p.extra["n_single"] else None, p.extra["n_single"]
            b.tiles, b.n_tiles = v["tiles"].data_ptr(), p.extra["n_tiles"]
            b.gather, b.n_gather = v["gather"].data_ptr(), p.extra["n_gather"]
        self._run(b)
        n = min(p.n_want, self.B_max - row0)
        if n:
            self.head(v, 0, n, row0)
        return n

    def head(self, v: dict, first: int, n: int, row0: int) -> None:
        L.check(self.lib.bcg_stack_head(C.byref(self.model.struct), C.byref(self.ws), v["rows"].data_ptr() + 4 * first, n,
                                        row0, self.flags & L.GEMM_PDL, L.stream_ptr()), "bcg_stack_head")

    def _launches_per_step(self, decode: bool) -> int:
        n, d = 1, self.cfg.d_model
        for l in self.cfg.layers:
            if l.parallel:   # input projection, its split, attention, output projection, norm; scatter, two products, gate
                n += 5 + (4 if isinstance(l.mlp, MoeMlp) else 0)
                continue
            if l.composed:
                # input projection, attention's split (, pooled blocks) and kernel, state space or matrix memory (convolution,
                # split or gates' product,) recurrence and norm, output projection, norm; feed-forward: up, its unit where K is split, down, norm;
                # experts: router and shared rows, routing, scatter, two products, unit, shared output, norm
                att = l.one(GroupedAttention)
                n += 3 + (2 if att else 0) + int(bool(att and att.pool and not decode))
                n += (2 if decode else 3) if l.one(StateSpace) or l.one(MatrixMemory) else 0
                if isinstance(l.mlp, MoeMlp):
                    n += 6 + int(decode) + int(l.mlp.shared > 0) * (1 if decode else 2)
                elif l.mlp:
                    n += 3 + int(not l.mlp.glu or decode and L.splits_for(1, l.mlp.up_rows, d) > 1)
                continue
            # input projection, mixer (delta: low rank, decay projection, scan; attention: qkv, absorb, decode,
            # combine, up), output projection, norm; feed-forward: up, activation, down, norm
            n += (6 if isinstance(l.mixer, GeneralDelta) else 8) + (4 if l.mlp else 0)
        return n

    def launches_prefill(self) -> int:
        return self._launches_per_step(False) + 2

    def decode(self, row: dict, B: int, max_splits: int) -> None:
        b = self._batch(B, B)
        b.ids, b.positions, b.slot_map = row["next_ids"].data_ptr(), row["positions"].data_ptr(), row["slot_map"].data_ptr()
        b.block_table, b.state_slots = row["block_table"].data_ptr(), row["state_slot"].data_ptr()
        b.max_context = min(max_splits * SPLIT_TOKENS, self.max_model_len)
        self._run(b)
        L.check(self.lib.bcg_stack_head(C.byref(self.model.struct), C.byref(self.ws), None, B, 0,
                                        self.flags & L.GEMM_PDL, L.stream_ptr()), "bcg_stack_head")

    def launches_per_decode_step(self, B: int) -> int:
        return self._launches_per_step(True) + 1


def make_executor(cfg, lcfg, weights, dev, **kw):
    from .stack import StackConfig
    if isinstance(cfg, StackConfig):
        keep = ("max_rows", "T_max", "max_model_len", "logit_rows", "flags")
        return StackExecutor(cfg, weights, dev, **{k: kw[k] for k in keep})
    return DenseExecutor(cfg, lcfg, weights, dev, **kw)
