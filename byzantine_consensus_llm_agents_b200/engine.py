"""The inference engine behind VLLMAgent: what `vllm.LLM.generate` is to the reference
(vllm_agent.py:144,195,331,430,502), rebuilt for one B200.

Host side (this file, plain Python): tokenise, look prompts up in the block-hash prefix cache,
lay out KV pages, build the ragged prefill batch, launch.  Device side (libbcg_b200.so): the
whole model forward, paged attention, grammar-masked sampling and ALL per-token bookkeeping —
after prefill the decode loop is a CUDA graph replayed once per token with no host round trip;
the host only polls a single counter every few steps to stop early.

Differences from the engine the reference reaches (deliberate):
  * every row of a call is decoded together, each with its own grammar (the reference falls
    back to one-prompt-at-a-time when schemas differ, vllm_agent.py:417-455) and without the
    `max_num_seqs=4` cap (config.py:38) — per-row results are batch-invariant, so this changes
    scheduling, not outputs;
  * KV pages of a prompt's full 16-token blocks stay cached ACROSS calls and rounds, keyed by a
    hash chain over token ids (same idea as vLLM's enable_prefix_caching): per-agent system
    prompts and identical retry prompts (main.py:293-317) are not prefilled twice.
"""
from __future__ import annotations

import ctypes as C
import hashlib
import json
import math
import struct
import time
from collections import OrderedDict
from dataclasses import dataclass, field
from typing import Dict, List, Optional, Sequence

import numpy as np
import torch

from . import grammar as G
from . import lib as L
from .executors import PAGE, PREFILL_TILE, SPLIT_TOKENS, Entry, block_pages_for, make_executor
from .model import ModelConfig, Weights
from .tokenizer import CachedEncoder

MAX_GRAMMARS = 64
POLL_EVERY = 8      # tensor-parallel engines: steps between two synchronised looks at the active-row count
IN_FLIGHT = 2       # single-GPU engines: decode steps queued ahead of the one whose result the host has seen


def row_seed(base_seed: int, call_index: int, row: int):
    """Per-row Philox key (splitmix-style mix); restated in oracle/engine.py."""
    x = (base_seed * 0x9E3779B97F4A7C15 + call_index * 0xBF58476D1CE4E5B9 + row * 0x94D049BB133111EB
         + 0x2545F4914F6CDD1D) & 0xFFFFFFFFFFFFFFFF
    x ^= x >> 30
    x = (x * 0xBF58476D1CE4E5B9) & 0xFFFFFFFFFFFFFFFF
    x ^= x >> 27
    x = (x * 0x94D049BB133111EB) & 0xFFFFFFFFFFFFFFFF
    x ^= x >> 31
    return x & 0xFFFFFFFF, x >> 32


@dataclass
class Request:
    prompt: str
    schema: Optional[dict] = None
    temperature: float = 0.0
    max_tokens: int = 256
    forced: Optional[Sequence[int]] = None     # teacher-forced ids (parity tests)
    prompt_ids: Optional[List[int]] = None     # pre-tokenised prompt (tests / bench)
    seed: Optional[Sequence[int]] = None       # explicit Philox key (lo, hi); default: row_seed()


@dataclass
class Result:
    text: str
    token_ids: List[int]
    chosen: List[int]
    finish: str
    prompt_tokens: int
    cached_tokens: int


_FINISH = {0: "length", 1: "stop", 2: "length", 3: "dead"}


class PagePool:
    """Free list + block-hash prefix cache over the physical KV pages."""

    def __init__(self, n_pages: int):
        self.n_pages = n_pages
        self.free = list(range(n_pages - 1, -1, -1))
        self.cached: "OrderedDict[bytes, int]" = OrderedDict()  # hash -> page (LRU order)
        self.page_hash: Dict[int, bytes] = {}
        self.ref: Dict[int, int] = {}
        self.hits = 0
        self.misses = 0

    @staticmethod
    def chain(prev: bytes, block: Sequence[int]) -> bytes:
        return hashlib.blake2b(prev + struct.pack(f"<{len(block)}i", *block), digest_size=16).digest()

    def lookup(self, h: bytes) -> Optional[int]:
        p = self.cached.get(h)
        if p is not None:
            self.cached.move_to_end(h)
        return p

    def acquire(self, page: int) -> None:
        self.ref[page] = self.ref.get(page, 0) + 1

    def alloc(self) -> int:
        if not self.free:
            # evict least-recently-used cached pages nobody holds
            for h, p in list(self.cached.items()):
                if self.ref.get(p, 0) == 0:
                    del self.cached[h]
                    del self.page_hash[p]
                    self.free.append(p)
                    if len(self.free) >= 64:
                        break
        if not self.free:
            raise MemoryError("KV page pool exhausted")
        p = self.free.pop()
        self.ref[p] = 1
        return p

    def publish(self, page: int, h: bytes) -> None:
        """Make a fully written prompt page reusable by later requests."""
        if h not in self.cached and page not in self.page_hash:
            self.cached[h] = page
            self.page_hash[page] = h

    def release(self, page: int) -> None:
        r = self.ref.get(page, 0) - 1
        if r > 0:
            self.ref[page] = r
            return
        self.ref.pop(page, None)
        if page not in self.page_hash:
            self.free.append(page)

    def reset_cache(self) -> None:
        for h, p in list(self.cached.items()):
            if self.ref.get(p, 0) == 0:
                del self.cached[h]
                del self.page_hash[p]
                self.free.append(p)


class SlotPool:
    """State slots of recurrent layers.  A slot is not cleared when it changes hands: a sequence's first token
    (position 0) starts from a zero state, whatever the slot holds."""

    def __init__(self, n: int):
        self.n = n
        self.free = list(range(n - 1, -1, -1))

    def alloc(self) -> int:
        if not self.free:
            raise MemoryError("state slots exhausted")
        return self.free.pop()

    def release(self, slot: int) -> None:
        self.free.append(slot)


@dataclass
class LiveSequence:
    """A live sequence of the step interface (Engine.open / step / close)."""
    length: int = 0
    pages: List[int] = field(default_factory=list)
    blocks: List[List[int]] = field(default_factory=list)      # pages of pooled blocks, one list per block size
    slot: int = 0


class Engine:
    def __init__(self, cfg: ModelConfig, weights: Weights, tokenizer, *, max_model_len: int = 8192,
                 max_rows: int = 64, prefill_tokens: int = 16384, kv_pages: Optional[int] = None,
                 gpu_memory_utilization: float = 0.9, base_seed: int = 0, device: str = "cuda:0",
                 enable_prefix_cache: bool = True, use_cuda_graph: bool = True, pdl: bool = True,
                 fused_norm: bool = False, deferred_norm: Optional[bool] = None,
                 fused_rope: bool = False, state_slots: Optional[int] = None, logit_rows: int = 0,
                 tp_rank: int = 0, tp_size: int = 1, tp_fused_allreduce: bool = True, tp_group=None):
        """`cfg` is the FULL architecture (a ModelConfig, or a StackConfig with StackWeights).  `tokenizer` may be
        None for an engine that only steps given tokens (open / step / close_sequence).  With tp_size > 1 `weights` must
        be this rank's shard (Weights.shard / random_init_sharded) and bcg_tp_init must have been called
        (collective)."""
        if not torch.cuda.is_available():
            raise L.BcgError("the engine needs a CUDA device (sm_100a); there is no CPU fallback")
        self.lib = L.load()
        self.cfg, self.w, self.tk = cfg, weights, tokenizer
        self.tp_rank, self.tp_size = tp_rank, tp_size
        full_cfg = cfg
        lcfg = cfg.shard(tp_size)          # this rank's heads / d_ff / vocab
        self.lcfg = lcfg
        if tp_size > 1 and weights.cfg.n_heads != lcfg.n_heads:
            raise L.BcgError("tensor-parallel engine needs sharded weights (Weights.shard)")
        self.dev = torch.device(device)
        torch.cuda.set_device(self.dev)
        self.max_model_len = min(max_model_len, cfg.max_pos)
        self.max_rows = min(max_rows, 128)
        self.T_max = max(prefill_tokens, self.max_model_len)
        self.base_seed = base_seed
        self.calls = 0
        self.use_cuda_graph = use_cuda_graph
        # How decode runs the residual add + RMSNorm between projections (include/bcg_b200.h,
        # bcg_model_decode).  Default on one GPU: statistics kernel + 1/RMS in the next GEMM's epilogue
        # (1.5 % faster per step than the complete norm kernel).  TP engines with the fused all-reduce
        # do the same inside bcg_tp_add_norm_stats; with NCCL all-reduces they run the complete norm.
        self.tp_group = tp_group
        if deferred_norm is None:
            deferred_norm = tp_size == 1 and not fused_norm
        self.flags = ((L.GEMM_PDL if pdl else 0) | (L.STEP_FUSED_NORM if fused_norm else 0)
                      | (L.STEP_DEFERRED_NORM if deferred_norm else 0)
                      | (L.STEP_FUSED_ROPE if fused_rope else 0))
        self.max_blocks = (self.max_model_len + PAGE - 1) // PAGE
        self.max_steps = self.max_model_len

        B = self.max_rows
        f32, i32 = torch.float32, torch.int32
        z = lambda *s, dt=torch.bfloat16: torch.zeros(*s, dtype=dt, device=self.dev)
        self.exec = make_executor(cfg, lcfg, weights, self.dev, max_rows=B, T_max=self.T_max,
                                  max_model_len=self.max_model_len, logit_rows=logit_rows, flags=self.flags,
                                  tp_rank=tp_rank, tp_size=tp_size, tp_fused_allreduce=tp_fused_allreduce,
                                  tp_group=tp_group)
        self.buf, self.ws = self.exec.buf, self.exec.ws
        # ---- state slots and KV pages
        self.slots = SlotPool(state_slots or B)
        page_bytes = self.exec.page_bytes
        if kv_pages is None:
            free_b, total_b = torch.cuda.mem_get_info(self.dev)
            budget = int(total_b * gpu_memory_utilization) - (total_b - free_b) \
                - self.slots.n * self.exec.state_slot_bytes
            want = self.max_rows * self.max_blocks * 2
            kv_pages = max(self.max_blocks + 8, min(want, budget // max(page_bytes, 1)))
            if tp_size > 1:
                # every rank must run the SAME page pool (eviction, cache hits and prefill sizes are
                # decided per rank and have to agree): take the smallest budget of the replica
                import torch.distributed as dist
                t = torch.tensor([kv_pages], dtype=torch.int64)
                dist.all_reduce(t, op=dist.ReduceOp.MIN, group=tp_group)
                kv_pages = int(t.item())
        # pages of pooled blocks: as many as the tokens of all pages can fill, and a part of one per sequence
        block_pages = [kv_pages // p + max(self.slots.n, B) for p, _ in self.exec.block_pools]
        self.exec.alloc_cache(kv_pages, self.slots.n, block_pages)
        self.kv_layers, self.model = self.exec.kv_layers, self.exec.model
        self.pool = PagePool(kv_pages)
        self.block_pools = [PagePool(n) for n in block_pages]
        # pages alone restore a prefix only where no layer carries a recurrent state or pools blocks of tokens
        self.enable_prefix_cache = enable_prefix_cache and not self.exec.has_state and not block_pages
        # ---- per-row device state (bcg_sampler_args).  Everything the host writes at the start of a
        # call lives in ONE int32 block with a pinned host mirror, so a call costs one H2D copy
        # instead of one per field.
        fields = [("grammar_id", 1), ("state", 1), ("temperature", 1), ("seed", 2), ("max_tokens", 1),
                  ("n_out", 1), ("finished", 1), ("seq_lens", 1), ("state_slot", 1), ("block_table", self.exec.table_cols)]
        words = sum(w for _, w in fields) * B
        self._state_dev = z(words, dt=i32)
        self._state_host = torch.zeros(words, dtype=i32).pin_memory()
        self.row, self.row_host, off = {}, {}, 0
        for name, w in fields:
            dv, hv = self._state_dev[off:off + w * B], self._state_host[off:off + w * B].numpy()
            if w > 1:
                dv, hv = dv.view(B, w), hv.reshape(B, w)
            if name == "temperature":
                dv, hv = dv.view(f32), hv.view(np.float32)
            self.row[name], self.row_host[name] = dv, hv
            off += w * B
        self.row.update(
            out_tokens=z(B, self.max_steps, dt=i32), chosen=z(B, self.max_steps, dt=i32),
            forced=torch.full((B, self.max_steps), -1, dtype=i32, device=self.dev),
            next_ids=z(B, dt=i32), positions=z(B, dt=i32), slot_map=z(B, dt=i32))
        # Number of unfinished rows: the sampler's bookkeeping kernel writes it straight into pinned
        # HOST memory (mapped into the device's address space), so the host reads it without a copy.
        self.n_active_host = torch.zeros(1, dtype=i32).pin_memory()
        self.row["n_active"] = self.n_active_host
        # ---- staging of a ragged step's arrays (ids, positions, slots, work lists, block table), one copy each
        self._pf_dev = z(self.exec.staging_words, dt=i32)
        self._pf_host = torch.zeros(self.exec.staging_words, dtype=i32).pin_memory()
        # ---- tokenizer / grammar tables on the device
        if tokenizer is not None:
            tok_bytes = G.grammar_token_bytes(tokenizer)
            lens = np.fromiter((len(x) for x in tok_bytes), np.int64, count=cfg.vocab)
            offs = np.zeros(cfg.vocab + 1, np.int32)
            offs[1:] = np.cumsum(lens)
            blob = np.frombuffer(b"".join(tok_bytes) or b"\0", dtype=np.uint8).copy()
            self.tok_bytes = torch.from_numpy(blob).to(self.dev)
            self.tok_offsets = torch.from_numpy(offs).to(self.dev)
            self.mask_words = (cfg.vocab + 31) // 32
        self.grammars: Dict[str, int] = {}
        self.grammar_objs: List[G.CompiledGrammar] = []
        self._gram_dev = []
        self.mask_ptrs = torch.zeros(MAX_GRAMMARS, dtype=torch.int64, device=self.dev)
        self.trans_ptrs = torch.zeros(MAX_GRAMMARS, dtype=torch.int64, device=self.dev)
        self._graphs: Dict[tuple, torch.cuda.CUDAGraph] = {}
        self.stats = dict(calls=0, prompts=0, prompt_tokens=0, cached_tokens=0, prefill_tokens=0,
                          decode_steps=0, generated_tokens=0, prefill_s=0.0, decode_s=0.0, host_s=0.0,
                          gpu_launches=0, h2d_bytes=0, d2h_bytes=0)
        self._capture_stream = torch.cuda.Stream(self.dev)
        self._encode = CachedEncoder(tokenizer) if tokenizer is not None else None    # retries resubmit identical prompts
        # parity tests: when set to a list, the logits of every step are appended (forces the
        # eager, graph-less decode loop)
        self.debug_logits: Optional[list] = None

    # ------------------------------------------------------------------ grammars
    def grammar_index(self, schema: Optional[dict]) -> int:
        if schema is None:
            return -1
        key = json.dumps(schema, sort_keys=False)
        gi = self.grammars.get(key)
        if gi is None:
            if len(self.grammar_objs) >= MAX_GRAMMARS:
                raise L.BcgError("too many distinct schemas in one engine")
            g = G.compile_schema(schema, self.tk)
            masks = torch.from_numpy(g.masks).to(self.dev).contiguous()
            trans = torch.from_numpy(g.trans).to(self.dev).contiguous()
            self._gram_dev.append((masks, trans))
            gi = len(self.grammar_objs)
            self.grammar_objs.append(g)
            self.grammars[key] = gi
            self.mask_ptrs[gi] = masks.data_ptr()
            self.trans_ptrs[gi] = trans.data_ptr()
        return gi

    # ------------------------------------------------------------------ sampler / steps
    def _sampler_args(self, B: int, use_forced: bool) -> L.SamplerArgs:
        r, a = self.row, L.SamplerArgs()
        a.logits, a.ld_logits = self.buf["logits"].data_ptr(), self.lcfg.vocab
        a.B, a.V, a.mask_words, a.max_steps = B, self.lcfg.vocab, self.mask_words, self.max_steps
        stops = list(self.tk.stop_ids) + [-1]
        a.eos_id0, a.eos_id1 = stops[0], stops[1]
        a.page_size, a.max_blocks_per_seq = PAGE, self.exec.table_cols
        a.grammar_id = r["grammar_id"].data_ptr()
        a.mask_tables, a.trans_tables = self.mask_ptrs.data_ptr(), self.trans_ptrs.data_ptr()
        a.tok_bytes, a.tok_offsets = self.tok_bytes.data_ptr(), self.tok_offsets.data_ptr()
        a.temperature, a.seed, a.max_tokens = r["temperature"].data_ptr(), r["seed"].data_ptr(), r["max_tokens"].data_ptr()
        a.forced = r["forced"].data_ptr() if use_forced else None
        a.state, a.n_out, a.finished = r["state"].data_ptr(), r["n_out"].data_ptr(), r["finished"].data_ptr()
        a.out_tokens, a.chosen = r["out_tokens"].data_ptr(), r["chosen"].data_ptr()
        a.next_ids, a.positions = r["next_ids"].data_ptr(), r["positions"].data_ptr()
        a.seq_lens, a.slot_map = r["seq_lens"].data_ptr(), r["slot_map"].data_ptr()
        a.block_table, a.n_active = r["block_table"].data_ptr(), r["n_active"].data_ptr()
        if self.tp_size > 1:   # vocab-parallel sampling: local shard + one candidate per row exchanged
            a.tp_rank, a.tp_size, a.vocab_base = self.tp_rank, self.tp_size, self.tp_rank * self.lcfg.vocab
        return a

    def _sample(self, B: int, use_forced: bool) -> None:
        a = self._sampler_args(B, use_forced)
        L.check(self.lib.bcg_mask_sample(C.byref(a), L.stream_ptr()), "bcg_mask_sample")

    def _decode_step(self, B: int, max_splits: int, use_forced: bool) -> None:
        self.exec.decode(self.row, B, max_splits)
        self._sample(B, use_forced)

    def launches_per_decode_step(self, B: int) -> int:
        return self.exec.launches_per_decode_step(B) + 2     # sampler + active count

    def _graph_for(self, B: int, max_splits: int, use_forced: bool):
        key = (B, max_splits, use_forced)
        g = self._graphs.get(key)
        if g is None:
            # The graph replays real state transitions, so capture must not disturb a live batch:
            # warm-up happens in _warmup() on scratch state; here we only record.
            g = torch.cuda.CUDAGraph()
            with torch.cuda.graph(g, stream=self._capture_stream):
                self._decode_step(B, max_splits, use_forced)
            self._graphs[key] = g
        return g

    # ------------------------------------------------------------------ generation
    def generate(self, requests: List[Request]) -> List[Result]:
        if self.tk is None:
            raise L.BcgError("an engine without a tokenizer only steps given tokens (open / step / close_sequence)")
        if self.lcfg.vocab % 4:
            raise L.BcgError(f"the sampler needs a vocabulary that is a multiple of 4 (got {self.lcfg.vocab})")
        out: List[Result] = []
        for i in range(0, len(requests), self.max_rows):
            out.extend(self._generate_wave(requests[i:i + self.max_rows], i))
        self.calls += 1
        self.stats["calls"] += 1
        return out

    def _generate_wave(self, reqs: List[Request], row0: int) -> List[Result]:
        t_host0 = time.perf_counter()
        cfg, B = self.cfg, len(reqs)
        r = self.row
        ids_list, cached, pages_of, hashes_of, slots_of, blocks_of = [], [], [], [], [], []
        use_forced = any(q.forced is not None for q in reqs)
        for q in reqs:
            ids = list(q.prompt_ids) if q.prompt_ids is not None else self._encode(q.prompt)
            if len(ids) + q.max_tokens > self.max_model_len:
                raise L.BcgError(f"prompt ({len(ids)} tokens) + max_tokens ({q.max_tokens}) exceeds "
                                 f"max_model_len ({self.max_model_len})")
            if not ids:
                raise L.BcgError("empty prompt")
            ids_list.append(ids)
        # ---- page layout + prefix-cache lookup
        try:
            for ids, q in zip(ids_list, reqs):
                n_full = len(ids) // PAGE
                hs, h = [], b"\0" * 16
                for j in range(n_full):
                    h = PagePool.chain(h, ids[j * PAGE:(j + 1) * PAGE])
                    hs.append(h)
                pages, hit = [], 0
                if self.enable_prefix_cache:
                    for j in range(n_full):
                        if (j + 1) * PAGE >= len(ids):
                            break  # always compute at least the last prompt token
                        p = self.pool.lookup(hs[j])
                        if p is None:
                            break
                        self.pool.acquire(p)
                        pages.append(p)
                        hit += 1
                total_pages = (len(ids) + q.max_tokens + PAGE - 1) // PAGE
                while len(pages) < total_pages:
                    pages.append(self.pool.alloc())
                pages_of.append(pages)
                blocks_of.append([[] for _ in self.block_pools])
                self._grow_blocks(blocks_of[-1], len(ids) + q.max_tokens)
                hashes_of.append(hs)
                cached.append(hit * PAGE)
                slots_of.append(self.slots.alloc() if self.exec.has_state else 0)
        except Exception:
            self._release(pages_of, slots_of, blocks_of)
            raise

        try:
            results = self._run(reqs, ids_list, cached, pages_of, blocks_of, hashes_of, slots_of, use_forced, row0, t_host0)
        finally:
            self._release(pages_of, slots_of, blocks_of)
        return results

    def _grow_blocks(self, blocks: List[List[int]], tokens: int) -> None:
        """Gives a sequence the pages of pooled blocks that `tokens` tokens fill."""
        for (size, _), pool, mine in zip(self.exec.block_pools, self.block_pools, blocks):
            while len(mine) < block_pages_for(tokens, size):
                mine.append(pool.alloc())

    def _table_row(self, row: np.ndarray, pages: List[int], blocks: List[List[int]]) -> None:
        """A sequence's row of the block table.  Pages of pooled blocks are numbered behind the tokens' pages."""
        row[:len(pages)] = pages
        for (_, col), mine in zip(self.exec.block_pools, blocks):
            row[col:col + len(mine)] = [self.pool.n_pages + p for p in mine]

    def _release(self, pages_of, slots_of, blocks_of) -> None:
        for pages in pages_of:
            for p in pages:
                self.pool.release(p)
        for blocks in blocks_of:
            for pool, mine in zip(self.block_pools, blocks):
                for p in mine:
                    pool.release(p)
        if self.exec.has_state:
            for s in slots_of:
                self.slots.release(s)

    def _run(self, reqs, ids_list, cached, pages_of, blocks_of, hashes_of, slots_of, use_forced, row0, t_host0):
        cfg, B, r, dev = self.cfg, len(reqs), self.row, self.dev
        i32 = torch.int32
        bt = np.zeros((B, self.exec.table_cols), np.int32)
        for b, pages in enumerate(pages_of):
            self._table_row(bt[b], pages, blocks_of[b])
        gids = [self.grammar_index(q.schema) for q in reqs]
        seeds = np.array([tuple(q.seed) if q.seed is not None else row_seed(self.base_seed, self.calls, row0 + b)
                          for b, q in enumerate(reqs)], np.uint32)
        # the previous call's copy out of the pinned mirror has long completed (every call ends with
        # a device synchronisation), so the mirror may be rewritten in place
        h = self.row_host
        h["grammar_id"][:B] = gids
        h["state"][:B] = 0
        h["temperature"][:B] = [q.temperature for q in reqs]
        h["max_tokens"][:B] = [q.max_tokens for q in reqs]
        h["n_out"][:B] = 0
        h["finished"][:B] = 0
        h["seq_lens"][:B] = [len(x) for x in ids_list]
        h["state_slot"][:B] = slots_of
        h["seed"][:B] = seeds.view(np.int32).reshape(B, 2)
        h["block_table"][:B] = bt
        self._state_dev.copy_(self._state_host, non_blocking=True)     # ONE copy for all per-row state
        self.stats["h2d_bytes"] += self._state_host.numel() * 4
        if use_forced:
            f = np.full((B, self.max_steps), -1, np.int32)
            for b, q in enumerate(reqs):
                if q.forced is not None:
                    f[b, :len(q.forced)] = np.asarray(q.forced, np.int32)
            r["forced"][:B].copy_(torch.from_numpy(f))
            self.stats["h2d_bytes"] += f.nbytes

        # ---- prefill: the uncached part of every prompt, in groups that fit a launch
        ev0, ev1, ev2 = (torch.cuda.Event(enable_timing=True) for _ in range(3))
        ev0.record()
        entries = [Entry(ids[c:], c, bt[b], slots_of[b], (len(ids) - c - 1,))
                   for b, (ids, c) in enumerate(zip(ids_list, cached))]
        b0 = 0
        for group in self._groups(entries):
            self._launch_group(group, b0)       # last-token logits go straight to the rows of these prompts
            b0 += len(group)
        # publish freshly written full prompt pages for later calls
        if self.enable_prefix_cache:
            for b in range(B):
                for j, h in enumerate(hashes_of[b]):
                    self.pool.publish(pages_of[b][j], h)
        if self.debug_logits is not None:
            self.debug_logits.append(self._logits_rows(B))
        self._sample(B, use_forced)          # first token of every row
        self.stats["gpu_launches"] += 2
        ev1.record()
        self.stats["host_s"] += time.perf_counter() - t_host0

        # ---- decode loop: one graph replay per token, no host sync except the poll
        max_new = max(q.max_tokens for q in reqs)
        max_len = max(len(x) + q.max_tokens for x, q in zip(ids_list, reqs))
        max_splits = max(1, (max_len + SPLIT_TOKENS - 1) // SPLIT_TOKENS)
        steps = 0
        if max_new > 1:
            per_step = self.launches_per_decode_step(B)
            key = (B, max_splits, use_forced)
            graph = self._graphs.get(key)
            done = False
            use_graph = self.use_cuda_graph and self.debug_logits is None
            if not use_graph:
                graph = None
            if use_graph and graph is None:
                # first use of this shape: one eager step (it is a real step and also performs the
                # kernels' one-time attribute set-up), then record — recording executes nothing.
                self._decode_step(B, max_splits, use_forced)
                steps += 1
                self.stats["gpu_launches"] += per_step
                graph = self._graph_for(B, max_splits, use_forced)
            def one_step():
                if graph is not None:
                    graph.replay()
                else:
                    self._decode_step(B, max_splits, use_forced)
                    if self.debug_logits is not None:
                        self.debug_logits.append(self._logits_rows(B))

            if self.tp_size == 1:
                # The bookkeeping kernel of every step leaves the number of unfinished rows in pinned
                # host memory.  The host keeps at most IN_FLIGHT steps queued: before launching step
                # k it waits for step k - IN_FLIGHT and looks at the counter, so a call whose rows
                # have all finished runs at most IN_FLIGHT dead steps (it used to poll every 16
                # steps: ~8 dead steps of 5.5 ms on average for every call that ends early) and the
                # GPU never waits for the host (one step is queued behind the running one).
                ring = [torch.cuda.Event() for _ in range(IN_FLIGHT + 1)]
                launched = 0
                while steps < max_new - 1:
                    one_step()
                    ring[launched % len(ring)].record()
                    launched += 1
                    steps += 1
                    if launched >= IN_FLIGHT:
                        ring[(launched - IN_FLIGHT) % len(ring)].synchronize()
                        if int(self.n_active_host[0]) == 0:
                            break
                self.stats["gpu_launches"] += launched * per_step
            else:
                # Tensor parallelism: every rank must stop after the SAME step (a rank that ran one
                # step more would wait for peers that never come), so the ranks decide at fixed step
                # counts on a fully synchronised counter, which is identical everywhere.
                while steps < max_new - 1 and not done:
                    n = min(POLL_EVERY, max_new - 1 - steps)
                    for _ in range(n):
                        one_step()
                    steps += n
                    self.stats["gpu_launches"] += n * per_step
                    torch.cuda.current_stream().synchronize()
                    done = int(self.n_active_host[0]) == 0
        ev2.record()
        torch.cuda.synchronize()
        t_host1 = time.perf_counter()
        n_out = r["n_out"][:B].cpu().numpy()
        fin = r["finished"][:B].cpu().numpy()
        width = int(n_out.max()) if B else 0
        toks = r["out_tokens"][:B, :width].cpu().numpy()
        chosen = r["chosen"][:B, :width].cpu().numpy()
        self.stats["d2h_bytes"] += n_out.nbytes + fin.nbytes + toks.nbytes + chosen.nbytes
        results = []
        stop = set(self.tk.stop_ids)
        for b in range(B):
            t = toks[b, :n_out[b]].tolist()
            text = self.tk.decode([x for x in t if x not in stop])
            results.append(Result(text, t, chosen[b, :n_out[b]].tolist(), _FINISH.get(int(fin[b]), "length"),
                                  len(ids_list[b]), cached[b]))
        st = self.stats
        st["prompts"] += B
        st["prompt_tokens"] += sum(len(x) for x in ids_list)
        st["cached_tokens"] += sum(cached)
        st["prefill_tokens"] += sum(len(x) - c for x, c in zip(ids_list, cached))
        st["decode_steps"] += steps
        st["generated_tokens"] += int(n_out.sum())
        st["prefill_s"] += ev0.elapsed_time(ev1) / 1e3
        st["decode_s"] += ev1.elapsed_time(ev2) / 1e3
        st["host_s"] += time.perf_counter() - t_host1
        return results

    def _logits_rows(self, B: int) -> torch.Tensor:
        """[B, V] logits of the current step (parity tests only; under TP the vocabulary shards are
        gathered over the control group — the product path never moves logits between ranks)."""
        if self.tp_size == 1:
            return self.buf["logits"][:B, :self.cfg.vocab].clone()
        import torch.distributed as dist
        mine = self.buf["logits"][:B].cpu()
        parts = [torch.empty_like(mine) for _ in range(self.tp_size)]
        dist.all_gather(parts, mine, group=self.tp_group)
        return torch.cat(parts, dim=1).to(self.dev)

    # ------------------------------------------------------------------ ragged steps
    def _groups(self, entries: List[Entry]):
        """Consecutive entries that fit one launch (tokens, gathered keys, rows)."""
        group, T, K = [], 0, 0
        for e in entries:
            t, k = self.exec.cost(e)
            if group and (T + t > self.T_max or K + k > max(self.exec.K_max, 0) and k or len(group) >= self.max_rows):
                yield group
                group, T, K = [], 0, 0
            group.append(e)
            T, K = T + t, K + k
        if group:
            yield group

    def _launch_group(self, entries: List[Entry], row0: int):
        """Stage and launch one ragged step; wanted logits from logits row `row0`.  Returns (plan, device
        views, how many wanted logits that left in the buffer)."""
        plan = self.exec.plan(entries)
        # one pinned staging block, one H2D copy per launch.  A launch's copy must have left the pinned
        # block before the next one refills it.
        if getattr(self, "_pf_event", None) is not None:
            self._pf_event.synchronize()
        hs, o0, views = self._pf_host.numpy(), 0, {}
        for name, arr in plan.arrays.items():
            a = np.asarray(arr, dtype=np.int32)
            hs[o0:o0 + a.size] = a
            views[name] = self._pf_dev[o0:o0 + a.size]
            o0 += (a.size + 3) // 4 * 4        # keep every array 16-byte aligned
        self._pf_dev[:o0].copy_(self._pf_host[:o0], non_blocking=True)
        self._pf_event = torch.cuda.Event()
        self._pf_event.record()
        self.stats["h2d_bytes"] += o0 * 4
        done = self.exec.launch(plan, views, row0)
        self.stats["gpu_launches"] += self.exec.launches_prefill()
        return plan, views, done

    # The step interface: the caller brings the tokens, the engine keeps pages and states.  The same launches
    # as generate(): a batch of single tokens is a decode step, anything else a ragged step.
    def open(self) -> LiveSequence:
        return LiveSequence(blocks=[[] for _ in self.block_pools], slot=self.slots.alloc() if self.exec.has_state else 0)

    def close_sequence(self, seq: LiveSequence) -> None:
        """Gives a sequence's pages and state slot back."""
        self._release([seq.pages], [seq.slot], [seq.blocks])
        seq.pages, seq.blocks, seq.length = [], [[] for _ in self.block_pools], 0

    def step(self, work) -> torch.Tensor:
        """work: [(LiveSequence, token ids, places among them whose logits are wanted)], one batch.  Returns the
        wanted logits [n, vocab] (fp32, on the device) in that order."""
        entries: List[Entry] = []
        for seq, tokens, want in work:
            end = seq.length + len(tokens)
            if not tokens:
                raise L.BcgError("a step's entry needs at least one token")
            if end > self.max_model_len:
                raise L.BcgError(f"sequence of {end} tokens exceeds max_model_len ({self.max_model_len})")
            while len(seq.pages) * PAGE < end:
                seq.pages.append(self.pool.alloc())
            self._grow_blocks(seq.blocks, end)
            row = np.zeros(self.exec.table_cols, np.int32)
            self._table_row(row, seq.pages, seq.blocks)
            done = 0
            while done < len(tokens):           # a portion longer than a launch takes is cut
                n = min(len(tokens) - done, self.exec.max_tokens_of(seq.length + done))
                entries.append(Entry(tokens[done:done + n], seq.length + done, row, seq.slot,
                                     [w - done for w in want if done <= w < done + n]))
                done += n
        out = []
        for group in self._groups(entries):
            plan, views, done = self._launch_group(group, 0)
            out.append(self.buf["logits"][:done, :self.lcfg.vocab].clone())
            while done < plan.n_want:
                n = min(plan.n_want - done, self.exec.B_max)
                self.exec.head(views, done, n, 0)
                out.append(self.buf["logits"][:n, :self.lcfg.vocab].clone())
                done += n
        for seq, tokens, _ in work:
            seq.length += len(tokens)
        return torch.cat(out)

    # ------------------------------------------------------------------ misc
    def reset_prefix_cache(self) -> None:
        self.pool.reset_cache()

    def close(self) -> None:
        self._graphs.clear()
        self.kv_layers = None
        self.buf = None
