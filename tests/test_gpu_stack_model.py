"""Layer-stack models through the engine: whole prompts, token by token, portions, mixed batches, reused pages
and slots, long decoding, greedy generation and trace replay — against the plain oracle."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from oracle import stack_ref as R

import stack_models as SM

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
# rms logit error over rms logit: of 95 % of the positions, and of every one.  (A head whose recurrent output
# nearly cancels is divided by its own small root mean square: such positions amplify bf16 rounding.)
TOL = {"float32": 3e-4, "bfloat16": 3e-2}
WORST = {"float32": 3e-4, "bfloat16": 0.2}

CONFIGS = {
    # attention first, a cache read by two layers with other windows and head counts, a layer without feed-forward
    "mixed": SM.config([SM.attn(), SM.delta(), SM.attn(kv_from=0, window=45, heads=5, dim=12, ff=None),
                        SM.attn(kv_from=0, window=3, vdim=8), SM.delta(heads=3, dim=36, ff=None)]),
    # everything on the tensor-core kernels, two caches, wide heads
    "tensor": SM.config([SM.delta(heads=3, dim=64, ff=256), SM.attn(4, 48, 16, 64, 112, 33, ff=256),
                         SM.attn(8, 32, 32, 32, 96, 70, base=1e6), SM.attn(2, 80, 16, 96, 112, 16, kv_from=1)], width=192, vocab=320),
    "attention-only": SM.config([SM.attn(window=1), SM.attn(2, 32, 32, 40, 32, 100)], width=64, vocab=101),
    "delta-only": SM.config([SM.delta(1, 8, ff=None), SM.delta(2, 128)], width=100, vocab=64, eps=1e-3),
    # sizes no vector load or tensor-core tile likes
    "odd": SM.config([SM.delta(3, 7, ff=45), SM.attn(3, 9, 6, 11, 13, 19, ff=51), SM.attn(5, 10, 6, 7, 13, 40, kv_from=1, ff=None)],
                     width=61, vocab=83),
    "one-each": SM.config([SM.attn(1, 8, 8, 8, 16, 5, ff=20)], width=36, vocab=36),
    # parallel layers: values mixed from the second layer on, a layer in between without, every kind of feed-forward
    "parallel": SM.parallel_config([SM.gattn(v_mix=False, mlp=SM.dense(96)), SM.gattn(window=1, mlp=SM.moe()),
                                    SM.gattn(2, 1, 16, 24, 45, v_mix=False), SM.gattn(3, 3, 40, 40, 400, every=64, mlp=SM.moe(4, 1, 24, 0.7))]),
    # everything on the tensor-core kernels
    "parallel-tensor": SM.parallel_config([SM.gattn(8, 2, 64, 32, 33, mlp=SM.moe(8, 3, 64)), SM.gattn(4, 1, 128, 64, 100, mlp=SM.dense(320)),
                                           SM.gattn(8, 2, 96, 32, 17, coef=-0.1, mlp=SM.moe(8, 2, 96, 3.0)), SM.gattn(2, 1, 256, 200, 70, v_mix=False)],
                                          width=192, vocab=320),
    # a group of more than 16 query heads, heads no tensor-core tile takes, one expert out of one
    "parallel-groups": SM.parallel_config([SM.gattn(20, 1, 16, 16, 64, mlp=SM.moe(1, 1, 16)), SM.gattn(36, 2, 8, 8, 30, mlp=SM.moe(9, 9, 8)),
                                           SM.gattn(2, 2, 264, 264, 50, v_mix=False)], width=96, vocab=96, eps=1e-3),
    # sizes no vector load or tile likes
    "parallel-odd": SM.parallel_config([SM.gattn(3, 1, 7, 11, 19, mlp=SM.dense(45)), SM.gattn(5, 5, 9, 6, 40, v_mix=False, mlp=SM.moe(5, 3, 21)),
                                        SM.gattn(3, 1, 13, 11, 130, every=1, mlp=SM.dense(51))], width=61, vocab=83),
    "parallel-one": SM.parallel_config([SM.gattn(1, 1, 8, 8, 5, mlp=SM.dense(20))], width=36, vocab=36, positions=300),
    # attention beside a state space, state spaces alone, with and without a feed-forward
    "side": SM.side_config([SM.mamba(), SM.both(mlp=SM.glu(70)), SM.mamba(heads=2, vdim=40, state=33, groups=1, norm_groups=1, conv=2, mlp=SM.glu(48, 0.4)),
                            SM.both(4, 1, 16, 24, every=64, coef=-0.1, conv=3)]),
    # everything on the tensor-core kernels, two blocks of head entries, more parts than groups and fewer
    "side-tensor": SM.side_config([SM.both(8, 2, 64, 32, mlp=SM.glu(320, 7.0), vdim_ssm=80, state=64), SM.mamba(heads=4, vdim=64, state=128, groups=1, norm_groups=8),
                                   SM.both(2, 1, 128, 128, every=1, vdim_ssm=16, state=144, groups=4, norm_groups=1)], width=192, vocab=320),
    # sizes no vector load or tile likes; one tap, five taps
    "side-odd": SM.side_config([SM.both(3, 1, 7, 11, mlp=SM.glu(45), vdim_ssm=9, state=7, groups=1, norm_groups=3, conv=5),
                                SM.mamba(heads=6, vdim=5, state=13, groups=3, norm_groups=5, conv=1), SM.both(5, 5, 9, 6, vdim_ssm=21, state=35, conv=2)],
                               width=61, vocab=83, eps=1e-3, scale=1.0),
    "side-wide": SM.side_config([SM.both(33, 1, 40, 8, heads_ssm=1, vdim_ssm=136, state=250, groups=1, norm_groups=1, mlp=SM.glu(16)),
                                 SM.both(2, 2, 264, 264, heads_ssm=1, vdim_ssm=8, state=8, groups=1, norm_groups=1)], width=96, vocab=96),
    "state-only": SM.side_config([SM.mamba(heads=1, vdim=8, state=16, groups=1, norm_groups=1), SM.mamba(heads=16, vdim=32, state=32, groups=8, norm_groups=16)], width=64, vocab=64),
    # pooled blocks of several sizes, longer than the window and shorter than a page's part, beside matrix memories
    "pooled": SM.output_norm_config([SM.pattn(mlp=SM.plain_moe()), SM.mlstm(mlp=SM.dense(70)), SM.pattn(4, 1, 16, 24, 5, 9, 8, base=100.0),
                                     SM.mlstm(2, 16, 72, 4.0, mlp=SM.plain_moe(5, 3, 24, 0)), SM.pattn(3, 3, 40, 16, 1, 1, 40, mlp=SM.plain_moe(4, 1, 20, 40))]),
    # everything on the tensor-core kernels
    "pooled-tensor": SM.output_norm_config([SM.mlstm(4, 64, 128, 12.0, mlp=SM.plain_moe(8, 3, 64, 80)), SM.pattn(8, 2, 64, 64, 33, 4, 64, mlp=SM.dense(320)),
                                            SM.mlstm(3, 128, 80, mlp=SM.dense(64)), SM.pattn(4, 4, 128, 128, 70, 16, 32, mlp=SM.plain_moe(8, 1, 128, 64)),
                                            SM.pattn(2, 1, 200, 248, 17, 3, 24), SM.mlstm(1, 200, 24)], width=192, vocab=320),
    # sizes no vector load or tile likes, groups of more than 16 query heads, heads beyond the tiles
    "pooled-odd": SM.output_norm_config([SM.pattn(3, 1, 7, 10, 19, 5, 6, mlp=SM.dense(45)), SM.mlstm(5, 9, 13, 1.5, mlp=SM.plain_moe(5, 3, 21, 11)),
                                         SM.pattn(33, 1, 13, 6, 40, 7, 0), SM.pattn(2, 2, 264, 260, 50, 24, 100), SM.mlstm(1, 250, 7)],
                                        width=61, vocab=83, eps=1e-3, scale=1.0),
    "pooled-one": SM.output_norm_config([SM.pattn(1, 1, 8, 8, 5, 2, 8, mlp=SM.dense(20))], width=36, vocab=36),
    "memory-only": SM.output_norm_config([SM.mlstm(1, 8, 16), SM.mlstm(2, 32, 64, 20.0, mlp=SM.plain_moe(9, 9, 8, 8))], width=64, vocab=64),
}
ATTENTION_MIX = ["mixed", "tensor", "parallel", "parallel-tensor", "side", "side-tensor", "pooled", "pooled-tensor"]


class Model:
    def __init__(self, name, dtype, **kw):
        self.cfg = CONFIGS[name]
        self.t = SM.tensors(self.cfg, seed=len(name))
        self.dtype = dtype
        self.eng = SM.engine(self.cfg, self.t, dtype, **kw)

    def tokens(self, n, seed=0):
        return torch.randint(0, self.cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()

    def oracle(self, toks):
        return R.forward(self.cfg, self.t, toks)

    def given_back(self):
        e = self.eng
        return all(len(p.free) == p.n_pages for p in [e.pool, *e.block_pools]) and len(e.slots.free) == e.slots.n

    def check(self, got, want):
        got, want = got.double().cpu(), want.double()
        assert got.shape == want.shape and torch.isfinite(got).all()
        d = got - want
        err = (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / want.std(-1).mean()
        assert err.max().item() < WORST[self.dtype], (err.max().item(), int(err.argmax()))
        assert err.quantile(0.95).item() < TOL[self.dtype], err.quantile(0.95).item()

    def feed(self, toks, sizes):
        """Logits of all tokens, fed in portions of the given sizes (the last size repeats)."""
        s, out, i, k = self.eng.open(), [], 0, 0
        while i < len(toks):
            n = min(sizes[min(k, len(sizes) - 1)], len(toks) - i)
            out.append(self.eng.step([(s, toks[i:i + n], list(range(n)))]))
            i, k = i + n, k + 1
        self.eng.close_sequence(s)
        return torch.cat(out)


@pytest.mark.parametrize("dtype", TOL)
@pytest.mark.parametrize("name", CONFIGS)
def test_prompt_tokens_and_portions(name, dtype):
    m = Model(name, dtype)
    toks = m.tokens(210)
    want = m.oracle(toks)
    for sizes in ([210], [1], [2], [130, 1], [1, 3, 2, 17, 64, 5, 16, 31], [7, 150, 4, 1]):
        m.check(m.feed(toks, sizes), want)
    assert m.given_back()


@pytest.mark.parametrize("name", ATTENTION_MIX)
def test_residual_after_every_depth(name):
    """The residual stream after each layer, by running the first layers only."""
    full, t = CONFIGS[name], SM.tensors(CONFIGS[name], seed=3)
    toks = torch.randint(0, full["vocab"], (60,), generator=torch.Generator().manual_seed(1)).tolist()
    layers = []
    R.forward(full, t, toks, collect=layers)
    for k in range(1, len(full["layers"]) + 1):
        cfg = {**full, "layers": full["layers"][:k]}
        eng = SM.engine(cfg, {n: x for n, x in t.items() if not n.startswith("l") or int(n[1:n.index(".")]) < k}, "float32")
        eng.step([(eng.open(), toks, [])])
        got = eng.buf["residual"][:60 * full["width"]].view(60, -1).double().cpu()
        assert (got - layers[k - 1]).abs().max() < 2e-4 * layers[k - 1].abs().max(), k


@pytest.mark.parametrize("dtype", TOL)
@pytest.mark.parametrize("name", ATTENTION_MIX)
def test_unequal_requests_in_one_batch_equal_each_alone(name, dtype):
    """Four live requests, portions beside single tokens; pages and slots of finished ones are used again."""
    m = Model(name, dtype, tokens=448)
    rng = np.random.default_rng(7)
    todo = [(m.tokens(n, seed=n), m) for n in (100, 1, 37, 64, 129, 16, 17, 2, 80)]
    want = {len(t): m.oracle(t) for t, _ in todo}
    live, got, queue = {}, {}, [t for t, _ in todo]
    while queue or live:
        while queue and len(live) < 4:
            t = queue.pop(0)
            live[len(t)] = [m.eng.open(), t, 0]
            got[len(t)] = []
        work, order = [], []
        for n, (s, t, at) in live.items():
            if len(live) > 1 and rng.random() < 0.25:
                continue                                             # left out of this step, goes on later
            k = min(int(rng.choice([1, 1, 2, 5, 33, 64])), n - at)
            work.append((s, t[at:at + k], list(range(k))))
            order.append((n, k))
        if not work:
            continue
        out = m.eng.step(work)
        for n, k in order:
            got[n].append(out[:k])
            out = out[k:]
            live[n][2] += k
            if live[n][2] == n:
                m.eng.close_sequence(live.pop(n)[0])
    for n, parts in got.items():
        m.check(torch.cat(parts), want[n])
    assert m.given_back()


def test_wanted_places_only_and_in_order():
    m = Model("mixed", "float32", logit_rows=3)           # fewer logit rows than wanted: several head launches
    a, b = m.tokens(50, 1), m.tokens(30, 2)
    sa, sb = m.eng.open(), m.eng.open()
    out = m.eng.step([(sa, a, [0, 49, 7, 8, 9]), (sb, b, [29, 3])])
    want = torch.cat([m.oracle(a)[[0, 49, 7, 8, 9]], m.oracle(b)[[29, 3]]])
    m.check(out, want)
    assert m.eng.step([(sa, [1, 2], [])]).shape == (0, m.cfg["vocab"])


def test_step_longer_than_a_launch_is_cut():
    m = Model("tensor", "float32", tokens=256, kv_pages=48)
    a, b = m.tokens(250, 1), m.tokens(200, 2)
    sa, sb = m.eng.open(), m.eng.open()
    out = m.eng.step([(sa, a, [249]), (sb, b, [0, 199])])
    m.check(out, torch.cat([m.oracle(a)[[249]], m.oracle(b)[[0, 199]]]))


def test_pool_is_as_large_as_asked_and_says_when_it_is_full():
    m = Model("mixed", "bfloat16", tokens=64)
    s = m.eng.open()
    m.eng.step([(s, m.tokens(64), [])])
    with pytest.raises(Exception, match="max_model_len"):
        m.eng.step([(s, [1], [])])
    with pytest.raises(MemoryError):
        m.eng.step([(m.eng.open(), [1], [])])
    m.eng.close_sequence(s)
    m.eng.step([(m.eng.open(), m.tokens(64), [])])


@pytest.mark.parametrize("dtype", TOL)
@pytest.mark.parametrize("name", ["mixed", "parallel", "side", "pooled", "pooled-tensor"])
def test_long_decoding(name, dtype):
    """Windows pass over decoded tokens many times over; the state is carried through every one of them."""
    m = Model(name, dtype)
    toks = m.tokens(400, 9)
    m.check(m.feed(toks, [3, 1]), m.oracle(toks))


@pytest.mark.parametrize("dtype", ["float32"])
@pytest.mark.parametrize("name", ["mixed", "state-only", "memory-only"])
def test_a_far_token_is_remembered(name, dtype):
    """Slow decays: logits hundreds of tokens later depend on the first ones (a lost state would show)."""
    m = Model(name, dtype)
    shift = {"mixed": {"l1.mix.w0": -6.0, "l4.mix.w0": -6.0}, "state-only": {"l0.mix.A_log": -6.0, "l1.mix.A_log": -6.0},
             "memory-only": {"l0.mix.f.b": 8.0, "l1.mix.f.b": 8.0, "l0.mix.i.b": -3.0, "l1.mix.i.b": -3.0}}
    for n, by in shift[name].items():
        m.t[n] += by
    m.eng = SM.engine(m.cfg, m.t, dtype)
    toks = m.tokens(300, 4)
    want = m.oracle(toks)
    other = m.oracle(m.tokens(8, 5) + toks[8:])
    assert (want[-1] - other[-1]).std() / want[-1].std() > 50 * TOL[dtype]
    for sizes in ([300], [90, 2, 1]):
        m.check(m.feed(toks, sizes), want)


def test_learned_positions_end_where_the_table_does():
    m = Model("parallel-one", "float32")                  # 300 positions, pages for 512 tokens
    toks = m.tokens(301)
    s = m.eng.open()
    out = m.eng.step([(s, toks[:300], [0, 299])])
    m.check(out, m.oracle(toks[:300])[[0, 299]])
    with pytest.raises(Exception, match="max_model_len"):
        m.eng.step([(s, toks[300:], [0])])


@pytest.mark.parametrize("dtype", TOL)
@pytest.mark.parametrize("name", ["parallel-tensor", "side-tensor", "pooled-tensor"])
def test_prompts_of_many_tiles(name, dtype):
    """More tokens than one row tile of the products, several prompt tiles and chunks, windows across them."""
    m = Model(name, dtype, tokens=1024, max_model_len=512)
    a, b = m.tokens(500, 1), m.tokens(333, 2)
    sa, sb = m.eng.open(), m.eng.open()
    out = [m.eng.step([(sa, a[:400], list(range(400))), (sb, b[:3], [0, 1, 2])]),
           m.eng.step([(sb, b[3:], list(range(330))), (sa, a[400:], list(range(100)))])]
    want = torch.cat([m.oracle(a)[:400], m.oracle(b), m.oracle(a)[400:]])
    m.check(torch.cat(out), want)


@pytest.mark.parametrize("dtype", TOL)
def test_one_expert_takes_every_token(dtype):
    """All rows of a batch on one expert, the others empty."""
    m = Model("parallel-tensor", dtype)
    for i in (0, 2):
        r = m.t[f"l{i}.mlp.router"]
        r[:, :] = 0.01 * r
        r[5, -8:] = 0
        others = [e for e in range(8) if e != 5]
        r[others, -8:] = torch.eye(8)[others].to(r.dtype)
        m.t["embed"][:, -8:] = torch.tensor([1.0, -1.0, 0.5, -0.5, 0.0, 0.0, -2.0, -3.0]).to(r.dtype)   # 5's logit: third
    m.eng = SM.engine(m.cfg, m.t, dtype)
    toks = m.tokens(200)
    m.check(m.feed(toks, [160, 1]), m.oracle(toks))


# ------------------------------------------------------------------------------------------ generation
GEN = SM.config([SM.delta(heads=2, dim=32), SM.attn(4, 32, 32, 32, 64, 24), SM.attn(2, 32, 32, 64, 64, 40, kv_from=1), SM.delta(2, 40)],
                width=128, vocab=1024)
GENS = {"Bekopel": GEN, "Lerazen": SM.parallel_config([SM.gattn(4, 2, 32, 32, 24, mlp=SM.dense(96)), SM.gattn(4, 1, 64, 64, 40, mlp=SM.moe(8, 2, 48)),
                                                       SM.gattn(2, 2, 40, 48, 1000, v_mix=False, mlp=SM.moe(4, 1, 32))],
                                                      width=128, vocab=1024, positions=600),
        "Merulorn": SM.side_config([SM.mamba(heads=4, vdim=32, state=32), SM.both(4, 2, 32, 32, mlp=SM.glu(96)), SM.mamba(heads=2, vdim=64, state=40, norm_groups=1),
                                    SM.both(2, 1, 64, 64, vdim_ssm=16, mlp=SM.glu(64, 0.7))], width=128, vocab=1024),
        "Vosolorn": SM.output_norm_config([SM.pattn(4, 2, 32, 32, 24, 3, 16, mlp=SM.plain_moe(8, 2, 48, 32)), SM.mlstm(2, 32, 48, mlp=SM.dense(96)),
                                           SM.mlstm(4, 16, 64), SM.pattn(2, 1, 64, 64, 16, 8, 64, mlp=SM.plain_moe(4, 1, 32, 16))], width=128, vocab=1024)}


def _greedy(cfg, t, ids, out):
    """The oracle's greedy continuation, following `out` where two logits are within rounding of each other."""
    lg = R.forward(cfg, t, ids + out[:-1])[len(ids) - 1:]
    for i, tok in enumerate(out):
        top = lg[i].max()
        assert top - lg[i][tok] < 0.15 * lg[i].std(), (i, tok, int(lg[i].argmax()))
    return [int(x.argmax()) for x in lg]


@pytest.mark.parametrize("graph", [False, True])
@pytest.mark.parametrize("dtype", TOL)
@pytest.mark.parametrize("design", GENS)
def test_greedy_generation_through_the_scheduler(design, dtype, graph):
    from byzantine_consensus_llm_agents_b200.engine import Request
    from byzantine_consensus_llm_agents_b200.tokenizer import get_tokenizer
    cfg = GENS[design]
    t = SM.tensors(cfg, seed=2)
    tk = get_tokenizer("qwen3", cfg["vocab"])
    eng = SM.engine(cfg, t, dtype, tokens=256, rows=3, tokenizer=tk, kv_pages=64, use_cuda_graph=graph)
    g = torch.Generator().manual_seed(0)
    prompts = [torch.randint(0, 700, (n,), generator=g).tolist() for n in (70, 1, 16, 33, 5)]    # two waves of rows
    res = eng.generate([Request("", prompt_ids=p, max_tokens=m) for p, m in zip(prompts, (40, 60, 25, 30, 64))])
    again = eng.generate([Request("", prompt_ids=prompts[3], max_tokens=30)])[0]
    same = 0
    for p, r in zip(prompts, res):
        assert r.token_ids and r.finish in ("length", "stop")
        want = _greedy(cfg, t, p, r.token_ids)
        same += sum(a == b for a, b in zip(want, r.token_ids))
    total = sum(len(r.token_ids) for r in res)
    assert same >= total * (0.995 if dtype == "float32" else 0.9), (same, total)
    if dtype == "float32":
        assert again.token_ids == res[3].token_ids
    # a prefix is taken from its pages where they are all there is to it
    assert again.cached_tokens == (0 if eng.exec.has_state else 32)
    assert all(len(p.free) == p.n_pages for p in eng.block_pools)
    assert len(eng.slots.free) == eng.slots.n and len(eng.pool.free) + len(eng.pool.cached) == eng.pool.n_pages


@pytest.mark.parametrize("design", GENS)
def test_adapter_generates_from_a_model_directory(design, tmp_path):
    """The agents' entry point: a directory as model name, a JSON schema, greedy."""
    from byzantine_consensus_llm_agents_b200 import vllm_agent as VA
    from byzantine_consensus_llm_agents_b200.stack import StackWeights
    GEN = GENS[design]
    t = SM.tensors(GEN, seed=2)
    d = SM.save(GEN, t, tmp_path / "stack-model")
    schema = {"type": "object", "properties": {"decision": {"type": "string", "enum": ["stop", "continue"]}},
              "required": ["decision"], "additionalProperties": False}
    mc = {"max_model_len": 512, "gpu_memory_utilization": 0.5, "kv_pages": 200, "engine_max_rows": 4,
          "tensor_parallel_size": 1, "max_num_seqs": 4, "seed": 3}
    rows = [("You are agent_%d." % i, "Vote now.", schema if i % 2 else None) for i in range(6)]

    def play(name):
        a = VA.VLLMAgent("agent_0", name, mc)
        out = [a.generate_json("Vote now.", schema, temperature=0.0, max_tokens=40, system_prompt="You are agent_0.")]
        out += a.batch_generate_json([r for r in rows if r[2]], temperature=0.7, max_tokens=40)
        return out + a.batch_generate([s + u for s, u, _ in rows], temperature=0.0, max_tokens=20)
    try:
        from_dir = play(str(d))
        assert all("raw" not in r or r["raw"].startswith("{") for r in from_dir if isinstance(r, dict))
        VA.register_model("test/stack", SM.stack_config(GEN, t),
                          lambda cfg, dev: StackWeights.from_tensors(cfg, t.__getitem__, dev))
        assert play("test/stack") == from_dir
    finally:
        VA.VLLMAgent.shutdown()


# ------------------------------------------------------------------------------------------ trace replay
@pytest.mark.parametrize("dtype", TOL)
@pytest.mark.parametrize("name", ["tensor", "parallel-tensor", "side-tensor", "pooled-tensor"])
def test_trace_replay_program(tmp_path, name, dtype):
    cfg = CONFIGS[name]
    t = SM.tensors(cfg, seed=11)
    d, out = SM.save(cfg, t, tmp_path / "m"), tmp_path / "out"
    out.mkdir()
    toks = {i: torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(n)).tolist()
            for i, n in (("a", 90), ("b", 40), ("c", 64), ("d", 120))}
    plan = [([("a", 60, [0, 59]), ("b", 40, [39])], ["b"]), ([("a", 1, [0]), ("c", 64, [])], ["c"]),
            ([("a", 1, []), ("d", 20, [3])], []), ([("d", 2, [1])], []), ([("a", 28, [27]), ("d", 98, [97, 0])], ["a", "d"])]
    at, lines, want = {}, [], {}
    for n, (entries, end) in enumerate(plan):
        e = []
        for i, k, w in entries:
            lo = at.get(i, 0)
            e.append({"id": i, "tokens": toks[i][lo:lo + k], "want": w})
            want.setdefault(n, []).extend((i, lo + x) for x in w)
            at[i] = lo + k
        lines.append(json.dumps({"step": n, "entries": e, "end": end}))
    p = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(d), "--dtype", dtype, "--out", str(out),
                        "--max-tokens", "256"], input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [x for x in p.stdout.splitlines() if x.startswith("done")] == [f"done {n}" for n in range(len(plan))]
    ref = {i: R.forward(cfg, t, x) for i, x in toks.items()}
    for n, w in want.items():
        f = out / f"{n}.f32"
        assert f.exists() == bool(w)
        if w:
            got = torch.from_numpy(np.fromfile(f, "<f4")).view(len(w), cfg["vocab"]).double()
            exp = torch.stack([ref[i][k] for i, k in w])
            assert ((got - exp).pow(2).mean(-1).sqrt() / exp.std(-1)).max() < WORST[dtype]


def test_dense_models_step_and_refuse_float32(tmp_path):
    """The step interface over a uniform dense decoder: portions and mixed batches equal whole prompts."""
    from byzantine_consensus_llm_agents_b200 import trace
    from byzantine_consensus_llm_agents_b200.engine import Engine
    from byzantine_consensus_llm_agents_b200.model import ModelConfig, Weights
    from oracle.model import build_hf_model, full_logits
    cfg = ModelConfig("dense", n_layers=2, d_model=256, n_heads=4, n_kv_heads=2, d_ff=512, vocab=4096)
    hf = build_hf_model(cfg, seed=0)
    w = Weights.from_hf_state_dict(cfg, hf.state_dict(), torch.device("cuda:0"))
    eng = Engine(cfg, w, None, max_model_len=256, max_rows=4, prefill_tokens=256, kv_pages=40)
    a, b = list(range(5, 155)), list(range(900, 960))
    sa, sb = eng.open(), eng.open()
    out = [eng.step([(sa, a[:70], [69, 3])]), eng.step([(sa, a[70:71], [0]), (sb, b, list(range(60)))]), eng.step([(sa, a[71:], [78])])]
    ra, rb = full_logits(hf, a), full_logits(hf, b)
    want = torch.cat([ra[[69, 3]], ra[[70]], rb, ra[[149]]])
    assert (torch.cat(out).cpu() - want).abs().max() < 2e-2
    hf.save_pretrained(str(tmp_path / "hf"), safe_serialization=True)
    assert trace.build_engine(str(tmp_path / "hf"), "float32", 256) is None
