"""Attention over a window and pooled blocks, its input split (norms and rotations head by head, means of blocks), plain experts
with a shared one, gelu units and products, one by one against the plain oracle (oracle/stack_ref.py)."""
import ctypes as C

import numpy as np
import pytest
import torch

from byzantine_consensus_llm_agents_b200 import lib as L
from byzantine_consensus_llm_agents_b200.executors import PAGE, Entry
from oracle import stack_ref as R

import stack_models as SM
from test_gpu_state_space import OneLayer, close, gen

pytestmark = pytest.mark.gpu
DT = {"float32": (L.DT_F32, torch.float32, 3e-5), "bfloat16": (L.DT_BF16, torch.bfloat16, 1e-2)}
SIZES = {   # heads, kv_heads, dim, vdim, rotated dims
    "odd": (3, 1, 10, 14, 6), "small": (6, 3, 16, 24, 16), "even": (8, 2, 64, 64, 32), "usual": (8, 2, 128, 128, 128), "wide": (4, 2, 192, 256, 64),
    "max": (2, 1, 256, 136, 254), "group": (20, 1, 64, 128, 2), "odd-group": (33, 1, 40, 8, 0), "huge": (2, 1, 264, 300, 100), "one": (1, 1, 8, 8, 8)}


class Attention(OneLayer):
    make = staticmethod(SM.output_norm_config)

    def __init__(self, size, window, pool, dtype, tokens=512, **kw):
        H, G, dim, vdim, dims = SIZES[size]
        super().__init__(SM.pattn(H, G, dim, vdim, window, pool, dims, base=1e3, scale=dim ** -0.5), dtype, width=32, tokens=tokens, seed=H + dim, **kw)
        self.m, self.window, self.pool = self.cfg["layers"][0]["mixer"], window, pool
        self.cache = list(self.x.caches[0].values())

    def table(self, n, pages, block_pages):
        """Block table of a sequence of n tokens; pages are taken from the lists."""
        bt, e = np.zeros(self.x.table_cols, np.int32), self.eng
        bt[:-(-n // PAGE)] = [pages.pop() for _ in range(-(-n // PAGE))]
        col, k = self.x.block_pools[0][1], -(-(n // self.pool) // PAGE)
        bt[col:col + k] = [e.pool.n_pages + block_pages.pop() for _ in range(k)]
        return bt

    def page_lists(self):
        r = np.random.default_rng(0)
        return list(r.permutation(self.eng.pool.n_pages)), list(r.permutation(self.eng.block_pools[0].n_pages))

    def rows(self, cache, bt, col, n, ld):
        """Entries 0 .. n - 1 of a sequence behind column `col` of its table: [n, kv_heads, ld]."""
        out = [cache[int(bt[col + j // PAGE]), :, j % PAGE, :ld] for j in range(n)]
        return torch.stack(out) if out else cache.new_zeros(0, cache.shape[1], ld)

    def fill(self, cache, bt, col, x):
        for j in range(-(-len(x) // PAGE)):
            part = x[j * PAGE:(j + 1) * PAGE].transpose(0, 1)
            cache[int(bt[col + j]), :, :part.shape[1], :part.shape[2]] = part.to(cache.dtype).cuda()

    def run(self, seqs, mode=0):
        """seqs: [(keys [n, G, dim], values [n, G, vdim], queries [k, H, dim] of its last k tokens)]."""
        m, e = self.m, self.eng
        pages, block_pages = self.page_lists()
        for c in self.cache:
            c.copy_(torch.randn(c.shape, generator=gen(1)).to(self.td) * 50)       # rows nobody wrote must not matter
        r = lambda x: x.to(self.td).double()
        entries, want = [], []
        for k, v, q in seqs:
            n = len(k)
            bt = self.table(n, pages, block_pages)
            blocks = [R.block_means(r(x), self.pool) for x in (k, v)]
            for c, x, mean in zip(self.cache, (k, v), blocks):
                self.fill(c, bt, 0, x)
                self.fill(c, bt, self.x.block_pools[0][1], mean)
            entries.append(Entry([0] * len(q), n - len(q), bt))
            want += [self.oracle(n - len(q) + i, r(k), r(v), *[r(x) for x in blocks], r(q)[i]) for i in range(len(q))]
        p, b = self.batch(entries)
        q = torch.zeros(p.T, m["heads"], self.layer.q_ld)
        q[..., :m["dim"]] = torch.cat([q for _, _, q in seqs])
        self.set("q", q)
        L.check(e.lib.bcg_grouped_attention(*self.args(C.byref(b), 0, mode)))
        out = self.get("mix", p.T, self.layer.mix_ld)[:, :m["heads"] * m["vdim"]].reshape(p.T, m["heads"], m["vdim"])
        return out, torch.stack(want)

    def oracle(self, pos, k, v, kb, vb, q):
        """The query at position pos; k, v: the sequence, kb, vb: its blocks."""
        m, n = self.m, len(k)
        ok = torch.cat([R.window_visible(n, self.window), R.blocks_visible(n, len(kb), self.window, self.pool)], dim=1)[pos]
        mine = torch.arange(m["heads"]) // (m["heads"] // m["kv_heads"])
        s = torch.einsum("hd,jhd->hj", q, torch.cat([k, kb])[:, mine]) * m["scale"]
        o = torch.einsum("hj,jhv->hv", R.softmax_with_sink(s[:, None], ok[None])[:, 0], torch.cat([v, vb])[:, mine])
        return R.rotate_pairs(o[None], torch.tensor([pos]), m["vdim"], 1e3, back=True)[0]


def _seqs(a, shapes, seed, gain=2.0):
    m, g = a.m, gen(seed)
    return [(torch.randn(n, m["kv_heads"], m["dim"], generator=g), torch.randn(n, m["kv_heads"], m["vdim"], generator=g),
             torch.randn(k, m["heads"], m["dim"], generator=g) * gain) for n, k in shapes]


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("size", SIZES)
@pytest.mark.parametrize("window,pool", [(1, 1), (1, 3), (17, 4), (40, 64), (65, 16), (130, 5), (300, 8)])
def test_window_and_blocks_share_one_softmax(size, window, pool, dtype):
    """Whole prompts, portions and single tokens, mixed; pages in any order."""
    if dtype == "float32" and size not in ("odd", "even", "odd-group"):
        pytest.skip("one kernel for all sizes")
    a = Attention(size, window, pool, dtype, tokens=1024)
    for shapes in ([(150, 150), (41, 1), (210, 2), (90, 33)], [(300, 1), (1, 1), (64, 1), (129, 1), (17, 1)]):
        got, want = a.run(_seqs(a, shapes, window + pool))
        close(got, want, DT[dtype][2])


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("context", [70, 333, 2000])
def test_single_tokens_at_many_cluster_sizes(context, dtype):
    a = Attention("even", 48, 3, dtype, tokens=2048)
    for n in (1, 4):
        got, want = a.run(_seqs(a, [(context - 7 * i, 1) for i in range(n)][:1 if context > 700 else n], context))
        close(got, want, DT[dtype][2])


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("size,window,pool", [("small", 16, 5), ("usual", 63, 16), ("usual", 64, 16), ("even", 33, 32), ("huge", 20, 7), ("wide", 64, 3)])
@pytest.mark.parametrize("portion", [1, 2, 40])
def test_one_loud_key_at_the_edges(size, window, pool, portion, dtype):
    """One key outweighs all others where it is seen: as the window's first token, the last one in front of it, in the last
    block that has left the window and in the first one that has not yet."""
    a = Attention(size, window, pool, dtype)
    m, n = a.m, 200
    pos = n - 1                                         # the query that is checked
    first = pos - window + 1                            # first token of its window
    gone = first // pool                                # blocks it sees
    edges = {first: True, first - 1: first % pool == 0, gone * pool - 1: True, gone * pool: gone * pool >= first, gone * pool - pool: True}
    for key, seen in edges.items():
        (k, v, q), = _seqs(a, [(n, portion)], key, gain=0.2)
        d = torch.nn.functional.normalize(torch.randn(m["dim"], generator=gen(5)), dim=0)
        q[-1] += 6.0 * d
        k[key] += 5.0 * pool ** 0.5 * m["dim"] ** 0.5 * d    # loud alone and as a part of its block's mean
        v[key] += 20.0
        got, want = a.run([(k, v, q)])
        quiet = v.clone()
        quiet[key] -= 20.0
        _, without = a.run([(k, quiet, q)])
        assert ((want[-1] - without[-1]).abs().max() > 0.3) == seen, (key, first)
        close(got, want, 1.5 * DT[dtype][2])


# ------------------------------------------------------------------------------------------ input split
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("size", SIZES)
@pytest.mark.parametrize("sizes", [[100], [1], [2, 33, 1, 1, 17]])
def test_heads_are_normed_rotated_and_pooled(size, sizes, dtype):
    """Queries, cached keys and values, and the means of every block that is whole, however the sequence was cut."""
    a = Attention(size, 20, 6, dtype)
    H, G, dim, vdim, dims = SIZES[size]
    n, ld, cols = 100, a.eng.cfg.in_rows(0), H * dim + G * (dim + vdim)
    x = torch.randn(n, cols, generator=gen(dim))
    w = {k[len("l0.mix."):]: t.double() for k, t in a.t.items() if k.startswith("l0.mix.")}
    pos = torch.arange(n)
    q, k, v = torch.split(x.double(), [H * dim, G * dim, G * vdim], dim=1)
    q = R.rotate_pairs(R.rms_norm(q.view(n, H, dim), 1e-5, w["q.norm"]), pos, dims, 1e3)
    k = R.rotate_pairs(R.rms_norm(k.view(n, G, dim), 1e-5, w["k.norm"]), pos, dims, 1e3)
    v = R.rotate_pairs(v.view(n, G, vdim), pos, vdim, 1e3)
    bt = a.table(n, *a.page_lists())
    at, i, got_q = 0, 0, []
    while at < n:
        t = min(sizes[min(i, len(sizes) - 1)], n - at)
        slabs = 1 + i % 5
        p, b = a.batch([Entry([0] * t, at, bt)])
        full = torch.zeros(slabs, t, ld)
        rest = x[at:at + t]
        for s in range(slabs - 1):
            full[s, :, :cols] = torch.randn(t, cols, generator=gen(s))
            rest = rest - full[s, :, :cols]
        full[slabs - 1, :, :cols] = rest
        a.set("proj", full)
        L.check(a.eng.lib.bcg_grouped_in(*a.args(C.byref(b), 0, slabs, t * ld, ld, 0)))
        got_q.append(a.get("q", t, H, a.layer.q_ld)[..., :dim])
        at, i = at + t, i + 1
    tol = DT[dtype][2]
    close(torch.cat(got_q), q, tol)
    col = a.x.block_pools[0][1]
    for c, want, width in zip(a.cache, (k, v), (dim, vdim)):
        held = a.rows(c, bt, 0, n, width).double().cpu()
        close(held, want, tol)
        mean = a.rows(c, bt, col, n // 6, width)
        close(mean, R.block_means(held, 6), 4e-3 if dtype == "bfloat16" else 1e-6)      # means of what the cache holds


@pytest.mark.parametrize("dtype", DT)
def test_far_positions_turn_exactly(dtype):
    a = Attention("small", 20, 6, dtype, tokens=16384)
    H, G, dim, vdim, dims = SIZES["small"]
    ld, cols = a.eng.cfg.in_rows(0), H * dim + G * (dim + vdim)
    bt = np.zeros(a.x.table_cols, np.int32)
    p, b = a.batch([Entry([0] * 2, 16001, bt)])
    x = torch.randn(2, cols, generator=gen(1))
    full = torch.zeros(1, 2, ld)
    full[0, :, :cols] = x
    a.set("proj", full)
    L.check(a.eng.lib.bcg_grouped_in(*a.args(C.byref(b), 0, 1, 2 * ld, ld, 0)))
    q = R.rms_norm(x[:, :H * dim].double().view(2, H, dim), 1e-5, a.t["l0.mix.q.norm"].double())
    close(a.get("q", 2, H, a.layer.q_ld)[..., :dim], R.rotate_pairs(q, torch.tensor([16001, 16002]), dims, 1e3), DT[dtype][2])


def test_finished_rows_write_no_blocks():
    a = Attention("even", 20, 6, "bfloat16")
    bt = a.table(12, *a.page_lists())
    p, b = a.batch([Entry([0], 11, bt), Entry([0], 5, bt)])
    a.keep["slots"][:] = -1
    before = [c.clone() for c in a.cache]
    a.set("proj", torch.randn(1, 2, a.eng.cfg.in_rows(0)))
    ld = a.eng.cfg.in_rows(0)
    L.check(a.eng.lib.bcg_grouped_in(*a.args(C.byref(b), 0, 1, 2 * ld, ld, 0)))
    torch.cuda.synchronize()
    assert all(torch.equal(x, y) for x, y in zip(before, a.cache))


# ------------------------------------------------------------------------------------------ experts
class Experts(OneLayer):
    make = staticmethod(SM.output_norm_config)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("width,experts,top,ff,shared", [(64, 8, 1, 64, 64), (64, 8, 3, 48, 0), (72, 5, 5, 20, 33), (61, 7, 2, 13, 8), (128, 40, 4, 160, 16),
                                                         (1024, 4, 2, 256, 512)])
@pytest.mark.parametrize("T", [1, 7, 60, 128, 129, 300])
def test_plain_experts(dtype, width, experts, top, ff, shared, T):
    """Routing by biased logits, weights of the chosen ones only, every expert's rows, the shared unit."""
    o = Experts(SM.mlstm(1, 8, 8, mlp=SM.plain_moe(experts, top, ff, shared)), dtype, width=width, seed=ff, prefill_tokens=512)
    f, tol = o.eng.cfg.layers[0].mlp, 1.5 * DT[dtype][2]
    g = gen(T + width)
    x = torch.randn(T, width, generator=g).to(o.td)
    z = torch.stack([torch.randperm(experts, generator=g) for _ in range(T)]).float() * 0.7 - 1.0      # logits without the bias, far apart
    up = torch.randn(T, max(shared, 1), generator=g)
    n = f.router_rows + f.shared_ld
    slabs = 2 if T <= 128 else 1
    full = torch.zeros(slabs, T, n)
    full[:, :, :experts] = z / slabs
    full[-1, :, f.router_rows:f.router_rows + shared] = up[:, :shared]
    o.set("proj", full)
    o.set("xn", x)
    o.x.buf["moe_counts"].zero_()
    L.check(o.eng.lib.bcg_expert_in(*o.args(0, T, slabs, T * n, n, 1)))
    splits = C.c_int()
    L.check(o.eng.lib.bcg_experts(*o.args(0, T, C.byref(splits))))
    bias = o.t["l0.mlp.router.b"].double()
    pick, weight = R.route_softmax(z.double(), torch.eye(experts, dtype=torch.float64), bias, top)
    got_e, got_w = o.get("moe_expert", T, top).long(), o.get("moe_weight", T, top).double()
    assert torch.equal(got_e.sort(1).values, pick.sort(1).values)
    dense = lambda e, w: torch.zeros(T, experts, dtype=torch.float64).scatter(1, e, w)
    close(dense(got_e, got_w), dense(pick, weight), 1e-5)
    assert torch.equal(o.get("moe_counts", experts).long(), torch.bincount(pick.flatten(), minlength=experts))
    rows = o.get("moe_row", T, top)
    assert sorted(rows.flatten().tolist()) == list(range(T * top))
    out = o.get("moe_out", splits.value, T * top, width).double().sum(0)
    w = lambda e, m: o.t[f"l0.mlp.e{e}.{m}"].double()
    want = torch.zeros(T * top, width, dtype=torch.float64)
    for e in range(experts):
        t, k = (got_e == e).nonzero(as_tuple=True)
        want[rows[t, k].long()] = R.gelu_erf(x[t].double() @ w(e, "up").T) @ w(e, "down").T
    close(out, want, tol)
    if shared:
        act = o.get("act", T, f.shared_ld)
        close(act[:, :shared], R.gelu_erf(up.double()), tol)
        assert not act[:, shared:].any()


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("gated", [0, 1])
@pytest.mark.parametrize("T,ff,parts", [(1, 16, 1), (3, 96, 4), (5, 2048, 6), (150, 640, 1)])
def test_gelu_units_of_slabs(dtype, gated, T, ff, parts):
    code, td, tol = DT[dtype]
    z = torch.randn(parts, T, (1 + gated) * ff, generator=gen(ff)) * 2.0
    out = torch.empty(T, ff, dtype=td, device="cuda")
    Z = z.cuda()
    L.check(L.load().bcg_gelu_unit(Z.data_ptr(), parts, T * (1 + gated) * ff, out.data_ptr(), code, T, ff, gated, L.stream_ptr()))
    s = z.double().sum(0)
    if gated:
        s = s.view(T, ff // 16, 2, 16)
        want = (R.gelu_tanh(s[:, :, 0]) * s[:, :, 1]).reshape(T, ff)
    else:
        want = R.gelu_erf(s)
    close(out, want, tol)


@pytest.mark.parametrize("gated", [0, 1])
@pytest.mark.parametrize("M,N,K", [(129, 64, 64), (300, 96, 200), (700, 256, 128), (600, 2080, 192), (513, 2048, 64)])
def test_gelu_products(M, N, K, gated):
    g = gen(M + N)
    x, w = torch.randn(M, K, generator=g).bfloat16(), (torch.randn(N, K, generator=g) * 2 * K ** -0.5).bfloat16()
    out = torch.empty(M, N // (1 + gated), dtype=torch.bfloat16, device="cuda")
    X, W = x.cuda(), w.cuda()
    L.check(L.load().bcg_gemm_bf16_gelu(X.data_ptr(), W.data_ptr(), out.data_ptr(), M, N, K, gated, 0, L.stream_ptr()))
    z = x.double() @ w.double().T
    if gated:
        z = z.view(M, N // 32, 2, 16)
        want = (R.gelu_tanh(z[:, :, 0]) * z[:, :, 1]).reshape(M, N // 2)
    else:
        want = R.gelu_erf(z)
    close(out, want, 1e-2)


def test_gelu_far_from_zero():
    z = torch.linspace(-40, 40, 1600).view(1, 1600)
    for gated in (0, 1):
        out = torch.empty(1, 1600 // (1 + gated), device="cuda")
        Z = z.cuda()
        L.check(L.load().bcg_gelu_unit(Z.data_ptr(), 1, 1600, out.data_ptr(), L.DT_F32, 1, 1600 // (1 + gated), gated, L.stream_ptr()))
        s = z.double().view(1, -1, 2, 16)
        want = (R.gelu_tanh(s[:, :, 0]) * s[:, :, 1]).reshape(1, -1) if gated else R.gelu_erf(z.double())
        assert torch.isfinite(out).all()
        close(out, want, 1e-6)
