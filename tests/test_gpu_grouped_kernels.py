"""The kernels of parallel layers one by one — grouped attention with a distance bias, its input split, experts,
the residual addition, the squared-relu product — against the plain oracle (oracle/stack_ref.py)."""
import ctypes as C

import numpy as np
import pytest
import torch

from byzantine_consensus_llm_agents_b200 import lib as L
from byzantine_consensus_llm_agents_b200.executors import Entry
from oracle import stack_ref as R

import stack_models as SM

pytestmark = pytest.mark.gpu
DT = {"float32": (L.DT_F32, torch.float32, 3e-5), "bfloat16": (L.DT_BF16, torch.bfloat16, 1e-2)}


def gen(seed):
    return torch.Generator().manual_seed(seed)


def close(got, want, tol):
    got, want = got.double().cpu(), want.double()
    assert torch.isfinite(got).all()
    err = (got - want).abs().max().item() / max(want.abs().max().item(), 1e-6)
    assert err < tol, err


class OneLayer:
    """A one-layer model inside an engine; its buffers are set and read by hand."""

    def __init__(self, layer, dtype, width=64, seed=0, tokens=512, **kw):
        self.cfg = SM.parallel_config([layer], width=width, vocab=16, positions=tokens)
        self.t = SM.tensors(self.cfg, seed=seed)
        self.eng = SM.engine(self.cfg, self.t, dtype, tokens=tokens, rows=kw.pop("rows", 4), **kw)
        self.m, self.td, self.x = layer["mixer"], self.eng.cfg.torch_dtype, self.eng.exec
        self.layer = self.x.model.struct.layers[0]

    def args(self, *rest):
        return (C.byref(self.x.model.struct), C.byref(self.x.ws), *rest, L.stream_ptr())

    def set(self, name, value):
        b = self.x.buf[name]
        b[:value.numel()] = value.to(b.dtype).flatten().cuda()

    def get(self, name, *shape):
        torch.cuda.synchronize()
        n = int(np.prod(shape))
        return self.x.buf[name].flatten()[:n].view(*shape).cpu()

    def batch(self, entries):
        p = self.x.plan(entries)
        v = {k: torch.as_tensor(np.asarray(a, np.int32)).cuda() for k, a in p.arrays.items()}
        b = self.x._batch(p.T, p.n_seqs)
        b.positions, b.slot_map, b.ids = v["pos"].data_ptr(), v["slots"].data_ptr(), v["ids"].data_ptr()
        b.row_seq, b.seq_start, b.block_table = v["row_seq"].data_ptr(), v["seq_start"].data_ptr(), v["bt"].data_ptr()
        b.max_context = p.extra["context"]
        b.single_rows, b.n_single = v["singles"].data_ptr() if p.extra["n_single"] else None, p.extra["n_single"]
        b.tiles, b.n_tiles = v["tiles"].data_ptr(), p.extra["n_tiles"]
        self.keep = v
        return p, b


# ------------------------------------------------------------------------------------------ attention
SIZES = {   # heads, kv_heads, dim, vdim
    "plain": (3, 1, 10, 20), "small": (6, 3, 16, 24), "even": (8, 2, 64, 64), "usual": (8, 2, 128, 128), "wide": (4, 2, 192, 256),
    "max": (2, 1, 256, 136), "group": (20, 1, 64, 128), "odd-group": (33, 1, 40, 8), "huge": (2, 1, 264, 300), "one": (1, 1, 8, 8)}


class Attention(OneLayer):
    def __init__(self, size, window, dtype, tokens=512, **kw):
        H, G, dim, vdim = SIZES[size]
        super().__init__(SM.gattn(H, G, dim, vdim, window, v_mix=False, scale=dim ** -0.5), dtype, width=32, tokens=tokens,
                         seed=H + dim, state_slots=4, **kw)
        self.window = window

    def run(self, seqs, mode=0):
        """seqs: [(keys [n, G, dim], values [n, G, vdim], queries [k, H, dim] of its last k tokens)]."""
        m, e = self.m, self.eng
        ck, cv = self.x.caches[0].values()
        junk = torch.randn(ck.shape[:3], generator=gen(1))[..., None].to(self.td).cuda() * 50
        ck[..., :m["dim"]] = junk             # rows nobody wrote must not matter
        cv[..., :m["vdim"]] = junk
        pages = list(np.random.default_rng(0).permutation(ck.shape[0]))
        entries = []
        for k, v, q in seqs:
            n = len(k)
            bt = np.zeros(e.max_blocks, np.int32)
            bt[:-(-n // 16)] = [pages.pop() for _ in range(-(-n // 16))]
            for j in range(-(-n // 16)):
                rows = min(16, n - j * 16)
                ck[int(bt[j]), :, :rows, :m["dim"]] = k[j * 16:j * 16 + rows].transpose(0, 1).to(self.td).cuda()
                cv[int(bt[j]), :, :rows, :m["vdim"]] = v[j * 16:j * 16 + rows].transpose(0, 1).to(self.td).cuda()
            entries.append(Entry([0] * len(q), n - len(q), bt))
        p, b = self.batch(entries)
        q_ld = self.layer.q_ld
        q = torch.zeros(p.T, m["heads"], q_ld)
        q[..., :m["dim"]] = torch.cat([q for _, _, q in seqs])
        self.set("q", q)
        L.check(e.lib.bcg_grouped_attention(*self.args(C.byref(b), 0, mode)))
        out = self.get("mix", p.T, self.layer.mix_ld)[:, :m["heads"] * m["vdim"]].reshape(p.T, m["heads"], m["vdim"])
        r = lambda x: x.to(self.td).double()
        return out, [(len(k) - len(q) + i, r(k), r(v), r(q)[i]) for k, v, q in seqs for i in range(len(q))]

    def oracle(self, pos, k, v, q, window=None):
        m, w = self.m, self.window if window is None else window
        lo = max(0, pos - w + 1) if w else 0
        mine = torch.arange(m["heads"]) // (m["heads"] // m["kv_heads"])
        k, v = k[lo:pos + 1, mine], v[lo:pos + 1, mine]
        s = torch.einsum("hd,jhd->hj", q, k) * m["scale"]
        s = s - R.head_slopes(m["heads"])[:, None] * (pos - torch.arange(lo, pos + 1))
        return torch.einsum("hj,jhv->hv", torch.softmax(s, -1), v)


def _seqs(a, shapes, seed, gain=2.0):
    m, g = a.m, gen(seed)
    return [(torch.randn(n, m["kv_heads"], m["dim"], generator=g), torch.randn(n, m["kv_heads"], m["vdim"], generator=g),
             torch.randn(k, m["heads"], m["dim"], generator=g) * gain) for n, k in shapes]


def _check(a, seqs, tol, mode=0):
    out, meta = a.run(seqs, mode)
    assert torch.isfinite(out.float()).all()
    want = torch.stack([a.oracle(*x) for x in meta])
    err = (out.double() - want).flatten(1).norm(dim=1) / want.flatten(1).norm(dim=1).clamp_min(1e-3 * want.norm() / len(want) ** 0.5)
    assert err.max().item() < tol, (err.max().item(), int(err.argmax()))
    return out, meta


@pytest.mark.parametrize("size", SIZES)
@pytest.mark.parametrize("window", [1, 2, 16, 17, 65, 130, 400, 0])
def test_grouped_attention_bf16(size, window):
    """Portions with and without history, two-token portions and single tokens in one batch."""
    a = Attention(size, window, "bfloat16")
    seqs = _seqs(a, ((150, 150), (97, 30), (90, 1), (66, 2)), window)
    _check(a, seqs, 2e-2)
    _check(a, seqs, 2e-2, mode=1)
    _check(a, [(k, v, q[-1:]) for k, v, q in seqs], 2e-2)


@pytest.mark.parametrize("size", ["plain", "even", "odd-group", "huge"])
@pytest.mark.parametrize("window", [1, 17, 64, 400])
def test_grouped_attention_fp32(size, window):
    a = Attention(size, window, "float32")
    _check(a, _seqs(a, ((300, 20), (40, 40), (9, 1)), window), 3e-6)


@pytest.mark.parametrize("context", [1, 15, 16, 17, 333, 2000])
@pytest.mark.parametrize("window", [0, 700])
def test_single_tokens_at_many_cluster_sizes(context, window):
    """Few and many rows (one to eight CTAs share a token's pages), contexts from one key to many pages."""
    a = Attention("usual", window, "bfloat16", tokens=2048, rows=40, kv_pages=40 * 128)
    for rows in (1, 3, 40):
        _check(a, _seqs(a, [(max(1, context - 7 * i % context), 1) for i in range(rows)], rows), 2e-2)


@pytest.mark.parametrize("size", ["small", "usual", "max", "huge"])
@pytest.mark.parametrize("window", [16, 63, 64, 100])
@pytest.mark.parametrize("portion", [1, 2, 40])
def test_window_edge_holds_one_loud_key(size, window, portion):
    """A key whose score dwarfs all others, distance bias included, sits just inside, then just outside, the last
    query's window; the answer must follow it, and a window off by one would show."""
    a = Attention(size, window, "bfloat16")
    m, n = a.m, 203
    for inside in (True, False):
        (k, v, q), = _seqs(a, ((n, portion),), window, 1.0)
        q[..., 0] = 1.0
        k *= 0.1
        edge = n - window - (0 if inside else 1)
        k[edge, :, 0] = (40.0 + window) / m["scale"]
        out, meta = _check(a, [(k, v, q)], 2e-2)
        pos, kk, vv, qq = meta[-1]
        loud = vv[edge, torch.arange(m["heads"]) // (m["heads"] // m["kv_heads"])]
        near = (out[-1].double() - loud).norm() / loud.norm()
        assert (near < 0.02) == inside, near.item()
        wrong = a.oracle(pos, kk, vv, qq, window=window + (-1 if inside else 1))
        assert (wrong - out[-1].double()).norm() / loud.norm() > 0.2


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("portion", [1, 3, 70])
def test_distance_bias_decides_between_equal_keys(dtype, portion):
    """All keys score the same: the weights are the bias alone, a geometric series from the newest key back, and
    the flattest head still hears keys hundreds of tokens away."""
    a = Attention("even", 0, dtype)
    (k, v, q), = _seqs(a, ((470, portion),), 5)
    k[:] = 0
    v[:] = 0
    v[100] = 1000.0                                        # far from every query of the portion
    out, meta = _check(a, [(k, v, q)], 2e-2 if dtype == "bfloat16" else 1e-5)
    got = out[-1].double()[:, 0]
    s = R.head_slopes(8)
    want = 1000 * torch.exp(-s * 369) * (1 - torch.exp(-s)) / (1 - torch.exp(-s * 470))
    assert got[-1] > 0.5 and got[0] == 0 and ((got - want).abs() / want.max()).max() < 2e-2


# ------------------------------------------------------------------------------------------ inputs
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("heads,kv,dim,vdim,ff,experts", [(3, 1, 7, 11, 45, 0), (8, 2, 64, 32, 96, 0), (4, 4, 20, 8, 0, 6), (2, 1, 260, 4, 0, 40), (2, 2, 16, 4, 0, 70)])
def test_projection_is_split_biased_and_stored(dtype, heads, kv, dim, vdim, ff, experts):
    mlp = SM.dense(ff) if ff else SM.moe(experts, 45 if experts > 45 else 3, 16)
    o = OneLayer(SM.gattn(heads, kv, dim, vdim, coef=0.7, every=9, mlp=mlp), dtype, seed=dim, width=96)
    td, tol, l = o.td, (4e-3 if dtype == "bfloat16" else 2e-6), o.layer
    starts = [40, 0, 7]
    entries, lens, used = [], [5, 1, 20], []
    for s, (at, n) in enumerate(zip(starts, lens)):
        bt = np.zeros(o.eng.max_blocks, np.int32)
        bt[:4] = [s * 4 + 3, s * 4 + 1, s * 4, s * 4 + 2]
        entries.append(Entry([0] * n, at, bt))
        used += [(bt[(at + i) // 16], (at + i) % 16) for i in range(n)]
    p, b = o.batch(entries)
    T, n_in, parts = p.T, l.n_in, 3
    proj = torch.randn(parts, T, n_in, generator=gen(T))
    o.set("proj", proj)
    first = torch.randn(T, kv * vdim, generator=gen(9))
    l.v_mix = 0.3
    for role in (0, L.VALUES_FIRST, L.VALUES_MIX):
        l.v_role = role
        o.set("v_first", first)
        for c in o.x.caches[0].values():
            c.zero_()
        o.set("moe_counts", torch.zeros(experts + 8))
        L.check(o.eng.lib.bcg_grouped_in(*o.args(C.byref(b), 0, parts, T * n_in, n_in, 1)))
        y = proj.double().sum(0)
        nq, nk, nv = heads * dim, kv * dim, kv * vdim
        bias = lambda n: o.t[f"l0.mix.{n}.b"].double()
        pos = torch.tensor([at + i for at, n in zip(starts, lens) for i in range(n)])
        q = (y[:, :nq] + bias("q")) * R.query_temperature(pos, 0.7, 9)[:, None]
        k, v = y[:, nq:nq + nk] + bias("k"), y[:, nq + nk:nq + nk + nv] + bias("v")
        close(o.get("q", T, heads, l.q_ld)[..., :dim], q.view(T, heads, dim), tol)
        own = v
        if role == L.VALUES_MIX:
            v = R.mix_values(v, first.double(), 0.3)
        close(o.get("v_first", T, nv), own if role == L.VALUES_FIRST else first, 2e-6)
        ck, cv = (c.cpu() for c in o.x.caches[0].values())
        close(torch.stack([ck[pg, :, r, :dim] for pg, r in used]), k.view(T, kv, dim), tol)
        close(torch.stack([cv[pg, :, r, :vdim] for pg, r in used]), v.view(T, kv, vdim), tol)
        for c, n in ((ck, dim), (cv, vdim)):                # nothing else is touched
            for pg, r in used:
                c[pg, :, r, :n] = 0
            assert not c.any()
        if ff:
            act = o.get("mix", T, l.mix_ld)[:, l.act_col:l.act_col + ff]
            close(act, R.squared_relu(y[:, l.n_qkv:l.n_qkv + ff]), tol)
        else:
            z = y[:, l.router_col:l.router_col + experts]
            top = l.top
            w, e = torch.topk(torch.sigmoid(z), top)
            assert torch.equal(o.get("moe_expert", T, top).long(), e)
            close(o.get("moe_weight", T, top), w, 2e-6)
            counts = o.get("moe_counts", experts)
            assert torch.equal(counts.long(), torch.bincount(e.flatten(), minlength=experts))
            rank = o.get("moe_rank", T, top)
            for x in range(experts):                        # every expert's rows are numbered without gaps
                assert sorted(rank[e == x].tolist()) == list(range(int(counts[x])))


def test_finished_rows_write_nothing():
    o = OneLayer(SM.gattn(4, 2, 16, 16, mlp=SM.dense(32)), "bfloat16")
    p, b = o.batch([Entry([0], 5, np.full(o.eng.max_blocks, 3, np.int32))])
    o.keep["slots"].fill_(-1)
    o.set("proj", torch.ones(o.layer.n_in))
    L.check(o.eng.lib.bcg_grouped_in(*o.args(C.byref(b), 0, 1, 0, o.layer.n_in, 1)))
    torch.cuda.synchronize()
    assert not any(c.any() for c in o.x.caches[0].values())


def test_temperature_steps_at_multiples():
    pos = torch.tensor([0, 1, 254, 255, 256, 511, 512])
    t = R.query_temperature(pos, 0.5, 256)
    want = [0, 0, 0, 1, 1, 2, 2]
    assert torch.allclose(t, torch.tensor([1 + 0.5 * np.log(n + 1) for n in want], dtype=torch.float64))
    o = OneLayer(SM.gattn(1, 1, 4, 4, coef=0.5, every=256), "float32", tokens=528)
    for x, n in zip(pos.tolist(), want):
        p, b = o.batch([Entry([0], x, np.zeros(o.eng.max_blocks, np.int32))])
        o.set("proj", torch.ones(o.layer.n_in))
        L.check(o.eng.lib.bcg_grouped_in(*o.args(C.byref(b), 0, 1, 0, o.layer.n_in, 1)))
        close(o.get("q", 4), (1 + o.t["l0.mix.q.b"].double()) * (1 + 0.5 * np.log(n + 1)), 1e-6)


# ------------------------------------------------------------------------------------------ experts
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("width,experts,top,ff,limit", [(64, 8, 1, 64, 2.0), (64, 8, 3, 48, 0.5), (72, 5, 5, 20, 1.0), (61, 7, 2, 13, 7.0),
                                                        (128, 40, 4, 160, 1.5), (1024, 4, 2, 256, 3.0)])
@pytest.mark.parametrize("T", [1, 7, 20, 60, 128, 129, 300])
def test_experts(dtype, width, experts, top, ff, limit, T):
    """Any number of tokens, experts with none, few and many rows; the weight scales the expert's input."""
    o = OneLayer(SM.gattn(1, 1, 8, 8, mlp=SM.moe(experts, top, ff, limit)), dtype, width=width, seed=ff)
    g = gen(T + width)
    x = torch.randn(T, width, generator=g).to(o.td).double()
    pick = torch.stack([torch.randperm(max(top, experts * 2 // 3), generator=g)[:top] for _ in range(T)])   # some experts stay empty
    weight = torch.rand(T, top, generator=g).double() + 0.3
    counts = torch.bincount(pick.flatten(), minlength=experts)
    rank, seen = torch.zeros(T, top), [0] * experts
    for t in reversed(range(T)):                            # any numbering of an expert's rows will do
        for k in range(top):
            rank[t, k] = seen[pick[t, k]]
            seen[pick[t, k]] += 1
    for n, v in (("xn", x), ("moe_expert", pick), ("moe_rank", rank), ("moe_weight", weight), ("moe_counts", counts)):
        o.set(n, v)
    splits = C.c_int()
    L.check(o.eng.lib.bcg_experts(*o.args(0, T, C.byref(splits))))
    rows = o.get("moe_row", T, top)
    assert sorted(rows.flatten().tolist()) == list(range(T * top))
    out = o.get("moe_out", splits.value, T * top, width).double().sum(0)
    w32 = weight.float().double()
    for t in range(T):
        for k in range(top):
            e, h = int(pick[t, k]), w32[t, k] * x[t]
            f = lambda n: o.t[f"l0.mlp.e{e}.{n}"].double()
            y = f("down") @ R.clamped_glu(f("gate") @ h, f("up") @ h, limit)
            close(out[rows[t, k]], y, 1.5e-2 if dtype == "bfloat16" else 3e-5)


def test_more_experts_than_the_tensor_core_product_takes():
    """600 experts, bf16: the CUDA-core product; prompt and decode sizes."""
    n, d = 600, 608
    o = OneLayer(SM.gattn(1, 1, 8, 8, mlp=SM.moe(n, 2, 16, 1.0)), "bfloat16", width=d)
    for T in (3, 140):
        g = gen(T)
        x = torch.randn(T, d, generator=g).to(o.td).double()
        pick = torch.stack([torch.randperm(n, generator=g)[:2] for _ in range(T)])
        rank, seen = torch.zeros(T, 2), [0] * n
        for t in range(T):
            for k in range(2):
                rank[t, k] = seen[pick[t, k]]
                seen[pick[t, k]] += 1
        for name, v in (("xn", x), ("moe_expert", pick), ("moe_rank", rank), ("moe_weight", torch.full((T, 2), 0.5)),
                        ("moe_counts", torch.bincount(pick.flatten(), minlength=n))):
            o.set(name, v)
        splits = C.c_int()
        L.check(o.eng.lib.bcg_experts(*o.args(0, T, C.byref(splits))))
        assert splits.value == 1
        rows, out = o.get("moe_row", T, 2), o.get("moe_out", T * 2, d)
        for t in range(0, T, 13):
            e, h = int(pick[t, 1]), 0.5 * x[t]
            f = lambda q: o.t[f"l0.mlp.e{e}.{q}"].double()
            close(out[rows[t, 1]], f("down") @ R.clamped_glu(f("gate") @ h, f("up") @ h, 1.0), 1.5e-2)


# ------------------------------------------------------------------------------------------ norm, product
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("T,d,parts,per_row,row_parts", [(1, 4, 1, 0, 1), (3, 77, 2, 3, 2), (5, 2048, 4, 8, 3), (200, 1536, 1, 2, 1)])
def test_residual_norm_adds_bias_and_expert_rows(dtype, T, d, parts, per_row, row_parts):
    code, td, tol = DT[dtype]
    g = gen(T + d)
    x, y, bias, wn = (torch.randn(*s, generator=g) for s in ((T, d), (parts, T, d), (d,), (d,)))
    n = max(T * per_row, 1)
    rows, index = torch.randn(row_parts, n, d, generator=g), torch.randperm(n, generator=g)[:T * per_row].view(T, per_row)
    weight, wp = torch.rand(T, max(per_row, 1), generator=g)[:, :per_row], torch.randn(d, generator=g)
    Y, B, W, E, I, F, P = (v.cuda() for v in (y, bias, wn, rows, index.int(), weight.contiguous(), wp))
    ptr = lambda v, there=True: v.data_ptr() if there else None
    # as it stands; weighted rows behind a norm of their own, the stream itself passed on; weighted rows alone
    for weighted, with_delta, post, nxt in ((False, True, False, True), (True, True, True, False), (True, False, True, True)):
        if not with_delta and not per_row:
            continue
        R_, xn = x.cuda(), torch.zeros(T, d, dtype=td, device="cuda")
        L.check(L.load().bcg_residual_norm(R_.data_ptr(), ptr(Y, with_delta), parts, T * d, ptr(B, with_delta), ptr(E, per_row),
                                           ptr(I, per_row), ptr(F, per_row and weighted), per_row, row_parts, n * d, ptr(P, post),
                                           ptr(W, nxt), xn.data_ptr(), code, T, d, 1e-3, L.stream_ptr()))
        factor = weight.double()[..., None] if weighted else 1.0
        add = (factor * rows.double().sum(0)[index]).sum(1)
        if with_delta:
            add = add + y.double().sum(0) + bias.double()
        want = x.double() + (R.rms_norm(add, 1e-3, wp.double()) if post else add)
        close(R_, want, 3e-6)
        close(xn, R.rms_norm(want, 1e-3, wn.double()) if nxt else want, tol)


@pytest.mark.parametrize("M,N,K", [(129, 48, 64), (300, 96, 200), (700, 256, 128), (600, 2080, 192), (513, 2048, 64)])
def test_squared_relu_product(M, N, K):
    g = gen(M)
    x, w = torch.randn(M, K, generator=g).bfloat16(), torch.randn(N, K, generator=g).bfloat16()
    out = torch.full((M, N + 16), 7.0, dtype=torch.bfloat16, device="cuda")
    X, W = x.cuda(), w.cuda()
    L.check(L.load().bcg_gemm_bf16_tn(X.data_ptr(), W.data_ptr(), out.data_ptr(), M, N, K, K, K, N + 16, L.EPI_RELU2, 1, 0,
                                      L.stream_ptr()))
    close(out[:, :N], R.squared_relu(x.double() @ w.double().T), 4e-3)
    assert (out[:, N:] == 7.0).all()
    assert L.load().bcg_gemm_bf16_tn(X.data_ptr(), W.data_ptr(), out.data_ptr(), 4, N, K, K, K, N + 16, L.EPI_RELU2, 1, 0,
                                     L.stream_ptr()) == 1
