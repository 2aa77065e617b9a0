"""The kernels of layer stacks one by one, against the plain oracle (oracle/stack_ref.py) on the same inputs."""
import ctypes as C

import numpy as np
import pytest
import torch

from byzantine_consensus_llm_agents_b200 import lib as L
from byzantine_consensus_llm_agents_b200.executors import Entry
from oracle import stack_ref as R

import stack_models as SM

pytestmark = pytest.mark.gpu
DT = {"float32": (L.DT_F32, torch.float32, 3e-5), "bfloat16": (L.DT_BF16, torch.bfloat16, 8e-3)}


def dev(x):
    return x.cuda().contiguous()


def gen(seed):
    return torch.Generator().manual_seed(seed)


def close(got, want, tol):
    got, want = got.double().cpu(), want.double()
    assert torch.isfinite(got).all()
    err = (got - want).abs().max().item() / max(want.abs().max().item(), 1e-6)
    assert err < tol, err


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("M,N,K", [(1, 1, 1), (3, 70, 33), (65, 64, 16), (130, 129, 200)])
def test_gemm_any(dtype, M, N, K):
    code, td, _ = DT[dtype]
    g = gen(M + N)
    x, w = torch.randn(M, K, generator=g).to(td), torch.randn(N, K, generator=g).bfloat16()
    out = torch.full((M, N + 3), 7.0, device="cuda")
    X, W = dev(x), dev(w)
    L.check(L.load().bcg_gemm_any(X.data_ptr(), code, W.data_ptr(), out.data_ptr(), M, N, K, K, K, N + 3, L.stream_ptr()))
    close(out[:, :N], x.double() @ w.double().T, 2e-6)
    assert (out[:, N:] == 7.0).all()


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("T,d,parts", [(1, 4, 1), (3, 80, 2), (5, 2048, 5), (128, 1028, 1), (200, 1536, 1), (2, 16384, 9),
                                        (3, 77, 2), (2, 1501, 3)])
def test_sandwich_norm(dtype, T, d, parts):
    code, td, tol = DT[dtype]
    g = gen(T + d)
    x, y = torch.randn(T, d, generator=g) * 3, torch.randn(parts, T, d, generator=g) * 5
    wp, wn = torch.randn(d, generator=g), torch.randn(d, generator=g)
    for post, nxt in ((wp, wn), (None, wn), (wp, None)):
        res, xn = dev(x), torch.zeros(T, d, dtype=td, device="cuda")
        Y, P, Q = dev(y), dev(wp), dev(wn)
        L.check(L.load().bcg_sandwich_norm(res.data_ptr(), Y.data_ptr(), parts, T * d, P.data_ptr() if post is not None else None,
                                           Q.data_ptr() if nxt is not None else None, xn.data_ptr(), code, T, d, 1e-3,
                                           L.stream_ptr()))
        add = y.double().sum(0)
        want = x.double() + (R.rms_norm(add, 1e-3, wp.double()) if post is not None else add)
        close(res, want, 2e-6)
        if nxt is not None:
            close(xn, R.rms_norm(want, 1e-3, wn.double()), tol)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("T,ff,parts", [(1, 8, 1), (3, 96, 3), (4, 4096, 2), (150, 1280, 1), (3, 99, 2), (5, 1155, 2)])
def test_poly_norm(dtype, T, ff, parts):
    code, td, tol = DT[dtype]
    g = gen(T + ff)
    z = torch.randn(parts, T, ff, generator=g)
    z[0, 0] *= 1e-3                                  # eps matters in this row
    for coef in ([0.7, 0, 0, 0], [0, 0.7, 0, 0], [0, 0, 0.7, 0], [0, 0, 0, 0.7], [0.9, -0.5, 0.3, 0.2]):
        out, Z, Cf = torch.zeros(T, ff, dtype=td, device="cuda"), dev(z), torch.tensor(coef, device="cuda")
        L.check(L.load().bcg_poly_norm(Z.data_ptr(), parts, T * ff, Cf.data_ptr(), out.data_ptr(), code, T, ff, 1e-5,
                                       L.stream_ptr()))
        close(out, R.poly_norm(z.double().sum(0), coef, 1e-5), tol)


# ------------------------------------------------------------------------------------------ delta rule
class Delta:
    """One delta-rule layer's operands for ragged sequences, and the oracle's answer."""

    def __init__(self, heads, dim, lens, parts=1, seed=0):
        g = gen(seed)
        self.H, self.D, self.lens, self.parts = heads, dim, lens, parts
        n, T = heads * dim, sum(lens)
        self.proj = torch.randn(T, 5 * n + 8, generator=g)
        self.decay = torch.randn(T, n, generator=g) * 2 - 2
        self.db, self.rb, self.nw = (torch.randn(n, generator=g) for _ in range(3))

    def oracle(self, s, lo, hi, state):
        n, t0 = self.H * self.D, sum(self.lens[:s])
        p = self.proj[t0 + lo:t0 + hi].double()
        sp = lambda x: x.reshape(hi - lo, self.H, self.D)
        w = torch.exp(-np.exp(-0.5) * torch.sigmoid(self.decay[t0 + lo:t0 + hi].double() + self.db.double()))
        a = torch.sigmoid(p[:, 4 * n:5 * n] + self.rb.double())
        o, st = R.delta_scan(sp(p[:, :n]), sp(p[:, n:2 * n]), sp(p[:, 2 * n:3 * n]), sp(w), sp(a), state)
        o = R.rms_norm(o, 1e-5).reshape(hi - lo, n) * self.nw.double() * torch.sigmoid(p[:, 3 * n:4 * n])
        return o, st

    def run(self, pieces, states, code, td):
        """pieces: [(sequence, lo, hi)] -> rows of all pieces; `states` [slots, H, D, D], slot = sequence."""
        idx = torch.cat([torch.arange(lo, hi) + sum(self.lens[:s]) for s, lo, hi in pieces])
        pos = torch.cat([torch.arange(lo, hi) for _, lo, hi in pieces])
        start = np.cumsum([0] + [hi - lo for _, lo, hi in pieces])
        split = lambda x: dev(torch.stack([x[idx] / self.parts] * self.parts))
        P, Dc = split(self.proj), split(self.decay)
        one = all(hi - lo == 1 for _, lo, hi in pieces)
        l = L.Layer()
        l.mixer, l.heads, l.dim, l.cache = L.MIXER_GENERAL_DELTA, self.H, self.D, states.data_ptr()
        keep = [dev(x) for x in (self.db, self.rb, self.nw)]
        l.decay_bias, l.rate_bias, l.out_norm = (x.data_ptr() for x in keep)
        i32 = lambda x: torch.as_tensor(x).int().cuda()
        posd, slot, st = i32(pos), i32(torch.zeros(len(idx))), i32([s for s, _, _ in pieces])
        sd = None if one else i32(start)
        n, T = self.H * self.D, len(idx)
        out = torch.zeros(T, n, dtype=td, device="cuda")
        L.check(L.load().bcg_delta_scan(C.byref(l), P.data_ptr(), self.parts, T * P.shape[-1], P.shape[-1], Dc.data_ptr(),
                                        self.parts, T * n, posd.data_ptr(), slot.data_ptr(),
                                        None if one else sd.data_ptr(), st.data_ptr(), len(pieces), out.data_ptr(), code,
                                        1e-5, L.stream_ptr()))
        torch.cuda.synchronize()
        return out


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("heads,dim", [(1, 4), (3, 24), (2, 32), (5, 48), (2, 64), (3, 100), (2, 128), (1, 200), (1, 256),
                                       (90, 64), (90, 128)])
def test_delta_scan_whole_portions_and_tokens(dtype, heads, dim):
    code, td, tol = DT[dtype]
    lens = [1, 16, 17, 37] if heads < 50 else [1, 19]
    d = Delta(heads, dim, lens, parts=2, seed=dim)
    want = [d.oracle(s, 0, n, None) for s, n in enumerate(lens)]
    dirty = lambda: torch.full((len(lens), heads, dim, dim), 3.0, device="cuda")     # position 0 starts from zero
    st = dirty()
    close(d.run([(s, 0, n) for s, n in enumerate(lens)], st, code, td), torch.cat([o for o, _ in want]), max(tol, 2e-4))
    for s in range(len(lens)):
        close(st[s], want[s][1], 2e-5)
    # cut anywhere: a portion, two tokens, then one by one, beside another sequence's portion
    st, s, n = dirty(), len(lens) - 1, lens[-1]
    got = [d.run([(0, 0, 1), (s, 0, 5)], st, code, td)[1:], d.run([(s, 5, 7)], st, code, td)]
    got += [d.run([(s, i, i + 1)], st, code, td) for i in range(7, n)]
    close(torch.cat(got), want[s][0], max(tol, 2e-4))
    close(st[s], want[s][1], 2e-5)
    assert len(lens) < 3 or (st[1] == 3.0).all()          # slots of other sequences stay as they are


def test_delta_scan_leaves_the_state_of_finished_rows():
    d = Delta(2, 32, [3])
    st = torch.full((1, 2, 32, 32), 2.0, device="cuda")
    l, i32 = L.Layer(), lambda *x: torch.tensor(x, dtype=torch.int32, device="cuda")
    l.mixer, l.heads, l.dim, l.cache = L.MIXER_GENERAL_DELTA, 2, 32, st.data_ptr()
    b = [dev(x) for x in (d.proj, d.decay, d.db, d.rb, d.nw)]
    l.decay_bias, l.rate_bias, l.out_norm = (x.data_ptr() for x in b[2:])
    out, pos, slot, ss = torch.zeros(1, 64, device="cuda"), i32(5), i32(-1), i32(0)
    L.check(L.load().bcg_delta_scan(C.byref(l), b[0].data_ptr(), 1, 0, d.proj.shape[1], b[1].data_ptr(), 1, 0,
                                    pos.data_ptr(), slot.data_ptr(), None, ss.data_ptr(), 1, out.data_ptr(), L.DT_F32, 1e-5,
                                    L.stream_ptr()))
    torch.cuda.synchronize()
    assert (st == 2.0).all()


def test_delta_scan_keeps_a_long_memory():
    """Channels that hardly decay: after thousands of tokens the state still carries the first ones, with no drift."""
    n = 3000
    d = Delta(1, 32, [n], seed=5)
    d.decay[:] = torch.randn(d.decay.shape, generator=gen(6)) - 12.0
    d.proj[1:, 32:96] = 0.0               # only the first token writes
    d.db[:] = 0.0
    st = torch.zeros(1, 1, 32, 32, device="cuda")
    out = d.run([(0, 0, n)], st, L.DT_F32, torch.float32)
    o, s = d.oracle(0, 0, n, None)
    assert s.abs().max() > 0.5
    close(st[0], s, 5e-5)
    close(out[-50:], o[-50:], 2e-4)


# ------------------------------------------------------------------------------------------ latent attention
SIZES = {   # heads, dim, rot_dim, vdim, kv_rank
    "plain": (3, 10, 6, 20, 20), "small": (5, 16, 16, 24, 48), "even": (6, 32, 32, 40, 80), "wide-v": (2, 48, 16, 200, 112),
    "large": (33, 128, 64, 128, 512), "max": (2, 192, 64, 256, 128), "one": (1, 8, 8, 8, 16), "tall": (40, 64, 64, 64, 64)}


class Attention:
    """One attention layer inside an engine, its queries and cache set by hand."""

    def __init__(self, size, window, dtype, tokens=512):
        H, dim, rot, vdim, rank = SIZES[size]
        self.m = dict(heads=H, dim=dim, rot_dim=rot, vdim=vdim, rank=rank, window=window, scale=(dim + rot) ** -0.5)
        cfg = SM.config([SM.attn(H, dim, rot, vdim, rank, window, scale=self.m["scale"], ff=None)], width=32, vocab=16)
        self.t = SM.tensors(cfg, seed=H + dim)
        self.eng = SM.engine(cfg, self.t, dtype, tokens=tokens, rows=4, state_slots=4)
        self.td = self.eng.cfg.torch_dtype
        self.sink = self.t["l0.mix.sink"].double()
        self.uk = self.t["l0.mix.uk"].double().view(H, dim, rank)
        self.uv = self.t["l0.mix.uv"].double().view(H, vdim, rank)

    def run(self, seqs, mode=0):
        """seqs: [(latent rows [n, rank + rot], queries [m, H, dim + rot] of its last m tokens)] -> values of all."""
        m, e = self.m, self.eng
        cache = e.exec.caches[0]
        cache.fill_(float("nan"))           # pages nobody wrote must not matter
        pages = list(np.random.default_rng(0).permutation(cache.shape[0]))
        entries, qs = [], []
        for rows, q in seqs:
            n = len(rows)
            bt = np.zeros(e.max_blocks, np.int32)
            k = -(-n // 16)
            bt[:k] = [pages.pop() for _ in range(k)]
            for j in range(k):
                part = rows[j * 16:(j + 1) * 16]
                cache[int(bt[j]), :len(part)] = part.to(self.td).cuda()
            entries.append(Entry([0] * len(q), n - len(q), bt))
            qs.append(q)
        p = e.exec.plan(entries)
        v = {k: torch.as_tensor(np.asarray(a, np.int32)).cuda() for k, a in p.arrays.items()}
        q = torch.cat(qs)
        row = e.exec.model.struct.layers[0].q_ld or m["dim"] + m["rot_dim"]
        qb = torch.zeros(p.T, m["heads"], row, dtype=self.td, device="cuda")
        qb[..., :q.shape[-1]] = q.to(self.td).cuda()
        e.buf["q"][:qb.numel()] = qb.flatten()
        b = e.exec._batch(p.T, p.n_seqs)
        b.positions, b.slot_map, b.ids = v["pos"].data_ptr(), v["slots"].data_ptr(), v["ids"].data_ptr()
        b.row_seq, b.seq_start, b.block_table = v["row_seq"].data_ptr(), v["seq_start"].data_ptr(), v["bt"].data_ptr()
        b.max_context = p.extra["context"]
        b.single_rows, b.n_single = v["singles"].data_ptr() if p.extra["n_single"] else None, p.extra["n_single"]
        b.tiles, b.n_tiles = v["tiles"].data_ptr(), p.extra["n_tiles"]
        b.gather, b.n_gather = v["gather"].data_ptr(), p.extra["n_gather"]
        L.check(e.lib.bcg_latent_attention(C.byref(e.exec.model.struct), C.byref(e.ws), C.byref(b), 0, mode, L.stream_ptr()))
        torch.cuda.synchronize()
        out = e.buf["mix"][:p.T * m["heads"] * m["vdim"]].view(p.T, m["heads"], m["vdim"]).cpu()
        return out, [(s - len(q) + i, r.to(self.td).double(), q.to(self.td).double()[i])
                     for r, q in seqs for s in [len(r)] for i in range(len(q))]

    def oracle(self, pos, rows, q, window=None):
        m = self.m
        w = m["window"] if window is None else window
        rows = rows[max(0, pos - w + 1):pos + 1]
        c, kr = rows[:, :m["rank"]], rows[:, m["rank"]:]
        kn = torch.einsum("jr,hdr->hjd", c, self.uk)
        s = (torch.einsum("hd,hjd->hj", q[:, :m["dim"]], kn) + q[:, m["dim"]:] @ kr.T) * m["scale"]
        p = R.softmax_with_sink(s[:, None], torch.ones(1, len(rows), dtype=torch.bool), self.sink)[:, 0]
        return torch.einsum("hj,jr,hvr->hv", p, c, self.uv)


def _check(att, seqs, tol, mode=0):
    out, meta = att.run(seqs, mode)
    assert torch.isfinite(out.float()).all()
    want = torch.stack([att.oracle(*x) for x in meta])
    err = (out.double() - want).flatten(1).norm(dim=1) / want.flatten(1).norm(dim=1).clamp_min(1e-3 * want.norm() / len(want) ** 0.5)
    assert err.max().item() < tol, (err.max().item(), int(err.argmax()))
    return out, meta


@pytest.mark.parametrize("size", SIZES)
@pytest.mark.parametrize("window", [1, 2, 17, 64, 65, 130, 400])
def test_latent_attention_bf16(size, window):
    """Portions with and without history, two-token portions and single tokens in one batch."""
    a = Attention(size, window, "bfloat16")
    g = gen(window)
    m = a.m
    seqs = [(torch.randn(n, m["rank"] + m["rot_dim"], generator=g), torch.randn(k, m["heads"], m["dim"] + m["rot_dim"], generator=g) * 2)
            for n, k in ((150, 150), (97, 30), (90, 1), (66, 2))]
    _check(a, seqs, 2e-2)
    _check(a, seqs, 2e-2, mode=1)
    _check(a, [(r, q[-1:]) for r, q in seqs], 2e-2)


@pytest.mark.parametrize("size", ["plain", "even", "wide-v"])
@pytest.mark.parametrize("window", [1, 17, 64, 400])
def test_latent_attention_fp32(size, window):
    a = Attention(size, window, "float32")
    g = gen(window)
    m = a.m
    seqs = [(torch.randn(n, m["rank"] + m["rot_dim"], generator=g), torch.randn(k, m["heads"], m["dim"] + m["rot_dim"], generator=g) * 2)
            for n, k in ((300, 20), (40, 40), (9, 1))]
    _check(a, seqs, 3e-6)


@pytest.mark.parametrize("size", ["small", "large", "max"])
@pytest.mark.parametrize("window", [16, 63, 64, 100])
@pytest.mark.parametrize("portion", [1, 2, 40])
def test_window_edge_holds_one_loud_key(size, window, portion):
    """A key whose score dwarfs all others sits just inside, then just outside, the last query's window; the
    answer must follow it, and the query before sees it in both cases."""
    a = Attention(size, window, "bfloat16")
    m, g = a.m, gen(window)
    n = 203
    q = torch.randn(portion, m["heads"], m["dim"] + m["rot_dim"], generator=g)
    q[..., m["dim"]:] = 1.0                      # the rotated part carries the loud score
    for inside in (True, False):
        rows = torch.randn(n, m["rank"] + m["rot_dim"], generator=g)
        rows[:, m["rank"]:] *= 0.1
        edge = n - window - (0 if inside else 1)
        rows[edge, m["rank"]:] = 30.0 / (m["scale"] * m["rot_dim"])
        out, meta = _check(a, [(rows, q)], 2e-2)
        pos, r, qq = meta[-1]
        loud = torch.einsum("r,hvr->hv", r[edge, :m["rank"]], a.uv)
        near = (out[-1].double() - loud).norm() / loud.norm()
        assert (near < 0.02) == inside, near.item()
        wrong = a.oracle(pos, r, qq, window=window + (-1 if inside else 1))       # a window off by one would show
        assert (wrong - out[-1].double()).norm() / loud.norm() > 0.2


@pytest.mark.parametrize("size", ["plain", "even", "large"])
def test_sink_takes_its_share(size):
    """Few visible keys and a large sink: leaving it out changes everything."""
    a = Attention(size, 8, "bfloat16")
    a.sink += 4.0
    new = a.sink.float().cuda()
    a.eng.w.layers[0]["sink"].copy_(new)
    m, g = a.m, gen(3)
    seqs = [(torch.randn(n, m["rank"] + m["rot_dim"], generator=g), torch.randn(k, m["heads"], m["dim"] + m["rot_dim"], generator=g))
            for n, k in ((1, 1), (5, 5), (30, 1), (3, 2))]
    out, meta = _check(a, seqs, 2.5e-2)
    keep = a.sink
    a.sink = torch.full_like(keep, -1e4)
    assert ((torch.stack([a.oracle(*x) for x in meta]) - out.double()).norm() / out.double().norm()) > 1.0
