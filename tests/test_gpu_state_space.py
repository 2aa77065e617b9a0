"""The kernels of state-space layers and of the attention beside them, one by one — convolution, recurrence, gated norm;
query and key norms, output gates, attention without a distance bias; clamped units; sinusoidal positions — against the
plain oracle (oracle/stack_ref.py)."""
import ctypes as C

import numpy as np
import pytest
import torch

from byzantine_consensus_llm_agents_b200 import lib as L
from byzantine_consensus_llm_agents_b200.executors import Entry
from oracle import stack_ref as R

import stack_models as SM

pytestmark = pytest.mark.gpu
DT = {"float32": (L.DT_F32, torch.float32, 2e-5), "bfloat16": (L.DT_BF16, torch.bfloat16, 1.5e-2)}


def gen(seed):
    return torch.Generator().manual_seed(seed)


def close(got, want, tol):
    got, want = got.double().cpu(), want.double()
    assert got.shape == want.shape and torch.isfinite(got).all()
    err = (got - want).abs().max().item() / max(want.abs().max().item(), 1e-6)
    assert err < tol, err


class OneLayer:
    """A one-layer model inside an engine; its buffers are set and read by hand."""
    make = staticmethod(SM.side_config)

    def __init__(self, layer, dtype, width=64, seed=0, tokens=512, rows=6, **kw):
        self.cfg = self.make([layer], width=width, vocab=16)
        self.t = SM.tensors(self.cfg, seed=seed)
        self.t.update(kw.pop("tensors", {}))
        self.eng = SM.engine(self.cfg, self.t, dtype, tokens=tokens, rows=rows, **kw)
        self.x, self.td, self.tol = self.eng.exec, DT[dtype][1], DT[dtype][2]
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
        """entries: [(tokens, start, slot)] or Entry objects; every sequence has pages of its own."""
        out = []
        for i, e in enumerate(entries):
            if not isinstance(e, Entry):
                bt = np.zeros(self.eng.max_blocks, np.int32)
                bt[:4] = np.arange(4) + 4 * (i % 8)
                e = Entry([0] * e[0], e[1], bt, e[2])
            out.append(e)
        p = self.x.plan(out)
        v = {k: torch.as_tensor(np.asarray(a, np.int32)).cuda() for k, a in p.arrays.items()}
        b = self.x._batch(p.T, p.n_seqs)
        b.positions, b.slot_map, b.ids, b.block_table = (v[k].data_ptr() for k in ("pos", "slots", "ids", "bt"))
        b.state_slots = v["state_slots"].data_ptr()
        if p.T != p.n_seqs:
            b.row_seq, b.seq_start = v["row_seq"].data_ptr(), v["seq_start"].data_ptr()
        b.max_context = p.extra["context"]
        b.single_rows, b.n_single = v["singles"].data_ptr() if p.extra["n_single"] else None, p.extra["n_single"]
        b.tiles, b.n_tiles = v["tiles"].data_ptr(), p.extra["n_tiles"]
        self.keep = v
        return p, b


# ------------------------------------------------------------------------------------------ state space
SIZES = {  # heads, vdim, state, groups, norm_groups, conv
    "usual": (4, 64, 128, 2, 2, 4), "small": (4, 16, 16, 4, 1, 4), "blocks": (2, 136, 64, 1, 2, 3), "wide": (2, 64, 256, 1, 1, 2),
    "odd": (3, 11, 13, 3, 3, 4), "halves": (2, 66, 50, 1, 4, 5), "one": (1, 8, 8, 1, 1, 1), "parts": (8, 24, 36, 2, 48, 4), "row": (2, 1, 200, 2, 2, 3),
    "many": (72, 16, 20, 8, 4, 3), "many-blocks": (40, 72, 24, 4, 1, 5),
    "large-part": (16, 72, 16, 2, 1, 2), "larger-part": (40, 56, 8, 1, 1, 3)}


class StateSpace(OneLayer):
    def __init__(self, size, dtype, **kw):
        m = dict(zip(("heads", "vdim", "state", "groups", "norm_groups", "conv"), SIZES[size]))
        super().__init__(SM.mamba(**m), dtype, tokens=1024, **kw)
        self.m = m
        self.w = {n[len("l0.mix."):]: x.double() for n, x in self.t.items() if n.startswith("l0.mix.")}
        n = m["heads"] * m["vdim"]
        self.inner, self.rows = n, n + n + 2 * m["groups"] * m["state"] + m["heads"]
        self.ld = self.eng.cfg.in_rows(0)
        self.state, self.conv = (self.x.caches[0][k] for k in ("ssm_state", "conv_state"))

    def junk(self):
        """What slots hold before a sequence starts must not matter."""
        self.state.normal_().mul_(100)
        self.conv.normal_().mul_(100)

    def run(self, shapes, proj, slabs=1, mode=0):
        """shapes: [(tokens, start, slot)]; proj [T, rows].  Returns the normed outputs [T, inner]."""
        p, b = self.batch(shapes)
        full = torch.zeros(slabs, p.T, self.ld)
        parts = torch.randn(slabs - 1, p.T, self.rows, generator=gen(9)) if slabs > 1 else proj.new_zeros(0, p.T, self.rows)
        full[:slabs - 1, :, :self.rows] = parts
        full[slabs - 1, :, :self.rows] = proj - parts.sum(0)
        self.set("proj", full)
        L.check(self.eng.lib.bcg_state_space(*self.args(C.byref(b), 0, slabs, p.T * self.ld, self.ld, mode)))
        return self.get("mix", p.T, self.layer.mix_ld)[:, :self.inner]

    def oracle(self, proj):
        """One whole sequence: outputs, final state, the convolution's last inputs."""
        m, w, n, t = self.m, self.w, self.inner, len(proj)
        z, xbc, dt = torch.split(proj.double(), [n, self.rows - n - m["heads"], m["heads"]], dim=-1)
        out = R.silu(R.causal_conv(xbc, w["conv"], w["conv.b"]))
        x, B, Cc = torch.split(out, [n, m["groups"] * m["state"], m["groups"] * m["state"]], dim=-1)
        step = torch.nn.functional.softplus(dt + w["dt_bias"], threshold=1e9)
        y, S = R.ssm_scan(x.view(t, m["heads"], -1), B.view(t, m["groups"], -1), Cc.view(t, m["groups"], -1), step, w["A_log"], w["D"])
        last = torch.cat([xbc.new_zeros(m["conv"], xbc.shape[1]), xbc])[len(xbc) + 1:]
        return R.part_norm(y.reshape(t, n) * R.silu(z), m["norm_groups"], 1e-5, w["norm"]), S.transpose(1, 2), last

    def feed(self, proj, sizes, slot, slabs=1, mode=0):
        out, at, k = [], 0, 0
        while at < len(proj):
            n = min(sizes[min(k, len(sizes) - 1)], len(proj) - at)
            out.append(self.run([(n, at, slot)], proj[at:at + n], slabs, mode))
            at, k = at + n, k + 1
        return torch.cat(out)

    def check(self, got, want, tol):
        """Rows relative to themselves: a row that nearly cancels is divided by its own small root mean square."""
        err = (got.double() - want).norm(dim=1) / want.norm(dim=1)
        assert torch.isfinite(err).all() and err.median() < tol and err.quantile(0.95) < 3 * tol and err.max() < 12 * tol, (err.median(), err.max())


def _proj(a, t, seed=0):
    return torch.randn(t, a.rows, generator=gen(seed)) * 1.2


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("size", SIZES)
def test_portions_tokens_and_states(size, dtype):
    """A sequence whole, in portions that end inside and at chunks of 64, and token by token; junk in fresh slots."""
    a = StateSpace(size, dtype)
    proj = _proj(a, 200)
    want, S, last = a.oracle(proj)
    for slot, (sizes, slabs, mode) in enumerate((([200], 1, 0), ([64, 65, 63, 2], 1, 0), ([2], 3, 0), ([1], 2, 0), ([150, 1], 1, 1), ([3, 129, 1], 5, 0))):
        a.junk()
        a.check(a.feed(proj, sizes, slot, slabs, mode), want, a.tol)
        close(a.state[slot], S, a.tol)
        if a.m["conv"] > 1:
            close(a.conv[slot], last, 1e-5)


@pytest.mark.parametrize("dtype", DT)
def test_unequal_sequences_in_one_launch(dtype):
    """Fresh and continued sequences, portions beside single tokens; neighbours' states stay as they are."""
    a = StateSpace("usual", dtype)
    lens = {0: 150, 1: 40, 2: 129, 3: 66, 4: 5}
    proj = {s: _proj(a, n, s) for s, n in lens.items()}
    a.junk()
    before = a.state[5].clone()
    first = {0: 20, 1: 39, 2: 0, 3: 65, 4: 0}
    got = {s: [] for s in lens}
    for s, n in first.items():
        if n:
            got[s].append(a.run([(n, 0, s)], proj[s][:n]))
    order = [3, 0, 4, 1, 2]
    out = a.run([(lens[s] - first[s], first[s], s) for s in order], torch.cat([proj[s][first[s]:] for s in order]))
    for s in order:
        n = lens[s] - first[s]
        got[s].append(out[:n])
        out = out[n:]
        want, S, last = a.oracle(proj[s])
        a.check(torch.cat(got[s]), want, a.tol)
        close(a.state[s], S, a.tol)
        close(a.conv[s], last, 1e-5)
    assert torch.equal(a.state[5], before)


def test_single_tokens_in_one_launch_and_idle_rows():
    a = StateSpace("usual", "bfloat16")
    proj = [_proj(a, 30, s) for s in range(4)]
    for s in range(4):
        a.run([(29, 0, 3 - s)], proj[s][:29])
    before = a.state.clone(), a.conv.clone()
    p, b = a.batch([(1, 29, 3 - s) for s in range(4)])
    a.keep["slots"][1] = -1                                       # a finished row
    full = torch.zeros(4, a.ld)
    full[:, :a.rows] = torch.stack([x[29] for x in proj])
    a.set("proj", full)
    L.check(a.eng.lib.bcg_state_space(*a.args(C.byref(b), 0, 1, 0, a.ld, 0)))
    out = a.get("mix", 4, a.layer.mix_ld)[:, :a.inner]
    for s in (0, 2, 3):
        want, S, last = a.oracle(proj[s])
        a.check(out[s:s + 1], want[29:], a.tol)
        close(a.state[3 - s], S, a.tol)
        close(a.conv[3 - s], last, 1e-5)
    assert torch.equal(a.state[2], before[0][2]) and torch.equal(a.conv[2], before[1][2])


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("size", ["many", "many-blocks", "row"])
def test_more_single_tokens_than_ctas(size, dtype):
    """Several steps of fifteen sequences: long ones, one that starts, one that is finished."""
    n = 15
    a = StateSpace(size, dtype, rows=16)
    proj = [_proj(a, 6 if s == 4 else 12, s) for s in range(n)]
    a.junk()
    for s in range(n):
        if s != 4:
            a.run([(6, 0, s)], proj[s][:6])
    idle = a.state[9].clone(), a.conv[9].clone()
    got = [[] for _ in range(n)]
    for step in range(6):
        starts = [step if s == 4 else 6 + step for s in range(n)]
        p, b = a.batch([(1, starts[s], s) for s in range(n)])
        a.keep["slots"][9] = -1
        full = torch.zeros(n, a.ld)
        full[:, :a.rows] = torch.stack([proj[s][starts[s]] for s in range(n)])
        a.set("proj", full)
        L.check(a.eng.lib.bcg_state_space(*a.args(C.byref(b), 0, 1, 0, a.ld, 0)))
        out = a.get("mix", n, a.layer.mix_ld)[:, :a.inner]
        for s in range(n):
            got[s].append(out[s])
    for s in range(n):
        if s == 9:
            continue
        want, S, last = a.oracle(proj[s])
        a.check(torch.stack(got[s]), want[-6:], a.tol)
        close(a.state[s], S, a.tol)
        close(a.conv[s], last, 1e-5)
    assert torch.equal(a.state[9], idle[0]) and torch.equal(a.conv[9], idle[1])


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("sizes", [[700], [1], [600, 50, 2]])
def test_long_memory_does_not_drift(sizes, dtype):
    """Decays of a ten-thousandth per token and one loud token at the start: what is left of it after hundreds of tokens."""
    H = SIZES["usual"][0]
    slow = {"l0.mix.A_log": torch.full((H,), -5.0).bfloat16(), "l0.mix.dt_bias": torch.full((H,), -4.5).bfloat16()}
    a = StateSpace("usual", dtype, tensors=slow)
    proj = _proj(a, 700) * 0.3
    proj[0] = 8.0 * torch.sign(proj[0])
    want, S, _ = a.oracle(proj)
    assert (a.oracle(torch.cat([proj[1:2], proj[1:]]))[1] - S).abs().max() > 0.3 * S.abs().max()
    a.feed(proj, sizes, 0)
    close(a.state[0], S, a.tol)


@pytest.mark.parametrize("dtype", DT)
def test_large_steps_forget_at_once(dtype):
    """Steps without an upper limit: a state that is wiped at every other token, exponentials that underflow."""
    a = StateSpace("usual", dtype)
    proj = _proj(a, 140)
    proj[::2, -a.m["heads"]:] = 300.0
    want, S, _ = a.oracle(proj)
    for slot, sizes in enumerate(([140], [2], [1])):
        a.check(a.feed(proj, sizes, slot), want, a.tol)
        close(a.state[slot], S, a.tol)


def test_bad_state_space_arguments_are_refused():
    a = StateSpace("small", "bfloat16")
    p, b = a.batch([(4, 0, 0)])
    lib = a.eng.lib
    assert lib.bcg_state_space(*a.args(C.byref(b), 3, 1, 0, a.ld, 0)) == 1
    a.layer.ssm_n = 300
    assert lib.bcg_state_space(*a.args(C.byref(b), 0, 1, 0, a.ld, 0)) == 1 and b"256" in lib.bcg_last_error()


# ------------------------------------------------------------------------------------------ attention beside it
HEADS = {"small": (6, 3, 16, 24), "usual": (8, 2, 128, 128), "even": (4, 4, 64, 64), "group": (20, 1, 64, 128), "odd": (3, 1, 10, 11), "huge": (2, 1, 264, 300)}


class Attention(OneLayer):
    def __init__(self, size, dtype, **kw):
        H, G, dim, vdim = HEADS[size]
        super().__init__(SM.both(H, G, dim, vdim, scale=dim ** -0.5, heads_ssm=2, vdim_ssm=8, groups=1), dtype, tokens=1024, rows=4, **kw)
        self.a = self.cfg["layers"][0]["mixer"]["left"]

    def attend(self, seqs, gates, mode=0):
        """seqs: [(keys [n, G, dim], values, queries of the last tokens)]; gates: factors [T, heads]."""
        a, cache = self.a, self.x.caches[0]
        ck, cv = cache["cache"], cache["cache_v"]
        ck[..., :a["dim"]], cv[..., :a["vdim"]] = 50.0, -70.0          # rows nobody wrote must not matter
        pages, entries = list(np.random.default_rng(0).permutation(ck.shape[0])), []
        for k, v, q in seqs:
            n, bt = len(k), np.zeros(self.eng.max_blocks, np.int32)
            for j in range(-(-n // 16)):
                bt[j] = pages.pop()
                rows = min(16, n - j * 16)
                ck[int(bt[j]), :, :rows, :a["dim"]] = k[j * 16:j * 16 + rows].transpose(0, 1).to(self.td).cuda()
                cv[int(bt[j]), :, :rows, :a["vdim"]] = v[j * 16:j * 16 + rows].transpose(0, 1).to(self.td).cuda()
            entries.append(Entry([0] * len(q), n - len(q), bt))
        p, b = self.batch(entries)
        q = torch.zeros(p.T, a["heads"], self.layer.q_ld)
        q[..., :a["dim"]] = torch.cat([q for _, _, q in seqs])
        self.set("q", q)
        self.set("gates", gates)
        L.check(self.eng.lib.bcg_grouped_attention(*self.args(C.byref(b), 0, mode)))
        out = self.get("mix", p.T, self.layer.mix_ld)[:, :a["heads"] * a["vdim"]].reshape(p.T, a["heads"], a["vdim"])
        r, want = lambda x: x.to(self.td).double(), []
        for k, v, q in seqs:
            mine = torch.arange(a["heads"]) // (a["heads"] // a["kv_heads"])
            s = torch.einsum("ihd,jhd->hij", r(q), r(k)[:, mine]) * a["scale"]
            p_ = R.softmax_with_sink(s, R.window_visible(len(k), 0)[-len(q):])
            want.append(torch.einsum("hij,jhd->ihd", p_, r(v)[:, mine]))
        return out, torch.cat(want) * gates.double()[:, :, None]


def _seqs(a, shapes, seed=0):
    m, g = a.a, gen(seed)
    return [(torch.randn(n, m["kv_heads"], m["dim"], generator=g), torch.randn(n, m["kv_heads"], m["vdim"], generator=g),
             torch.randn(k, m["heads"], m["dim"], generator=g) * 2) for n, k in shapes]


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("size", HEADS)
def test_gated_attention_without_bias(size, dtype):
    a = Attention(size, dtype)
    for shapes in (((150, 150), (97, 30), (90, 1), (66, 2)), ((300, 1), (1, 1), (16, 1), (17, 1))):
        seqs = _seqs(a, shapes)
        gates = torch.rand(sum(k for _, k in shapes), a.a["heads"], generator=gen(4)) + 0.1
        for mode in (0, 1):
            out, want = a.attend(seqs, gates, mode)
            err = (out.double() - want).flatten(1).norm(dim=1) / want.flatten(1).norm(dim=1)
            assert torch.isfinite(err).all() and err.max() < (2e-2 if dtype == "bfloat16" else 3e-6), err.max()


@pytest.mark.parametrize("at", [0, 1, 15, 16, 63, 64, 127, 128, 255, 256, 390])
def test_one_loud_key_is_found(at):
    """One key among hundreds: first ones, page and block edges, far away; by a prompt's portion and by single tokens."""
    a = Attention("usual", "bfloat16")
    for shapes in (((400, 130),), ((400, 1),), ((392, 2),)):
        seqs = _seqs(a, shapes, at)
        k, v, q = seqs[0]
        k[at] = 4.0
        q[...] = 1.0
        gates = torch.ones(len(q), 8)
        out, want = a.attend(seqs, gates)
        close(out, want, 1.5e-2)
        if at <= len(k) - len(q):
            close(out[0], v[at][torch.arange(8) // 4], 3e-2)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("size", HEADS)
def test_input_split_norms_temperature_and_gates(size, dtype):
    a = Attention(size, dtype)
    m, w = a.a, {n[len("l0.mix.left."):]: x.double() for n, x in a.t.items() if n.startswith("l0.mix.left.")}
    H, G, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    cols, ld = H * dim + G * (dim + vdim) + H, a.eng.cfg.in_rows(0)
    for slabs, shapes in ((1, [(60, 2, 0), (1, 22, 1), (1, 45, 2)]), (3, [(1, 0, 0), (1, 22, 1), (1, 23, 2)])):
        for c in a.x.caches[0].values():
            c.zero_()
        p, b = a.batch(shapes)
        proj = torch.randn(slabs, p.T, ld, generator=gen(2))
        a.set("proj", proj)
        L.check(a.eng.lib.bcg_grouped_in(*a.args(C.byref(b), 0, slabs, p.T * ld, ld, 0)))
        x, pos = proj.double().sum(0), torch.as_tensor(p.arrays["pos"])
        q = R.rms_norm(x[:, :H * dim] + w["q.b"], 1e-5, w["q.norm"]).view(-1, H, dim)
        q = q * R.query_temperature(pos, m["q_temp"]["coef"], m["q_temp"]["every"])[:, None, None]
        k = R.rms_norm(x[:, H * dim:H * dim + G * dim] + w["k.b"], 1e-5, w["k.norm"]).view(-1, G, dim)
        v = (x[:, H * dim + G * dim:cols - H] + w["v.b"]).view(-1, G, vdim)
        tol = 6e-3 if dtype == "bfloat16" else 3e-6
        close(a.get("q", p.T, H, a.layer.q_ld)[..., :dim], q, tol)
        close(a.get("gates", p.T, H), 0.8 * torch.sigmoid(x[:, cols - H:cols]), 3e-6)
        slots = torch.as_tensor(p.arrays["slots"]).long()
        for c, want, n in ((a.x.caches[0]["cache"], k, dim), (a.x.caches[0]["cache_v"], v, vdim)):
            c = c.cpu()
            close(c[slots // 16, :, slots % 16, :n], want, tol)
            assert not c[..., n:].any()


def test_wide_norms_span_a_cluster():
    """A token's queries over a cluster of CTAs (few tokens) and in one CTA (many)."""
    a = OneLayer(SM.both(16, 4, 64, 64, heads_ssm=2, vdim_ssm=8, groups=1), "bfloat16", tokens=512)
    ld = a.eng.cfg.in_rows(0)
    proj = torch.randn(130, ld, generator=gen(1)) * torch.linspace(0.1, 5, 16 * 64 + ld - 16 * 64)
    rows = []
    for n in (3, 130):
        bt = np.arange(a.eng.max_blocks, dtype=np.int32)
        p, b = a.batch([Entry([0] * n, 0, bt)])
        a.set("proj", proj[:n])
        L.check(a.eng.lib.bcg_grouped_in(*a.args(C.byref(b), 0, 1, 0, ld, 0)))
        rows.append(a.get("q", n, 16 * 64)[:3])
    assert torch.allclose(rows[0].float(), rows[1].float(), rtol=1e-2)
    want = R.rms_norm(proj[:3, :1024].double() + a.t["l0.mix.left.q.b"].double(), 1e-5, a.t["l0.mix.left.q.norm"].double())
    close(rows[0], want, 6e-3)


# ------------------------------------------------------------------------------------------ feed-forward, embedding
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("T, ff, slabs", [(1, 16, 1), (5, 48, 3), (200, 720, 1), (1100, 32, 2)])
def test_clamped_unit(T, ff, slabs, dtype):
    dt, td, _ = DT[dtype]
    z = torch.randn(slabs, T, 2 * ff, generator=gen(T)) * 3
    z[0, 0, 0], z[0, 0, 16], z[0, -1, 3] = 40.0, -90.0, -200.0        # far over both clamps, and far below
    out = torch.empty(T, ff, dtype=td, device="cuda")
    zc = z.cuda()
    L.check(L.load().bcg_clamped_glu(zc.data_ptr(), slabs, T * 2 * ff, out.data_ptr(), dt, T, ff, 1.25, 1.702, L.stream_ptr()))
    s = z.double().sum(0).view(T, ff // 16, 2, 16)
    close(out, R.clamped_glu(s[:, :, 0].reshape(T, ff), s[:, :, 1].reshape(T, ff), 1.25), 6e-3 if dtype == "bfloat16" else 2e-6)


@pytest.mark.parametrize("M, N, K", [(3, 64, 64), (40, 224, 136), (128, 512, 64), (130, 96, 72), (300, 1024, 128), (700, 2112, 192), (600, 512, 64)])
def test_clamped_unit_as_an_epilogue(M, N, K):
    x, w = torch.randn(M, K, generator=gen(M)).bfloat16(), (torch.randn(N, K, generator=gen(N)) * 2 * K ** -0.5).bfloat16()
    xc, wc, out = x.cuda(), w.cuda(), torch.full((M, N // 2), 7.0, dtype=torch.bfloat16, device="cuda")
    L.check(L.load().bcg_gemm_bf16_glu(xc.data_ptr(), wc.data_ptr(), out.data_ptr(), M, N, K, 0.9, 1.702, 0, L.stream_ptr()))
    z = (x.double() @ w.double().T).view(M, N // 32, 2, 16)
    close(out, R.clamped_glu(z[:, :, 0].reshape(M, -1), z[:, :, 1].reshape(M, -1), 0.9), 1e-2)


@pytest.mark.parametrize("width", [64, 61])
def test_embedding_with_sinusoids_at_far_positions(width):
    """Scaled embedding plus sines and cosines, positions up to a hundred thousand: a layer that adds nothing."""
    a = OneLayer(SM.mamba(heads=1, vdim=8, state=8, groups=1, norm_groups=1), "float32", width=width,
                 tensors={"l0.mix.o": torch.zeros(width, 8, dtype=torch.bfloat16)})
    pos = [0, 1, 2, 511, 4096, 65537, 99999]
    p, b = a.batch([(1, 0, i % 6) for i in range(6)] + [(1, 0, 0)])
    a.keep["pos"][:] = torch.tensor(pos, dtype=torch.int32)
    a.keep["ids"][:] = torch.arange(7, dtype=torch.int32)
    L.check(a.eng.lib.bcg_stack_step(*a.args(C.byref(b))))
    want = a.t["embed"][:7].double() * 3.0 + R.sinusoid(torch.tensor(pos), width)
    assert (a.get("residual", 7, width).double() - want).abs().max() < 2e-6
    close(a.get("xn", 7, width), R.zero_norm(want, 1e-5, a.t["final.norm"].double()), 2e-6)
