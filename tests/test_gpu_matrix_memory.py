"""The matrix memory alone — split of the projection, chunks, tokens, denominators, gated head norm — against the plain
oracle (oracle/stack_ref.py)."""
import ctypes as C

import pytest
import torch

from byzantine_consensus_llm_agents_b200 import lib as L
from oracle import stack_ref as R

import stack_models as SM
from test_gpu_state_space import OneLayer, close, gen

pytestmark = pytest.mark.gpu
TOL = {"float32": 3e-5, "bfloat16": 1.5e-2}
SIZES = {   # heads, dim, vdim
    "usual": (4, 128, 256), "small": (4, 16, 32), "even": (3, 64, 64), "blocks": (2, 48, 136), "wide": (2, 256, 200), "flat": (5, 100, 24),
    "odd": (3, 11, 13), "odd-rows": (2, 36, 70), "odd-keys": (2, 50, 64), "one": (1, 8, 8), "row": (2, 200, 1), "column": (3, 1, 66), "many": (40, 24, 72)}


class Memory(OneLayer):
    make = staticmethod(SM.output_norm_config)

    def __init__(self, size, dtype, cap=9.0, **kw):
        H, D, V = SIZES[size]
        super().__init__(SM.mlstm(H, D, V, cap), dtype, tokens=1024, **kw)
        self.dims, self.cap, self.dtype = (H, D, V), cap, dtype
        self.w = {n[len("l0.mix."):]: x.double() for n, x in self.t.items() if n.startswith("l0.mix.")}
        self.rows, self.gate_col, self.ld = 2 * H * (D + V), self.eng.cfg.layers[0].mixer.gate_col, self.eng.cfg.in_rows(0)
        self.state, self.top = (self.x.caches[0][k] for k in ("mem_state", "mem_max"))

    def junk(self):
        """What slots hold before a sequence starts must not matter."""
        self.state.normal_().mul_(100)
        self.top.normal_().mul_(100)

    def proj(self, t, seed=0, gates=1.0):
        """Rows q | k | v | g and gates of t tokens; keys and queries share a part, so that outputs do not cancel."""
        H, D, V = self.dims
        x, g = torch.randn(t, self.rows, generator=gen(seed)), torch.randn(t, 2 * H, generator=gen(seed + 1)) * gates
        same = 1.5 * torch.randn(H * D, generator=gen(99))
        x[:, :H * D] += same
        x[:, H * D:2 * H * D] += same
        return torch.cat([x, g], dim=1)

    def run(self, shapes, proj, slabs=1, mode=0, idle=()):
        """shapes: [(tokens, start, slot)]; returns (gated outputs, denominators)."""
        H, D, V = self.dims
        p, b = self.batch(shapes)
        if idle:
            self.keep["slots"][list(idle)] = -1
        full = torch.zeros(slabs, p.T, self.ld)
        put = lambda dst, x: (dst[:, :self.rows].copy_(x[:, :self.rows]), dst[:, self.gate_col:self.gate_col + 2 * H].copy_(x[:, self.rows:]))
        rest = proj
        for s in range(slabs - 1):
            part = torch.randn(proj.shape, generator=gen(70 + s))
            put(full[s], part)
            rest = rest - part
        put(full[slabs - 1], rest)
        self.set("proj", full)
        L.check(self.eng.lib.bcg_matrix_memory(*self.args(C.byref(b), 0, slabs, p.T * self.ld, self.ld, mode)))
        return self.get("mix", p.T, self.layer.mix_ld)[:, :H * V], self.get("mem_den", p.T, H)

    def oracle(self, proj):
        """One whole sequence: outputs, denominators, (S, n, m) at its end."""
        H, D, V = self.dims
        t, x = len(proj), proj.double()
        q, k, v, g, zi, zf = torch.split(x, [H * D, H * D, H * V, H * V, H, H], dim=1)
        soft = lambda z: self.cap * torch.tanh(z / self.cap)
        log_i, log_f = soft(zi + self.w["i.b"]), torch.nn.functional.logsigmoid(soft(zf + self.w["f.b"]))
        q, k, v = q.view(t, H, D) * D ** -0.5, k.view(t, H, D), v.view(t, H, V)
        out, den, state = [], [], None
        for i in range(t):
            o, state = R.memory_scan(q[i:i + 1], k[i:i + 1], v[i:i + 1], log_i[i:i + 1], log_f[i:i + 1], state)
            out.append(o)
            den.append(torch.maximum((state[1] * q[i]).sum(-1).abs(), torch.exp(-state[2])) + 1e-6)
        y = R.rms_norm(torch.cat(out), 1e-5).reshape(t, H * V) * self.w["norm"] * torch.sigmoid(g)
        return y, torch.stack(den), state

    def feed(self, proj, sizes, slot, slabs=1, mode=0):
        out, at, k = [], 0, 0
        while at < len(proj):
            n = min(sizes[min(k, len(sizes) - 1)], len(proj) - at)
            out.append(self.run([(n, at, slot)], proj[at:at + n], slabs, mode))
            at, k = at + n, k + 1
        return tuple(torch.cat(x) for x in zip(*out))

    def check(self, got, want, slot=None, loose=1.0):
        (y, den), (wy, wd, (S, n, m)) = got, want
        tol = TOL[self.dtype] * loose
        err = (y.double() - wy).norm(dim=1) / wy.norm(dim=1)
        assert torch.isfinite(err).all() and err.median() < tol and err.quantile(0.95) < 3 * tol and err.max() < 12 * tol, (err.median(), err.max())
        close(den / wd.float(), torch.ones_like(wd), 6 * tol)
        if slot is not None:
            close(self.state[slot, :, :-1].cpu(), S.transpose(1, 2), tol)
            close(self.state[slot, :, -1].cpu(), n, tol)
            close(self.top[slot].cpu(), m[:, None].expand(self.top.shape[1:]), 2e-4)


@pytest.mark.parametrize("dtype", TOL)
@pytest.mark.parametrize("size", SIZES)
def test_portions_and_tokens(size, dtype):
    a = Memory(size, dtype)
    n = 90 if size in ("many", "wide") else 150
    proj = a.proj(n)
    want = a.oracle(proj)
    for slot, (sizes, slabs, mode) in enumerate([([n], 1, 0), ([1], 3, 0), ([2], 1, 0), ([65, 1, 2, 63, 1], 6, 0), ([40, 3, 64, 1], 2, 1)]):
        a.junk()
        a.check(a.feed(proj, sizes, slot, slabs, mode), want, slot)


@pytest.mark.parametrize("dtype", TOL)
@pytest.mark.parametrize("size", ["usual", "small", "even"])
def test_operands_that_are_activations_already(size, dtype):
    """What a product with bf16 output leaves: rows q | k | v | g, and a narrow matrix of gates."""
    a = Memory(size, dtype)
    H, n = a.dims[0], 140
    proj = a.proj(n, 11)
    assert a.gate_col == a.rows and a.eng.cfg.layers[0].mixer.x_ld == a.rows
    gates = torch.zeros(n, a.ld - a.gate_col)
    gates[:, :2 * H] = proj[:, a.rows:]
    a.junk()
    out, at = [], 0
    for t in (90, 50):
        p, b = a.batch([(t, at, 3)])
        a.set("ssm_x", proj[at:at + t, :a.rows])
        a.set("proj", gates[at:at + t])
        L.check(a.eng.lib.bcg_matrix_memory(*a.args(C.byref(b), 0, 1, 0, gates.shape[1], 2)))
        out.append((a.get("mix", t, a.layer.mix_ld)[:, :H * a.dims[2]], a.get("mem_den", t, H)))
        at += t
    a.check(tuple(torch.cat(x) for x in zip(*out)), a.oracle(proj), 3)
    p, b = a.batch([(2, 0, 0)])
    assert a.eng.lib.bcg_matrix_memory(*a.args(C.byref(b), 0, 2, 0, gates.shape[1], 2)) != 0


@pytest.mark.parametrize("dtype", TOL)
@pytest.mark.parametrize("cap", [1.5, 30.0])
@pytest.mark.parametrize("sizes", [[140], [1], [70, 1]])
def test_gates_far_above_and_below_the_maximum(sizes, cap, dtype):
    """Log gates over the whole range: single tokens that replace the memory, tokens that leave no trace, exp(-m) as denominator."""
    a = Memory("small", dtype, cap)
    proj = a.proj(140, 3, gates=12.0)
    a.junk()
    want = a.oracle(proj)
    assert (want[1] > 1.0).any() and want[2][2].max() > 0.9
    a.check(a.feed(proj, sizes, 1), want, 1, loose=2.0)


@pytest.mark.parametrize("dtype", TOL)
def test_the_maximum_starts_at_zero_and_bounds_the_denominator(dtype):
    """Input gates far below zero: m decays from 0, the denominator is exp(-m), outputs are small beside it."""
    a = Memory("even", dtype, 20.0)
    proj = a.proj(100, 5, gates=0.2)
    H, D, V = a.dims
    proj[:, a.rows:a.rows + H] -= 6.0
    want = a.oracle(proj)
    assert (want[1] > 0.99).all() and (want[2][2] < -1.0).any()
    for slot, sizes in enumerate(([100], [1], [64, 2, 1])):
        a.junk()
        a.check(a.feed(proj, sizes, slot), want, slot, loose=3.0)


@pytest.mark.parametrize("dtype", TOL)
@pytest.mark.parametrize("size", ["small", "wide", "odd"])
def test_a_long_memory_is_kept(size, dtype):
    """One loud token, then hundreds of quiet ones and forget gates near 1: it is read out at the end."""
    a = Memory(size, dtype, 15.0)
    t, (H, D, V) = 400, a.dims
    proj = a.proj(t, 7, gates=0.1)
    proj[:, a.rows:a.rows + H] -= 9.0
    proj[:, a.rows + H:] += 9.0
    proj[3, a.rows:a.rows + H] += 12.0
    want = a.oracle(proj)
    quiet = proj.clone()
    quiet[3, 2 * H * D:2 * H * D + H * V] *= -1
    assert (a.oracle(quiet)[0][-1] - want[0][-1]).norm() > want[0][-1].norm()
    for slot, sizes in enumerate(([t], [5, 1], [1, 100, 33, 2])):
        a.junk()
        a.check(a.feed(proj, sizes, slot), want, slot, loose=2.0)


@pytest.mark.parametrize("dtype", TOL)
@pytest.mark.parametrize("size", ["usual", "blocks", "odd"])
def test_unequal_sequences_in_one_launch(size, dtype):
    """Portions beside single tokens, slots in any order; then single tokens of all of them, one of them idle."""
    a = Memory(size, dtype)
    lens, slots = [70, 1, 2, 129], [4, 0, 5, 2]
    projs = [a.proj(n + 12, 20 + n) for n in lens]
    a.junk()
    untouched = a.state[[1, 3]].clone()
    first = a.run([(n, 0, s) for n, s in zip(lens, slots)], torch.cat([p[:n] for p, n in zip(projs, lens)]))
    first = [tuple(torch.split(x, lens)[i] for x in first) for i in range(4)]
    rest = [[] for _ in lens]
    for k in range(10):
        out = a.run([(1, n + k, s) for n, s in zip(lens, slots)], torch.stack([p[n + k] for p, n in zip(projs, lens)]), 1 + k % 4)
        for i in range(4):
            rest[i].append(tuple(x[i:i + 1] for x in out))
    before, top = a.state.clone(), a.top.clone()
    a.run([(1, n + 10, s) for n, s in zip(lens, slots)], torch.stack([p[n + 10] for p, n in zip(projs, lens)]), 2, idle=(0, 2))
    assert torch.equal(a.state[[4, 5]], before[[4, 5]]) and torch.equal(a.top[[4, 5]], top[[4, 5]])
    assert not torch.equal(a.state[2], before[2])
    a.state.copy_(before)
    a.top.copy_(top)
    for i, n in enumerate(lens):
        a.check(tuple(torch.cat(x) for x in zip(first[i], *rest[i])), a.oracle(projs[i][:n + 10]), slots[i])
    assert torch.equal(a.state[[1, 3]], untouched)


def test_too_many_key_channels_are_refused():
    a = Memory("one", "bfloat16")
    p, b = a.batch([(2, 0, 0)])
    a.layer.dim = 257
    assert a.eng.lib.bcg_matrix_memory(*a.args(C.byref(b), 0, 1, p.T * a.ld, a.ld, 0)) != 0
