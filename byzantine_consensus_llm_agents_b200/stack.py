"""Layer stacks: models whose layers differ in kind, described by composable specs.

A `StackConfig` lists layers; each has a mixer spec (`LatentAttention`, `GeneralDelta`, `GroupedAttention`, `StateSpace`,
`MatrixMemory`, or two of them `SideBySide`), optionally a feed-forward spec (`DenseMlp`, `MoeMlp`), and norms before, after,
or before and after every sublayer or, in a parallel layer, one norm in front of both.  Which design a model directory
holds is decided by config.json's "architecture" (`DESIGNS`, consulted by model.config_from_dir); a design is
a reader from its config.json to specs, everything below the specs is shared.  `StackWeights` loads and packs
the tensors for the kernels (include/bcg_b200.h, bcg_layer); there is nothing model-specific in the engine.

The reference has no counterpart: its engine only ever meets uniform dense decoders (config.py:20-25).
"""
from __future__ import annotations

import ctypes as C
import json
import math
from dataclasses import dataclass, field, replace
from pathlib import Path
from typing import Callable, Dict, Optional, Tuple

import torch

from . import lib as L


def _up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


# ------------------------------------------------------------------------------------------ specs
@dataclass(frozen=True)
class Rotary:
    """The first `dims` entries of the rotated part turn, frequencies base^(-2i/dims): entry i with dims / 2 + i or, with
    `pairs`, 2i with 2i + 1."""
    base: float
    dims: int
    pairs: bool = False


@dataclass(frozen=True)
class LatentAttention:
    """Attention over a compressed cache row (latent, shared rotated key part)."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot: Rotary
    window: int = 0                 # keys a query sees, itself included; 0 = all
    kv_from: Optional[int] = None   # layer whose cache rows this one reads; None = its own
    sink: bool = True

    @property
    def cache_row(self) -> int:
        return self.kv_rank + self.rot_dim

    @property
    def out_dim(self) -> int:
        return self.heads * self.vdim

    @property
    def q_ld(self) -> int:
        """Padded q/k head size of the expanded form, 0 when the sizes are not for it."""
        n = _up(self.dim + self.rot_dim, 64)
        return n if n <= 256 and self.v_pad and self.vdim % 8 == 0 and self.cache_row % 8 == 0 and self.scale > 0 else 0

    @property
    def v_pad(self) -> int:
        return next((v for v in (64, 128, 256) if self.vdim <= v), 0)

    @property
    def v_ld(self) -> int:
        return self.v_pad if self.q_ld else 0

    @property
    def q_row(self) -> int:
        return self.q_ld or self.dim + self.rot_dim

    def in_rows(self) -> int:
        return self.heads * (self.dim + self.rot_dim) + (self.cache_row if self.kv_from is None else 0)

    def tensors(self, d: int) -> Dict[str, tuple]:
        t = {"q": (self.heads * (self.dim + self.rot_dim), d), "uk": (self.heads * self.dim, self.kv_rank),
             "uv": (self.heads * self.vdim, self.kv_rank), "o": (d, self.out_dim)}
        if self.sink:
            t["sink"] = (self.heads,)
        if self.kv_from is None:
            t.update({"dkv": (self.cache_row, d), "dkv.norm": (self.kv_rank,)})
        return t


@dataclass(frozen=True)
class GeneralDelta:
    """Generalized delta rule: a [dim, dim] fp32 state per head, decay and removal rate per key channel."""
    heads: int
    dim: int
    decay_rank: int

    @property
    def out_dim(self) -> int:
        return self.heads * self.dim

    @property
    def rank_ld(self) -> int:
        return _up(self.decay_rank, 8)

    def in_rows(self) -> int:
        return 5 * self.out_dim + self.rank_ld

    def tensors(self, d: int) -> Dict[str, tuple]:
        n = self.out_dim
        return {"r": (n, d), "k": (n, d), "v": (n, d), "g": (n, d), "a": (n, d), "a.b": (n,), "w1": (self.decay_rank, d),
                "w2": (n, self.decay_rank), "w0": (n,), "norm": (n,), "o": (d, n)}


@dataclass(frozen=True)
class GroupedAttention:
    """Grouped-query attention: queries scaled by 1 + temp_coef * ln(floor((position + 1) / temp_every) + 1); optionally
    biased projections, a linear distance bias per head, RMS norms of a token's queries and of its keys over all heads at
    once or head by head, rotated queries and keys, rotated values whose sum is turned back, an output gate per head.
    Behind a window, means of whole blocks of `pool` tokens may stand for the tokens that have left it."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int = 0                 # keys a query sees, itself included; 0 = all
    temp_coef: float = 0.0
    temp_every: float = 1.0
    v_mix: bool = False             # the first such layer's values are mixed into the later ones'
    slopes: bool = True             # distance slope 2^(-8 (h + 1) / heads) of head h
    qk_norm: bool = False
    gate: bool = False              # head outputs times sigmoid of a projection
    out_bias: bool = True
    in_bias: bool = True
    head_norm: bool = False         # every head by its own root mean square, one weight for all heads
    rot: Optional[Rotary] = None    # queries and keys
    v_rot: Optional[Rotary] = None  # values; outputs are turned back by the query's position
    pool: int = 0                   # tokens of a block; 0: what has left the window is not seen

    @property
    def out_dim(self) -> int:
        return self.heads * self.vdim

    @property
    def q_ld(self) -> int:
        """Columns of a head in the query buffer and the key pages."""
        return _up(self.dim, 64) if self.dim <= 256 else _up(self.dim, 8)

    @property
    def v_ld(self) -> int:
        return next((v for v in (64, 128, 256) if self.vdim <= v), _up(self.vdim, 8))

    q_row = q_ld

    @property
    def by_head(self) -> bool:
        """Heads are normed or rotated one by one on the way from the projection."""
        return self.head_norm or self.rot is not None or self.v_rot is not None

    @property
    def cache_row(self) -> int:
        """Cache elements of one token."""
        return self.kv_heads * (self.q_ld + self.v_ld)

    @property
    def in_dim(self) -> int:
        """Rows of the input projection: q | k | v | gate."""
        return self.heads * self.dim + self.kv_heads * (self.dim + self.vdim) + (self.heads if self.gate else 0)

    def tensors(self, d: int) -> Dict[str, tuple]:
        out = {}
        for n, rows, cols in (("q", self.heads * self.dim, d), ("k", self.kv_heads * self.dim, d),
                              ("v", self.kv_heads * self.vdim, d), ("o", d, self.out_dim)):
            out[n] = (rows, cols)
            if self.out_bias if n == "o" else self.in_bias:
                out[n + ".b"] = (rows,)
        if self.head_norm:
            out.update({"q.norm": (self.dim,), "k.norm": (self.dim,)})
        if self.qk_norm:
            out.update({"q.norm": (self.heads * self.dim,), "k.norm": (self.kv_heads * self.dim,)})
        if self.gate:
            out["g"] = (self.heads, d)
        if self.v_mix:
            out["vmix"] = ()
        return out


@dataclass(frozen=True)
class StateSpace:
    """State-space mixer with one decay per head: x, B and C behind a causal convolution, a [vdim, state] fp32 state per
    head, gated outputs normed in `norm_groups` equal parts."""
    heads: int
    vdim: int
    state: int
    groups: int                     # head h uses B and C of group h / (heads / groups)
    norm_groups: int
    conv: int                       # taps

    @property
    def out_dim(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        """Channels of the convolution."""
        return self.out_dim + 2 * self.groups * self.state

    @property
    def x_ld(self) -> int:
        """Columns of the convolved channels, heads and groups padded."""
        return self.heads * _up(self.vdim, 8) + 2 * self.groups * _up(self.state, 8)

    @property
    def in_dim(self) -> int:
        """Rows of the input projection: z | x | B | C | step."""
        return self.out_dim + self.channels + self.heads

    @property
    def state_floats(self) -> int:
        return self.out_dim * self.state + (self.conv - 1) * self.channels

    def tensors(self, d: int) -> Dict[str, tuple]:
        n = self.out_dim
        return {"in": (self.in_dim, d), "conv": (self.channels, self.conv), "conv.b": (self.channels,), "dt_bias": (self.heads,),
                "A_log": (self.heads,), "D": (self.heads,), "norm": (n,), "o": (d, n)}


@dataclass(frozen=True)
class MatrixMemory:
    """Matrix memory with exponential gates: a [vdim, dim] fp32 state, a normalizer row and a running maximum of the log
    gates per head; log gates are limited softly to +-gate_cap."""
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    @property
    def out_dim(self) -> int:
        return self.heads * self.vdim

    @property
    def gate_col(self) -> int:
        """First gate row of the input projection q | k | v | output gate | input and forget gates."""
        return _up(2 * self.heads * (self.dim + self.vdim), 16)

    @property
    def in_dim(self) -> int:
        return self.gate_col + 2 * self.heads

    @property
    def x_ld(self) -> int:
        """Columns of the projections as activations, heads padded: q | k | v | output gate."""
        return 2 * self.heads * (_up(self.dim, 8) + _up(self.vdim, 8))

    @property
    def blocks(self) -> int:
        """Blocks of a head's state rows; each keeps the running maximum."""
        return (self.vdim + 63) // 64

    @property
    def state_floats(self) -> int:
        return self.heads * ((self.vdim + 1) * self.dim + self.blocks)

    def tensors(self, d: int) -> Dict[str, tuple]:
        nk, n, H = self.heads * self.dim, self.out_dim, self.heads
        return {"q": (nk, d), "k": (nk, d), "v": (n, d), "g": (n, d), "i": (H, d), "i.b": (H,), "f": (H, d), "f.b": (H,),
                "norm": (n,), "o": (d, n)}


@dataclass(frozen=True)
class SideBySide:
    """left_scale * left(h) + right_scale * right(h)."""
    left: GroupedAttention
    right: StateSpace
    left_scale: float = 1.0
    right_scale: float = 1.0

    def tensors(self, d: int) -> Dict[str, tuple]:
        return {f"{side}.{n}": s for side, m in (("left", self.left), ("right", self.right)) for n, s in m.tensors(d).items()}


@dataclass(frozen=True)
class DenseMlp:
    """down(act(up(x))); act is PolyNorm, whose four numbers are weights, or the square of relu, or a gated unit: gate
    clamped from above, linear part from both sides, gate * sigmoid(alpha * gate) * (linear + 1), or the tanh form of
    gelu of the gate times the linear part."""
    ff: int
    act: str = "poly_norm"          # or "relu2", "clamped_glu", "gelu_glu"
    limit: float = 0.0
    alpha: float = 1.702

    @property
    def glu(self) -> bool:
        return self.act in ("clamped_glu", "gelu_glu")

    @property
    def ff_ld(self) -> int:
        """Columns of the activations."""
        return _up(self.ff, 16) if self.glu else self.ff

    @property
    def up_rows(self) -> int:
        return 2 * self.ff_ld if self.glu else self.ff

    def tensors(self, d: int) -> Dict[str, tuple]:
        t = {"up": (self.ff, d), "down": (d, self.ff)}
        if self.glu:
            t["gate"] = (self.ff, d)
        if self.act == "poly_norm":
            t["act"] = (4,)
        return t


@dataclass(frozen=True)
class MoeMlp:
    """`experts` units of which a token uses the `top` with the largest router logits.  "clamped_glu" (parallel layers): gated
    units (gate clamped from above, linear part from both sides, sigmoid(alpha * gate)), a sigmoid score scales its expert's
    input.  "gelu" (other layers): down(gelu(up(x))) with the erf form, biased logits, the softmax over the chosen ones scales
    the outputs; beside them an expert of `shared` inner size that every token uses."""
    experts: int
    top: int
    ff: int
    limit: float = 0.0
    alpha: float = 1.702
    act: str = "clamped_glu"        # or "gelu"
    shared: int = 0                 # 0: none

    @property
    def ff_ld(self) -> int:
        return _up(self.ff, 16)

    @property
    def glu(self) -> bool:
        return self.act == "clamped_glu"

    @property
    def in_rows(self) -> int:
        """Rows of an expert's first matrix."""
        return 2 * self.ff_ld if self.glu else self.ff_ld

    @property
    def router_rows(self) -> int:
        """Layers that are not parallel: rows of the router in front of the shared expert's."""
        return _up(self.experts, 16)

    @property
    def shared_ld(self) -> int:
        return _up(self.shared, 16)

    def tensors(self, d: int) -> Dict[str, tuple]:
        t = {"router": (self.experts, d)}
        names = ("gate", "up", "down") if self.glu else ("up", "down")
        each = lambda p, ff: {f"{p}.{n}": (d, ff) if n == "down" else (ff, d) for n in names}
        if not self.glu:
            t["router.b"] = (self.experts,)
        for e in range(self.experts):
            t.update(each(f"e{e}", self.ff))
        if self.shared:
            t.update(each("shared", self.shared))
        return t


@dataclass(frozen=True)
class LayerSpec:
    mixer: object
    mlp: object = None
    parallel: bool = False          # x += mixer(h) + ff(h) with one norm h of x
    post_norm: bool = True          # the sublayers' outputs are normed too (layers that are not parallel)
    pre_norm: bool = True           # False: the sublayers read the stream itself; norm1 and norm2 are their outputs' norms
    layer_scale: bool = False       # the sublayers' outputs are multiplied by ls1 and ls2 (behind their norms)

    @property
    def mixers(self) -> tuple:
        """The mixers that read the layer's input: one, or two side by side."""
        return (self.mixer.left, self.mixer.right) if isinstance(self.mixer, SideBySide) else (self.mixer,)

    def one(self, kind):
        """The mixer of this kind, or None."""
        return next((m for m in self.mixers if isinstance(m, kind)), None)

    @property
    def composed(self) -> bool:
        """Grouped attention and / or a state-space mixer, or a matrix memory, behind one input projection."""
        return not self.parallel and all(isinstance(m, (GroupedAttention, StateSpace, MatrixMemory)) for m in self.mixers)

    @property
    def norms(self) -> tuple:
        """Checkpoint names of the norms and scales."""
        if self.parallel:
            return ("norm1",)
        parts = ("1", "2") if self.mlp else ("1",)
        out = tuple(f"norm{p}" for p in parts)
        if self.pre_norm and self.post_norm:
            out += tuple(f"norm{p}b" for p in parts)
        return out + (tuple(f"ls{p}" for p in parts) if self.layer_scale else ())


@dataclass(frozen=True)
class StackConfig:
    name: str
    d_model: int
    vocab: int
    layers: Tuple[LayerSpec, ...]
    rms_eps: float = 1e-5
    act_dtype: str = "bfloat16"      # or "float32": everything in true fp32
    family: str = "qwen3"            # tokenizer / chat-template family
    max_pos: int = 131072
    learned_pos: bool = False        # max_pos position vectors are added to the embedding
    sinusoid_pos: bool = False       # sines and cosines of position * 10000^(-2i / d_model) are added to the embedding
    embed_scale: float = 1.0
    norm_offset: float = 0.0         # added to the stored weights of the layers' and the final norm
    embed_norm: bool = False         # the embedding is normed
    tied_head: bool = False          # logits are products with the embedding
    logit_scale: float = 1.0

    def __post_init__(self):
        if self.act_dtype not in ("bfloat16", "float32"):
            raise ValueError(f"act_dtype {self.act_dtype!r}")
        for i, l in enumerate(self.layers):
            m = l.mixer
            att, ssm = l.one(GroupedAttention), l.one(StateSpace)
            if l.parallel and not isinstance(m, GroupedAttention):
                raise ValueError(f"{self.name}: layer {i}: parallel layers have grouped attention")
            if isinstance(l.mlp, MoeMlp) and l.mlp.glu != l.parallel:
                raise ValueError(f"{self.name}: layer {i}: gated experts come in parallel layers, plain ones in the others")
            if l.mlp and isinstance(l.mlp, DenseMlp) and (l.mlp.act == "relu2") != l.parallel:
                raise ValueError(f"{self.name}: layer {i}: activation {l.mlp.act!r} in this kind of layer")
            if l.parallel and (att.qk_norm or att.gate or att.by_head):
                raise ValueError(f"{self.name}: layer {i}: query and key norms, rotation and gates come in layers that are not parallel")
            if not l.pre_norm and (l.parallel or not l.post_norm):
                raise ValueError(f"{self.name}: layer {i}: norms in front of the sublayers, behind them, or both")
            mem = l.one(MatrixMemory)
            if mem and (isinstance(m, SideBySide) or not 0 < mem.dim <= 256 or mem.gate_cap <= 0):
                raise ValueError(f"{self.name}: layer {i}: a matrix memory stands alone and takes up to 256 key channels per head")
            if isinstance(m, SideBySide) and (att is None or ssm is None or att.out_bias):
                raise ValueError(f"{self.name}: layer {i}: side by side are grouped attention without output bias and a state-space mixer")
            if ssm and (ssm.heads % ssm.groups or ssm.out_dim % ssm.norm_groups or not 0 < ssm.state <= 256 or ssm.conv < 1):
                raise ValueError(f"{self.name}: layer {i}: state-space sizes (groups and parts that divide, up to 256 state entries)")
            if isinstance(l.mlp, MoeMlp) and not 0 < l.mlp.top <= l.mlp.experts <= 1024:
                raise ValueError(f"{self.name}: layer {i}: {l.mlp.top} of {l.mlp.experts} experts (at most 1,024)")
            if att:
                if att.by_head and (att.qk_norm or att.gate or att.v_mix or att.slopes or att.temp_coef):
                    raise ValueError(f"{self.name}: layer {i}: norms by head and rotation do not come with norms over all heads, "
                                     "gates, mixed values, distance bias or query temperature")
                if att.rot and (att.rot.dims % 2 or not 0 <= att.rot.dims <= att.dim):
                    raise ValueError(f"{self.name}: layer {i}: rotary dims {att.rot.dims} of {att.dim}")
                if att.v_rot and (not att.v_rot.pairs or att.v_rot.dims % 2 or not 0 <= att.v_rot.dims <= att.vdim):
                    raise ValueError(f"{self.name}: layer {i}: values rotate in pairs of neighbours")
                if att.pool and (att.window <= 0 or att.pool < 0 or att.slopes):
                    raise ValueError(f"{self.name}: layer {i}: pooled blocks stand behind a window, without distance bias")
                if att.heads % att.kv_heads:
                    raise ValueError(f"{self.name}: layer {i}: {att.heads} query heads on {att.kv_heads} key/value heads")
                if att.v_mix:
                    f = self.layers[self.v_first].one(GroupedAttention)
                    if f.kv_heads * f.vdim != att.kv_heads * att.vdim:
                        raise ValueError(f"{self.name}: layer {i} cannot mix in values of layer {self.v_first}")
            if isinstance(m, GeneralDelta) and m.dim > 256:
                raise ValueError(f"{self.name}: layer {i}: the delta-rule kernel takes up to 256 channels per head")
            if isinstance(m, LatentAttention):
                if m.rot.dims % 2 or m.rot.dims > m.rot_dim:
                    raise ValueError(f"{self.name}: layer {i}: rotary dims {m.rot.dims} of {m.rot_dim}")
                if m.kv_from is not None:
                    src = self.layers[m.kv_from].mixer if 0 <= m.kv_from < i else None
                    if not isinstance(src, LatentAttention) or src.kv_from is not None or src.kv_rank != m.kv_rank \
                            or src.rot_dim != m.rot_dim:
                        raise ValueError(f"{self.name}: layer {i} cannot read layer {m.kv_from}'s cache")

    @property
    def n_layers(self) -> int:
        return len(self.layers)

    @property
    def v_first(self) -> Optional[int]:
        """The layer whose values later layers mix in."""
        return next((i for i, l in enumerate(self.layers) if any(getattr(m, "v_mix", False) for m in l.mixers)), None)

    def mixers(self, *kinds) -> list:
        """All mixers of these kinds."""
        return [m for l in self.layers for m in l.mixers if isinstance(m, kinds)]

    @property
    def vocab_ld(self) -> int:
        return _up(self.vocab, 4)

    @property
    def has_state(self) -> bool:
        """True when a prefix's cache pages alone do not restore it (recurrent layers)."""
        return bool(self.mixers(GeneralDelta, StateSpace, MatrixMemory))

    @property
    def pools(self) -> Tuple[int, ...]:
        """Block sizes of pooled keys; each has pages and columns of the block table of its own."""
        return tuple(sorted({m.pool for m in self.mixers(GroupedAttention) if m.pool}))

    @property
    def max_window(self) -> int:
        """Largest attention window of the stack, 0 = unbounded."""
        w = [m.window for m in self.mixers(LatentAttention, GroupedAttention)]
        return 0 if not w or 0 in w else max(w)

    @property
    def torch_dtype(self):
        return torch.float32 if self.act_dtype == "float32" else torch.bfloat16

    @property
    def itemsize(self) -> int:
        return 4 if self.act_dtype == "float32" else 2

    @property
    def kv_bytes_per_token(self) -> int:
        return sum(m.cache_row for m in self.mixers(LatentAttention, GroupedAttention)
                   if getattr(m, "kv_from", None) is None) * self.itemsize

    def pool_bytes_per_block(self, pool: int) -> int:
        """Bytes of one pooled block of `pool` tokens, all layers that have such blocks."""
        return sum(m.cache_row for m in self.mixers(GroupedAttention) if m.pool == pool) * self.itemsize

    @property
    def state_bytes_per_row(self) -> int:
        return sum(4 * m.heads * m.dim ** 2 for m in self.mixers(GeneralDelta)) + \
            sum(4 * m.state_floats for m in self.mixers(StateSpace, MatrixMemory))

    def in_rows(self, i: int) -> int:
        """Rows of layer i's fused input projection, padded for the 256-wide GEMM tiles when it is large."""
        if self.layers[i].parallel:
            return self.qkv_rows(i) + self.up_rows(i)
        if self.layers[i].composed:
            ssm, mem = self.layers[i].one(StateSpace), self.layers[i].one(MatrixMemory)
            n = mem.in_dim if mem else self.ssm_col(i) + (ssm.in_dim if ssm else 0)
        else:
            n = self.layers[i].mixer.in_rows()
        return _up(n, 256 if n >= 2048 else 16)

    def ssm_col(self, i: int) -> int:
        """Composed layers: first state-space row of the input projection, behind the attention's."""
        att = self.layers[i].one(GroupedAttention)
        return _up(att.in_dim, 16) if att else 0

    def ssm_mix_col(self, i: int) -> int:
        """Composed layers: first state-space column of what the output projection reads."""
        att = self.layers[i].one(GroupedAttention)
        return _up(att.out_dim, 8) if att else 0

    def qkv_rows(self, i: int) -> int:
        """Parallel layers: padded rows of q | k | v | router."""
        f = self.layers[i].mlp
        n = self.layers[i].mixer.in_dim + (f.experts if isinstance(f, MoeMlp) else 0)
        return _up(n, 32 if n >= 2048 else 16)

    def up_rows(self, i: int) -> int:
        """Parallel layers: padded rows of a dense feed-forward's up matrix, behind the rows above."""
        f = self.layers[i].mlp
        return _up(f.ff, 32 if f.ff >= 2048 else 16) if isinstance(f, DenseMlp) else 0

    def mix_cols(self, i: int) -> Tuple[int, int]:
        """(first activation column, columns) of what layer i's output projection reads."""
        if self.layers[i].composed:
            own = self.layers[i].one(StateSpace) or self.layers[i].one(MatrixMemory)
            n = _up(self.ssm_mix_col(i) + (own.out_dim if own else 0), 8)
            return n, n
        n = self.layers[i].mixer.out_dim
        return (_up(n, 8), _up(n, 8) + self.up_rows(i)) if self.layers[i].parallel else (n, n)

    def tensor_shapes(self) -> Dict[str, tuple]:
        """Every tensor of the checkpoint, name -> shape."""
        d = self.d_model
        out = {"embed": (self.vocab, d), "final.norm": (d,)}
        if not self.tied_head:
            out["head"] = (self.vocab, d)
        if self.embed_norm:
            out["embed.norm"] = (d,)
        if self.learned_pos:
            out["pos"] = (self.max_pos, d)
        for i, l in enumerate(self.layers):
            out.update({f"l{i}.{n}": (d,) for n in l.norms})
            out.update({f"l{i}.mix.{n}": s for n, s in l.mixer.tensors(d).items()})
            if l.mlp:
                out.update({f"l{i}.mlp.{n}": s for n, s in l.mlp.tensors(d).items()})
        return out

    def decode_weight_bytes(self, rows: Optional[int] = None) -> int:
        """bf16 bytes of matrices streamed per decode step of `rows` tokens: experts by the number that so many tokens
        use on average when they choose at random (None: all of them)."""
        total = 0.0
        for n, s in self.tensor_shapes().items():
            if len(s) == 2 and n not in (("pos",) if self.tied_head else ("embed", "pos")):
                f = self.layers[int(n[1:n.index(".")])].mlp if ".mlp.e" in n else None
                used = 1.0 - (1.0 - f.top / f.experts) ** rows if f and rows is not None else 1.0
                total += 2 * s[0] * s[1] * used
        return round(total)

    def shard(self, tp_size: int) -> "StackConfig":
        if tp_size != 1:
            raise ValueError(f"{self.name}: tensor parallelism is not implemented for layer stacks")
        return self


# ------------------------------------------------------------------------------------------ designs
def _bekopel(c: dict, shape: Callable[[str], tuple], name: str) -> StackConfig:
    """config.json of the Bekopel design; `shape(tensor)` gives what only the checkpoint states."""
    layers = []
    for i, e in enumerate(c["layers"]):
        m, kind = e["mixer"], e["type"]
        if kind == "latent_attention":
            mixer = LatentAttention(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]),
                                    vdim=int(m["vdim"]), kv_rank=int(m["kv_rank"]), scale=float(m["scale"]),
                                    rot=Rotary(float(m["rot"]["base"]), int(m["rot"]["dims"])),
                                    window=int(m["mask"]["size"]),
                                    kv_from=None if m.get("kv_from") is None else int(m["kv_from"]))
        elif kind == "general_delta":
            mixer = GeneralDelta(heads=int(m["heads"]), dim=int(m["dim"]), decay_rank=int(shape(f"l{i}.mix.w1")[0]))
        else:
            raise ValueError(f"{name}: layer {i}: unknown mixer {kind!r}")
        f = e.get("mlp")
        if f is not None and f.get("kind") != "dense":
            raise ValueError(f"{name}: layer {i}: unknown feed-forward {f.get('kind')!r}")
        layers.append(LayerSpec(mixer, DenseMlp(int(f["ff"])) if f is not None else None))
    return StackConfig(name=name, d_model=int(c["width"]), vocab=int(c["vocab"]), layers=tuple(layers),
                       rms_eps=float(c["norm"]["eps"]))


def _lerazen(c: dict, shape: Callable[[str], tuple], name: str) -> StackConfig:
    """config.json of the Lerazen design."""
    layers = []
    for i, e in enumerate(c["layers"]):
        m, kind = e["mixer"], e["type"]
        if kind != "attention":
            raise ValueError(f"{name}: layer {i}: unknown mixer {kind!r}")
        temp = m.get("q_temp") or {"coef": 0.0, "every": 1}
        mixer = GroupedAttention(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                                 scale=float(m["scale"]), window=int((m.get("mask") or {"size": 0})["size"]),
                                 temp_coef=float(temp["coef"]), temp_every=float(temp["every"]),
                                 v_mix=bool(m.get("v_mix", False)))
        f = e.get("mlp")
        if f is None:
            mlp = None
        elif f.get("kind") == "dense":
            mlp = DenseMlp(int(f["ff"]), "relu2")
        elif f.get("kind") == "moe":
            mlp = MoeMlp(int(f["router"]["experts"]), int(f["router"]["top"]), int(f["expert"]["ff"]), float(f["expert"]["limit"]))
        else:
            raise ValueError(f"{name}: layer {i}: unknown feed-forward {f.get('kind')!r}")
        layers.append(LayerSpec(mixer, mlp, parallel=True))
    return StackConfig(name=name, d_model=int(c["width"]), vocab=int(c["vocab"]), layers=tuple(layers),
                       rms_eps=float(c["norm"]["eps"]), max_pos=int(c["max_positions"]), learned_pos=True)


def _state_space(m: dict) -> StateSpace:
    return StateSpace(heads=int(m["heads"]), vdim=int(m["vdim"]), state=int(m["state"]), groups=int(m["groups"]),
                      norm_groups=int(m["norm_groups"]), conv=int(m["conv"]))


def _merulorn(c: dict, shape: Callable[[str], tuple], name: str) -> StackConfig:
    """config.json of the Merulorn design."""
    layers = []
    for i, e in enumerate(c["layers"]):
        m, kind = e["mixer"], e["type"]
        if kind == "parallel":
            a = m["left"]
            temp = a.get("q_temp") or {"coef": 0.0, "every": 1}
            left = GroupedAttention(heads=int(a["heads"]), kv_heads=int(a["kv_heads"]), dim=int(a["dim"]), vdim=int(a["vdim"]),
                                    scale=float(a["scale"]), temp_coef=float(temp["coef"]), temp_every=float(temp["every"]),
                                    slopes=False, qk_norm=True, gate=True, out_bias=False)
            mixer = SideBySide(left, _state_space(m["right"]), float(m["left_scale"]), float(m["right_scale"]))
        elif kind == "mamba2":
            mixer = _state_space(m)
        else:
            raise ValueError(f"{name}: layer {i}: unknown mixer {kind!r}")
        f = e.get("mlp")
        if f is not None and f.get("kind") != "dense":
            raise ValueError(f"{name}: layer {i}: unknown feed-forward {f.get('kind')!r}")
        mlp = DenseMlp(int(f["ff"]), "clamped_glu", float(f["limit"])) if f is not None else None
        layers.append(LayerSpec(mixer, mlp, post_norm=False))
    return StackConfig(name=name, d_model=int(c["width"]), vocab=int(c["vocab"]), layers=tuple(layers),
                       rms_eps=float(c["norm"]["eps"]), sinusoid_pos=True, embed_scale=float(c["embedding"]["scale"]),
                       norm_offset=1.0)


def _vosolorn(c: dict, shape: Callable[[str], tuple], name: str) -> StackConfig:
    """config.json of the Vosolorn design."""
    layers = []
    for i, e in enumerate(c["layers"]):
        m, kind = e["mixer"], e["type"]
        if kind == "attention":
            mask, rot, vdim = m.get("mask") or {"size": 0}, m["rot"], int(m["vdim"])
            mixer = GroupedAttention(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=vdim,
                                     scale=float(m["scale"]), window=int(mask["size"]), slopes=False, out_bias=False, in_bias=False,
                                     head_norm=True, rot=Rotary(float(rot["base"]), int(rot["dims"]), True),
                                     v_rot=Rotary(float(rot["base"]), vdim, True), pool=int(mask.get("pool") or 0))
        elif kind == "mlstm":
            mixer = MatrixMemory(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), gate_cap=float(m["gate_cap"]))
        else:
            raise ValueError(f"{name}: layer {i}: unknown mixer {kind!r}")
        f = e.get("mlp")
        if f is None:
            mlp = None
        elif f.get("kind") == "dense":
            mlp = DenseMlp(int(f["ff"]), "gelu_glu")
        elif f.get("kind") == "moe":
            mlp = MoeMlp(int(f["router"]["experts"]), int(f["router"]["top"]), int(f["expert"]["ff"]), act="gelu",
                         shared=int((f.get("shared") or {"ff": 0})["ff"]))
        else:
            raise ValueError(f"{name}: layer {i}: unknown feed-forward {f.get('kind')!r}")
        layers.append(LayerSpec(mixer, mlp, pre_norm=False, layer_scale=True))
    return StackConfig(name=name, d_model=int(c["width"]), vocab=int(c["vocab"]), layers=tuple(layers),
                       rms_eps=float(c["norm"]["eps"]), embed_norm=True, tied_head=True, logit_scale=float(c["logit_scale"]))


DESIGNS: Dict[str, Callable] = {"Bekopel": _bekopel, "Lerazen": _lerazen, "Merulorn": _merulorn, "Vosolorn": _vosolorn}


def safetensors_shapes(path) -> Dict[str, tuple]:
    """Tensor shapes from a safetensors header (the data is not read)."""
    with open(path, "rb") as f:
        n = int.from_bytes(f.read(8), "little")
        head = json.loads(f.read(n))
    return {k: tuple(v["shape"]) for k, v in head.items() if k != "__metadata__"}


def config_from_dir(model_dir, c: dict) -> StackConfig:
    """StackConfig of a model directory whose config.json `c` names a design in DESIGNS."""
    path = Path(model_dir) / "model.safetensors"
    shapes: Dict[str, tuple] = {}

    def shape(n):
        if not shapes:
            shapes.update(safetensors_shapes(path))
        return shapes[n]
    return DESIGNS[c["architecture"]](c, shape, Path(model_dir).name)


def bekopel_preset(name: str, n_layers: int, d_model: int, ff: int, vocab: int, heads: int = 32, dim: int = 128,
                   rot_dim: int = 64, kv_rank: int = 512, window: int = 1024, decay_rank: int = 128,
                   max_pos: int = 32768) -> StackConfig:
    """Bekopel at sizes of a real model's layers (random-init presets, bench): groups of delta, latent attention,
    latent attention on the same cache, delta."""
    delta = GeneralDelta(d_model // 128, 128, decay_rank)
    layers = []
    for i in range(n_layers):
        if i % 4 in (1, 2):
            m = LatentAttention(heads, dim, rot_dim, dim, kv_rank, (dim + rot_dim) ** -0.5, Rotary(1e6, rot_dim), window,
                                None if i % 4 == 1 else i - 1)
        else:
            m = delta
        layers.append(LayerSpec(m, DenseMlp(ff)))
    return StackConfig(name, d_model, vocab, tuple(layers), max_pos=max_pos)


def lerazen_preset(name: str, n_layers: int, d_model: int, ff: int, vocab: int, heads: int = 32, kv_heads: int = 8,
                   dim: int = 128, window: int = 1024, experts: int = 0, top: int = 4, expert_ff: int = 1024,
                   max_pos: int = 32768) -> StackConfig:
    """Lerazen at sizes of a real model's layers (random-init presets, bench): dense feed-forwards, or, with
    `experts`, a dense one in the first layer and experts in the others."""
    m = GroupedAttention(heads, kv_heads, dim, dim, dim ** -0.5, window, 0.1, 8192, True)
    dense = DenseMlp(ff, "relu2")
    moe = MoeMlp(experts, top, expert_ff, 7.0) if experts else dense
    layers = tuple(LayerSpec(m, moe if i else dense, True) for i in range(n_layers))
    return StackConfig(name, d_model, vocab, layers, max_pos=max_pos, learned_pos=True)


def merulorn_preset(name: str, n_layers: int, d_model: int, ff: int, vocab: int, heads: int = 32, kv_heads: int = 8,
                    dim: int = 128, vdim: int = 64, state: int = 128, groups: int = 8, max_pos: int = 32768) -> StackConfig:
    """Merulorn at sizes of a real model's layers (random-init presets, bench): one layer in four has attention beside the
    state-space mixer and a feed-forward."""
    ssm = StateSpace(2 * d_model // vdim, vdim, state, groups, groups, 4)
    att = GroupedAttention(heads, kv_heads, dim, dim, dim ** -0.5, 0, 0.1, 8192, slopes=False, qk_norm=True, gate=True, out_bias=False)
    both = LayerSpec(SideBySide(att, ssm, 0.7, 0.7), DenseMlp(ff, "clamped_glu", 7.0), post_norm=False)
    layers = tuple(LayerSpec(ssm, None, post_norm=False) if i % 4 in (1, 2, 3) else both for i in range(n_layers))
    return StackConfig(name, d_model, vocab, layers, max_pos=max_pos, sinusoid_pos=True, embed_scale=d_model ** 0.5, norm_offset=1.0)


def vosolorn_preset(name: str, n_layers: int, d_model: int, ff: int, vocab: int, heads: int = 32, kv_heads: int = 8, dim: int = 128,
                    window: int = 512, pool: int = 16, mem_dim: int = 128, mem_vdim: int = 256, experts: int = 0, top: int = 8,
                    expert_ff: int = 1024, max_pos: int = 32768) -> StackConfig:
    """Vosolorn at sizes of a real model's layers (random-init presets, bench): one layer in four has attention, the others a
    matrix memory; dense feed-forwards, or, with `experts`, a dense one in the first layer and experts, one of them shared, in
    the others."""
    att = GroupedAttention(heads, kv_heads, dim, dim, dim ** -0.5, window, slopes=False, out_bias=False, in_bias=False, head_norm=True,
                           rot=Rotary(1e6, dim, True), v_rot=Rotary(1e6, dim, True), pool=pool)
    mem = MatrixMemory(d_model // mem_vdim, mem_dim, mem_vdim, 15.0)
    dense = DenseMlp(ff, "gelu_glu")
    moe = MoeMlp(experts, top, expert_ff, act="gelu", shared=expert_ff) if experts else dense
    layers = tuple(LayerSpec(mem if i % 4 else att, moe if i else dense, pre_norm=False, layer_scale=True) for i in range(n_layers))
    return StackConfig(name, d_model, vocab, layers, max_pos=max_pos, embed_norm=True, tied_head=True, logit_scale=d_model ** -0.5)


# ------------------------------------------------------------------------------------------ weights
def head_slopes(heads: int, device) -> torch.Tensor:
    """[heads] fp32 distance slopes 2^(-8 (h + 1) / heads)."""
    h = torch.arange(1, heads + 1, dtype=torch.float64)
    return torch.exp2(-8.0 * h / heads).float().to(device)


def position_turns(width: int, device) -> torch.Tensor:
    """[(width + 1) // 2] fp64: turns per position of the sinusoids, 10000^(-2i / width) / 2 pi."""
    i = torch.arange((width + 1) // 2, dtype=torch.float64)
    return (10000.0 ** (-2.0 * i / width) / (2.0 * math.pi)).to(device)


def rope_table(rot: Rotary, n_pos: int, device) -> torch.Tensor:
    """[n_pos, dims] fp32: cos of the dims/2 angles, then sin (angles formed in fp64, rounded once)."""
    half = rot.dims // 2
    f = rot.base ** (-2.0 * torch.arange(half, dtype=torch.float64) / rot.dims)
    ang = torch.arange(n_pos, dtype=torch.float64)[:, None] * f[None, :]
    return torch.cat([ang.cos(), ang.sin()], dim=1).float().contiguous().to(device)


@dataclass
class StackWeights:
    """Tensors packed for the kernels: per layer a dict of device tensors named after bcg_layer's fields."""
    cfg: StackConfig
    embed: torch.Tensor
    lm_head: torch.Tensor
    final_norm: torch.Tensor
    layers: list = field(default_factory=list)
    pos_embed: Optional[torch.Tensor] = None
    pos_turns: Optional[torch.Tensor] = None
    embed_norm: Optional[torch.Tensor] = None

    @staticmethod
    def from_tensors(cfg: StackConfig, get: Callable[[str], torch.Tensor], device) -> "StackWeights":
        """`get(name)` returns a checkpoint tensor (CPU or device, any float dtype)."""
        want = cfg.tensor_shapes()

        def raw(n):
            t = get(n)
            if tuple(t.shape) != want[n]:
                raise ValueError(f"{cfg.name}: tensor {n} has shape {tuple(t.shape)}, expected {want[n]}")
            return t.detach().to(device)

        bf = lambda t: t.to(torch.bfloat16).contiguous()
        f32 = lambda t: t.float().contiguous()

        def rows(t, n):
            return t if t.shape[0] == n else torch.cat([t, t.new_zeros(n - t.shape[0], *t.shape[1:])])

        norm = lambda n: f32(raw(n)) + cfg.norm_offset
        embed = bf(raw("embed"))
        head = rows(embed, cfg.vocab_ld) if cfg.tied_head else bf(rows(raw("head"), cfg.vocab_ld))
        # the factor of the logits joins the final norm's weight
        w = StackWeights(cfg, embed, head, norm("final.norm") * cfg.logit_scale)
        if cfg.embed_norm:
            w.embed_norm = norm("embed.norm")
        if cfg.sinusoid_pos:
            w.pos_turns = position_turns(cfg.d_model, device)
        if cfg.learned_pos:
            w.pos_embed = bf(raw("pos"))
        for i, l in enumerate(cfg.layers):
            m, g = l.mixer, lambda n: raw(f"l{i}.mix.{n}")
            if l.parallel:
                w.layers.append(StackWeights._parallel(cfg, i, raw, norm, bf, f32, rows))
                continue
            t = {}
            for part in ("1", "2") if l.mlp else ("1",):        # a scale joins the weight of the norm in front of it
                scale = f32(raw(f"l{i}.ls{part}")) if l.layer_scale else 1.0
                if l.pre_norm:
                    t[f"norm{part}"] = norm(f"l{i}.norm{part}")
                if l.post_norm:
                    t[f"norm{part}b"] = norm(f"l{i}.norm{part}" + ("b" if l.pre_norm else "")) * scale
            if l.composed:
                t.update(StackWeights._composed(cfg, i, raw, bf, f32, rows))
            elif isinstance(m, LatentAttention):
                t["w_out"] = bf(g("o"))
                own = m.kv_from is None
                t["w_in"] = bf(rows(torch.cat([g("q"), g("dkv")]) if own else g("q"), cfg.in_rows(i)))
                if own:
                    t["latent_norm"] = f32(g("dkv.norm"))
                if m.sink:
                    t["sink"] = f32(g("sink"))
                t["w_uk"], t["w_uv"] = bf(g("uk")), bf(g("uv"))
                if m.q_ld and cfg.act_dtype == "bfloat16":
                    t["w_expand"] = StackWeights.expansion(m, t["w_uk"], t["w_uv"])
            else:
                t["w_out"] = bf(g("o"))
                w1 = rows(g("w1"), m.rank_ld)
                t["w_in"] = bf(rows(torch.cat([g("r"), g("k"), g("v"), g("g"), g("a"), w1]), cfg.in_rows(i)))
                w2 = g("w2")
                t["w_decay"] = bf(torch.cat([w2, w2.new_zeros(w2.shape[0], m.rank_ld - m.decay_rank)], dim=1))
                t["decay_bias"], t["rate_bias"], t["out_norm"] = f32(g("w0")), f32(g("a.b")), f32(g("norm"))
            if isinstance(l.mlp, MoeMlp):
                t.update(StackWeights._experts(cfg, i, raw, bf, f32, rows))
            elif l.mlp and l.mlp.glu:
                t["w_up"] = StackWeights.glu_rows(*(rows(bf(raw(f"l{i}.mlp.{n}")), l.mlp.ff_ld) for n in ("gate", "up")))
                t["w_down"] = torch.zeros(cfg.d_model, l.mlp.ff_ld, dtype=torch.bfloat16, device=device)
                t["w_down"][:, :l.mlp.ff] = bf(raw(f"l{i}.mlp.down"))
            elif l.mlp:
                t.update(w_up=bf(raw(f"l{i}.mlp.up")), w_down=bf(raw(f"l{i}.mlp.down")), act_coef=f32(raw(f"l{i}.mlp.act")))
            w.layers.append(t)
        return w

    @staticmethod
    def glu_rows(gate: torch.Tensor, up: torch.Tensor) -> torch.Tensor:
        """Gate and up rows (a multiple of 16 of each) interleaved by 16."""
        n, d = gate.shape
        return torch.stack([gate.view(n // 16, 16, d), up.view(n // 16, 16, d)], dim=1).reshape(2 * n, d)

    @staticmethod
    def _composed(cfg: StackConfig, i: int, raw, bf, f32, rows) -> dict:
        """Grouped attention (q | k | v | gate) and a state-space mixer (z | x | B | C | step) in one input matrix, their
        output matrices side by side.  Scales of the two join the gate and the state-space norm."""
        l, d = cfg.layers[i], cfg.d_model
        att, ssm, both = l.one(GroupedAttention), l.one(StateSpace), isinstance(l.mixer, SideBySide)
        left = lambda n: raw(f"l{i}.mix." + ("left." if both else "") + n)
        right = lambda n: raw(f"l{i}.mix." + ("right." if both else "") + n)
        if l.one(MatrixMemory):
            return StackWeights._memory(cfg, i, right, bf, f32, rows)
        w_in, t = [], {}
        some = left("o") if att else right("o")
        w_out = torch.zeros(d, cfg.mix_cols(i)[1], dtype=torch.bfloat16, device=some.device)
        if att:
            w_in.append(rows(torch.cat([left(n) for n in ("q", "k", "v")] + ([left("g")] if att.gate else [])), cfg.ssm_col(i)))
            w_out[:, :att.out_dim] = bf(left("o"))
            if att.in_bias:
                t["in_bias"] = f32(torch.cat([left("q.b"), left("k.b"), left("v.b")]))
            if att.out_bias:
                t["out_bias"] = f32(left("o.b"))
            if att.qk_norm or att.head_norm:
                t["q_norm"], t["k_norm"] = f32(left("q.norm")), f32(left("k.norm"))
            if att.slopes:
                t["slopes"] = head_slopes(att.heads, some.device)
            if att.v_mix:
                t["vmix"] = f32(left("vmix"))
        if ssm:
            w_in.append(right("in"))
            at = cfg.ssm_mix_col(i)
            w_out[:, at:at + ssm.out_dim] = bf(right("o"))
            t.update(conv_w=f32(right("conv").T), conv_b=f32(right("conv.b")), step_bias=f32(right("dt_bias")),
                     decay_rate=right("A_log").double().exp().float().contiguous(), skip=f32(right("D")),
                     ssm_norm=f32(right("norm")) * (l.mixer.right_scale if both else 1.0))
        t["w_in"], t["w_out"] = bf(rows(torch.cat(w_in), cfg.in_rows(i))), w_out
        return t

    @staticmethod
    def _memory(cfg: StackConfig, i: int, get, bf, f32, rows) -> dict:
        """q | k | v | output gate, then the input and forget gates, in one input matrix."""
        m = cfg.layers[i].mixer
        w_in = torch.cat([rows(torch.cat([get(n) for n in ("q", "k", "v", "g")]), m.gate_col), get("i"), get("f")])
        w_out = torch.zeros(cfg.d_model, cfg.mix_cols(i)[1], dtype=torch.bfloat16, device=w_in.device)
        w_out[:, :m.out_dim] = bf(get("o"))
        return {"w_in": bf(rows(w_in, cfg.in_rows(i))), "w_out": w_out, "mem_bias": f32(torch.cat([get("i.b"), get("f.b")])),
                "mem_norm": f32(get("norm"))}

    @staticmethod
    def _experts(cfg: StackConfig, i: int, raw, bf, f32, rows) -> dict:
        """Plain experts: the router and the shared expert's rows in one matrix, the others' one after another."""
        f, d = cfg.layers[i].mlp, cfg.d_model
        g = lambda n: raw(f"l{i}.mlp.{n}")
        up = [rows(g("router"), f.router_rows)] + ([rows(g("shared.up"), f.shared_ld)] if f.shared else [])
        t = {"w_up": bf(torch.cat(up)), "router_bias": f32(g("router.b"))}
        z = lambda *s: torch.zeros(*s, dtype=torch.bfloat16, device=t["w_up"].device)
        if f.shared:
            t["w_down"] = z(d, f.shared_ld)
            t["w_down"][:, :f.shared] = bf(g("shared.down"))
        t["w_experts_in"], t["w_experts_out"] = z(f.experts, f.ff_ld, d), z(f.experts, d, f.ff_ld)
        for e in range(f.experts):
            t["w_experts_in"][e, :f.ff] = bf(g(f"e{e}.up"))
            t["w_experts_out"][e, :, :f.ff] = bf(g(f"e{e}.down"))
        return t

    @staticmethod
    def _parallel(cfg: StackConfig, i: int, raw, norm, bf, f32, rows) -> dict:
        """A parallel layer: q | k | v | router, then the up rows, in one matrix; o and down side by side in another;
        experts one after another, gate and up rows interleaved by 16."""
        l, d = cfg.layers[i], cfg.d_model
        m, f, dense = l.mixer, l.mlp, isinstance(l.mlp, DenseMlp)
        g, ffn = lambda n: raw(f"l{i}.mix.{n}"), lambda n: raw(f"l{i}.mlp.{n}")
        top = [g("q"), g("k"), g("v")] + ([ffn("router")] if isinstance(f, MoeMlp) else [])
        w_in = rows(torch.cat(top), cfg.qkv_rows(i))
        act_col, cols = cfg.mix_cols(i)
        w_out = torch.zeros(d, cols, dtype=torch.bfloat16, device=w_in.device)
        w_out[:, :m.out_dim] = bf(g("o"))
        if dense:
            w_in = torch.cat([w_in, rows(ffn("up"), cfg.up_rows(i))])
            w_out[:, act_col:act_col + f.ff] = bf(ffn("down"))
        t = {"norm1": norm(f"l{i}.norm1"), "w_in": bf(w_in), "w_out": w_out, "out_bias": f32(g("o.b")),
             "in_bias": f32(torch.cat([g("q.b"), g("k.b"), g("v.b")]))}
        if m.slopes:
            t["slopes"] = head_slopes(m.heads, w_in.device)
        if m.v_mix:
            t["vmix"] = f32(g("vmix"))
        if isinstance(f, MoeMlp):
            n = f.ff_ld
            t["w_experts_in"] = torch.zeros(f.experts, 2 * n, d, dtype=torch.bfloat16, device=w_in.device)
            t["w_experts_out"] = torch.zeros(f.experts, d, n, dtype=torch.bfloat16, device=w_in.device)
            for e in range(f.experts):
                t["w_experts_in"][e] = StackWeights.glu_rows(*(rows(bf(ffn(f"e{e}.{x}")), n) for x in ("gate", "up")))
                t["w_experts_out"][e, :, :f.ff] = bf(ffn(f"e{e}.down"))
        return t

    @staticmethod
    def expansion(m: LatentAttention, uk: torch.Tensor, uv: torch.Tensor) -> torch.Tensor:
        """[heads * (q_ld + v_ld), cache_row]: cache row -> every head's key (up-projected latent, the rotated
        part through an identity block, zero padding), then every head's value."""
        k = uk.new_zeros(m.heads, m.q_ld, m.cache_row)
        k[:, :m.dim, :m.kv_rank] = uk.view(m.heads, m.dim, m.kv_rank)
        k[:, m.dim:m.dim + m.rot_dim, m.kv_rank:] = torch.eye(m.rot_dim, dtype=uk.dtype, device=uk.device)
        v = uv.new_zeros(m.heads, m.v_ld, m.cache_row)
        v[:, :m.vdim, :m.kv_rank] = uv.view(m.heads, m.vdim, m.kv_rank)
        return torch.cat([k.flatten(0, 1), v.flatten(0, 1)]).contiguous()

    @staticmethod
    def from_safetensors_dir(cfg: StackConfig, model_dir, device) -> "StackWeights":
        from safetensors import safe_open
        with safe_open(str(Path(model_dir) / "model.safetensors"), "pt") as f:
            return StackWeights.from_tensors(cfg, f.get_tensor, device)

    @staticmethod
    def random_init(cfg: StackConfig, device, seed: int = 0) -> "StackWeights":
        """N(0, 0.02) matrices, unit norms, zero biases and sinks, identity-like activation; made on the device."""
        g = torch.Generator(device=device)
        g.manual_seed(seed)
        shapes = cfg.tensor_shapes()

        def get(n):
            s = shapes[n]
            if n.endswith(".act"):
                return torch.tensor([1.0, 0.5, 0.25, 0.0], device=device)
            if n.endswith(".vmix"):
                return torch.tensor(0.5, device=device)
            if n.endswith(".conv"):
                return torch.empty(*s, device=device).normal_(0.0, s[1] ** -0.5, generator=g)
            if n.endswith(".dt_bias"):      # steps around 0.02
                return torch.full(s, -4.0, device=device)
            if n.endswith(".D"):
                return torch.ones(*s, device=device)
            if n.endswith(".f.b"):          # memories of a few dozen tokens and more
                return torch.linspace(3.0, 6.0, s[0], device=device)
            if len(s) == 2:
                return torch.empty(*s, dtype=torch.bfloat16, device=device).normal_(0.0, 0.02, generator=g)
            leaf = n.rsplit(".", 1)[-1]
            one = leaf.startswith(("norm", "ls")) and not (cfg.norm_offset and ".mix." not in n)
            return (torch.ones if one else torch.zeros)(*s, device=device)
        return StackWeights.from_tensors(cfg, get, device)

    def nbytes(self) -> int:
        ts = [self.embed] + ([] if self.lm_head.data_ptr() == self.embed.data_ptr() else [self.lm_head]) + ([self.pos_embed] if self.pos_embed is not None else []) + [t for l in self.layers for t in l.values()]
        return sum(t.numel() * t.element_size() for t in ts)


# ------------------------------------------------------------------------------------------ handle
class StackHandle:
    """Host-side bcg_stack (include/bcg_b200.h) over StackWeights, caches and states.

    caches[i]: the latent pages [pages, page, cache_row] or the states [slots, heads, dim, dim] of layer i
    (None where the layer reads another layer's cache); for grouped attention and state-space mixers a dict of what
    there is of cache (keys [pages, kv_heads, page, q_ld]), cache_v (values [pages, kv_heads, page, v_ld]), ssm_state
    [slots, heads, vdim, state] and conv_state [slots, taps - 1, channels]; for matrix memories mem_state [slots, heads,
    vdim + 1, dim] and mem_max [slots, heads, blocks].  Pages of pooled blocks follow the others; pool_cols: block size ->
    first column of their page numbers in the block table."""

    def __init__(self, w: StackWeights, caches: list, n_pos: int, page_size: int, pool_cols: Optional[Dict[int, int]] = None):
        cfg = w.cfg
        self.w, self.caches = w, caches
        dev = w.embed.device
        self._rope: Dict[Rotary, torch.Tensor] = {}
        arr = (L.Layer * cfg.n_layers)()
        counts = 0

        def table(rot: Rotary) -> int:
            if rot not in self._rope:
                self._rope[rot] = rope_table(rot, n_pos, dev)
            return self._rope[rot].data_ptr()
        for i, (spec, t) in enumerate(zip(cfg.layers, w.layers)):
            a, m = arr[i], spec.mixer
            a.n_in = cfg.in_rows(i)
            src = i
            att, ssm, mem = spec.one(GroupedAttention), spec.one(StateSpace), spec.one(MatrixMemory)
            if att:
                if att.by_head:
                    a.by_head, a.rot_dims, a.v_rot_dims = 1, att.rot.dims if att.rot else 0, att.v_rot.dims if att.v_rot else 0
                    if a.rot_dims:
                        a.cos_sin, a.rot_pairs = table(att.rot), int(att.rot.pairs)
                    if a.v_rot_dims:
                        a.v_cos_sin = table(att.v_rot)
                if att.pool:
                    a.pool, a.pool_col = att.pool, pool_cols[att.pool]
                a.mixer, a.heads, a.dim = L.MIXER_GROUPED_ATTN, att.heads, att.dim
                a.kv_heads, a.vdim, a.q_ld, a.v_ld = att.kv_heads, att.vdim, att.q_ld, att.v_ld
                a.window, a.scale, a.owns_cache = att.window, att.scale, 1
                a.temp_coef, a.temp_every = att.temp_coef, att.temp_every
                if att.v_mix:
                    a.v_role = L.VALUES_FIRST if i == cfg.v_first else L.VALUES_MIX
                    a.v_mix = float(t["vmix"])
                if spec.parallel:
                    a.parallel, a.n_qkv, a.router_col = 1, cfg.qkv_rows(i), att.in_dim
                if att.gate:
                    a.gated, a.gate_col = 1, att.in_dim - att.heads
                    a.gate_scale = m.left_scale if isinstance(m, SideBySide) else 1.0
                a.act_col, a.mix_ld = cfg.mix_cols(i)
            if ssm:
                if not att:
                    a.mixer = L.MIXER_STATE_SPACE
                a.ssm_heads, a.ssm_vdim, a.ssm_n, a.ssm_groups = ssm.heads, ssm.vdim, ssm.state, ssm.groups
                a.ssm_norm_parts, a.ssm_taps, a.ssm_col, a.ssm_mix_col = ssm.norm_groups, ssm.conv, cfg.ssm_col(i), cfg.ssm_mix_col(i)
                a.mix_ld = cfg.mix_cols(i)[1]
            if mem:
                a.mixer, a.heads, a.dim, a.vdim = L.MIXER_MATRIX_MEMORY, mem.heads, mem.dim, mem.vdim
                a.gate_col, a.gate_cap, a.mix_ld = mem.gate_col, mem.gate_cap, cfg.mix_cols(i)[1]
            if att or ssm or mem:
                for n, x in caches[i].items():
                    setattr(a, n, x.data_ptr() if x.numel() else None)
            elif isinstance(m, LatentAttention):
                a.mixer, a.heads, a.dim = L.MIXER_LATENT_ATTN, m.heads, m.dim
                a.rot_dim, a.rot_dims, a.vdim, a.kv_rank = m.rot_dim, m.rot.dims, m.vdim, m.kv_rank
                a.window, a.scale, a.owns_cache = m.window, m.scale, int(m.kv_from is None)
                if "w_expand" in t:
                    a.q_ld, a.v_ld = m.q_ld, m.v_ld
                src = i if m.kv_from is None else m.kv_from
                a.cos_sin = table(m.rot)
            else:
                a.mixer, a.heads, a.dim, a.decay_rank = L.MIXER_GENERAL_DELTA, m.heads, m.dim, m.rank_ld
            if isinstance(spec.mlp, MoeMlp):
                f = spec.mlp
                a.experts, a.top, a.expert_ld, a.glu_limit, a.glu_alpha = f.experts, f.top, f.ff_ld, f.limit, f.alpha
                a.moe_counts_at = counts
                counts += f.experts
                if not f.glu:
                    a.ff_kind, a.ff, a.n_router = L.FF_EXPERTS, f.shared_ld, f.router_rows
            else:
                f = spec.mlp
                a.ff = f.ff_ld if f else 0
                if f and f.glu:
                    a.ff_kind = L.FF_GELU_GLU if f.act == "gelu_glu" else L.FF_CLAMPED_GLU
                    a.glu_limit, a.glu_alpha = f.limit, f.alpha
            for n, x in t.items():
                if n != "vmix":
                    setattr(a, n, x.data_ptr())
            if not (att or ssm or mem):
                a.cache = caches[src].data_ptr()
        self._layers = arr
        s = L.Stack()
        s.n_layers, s.d_model, s.vocab_ld, s.page_size, s.eps = cfg.n_layers, cfg.d_model, cfg.vocab_ld, page_size, cfg.rms_eps
        s.act_dtype = L.DT_F32 if cfg.act_dtype == "float32" else L.DT_BF16
        s.embed, s.lm_head, s.final_norm = w.embed.data_ptr(), w.lm_head.data_ptr(), w.final_norm.data_ptr()
        if w.pos_embed is not None:
            s.pos_embed, s.n_pos = w.pos_embed.data_ptr(), w.pos_embed.shape[0]
        s.embed_scale = cfg.embed_scale
        if w.embed_norm is not None:
            s.embed_norm = w.embed_norm.data_ptr()
        if w.pos_turns is not None:
            s.pos_turns = w.pos_turns.data_ptr()
        s.layers = C.cast(arr, C.POINTER(L.Layer))
        self.struct = s
