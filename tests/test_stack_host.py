"""Layer stacks, host side (no GPU): reading a design's configuration, packing weights, the oracle's own
consistency, work lists of ragged steps, pools."""
import numpy as np
import pytest
import torch

from byzantine_consensus_llm_agents_b200 import model as M
from byzantine_consensus_llm_agents_b200 import stack as S
from byzantine_consensus_llm_agents_b200.engine import SlotPool
from byzantine_consensus_llm_agents_b200.executors import Entry, StackExecutor
from oracle import stack_ref as R

import stack_models as SM

CFG = SM.config([SM.delta(), SM.attn(), SM.attn(kv_from=1, window=33, heads=2, ff=None), SM.delta(heads=1, dim=40, ff=None)])


def test_config_comes_from_the_directory(tmp_path):
    t = SM.tensors(CFG)
    c = M.config_from_dir(str(SM.save(CFG, t, tmp_path / "m")))
    assert isinstance(c, S.StackConfig) and M.weights_for(c) is S.StackWeights
    assert set(c.tensor_shapes()) == set(t)
    assert all(tuple(t[n].shape) == s for n, s in c.tensor_shapes().items())
    assert [type(l.mixer).__name__ for l in c.layers] == ["GeneralDelta", "LatentAttention", "LatentAttention", "GeneralDelta"]
    assert c.layers[2].mixer.kv_from == 1 and c.layers[2].mixer.window == 33 and c.layers[2].mlp is None
    assert c.layers[0].mixer.decay_rank == 12          # stated by the checkpoint only
    assert c.has_state and c.max_window == 33
    assert c.kv_bytes_per_token == 2 * (32 + 8)        # one cache for both attention layers
    assert c.state_bytes_per_row == 4 * (2 * 24 * 24 + 40 * 40)


@pytest.mark.parametrize("spoil, words", [
    (lambda c: c["layers"][0].update(type="other"), "unknown mixer"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "unknown feed-forward"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=0), "cannot read"),
    (lambda c: c["layers"][2]["mixer"].update(kv_rank=64), "cannot read"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=10), "rotary"),
    (lambda c: c["layers"][3]["mixer"].update(dim=300), "256 channels"),
])
def test_bad_configurations_are_refused(spoil, words):
    import copy
    c = copy.deepcopy(CFG)
    spoil(c)
    with pytest.raises(ValueError, match=words):
        SM.stack_config(c, SM.tensors(CFG))


def test_wrong_tensor_shape_is_refused():
    t = SM.tensors(CFG)
    c = SM.stack_config(CFG, t)
    t["l1.mix.uk"] = t["l1.mix.uk"][:-1]
    with pytest.raises(ValueError, match="l1.mix.uk"):
        S.StackWeights.from_tensors(c, t.__getitem__, "cpu")


def test_expansion_matrix_builds_keys_and_values():
    m = S.LatentAttention(heads=3, dim=20, rot_dim=12, vdim=40, kv_rank=28, scale=1.0, rot=S.Rotary(1e4, 12))
    uk, uv, row = torch.randn(60, 28), torch.randn(120, 28), torch.randn(5, 40)
    e = (row @ S.StackWeights.expansion(m, uk, uv).T)
    k, v = e[:, :3 * m.q_ld].view(5, 3, m.q_ld), e[:, 3 * m.q_ld:].view(5, 3, m.v_ld)
    assert torch.allclose(k[..., :20].flatten(1), row[:, :28] @ uk.T, atol=1e-5)
    assert torch.equal(k[..., 20:32], row[:, None, 28:].expand(5, 3, 12)) and not k[..., 32:].any()
    assert torch.allclose(v[..., :40].flatten(1), row[:, :28] @ uv.T, atol=1e-5) and not v[..., 40:].any()


def test_packed_rows_are_padded_with_zeros():
    t = SM.tensors(CFG)
    w = S.StackWeights.from_tensors(SM.stack_config(CFG, t), t.__getitem__, "cpu")
    l0, n = w.layers[0], 2 * 24
    assert l0["w_in"].shape[0] % 16 == 0 and torch.equal(l0["w_in"][5 * n:5 * n + 12], t["l0.mix.w1"])
    assert not l0["w_in"][5 * n + 12:].any() and l0["w_decay"].shape == (n, 16) and not l0["w_decay"][:, 12:].any()
    assert "latent_norm" not in w.layers[2] and w.layers[2]["w_in"].shape[0] == 48


# ---------------------------------------------------------------------------------------- parallel layers
PAR = SM.parallel_config([SM.gattn(v_mix=False, mlp=SM.dense(45)), SM.gattn(window=33, mlp=SM.moe(5, 2, 21, 0.75)), SM.gattn(mlp=None)], width=60)


def test_parallel_config_comes_from_the_directory(tmp_path):
    t = SM.tensors(PAR)
    c = M.config_from_dir(str(SM.save(PAR, t, tmp_path / "m")))
    assert isinstance(c, S.StackConfig) and set(c.tensor_shapes()) == set(t)
    assert all(tuple(t[n].shape) == s for n, s in c.tensor_shapes().items())
    assert all(l.parallel for l in c.layers) and c.v_first == 1 and not c.has_state and c.max_window == 33
    assert c.layers[0].mlp == S.DenseMlp(45, "relu2") and c.layers[1].mlp == S.MoeMlp(5, 2, 21, 0.75) and c.layers[2].mlp is None
    m = c.layers[1].mixer
    assert (m.heads, m.kv_heads, m.dim, m.vdim, m.window, m.temp_coef, m.temp_every) == (6, 3, 24, 40, 33, 0.4, 23.0)
    assert c.learned_pos and c.max_pos == PAR["max_positions"] and c.kv_bytes_per_token == 3 * 2 * 3 * (64 + 64)
    w = S.StackWeights.from_safetensors_dir(c, tmp_path / "m", "cpu")
    assert w.pos_embed.shape == (PAR["max_positions"], 60)
    # experts are streamed by the number of them that a step's tokens use
    dense = 2 * (c.decode_weight_bytes(1) - c.decode_weight_bytes(0)) // 2
    assert dense == 2 * 2 * 3 * 21 * 60 and c.decode_weight_bytes(1000) == c.decode_weight_bytes() > c.decode_weight_bytes(1)


def test_parallel_layers_are_packed_side_by_side():
    t = SM.tensors(PAR)
    c = SM.stack_config(PAR, t)
    w = S.StackWeights.from_tensors(c, t.__getitem__, "cpu")
    m, a, b = c.layers[0].mixer, *w.layers[:2]
    col, cols = c.mix_cols(0)
    assert c.qkv_rows(0) % 16 == 0 and a["w_in"].shape == (c.qkv_rows(0) + 48, 60) and a["w_out"].shape == (60, cols)
    assert torch.equal(a["w_in"][m.in_dim - 120:m.in_dim], t["l0.mix.v"]) and not a["w_in"][m.in_dim:c.qkv_rows(0)].any()
    assert torch.equal(a["w_in"][c.qkv_rows(0):c.qkv_rows(0) + 45], t["l0.mlp.up"]) and not a["w_in"][c.qkv_rows(0) + 45:].any()
    assert torch.equal(a["w_out"][:, :240], t["l0.mix.o"]) and torch.equal(a["w_out"][:, col:col + 45], t["l0.mlp.down"])
    assert not a["w_out"][:, col + 45:].any() and "vmix" not in a and "slopes" in a
    assert torch.equal(b["w_in"][m.in_dim:m.in_dim + 5], t["l1.mlp.router"]) and b["w_out"].shape == (60, 240)
    gate, up = b["w_experts_in"][3].view(2, 2, 16, 60).unbind(1)
    for x, n in ((gate, "gate"), (up, "up")):
        assert torch.equal(x.reshape(32, 60)[:21], t[f"l1.mlp.e3.{n}"]) and not x.reshape(32, 60)[21:].any()
    assert torch.equal(b["w_experts_out"][4, :, :21], t["l1.mlp.e4.down"]) and not b["w_experts_out"][:, :, 21:].any()
    assert torch.allclose(a["slopes"], 2.0 ** (-8 * torch.arange(1, 7) / 6))


@pytest.mark.parametrize("spoil, words", [
    (lambda c: c["layers"][0].update(type="other"), "unknown mixer"),
    (lambda c: c["layers"][0]["mlp"].update(kind="other"), "unknown feed-forward"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "key/value heads"),
    (lambda c: c["layers"][2]["mixer"].update(vdim=8), "cannot mix"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=6), "6 of 5 experts"),
])
def test_bad_parallel_configurations_are_refused(spoil, words):
    import copy
    c = copy.deepcopy(PAR)
    spoil(c)
    with pytest.raises(ValueError, match=words):
        SM.stack_config(c, SM.tensors(PAR))


def test_mixed_kinds_of_layers_are_refused():
    g = S.GroupedAttention(2, 1, 8, 8, 1.0)
    with pytest.raises(ValueError, match="parallel"):
        S.StackConfig("x", 16, 16, (S.LayerSpec(S.GeneralDelta(1, 8, 8), parallel=True),))
    with pytest.raises(ValueError, match="not parallel"):
        S.StackConfig("x", 16, 16, (S.LayerSpec(S.GroupedAttention(2, 1, 8, 8, 1.0, gate=True), parallel=True),))
    with pytest.raises(ValueError, match="side by side"):
        S.StackConfig("x", 16, 16, (S.LayerSpec(S.SideBySide(g, S.StateSpace(2, 8, 8, 1, 1, 2))),))
    with pytest.raises(ValueError, match="state-space sizes"):
        S.StackConfig("x", 16, 16, (S.LayerSpec(S.StateSpace(3, 8, 8, 2, 1, 2)),))
    with pytest.raises(ValueError, match="activation"):
        S.StackConfig("x", 16, 16, (S.LayerSpec(g, S.DenseMlp(8), True),))


def test_oracle_temperature_slopes_and_mixing():
    assert torch.allclose(R.head_slopes(4), torch.tensor([2.0 ** -2, 2.0 ** -4, 2.0 ** -6, 2.0 ** -8], dtype=torch.float64))
    t = R.query_temperature(torch.tensor([0, 2, 3, 4, 8]), 2.0, 4)
    assert torch.allclose(t, 1 + 2 * torch.log(torch.tensor([1.0, 1, 2, 2, 3], dtype=torch.float64)))
    v = R.mix_values(torch.tensor([1.0]), torch.tensor([3.0]), 0.25)
    assert v.item() == 1.5


def test_oracle_experts_scale_their_input():
    g = torch.Generator().manual_seed(0)
    w = {f"e{e}.{n}": torch.randn(*s, generator=g, dtype=torch.float64) for e in range(3) for n, s in (("gate", (4, 5)), ("up", (4, 5)), ("down", (5, 4)))}
    w["router"] = torch.tensor([[1.0, 0, 0, 0, 0], [0, 1.0, 0, 0, 0], [0, 0, 1.0, 0, 0]], dtype=torch.float64)
    h = torch.tensor([[0.3, -2.0, 1.1, 0.4, -0.7]], dtype=torch.float64)
    s = torch.sigmoid(h[0, :3])
    y = 0
    for e in (2, 0):
        gate, up = torch.clamp(w[f"e{e}.gate"] @ (s[e] * h[0]), max=0.6), torch.clamp(w[f"e{e}.up"] @ (s[e] * h[0]), -0.6, 0.6)
        y = y + w[f"e{e}.down"] @ (gate * torch.sigmoid(1.702 * gate) * (up + 1))
    assert torch.allclose(R.mixture(h, w, 2, 0.6)[0], y)


def test_preset_resolves_by_name():
    c = M.config_for("bekopel-8b")
    assert isinstance(c, S.StackConfig) and c.d_model == M.PRESETS["qwen3-8b"].d_model
    with pytest.raises(ValueError, match="tensor parallelism"):
        c.shard(2)
    c = M.config_for("lerazen-30b-a3b")
    assert M.config_for("vosolorn-8b").pools == (16,)
    assert M.config_for("merulorn-8b").layers[0].mixer.right.state == 128
    assert c.layers[0].mlp.act == "relu2" and c.layers[1].mlp.experts == 128 and c.v_first == 0


# ---------------------------------------------------------------------------------------- mixers side by side
SIDE = SM.side_config([SM.mamba(mlp=SM.glu(20, 0.5)), SM.both(heads=6, kv_heads=3, dim=7, vdim=9, mlp=None, conv=3), SM.mamba(heads=3, vdim=5, state=7, groups=1, norm_groups=5, conv=1)],
                      width=60, eps=1e-3, scale=2.5)


def test_side_config_comes_from_the_directory(tmp_path):
    t = SM.tensors(SIDE)
    c = M.config_from_dir(str(SM.save(SIDE, t, tmp_path / "m")))
    assert isinstance(c, S.StackConfig) and set(c.tensor_shapes()) == set(t)
    assert all(tuple(t[n].shape) == s for n, s in c.tensor_shapes().items())
    assert c.sinusoid_pos and c.embed_scale == 2.5 and c.norm_offset == 1.0 and c.rms_eps == 1e-3 and c.has_state
    assert c.layers[0].mixer == S.StateSpace(4, 24, 20, 2, 2, 4) and c.layers[0].mlp == S.DenseMlp(20, "clamped_glu", 0.5, 1.702)
    m = c.layers[1].mixer
    assert (m.left_scale, m.right_scale, m.right.conv) == (0.8, 1.3, 3) and c.layers[1].mlp is None
    assert m.left == S.GroupedAttention(6, 3, 7, 9, 2.0 * 7 ** -0.5, 0, 0.4, 23.0, slopes=False, qk_norm=True, gate=True, out_bias=False)
    assert c.kv_bytes_per_token == 2 * 3 * (64 + 64)
    ch = (96 + 80, 96 + 80, 15 + 14)
    assert c.state_bytes_per_row == 4 * (96 * 20 + 3 * ch[0] + 96 * 20 + 2 * ch[1] + 15 * 7)
    w = S.StackWeights.from_safetensors_dir(c, tmp_path / "m", "cpu")
    assert torch.equal(w.final_norm, 1 + t["final.norm"].float()) and torch.equal(w.layers[0]["norm2"], 1 + t["l0.norm2"].float())


def test_side_layers_are_packed_side_by_side():
    t = SM.tensors(SIDE)
    c = SM.stack_config(SIDE, t)
    w = S.StackWeights.from_tensors(c, t.__getitem__, "cpu")
    a, b, m = w.layers[1], w.layers[0], c.layers[1].mixer
    assert c.ssm_col(1) == 96 and m.left.in_dim == 42 + 21 + 27 + 6       # q | k | v | gate
    assert torch.equal(a["w_in"][90:96], t["l1.mix.left.g"]) and torch.equal(a["w_in"][96:96 + m.right.in_dim], t["l1.mix.right.in"])
    assert not a["w_in"][96 + m.right.in_dim:].any() and a["w_in"].shape[0] % 16 == 0
    assert c.ssm_mix_col(1) == 56 and c.mix_cols(1) == (152, 152) and a["w_out"].shape == (60, 152)
    assert torch.equal(a["w_out"][:, :54], t["l1.mix.left.o"]) and not a["w_out"][:, 54:56].any()
    assert torch.equal(a["w_out"][:, 56:], t["l1.mix.right.o"]) and "slopes" not in a and "out_bias" not in a
    assert torch.allclose(a["ssm_norm"], 1.3 * t["l1.mix.right.norm"].float()) and torch.equal(b["ssm_norm"], t["l0.mix.norm"].float())
    assert torch.equal(a["conv_w"][2], t["l1.mix.right.conv"][:, 2].float()) and a["conv_w"].is_contiguous()
    assert torch.allclose(b["decay_rate"], t["l0.mix.A_log"].float().exp())
    gate, up = b["w_up"].view(2, 2, 16, 60).unbind(1)
    for x, n in ((gate, "gate"), (up, "up")):
        assert torch.equal(x.reshape(32, 60)[:20], t[f"l0.mlp.{n}"]) and not x.reshape(32, 60)[20:].any()
    assert torch.equal(b["w_down"][:, :20], t["l0.mlp.down"]) and not b["w_down"][:, 20:].any()
    # sizes of the third layer: one group, output columns padded for the product
    assert c.mix_cols(2) == (16, 16) and c.layers[2].mixer.x_ld == 3 * 8 + 2 * 8


@pytest.mark.parametrize("spoil, words", [
    (lambda c: c["layers"][0].update(type="other"), "unknown mixer"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "unknown feed-forward"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=4), "key/value heads"),
    (lambda c: c["layers"][0]["mixer"].update(groups=3), "state-space sizes"),
    (lambda c: c["layers"][0]["mixer"].update(norm_groups=5), "state-space sizes"),
    (lambda c: c["layers"][0]["mixer"].update(state=257), "state-space sizes"),
])
def test_bad_side_configurations_are_refused(spoil, words):
    import copy
    c = copy.deepcopy(SIDE)
    spoil(c)
    with pytest.raises(ValueError, match=words):
        SM.stack_config(c, SM.tensors(SIDE))


# ---------------------------------------------------------------------------------------- norms on outputs only
POOLED = SM.output_norm_config([SM.pattn(6, 2, 10, 14, 33, 5, 6, mlp=SM.plain_moe(5, 2, 21, 11)), SM.mlstm(3, 7, 9, 4.5, mlp=SM.dense(20)),
                                SM.pattn(2, 2, 8, 8, 7, 40, 8), SM.mlstm(2, 24, 70, mlp=SM.plain_moe(3, 1, 16, 0))], width=60, eps=1e-3, scale=0.3)


def test_pooled_config_comes_from_the_directory(tmp_path):
    t = SM.tensors(POOLED)
    c = M.config_from_dir(str(SM.save(POOLED, t, tmp_path / "m")))
    assert isinstance(c, S.StackConfig) and set(c.tensor_shapes()) == set(t)
    assert all(tuple(t[n].shape) == s for n, s in c.tensor_shapes().items())
    assert c.embed_norm and c.tied_head and c.rms_eps == 1e-3 and c.has_state and c.pools == (5, 40) and c.max_window == 33
    m = c.layers[0].mixer
    assert m == S.GroupedAttention(6, 2, 10, 14, 2.0 * 10 ** -0.5, 33, slopes=False, out_bias=False, in_bias=False, head_norm=True,
                                   rot=S.Rotary(1e4, 6, True), v_rot=S.Rotary(1e4, 14, True), pool=5)
    assert c.layers[1].mixer == S.MatrixMemory(3, 7, 9, 4.5) and c.layers[1].mlp == S.DenseMlp(20, "gelu_glu")
    assert c.layers[0].mlp == S.MoeMlp(5, 2, 21, act="gelu", shared=11) and c.layers[3].mlp.shared == 0 and c.layers[2].mlp is None
    assert c.state_bytes_per_row == 4 * (3 * (10 * 7 + 1) + 2 * (71 * 24 + 2))
    w = S.StackWeights.from_safetensors_dir(c, tmp_path / "m", "cpu")
    # factors join the norms in front of them; the head is the embedding
    assert torch.allclose(w.final_norm, 0.3 * t["final.norm"].float()) and torch.equal(w.embed_norm, t["embed.norm"].float())
    assert torch.equal(w.lm_head[:200], t["embed"]) and "norm1" not in w.layers[0]
    assert torch.allclose(w.layers[0]["norm1b"], t["l0.norm1"].float() * t["l0.ls1"].float())
    assert torch.allclose(w.layers[3]["norm2b"], t["l3.norm2"].float() * t["l3.ls2"].float()) and "norm2b" not in w.layers[2]


def test_memory_and_plain_expert_rows_are_packed():
    t = SM.tensors(POOLED)
    c = SM.stack_config(POOLED, t)
    w = S.StackWeights.from_tensors(c, t.__getitem__, "cpu")
    a, b = w.layers[0], w.layers[1]
    m = c.layers[1].mixer
    assert m.gate_col == 96 and c.in_rows(1) == 112 and b["w_in"].shape == (112, 60)          # 2 * 3 * (7 + 9) rows, then the gates
    assert torch.equal(b["w_in"][21:42], t["l1.mix.k"]) and torch.equal(b["w_in"][69:96], t["l1.mix.g"])
    assert torch.equal(b["w_in"][96:102], torch.cat([t["l1.mix.i"], t["l1.mix.f"]])) and not b["w_in"][102:].any()
    assert torch.equal(b["w_out"][:, :27], t["l1.mix.o"]) and not b["w_out"][:, 27:].any()
    assert torch.equal(b["mem_bias"], torch.cat([t["l1.mix.i.b"], t["l1.mix.f.b"]]).float())
    f = c.layers[0].mlp
    assert (f.router_rows, f.shared_ld, f.ff_ld, f.in_rows) == (16, 16, 32, 32) and a["w_up"].shape == (32, 60)
    assert torch.equal(a["w_up"][:5], t["l0.mlp.router"]) and torch.equal(a["w_up"][16:27], t["l0.mlp.shared.up"])
    assert not a["w_up"][5:16].any() and not a["w_up"][27:].any() and torch.equal(a["w_down"][:, :11], t["l0.mlp.shared.down"])
    assert torch.equal(a["w_experts_in"][3, :21], t["l0.mlp.e3.up"]) and torch.equal(a["w_experts_out"][4, :, :21], t["l0.mlp.e4.down"])
    assert not a["w_experts_in"][:, 21:].any() and not a["w_experts_out"][:, :, 21:].any() and "w_down" not in w.layers[3]


@pytest.mark.parametrize("spoil, words", [
    (lambda c: c["layers"][0].update(type="other"), "unknown mixer"),
    (lambda c: c["layers"][1]["mlp"].update(kind="other"), "unknown feed-forward"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "key/value heads"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=12), "rotary dims 12 of 10"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "pooled blocks"),
    (lambda c: c["layers"][1]["mixer"].update(dim=257), "256 key channels"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=6), "6 of 5 experts"),
])
def test_bad_pooled_configurations_are_refused(spoil, words):
    import copy
    c = copy.deepcopy(POOLED)
    spoil(c)
    with pytest.raises(ValueError, match=words):
        SM.stack_config(c, SM.tensors(POOLED))


def test_pages_of_pooled_blocks():
    from byzantine_consensus_llm_agents_b200.executors import PAGE, block_pages_for
    assert [block_pages_for(n, 5) for n in (0, 4, 5, 5 * PAGE, 5 * PAGE + 4, 5 * PAGE + 5)] == [0, 0, 1, 1, 1, 2]


def test_oracle_matrix_memory_can_be_carried():
    g = torch.Generator().manual_seed(4)
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    q, k, v, i, f = rnd(9, 2, 3), rnd(9, 2, 3), rnd(9, 2, 5), 3 * rnd(9, 2), -rnd(9, 2).abs()
    whole, (S_, n, m) = R.memory_scan(q, k, v, i, f)
    y1, s1 = R.memory_scan(q[:4], k[:4], v[:4], i[:4], f[:4])
    y2, s2 = R.memory_scan(q[4:], k[4:], v[4:], i[4:], f[4:], s1)
    assert torch.allclose(whole, torch.cat([y1, y2])) and all(torch.allclose(a, b) for a, b in zip((S_, n, m), s2))
    # without a running maximum: the plain sums, scaled
    c = torch.cumsum(f, 0)
    w = torch.exp(i + c[-1] - c)[:, :, None]                # weight of token j at the end
    assert torch.allclose(n * m.exp()[:, None], (w * k).sum(0)) and (m >= c[-1]).all()
    nq = ((w * k).sum(0) * q[-1]).sum(-1)
    o = torch.einsum("jhd,jhe,hd->he", w * k, v, q[-1])
    want = o / (torch.maximum(nq.abs(), torch.ones_like(nq)) + 1e-6 * m.exp())[:, None]
    assert torch.allclose(whole[-1], want)
    assert torch.allclose(R.memory_gates(torch.ones(1, 1), {"i": torch.ones(1, 1), "i.b": torch.zeros(1), "f": torch.ones(1, 1) * 50,
                                                            "f.b": torch.zeros(1)}, 2.0)[0], torch.tensor(2 * np.tanh(0.5)).float())


def test_oracle_blocks_rotation_and_experts():
    # 3-token blocks behind a window of 4: block b is seen from position 3b + 6 on
    seen = R.blocks_visible(12, 4, 4, 3)
    assert [int(seen[:, b].float().argmax()) for b in range(2)] == [6, 9] and not seen[:, 2:].any()
    assert R.block_means(torch.arange(8.0)[:, None], 3).flatten().tolist() == [1.0, 4.0]
    x, pos = torch.randn(5, 2, 7, dtype=torch.float64), torch.tensor([0, 3, 4, 90, 7])
    y = R.rotate_pairs(x, pos, 4, 100.0)
    a = 3 * 100.0 ** -0.5
    assert torch.allclose(y[1, 0, 2:4], torch.stack([x[1, 0, 2] * np.cos(a) - x[1, 0, 3] * np.sin(a), x[1, 0, 3] * np.cos(a) + x[1, 0, 2] * np.sin(a)]))
    assert torch.equal(y[..., 4:], x[..., 4:]) and torch.allclose(R.rotate_pairs(y, pos, 4, 100.0, back=True), x)
    e, w = R.route_softmax(torch.tensor([[1.0, 2.0, 0.0]]), torch.eye(3), torch.tensor([0.0, -5.0, 2.0]), 2)
    assert e.tolist() == [[2, 0]] and torch.allclose(w, torch.softmax(torch.tensor([[2.0, 1.0]]), -1))
    z = torch.tensor([-1.5, 0.0, 2.0], dtype=torch.float64)
    assert torch.allclose(R.gelu_erf(z), torch.nn.functional.gelu(z)) and torch.allclose(R.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"))


def test_position_turns_are_the_oracles_frequencies():
    turns = S.position_turns(7, "cpu")
    pos = torch.tensor([0, 1, 17, 90001])
    ang = 2 * np.pi * pos.double()[:, None] * turns[None]
    want = R.sinusoid(pos, 7)
    assert torch.allclose(ang.sin(), want[:, 0::2], atol=1e-9) and torch.allclose(ang.cos()[:, :3], want[:, 1::2], atol=1e-9)


def test_oracle_state_space_can_be_carried():
    g = torch.Generator().manual_seed(3)
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    x, B, C, dt, A, D = rnd(9, 4, 3), rnd(9, 2, 5), rnd(9, 2, 5), rnd(9, 4).abs(), rnd(4), rnd(4)
    whole, s = R.ssm_scan(x, B, C, dt, A, D)
    y1, s1 = R.ssm_scan(x[:4], B[:4], C[:4], dt[:4], A, D)
    y2, s2 = R.ssm_scan(x[4:], B[4:], C[4:], dt[4:], A, D, s1)
    assert torch.allclose(whole, torch.cat([y1, y2])) and torch.allclose(s, s2)
    # head 2 uses group 1; one step by hand
    want = torch.exp(-torch.exp(A[2]) * dt[4, 2]) * s1[2] + dt[4, 2] * B[4, 1][:, None] * x[4, 2][None]
    assert torch.allclose(R.ssm_scan(x[4:5], B[4:5], C[4:5], dt[4:5], A, D, s1)[1][2], want)
    assert torch.allclose(y2[0, 2], want.T @ C[4, 1] + D[2] * x[4, 2])


def test_oracle_convolution_parts_and_heads():
    x, w, b = torch.tensor([[1.0], [2.0], [4.0]]), torch.tensor([[10.0, 1.0]]), torch.tensor([0.5])
    assert R.causal_conv(x, w, b).flatten().tolist() == [1.5, 12.5, 24.5]
    assert R.causal_conv(x[1:], w, b, x[:1]).flatten().tolist() == [12.5, 24.5]
    y = R.part_norm(torch.tensor([[3.0, 4.0, 0.0, 2.0]]), 2, 0.0, torch.tensor([1.0, 1.0, 1.0, 5.0]))
    assert torch.allclose(y, torch.tensor([[3.0, 4.0, 0.0, 10.0]]) / torch.tensor([12.5 ** 0.5] * 2 + [2.0 ** 0.5] * 2))
    assert torch.allclose(R.zero_norm(torch.tensor([[3.0, 4.0]]), 0.0, torch.tensor([0.0, -1.0])), torch.tensor([[3.0 / 12.5 ** 0.5, 0.0]]))


# ---------------------------------------------------------------------------------------- work lists
def _exec(history=10, D_max=4, K_max=1 << 20):
    x = StackExecutor.__new__(StackExecutor)
    x.history, x.D_max, x.K_max, x.T_max = history, D_max, K_max, 512
    return x


def test_plan_separates_portions_from_single_tokens():
    rows = np.arange(3 * 20, dtype=np.int32).reshape(3, 20)
    p = _exec().plan([Entry([7], 40, rows[0], 2, [0]), Entry(list(range(150)), 25, rows[1], 0, [0, 149]),
                      Entry([1, 2], 0, rows[2], 1, [])])
    a = p.arrays
    assert p.T == 153 and p.n_seqs == 3 and p.n_want == 3 and list(a["rows"]) == [0, 1, 150]
    assert list(a["seq_start"]) == [0, 1, 151, 153] and list(a["state_slots"]) == [2, 0, 1]
    assert list(a["singles"]) == [0, 151, 152] and p.extra["context"] == 41
    t = a["tiles"].reshape(-1, 8)
    assert [list(x[:5]) for x in t] == [[1, 25, 128, 0, 15], [129, 153, 22, 0, 15]]
    keys = np.arange(15, 175)                       # window history of ten keys, then the portion itself
    assert list(a["gather"]) == list(rows[1][keys // 16] * 16 + keys % 16)
    assert list(a["slots"][:2]) == [rows[0][2] * 16 + 8, rows[1][1] * 16 + 9]


def test_plan_keeps_a_place_for_every_single_token():
    rows = np.zeros((4, 20), np.int32)
    p = _exec(D_max=4).plan([Entry([1, 2, 3], 0, rows[i], i) for i in range(2)] + [Entry([1], 0, rows[i], i) for i in (2, 3)])
    assert len(p.arrays["singles"]) <= 4 and p.extra["n_tiles"] == 2


def test_slot_pool_reuses_and_refuses():
    p = SlotPool(2)
    a, b = p.alloc(), p.alloc()
    with pytest.raises(MemoryError):
        p.alloc()
    p.release(a)
    assert p.alloc() == a and a != b


# ---------------------------------------------------------------------------------------- oracle
def test_oracle_window_and_sink():
    v = R.window_visible(6, 3)
    assert v[5].tolist() == [False, False, False, True, True, True] and v[0].tolist() == [True] + [False] * 5
    s = torch.zeros(1, 2, 2, dtype=torch.float64)
    p = R.softmax_with_sink(s, R.window_visible(2, 2), torch.tensor([0.0], dtype=torch.float64))
    assert torch.allclose(p[0], torch.tensor([[0.5, 0.0], [1 / 3, 1 / 3]], dtype=torch.float64))


def test_oracle_delta_state_can_be_carried():
    g = torch.Generator().manual_seed(1)
    r, k, v = (torch.randn(9, 2, 5, generator=g, dtype=torch.float64) for _ in range(3))
    w, a = (torch.rand(9, 2, 5, generator=g, dtype=torch.float64) for _ in range(2))
    whole, s = R.delta_scan(r, k, v, w, a)
    o1, s1 = R.delta_scan(r[:4], k[:4], v[:4], w[:4], a[:4])
    o2, s2 = R.delta_scan(r[4:], k[4:], v[4:], w[4:], a[4:], s1)
    assert torch.allclose(whole, torch.cat([o1, o2])) and torch.allclose(s, s2)
    # one step by hand: removal uses the unit key and the old state
    u = k[4] / torch.sqrt((k[4] ** 2).sum(-1, keepdim=True) + 1e-6)
    seen = (u[:, :, None] * s1).sum(1)
    want = w[4][:, :, None] * s1 - (a[4] * u)[:, :, None] * seen[:, None] + k[4][:, :, None] * v[4][:, None]
    assert torch.allclose(R.delta_scan(r[4:5], k[4:5], v[4:5], w[4:5], a[4:5], s1)[1], want)


def test_oracle_rotation_turns_pairs():
    x = torch.tensor([[1.0, 0.0, 0.0, 2.0, 9.0]], dtype=torch.float64)
    y = R.rotate(x, torch.tensor([3]), 4, 100.0)
    c, s = np.cos(3.0), np.sin(3.0)
    c2, s2 = np.cos(0.3), np.sin(0.3)
    assert torch.allclose(y, torch.tensor([[c, -2 * s2, s, 2 * c2, 9.0]], dtype=torch.float64))
