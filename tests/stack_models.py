"""Small random layer-stack models for the tests: config.json dicts of the Bekopel, Lerazen, Merulorn and Vosolorn designs,
their tensors, and model directories.  Weights are scaled so that every mechanism moves the logits: scores spread over
several units, sinks that take a visible share, decays from fast to almost none, all four activation numbers set,
biases and mixed values of the size of what they join.  Routers are decisive: a few coordinates of the stream hold
a code of the token that no layer touches, and the router reads mostly those, so that rounding does not choose
another expert."""
import json

import torch


def attn(heads=3, dim=16, rot_dim=8, vdim=24, kv_rank=32, window=20, base=1e4, scale=None, kv_from=None, ff=96):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "mask": {"size": window},
         "rot": {"base": base, "dims": rot_dim}, "scale": scale or 2.0 * (dim + rot_dim) ** -0.5}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def delta(heads=2, dim=24, ff=96):
    return {"type": "general_delta", "mixer": {"heads": heads, "dim": dim},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=40, limit=1.5):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def gattn(heads=6, kv_heads=3, dim=24, vdim=40, window=20, coef=0.4, every=23, v_mix=True, scale=None, mlp=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window},
                      "q_temp": {"coef": coef, "every": every}, "scale": scale or 2.0 * dim ** -0.5, "v_mix": v_mix}}


def ssm(heads=4, vdim=24, state=20, groups=2, norm_groups=2, conv=4):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}


def glu(ff, limit=1.5):
    return {"kind": "dense", "ff": ff, "limit": limit}


def mamba(mlp=None, **kw):
    return {"type": "mamba2", "mixer": ssm(**kw), "mlp": mlp}


def both(heads=6, kv_heads=3, dim=24, vdim=40, coef=0.4, every=23, scale=None, left_scale=0.8, right_scale=1.3, mlp=None, heads_ssm=4,
         vdim_ssm=24, **kw):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "q_temp": {"coef": coef, "every": every},
            "scale": scale or 2.0 * dim ** -0.5}
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": left, "left_scale": left_scale, "right": ssm(heads_ssm, vdim_ssm, **kw), "right_scale": right_scale}}


def side_config(layers, width=80, vocab=200, eps=1e-5, scale=3.0):
    return {"architecture": "Merulorn", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width,
            "embedding": {"scale": scale}}


def side_tensors(cfg, seed=0):
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s, std=1.0, mean=0.0: torch.randn(*s, generator=g) * std + mean
    d, V = cfg["width"], cfg["vocab"]
    lin = lambda n, k, gain=1.0: rnd(n, k, std=gain * k ** -0.5)
    t = {"embed": rnd(V, d, std=0.5), "final.norm": rnd(d, std=0.2), "head": lin(V, d)}

    def state_space(p, m):
        H, n = m["heads"], m["heads"] * m["vdim"]
        ch = n + 2 * m["groups"] * m["state"]
        # decays from a few tokens to thousands of them
        t.update({p + "in": lin(n + ch + H, d), p + "conv": rnd(ch, m["conv"], std=m["conv"] ** -0.5), p + "conv.b": rnd(ch, std=0.2),
                  p + "dt_bias": torch.linspace(-3.0, 0.5, H), p + "A_log": torch.linspace(-5.0, 0.5, H)[torch.randperm(H, generator=g)],
                  p + "D": rnd(H, std=0.2, mean=0.8), p + "norm": rnd(n, std=0.2, mean=1.0), p + "o": lin(d, n)})
    for i, l in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", l["mixer"], l["mlp"]
        t[p + "norm1"] = rnd(d, std=0.2)
        if l["type"] == "parallel":
            a, q = m["left"], p + "mix.left."
            H, G = a["heads"], a["kv_heads"]
            for n, rows in (("q", H * a["dim"]), ("k", G * a["dim"]), ("v", G * a["vdim"])):
                t[q + n], t[q + n + ".b"] = lin(rows, d), rnd(rows, std=0.5)
            t.update({q + "q.norm": rnd(H * a["dim"], std=0.3, mean=1.0), q + "k.norm": rnd(G * a["dim"], std=0.3, mean=1.0),
                      q + "g": lin(H, d, 2.0), q + "o": lin(d, H * a["vdim"], 1.5)})
            state_space(p + "mix.right.", m["right"])
        else:
            state_space(p + "mix.", m)
        if f:
            t[p + "norm2"] = rnd(d, std=0.2)
            t.update({p + "mlp.gate": lin(f["ff"], d, 1.5), p + "mlp.up": lin(f["ff"], d, 1.5), p + "mlp.down": lin(d, f["ff"])})
    return {n: x.to(torch.bfloat16) for n, x in t.items()}


def parallel_config(layers, width=80, vocab=200, eps=1e-5, positions=512):
    return {"architecture": "Lerazen", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width,
            "max_positions": positions}


def parallel_tensors(cfg, seed=0):
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s, std=1.0, mean=0.0: torch.randn(*s, generator=g) * std + mean
    d, V = cfg["width"], cfg["vocab"]
    lin = lambda n, k, gain=1.0: rnd(n, k, std=gain * k ** -0.5)
    routers = [l["mlp"]["router"]["experts"] for l in cfg["layers"] if l["mlp"] and l["mlp"]["kind"] == "moe"]
    code = max(routers, default=0)               # the last coordinates of the stream

    def out(*s, gain=1.0):                        # output matrices and biases leave the code alone
        w = lin(*s, gain) if len(s) == 2 else rnd(*s, std=0.3)
        w[d - code:] = 0
        return w
    t = {"embed": rnd(V, d), "pos": rnd(cfg["max_positions"], d, std=0.5), "final.norm": rnd(d, std=0.1, mean=1.0), "head": lin(V, d)}
    if code:
        t["pos"][:, d - code:] = 0
        for v in range(V):
            t["embed"][v, d - code:] = torch.linspace(-3, 3, code)[torch.randperm(code, generator=g)]
    for i, l in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", l["mixer"], l["mlp"]
        t[p + "norm1"] = rnd(d, std=0.1, mean=1.0)
        t[p + "norm1"][d - code:] = 1
        H, G = m["heads"], m["kv_heads"]
        for n, rows in (("q", H * m["dim"]), ("k", G * m["dim"]), ("v", G * m["vdim"])):
            t[p + f"mix.{n}"], t[p + f"mix.{n}.b"] = lin(rows, d), rnd(rows, std=0.5)
        t[p + "mix.o"], t[p + "mix.o.b"] = out(d, H * m["vdim"], gain=1.5), out(d)
        if m["v_mix"]:
            t[p + "mix.vmix"] = torch.rand((), generator=g) * 0.5 + 0.25
        if f and f["kind"] == "dense":
            t[p + "mlp.up"], t[p + "mlp.down"] = lin(f["ff"], d), out(d, f["ff"])
        elif f:
            E, n = f["router"]["experts"], f["expert"]["ff"]
            router = lin(E, d, 0.02)
            router[:, d - code:] = 0
            for e, c in enumerate(torch.randperm(code, generator=g)[:E]):
                router[e, d - code + c] = 2.0
            t[p + "mlp.router"] = router
            for e in range(E):
                q = p + f"mlp.e{e}."
                t.update({q + "gate": lin(n, d, 3.0), q + "up": lin(n, d, 3.0), q + "down": out(d, n, gain=1.5)})
    return {n: x.to(torch.bfloat16) for n, x in t.items()}


def pattn(heads=6, kv_heads=3, dim=24, vdim=40, size=20, pool=6, dims=16, base=1e4, scale=None, mlp=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size, "pool": pool},
                      "rot": {"base": base, "dims": dims}, "scale": scale or 2.0 * dim ** -0.5}}


def mlstm(heads=3, dim=24, vdim=40, cap=9.0, mlp=None):
    return {"type": "mlstm", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def plain_moe(experts=6, top=2, ff=40, shared=24):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, **({"shared": {"ff": shared}} if shared else {})}


def output_norm_config(layers, width=80, vocab=200, eps=1e-5, scale=0.4):
    return {"architecture": "Vosolorn", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "logit_scale": scale}


def output_norm_tensors(cfg, seed=0):
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s, std=1.0, mean=0.0: torch.randn(*s, generator=g) * std + mean
    d, V = cfg["width"], cfg["vocab"]
    lin = lambda n, k, gain=1.0: rnd(n, k, std=gain * k ** -0.5)
    routers = [l["mlp"]["router"]["experts"] for l in cfg["layers"] if l["mlp"] and l["mlp"]["kind"] == "moe"]
    # the last coordinates of the stream: a constant, then the code
    code = max(routers, default=0)
    own = code + 1

    def out(*s, gain=1.0):                        # output matrices leave them alone
        w = lin(*s, gain)
        w[d - own:] = 0
        return w
    t = {"embed": rnd(V, d), "embed.norm": rnd(d, std=0.2, mean=1.0), "final.norm": rnd(d, std=0.2, mean=1.0)}
    t["embed.norm"][d - own:] = 1
    t["embed"][:, d - own] = 2
    if code:
        for v in range(V):
            t["embed"][v, d - code:] = torch.linspace(-3, 3, code)[torch.randperm(code, generator=g)]
    step = 12.0 / max(code - 1, 1) / (1 + 2.0 * code / d) ** 0.5        # between two neighbouring logits of a router
    for i, l in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", l["mixer"], l["mlp"]
        for n in ("norm1", "ls1") + (("norm2", "ls2") if f else ()):
            t[p + n] = rnd(d, std=0.2, mean=1.0 if n.startswith("norm") else 0.8)
        H = m["heads"]
        if l["type"] == "attention":
            G = m["kv_heads"]
            t.update({p + "mix.q": lin(H * m["dim"], d), p + "mix.k": lin(G * m["dim"], d), p + "mix.v": lin(G * m["vdim"], d),
                      p + "mix.q.norm": rnd(m["dim"], std=0.4, mean=1.2), p + "mix.k.norm": rnd(m["dim"], std=0.4, mean=1.2),
                      p + "mix.o": out(d, H * m["vdim"], gain=1.5)})
        else:
            n = H * m["vdim"]
            # Forget gates from a few tokens to thousands of them; input gates above and below the running maximum.  Keys and
            # queries share a part that every token has: a head's output, which is divided by its own root mean square, is a sum
            # with positive weights and does not cancel, so that rounding does not choose its sign.
            k, q, same = lin(H * m["dim"], d), lin(H * m["dim"], d), rnd(H * m["dim"])
            k[:, d - own], q[:, d - own] = same, same
            t.update({p + "mix.q": q, p + "mix.k": k, p + "mix.v": lin(n, d), p + "mix.g": lin(n, d),
                      p + "mix.i": lin(H, d, 1.5), p + "mix.i.b": torch.linspace(1.0, -2.0, H), p + "mix.f": lin(H, d),
                      p + "mix.f.b": torch.linspace(0.0, 8.0, H)[torch.randperm(H, generator=g)], p + "mix.norm": rnd(n, std=0.2, mean=1.0),
                      p + "mix.o": out(d, n)})
        if f and f["kind"] == "dense":
            t.update({p + "mlp.gate": lin(f["ff"], d, 1.5), p + "mlp.up": lin(f["ff"], d, 1.5), p + "mlp.down": out(d, f["ff"])})
        elif f:
            E, n = f["router"]["experts"], f["expert"]["ff"]
            router = lin(E, d, 0.02)
            router[:, d - code:] = 0
            for e, c in enumerate(torch.randperm(code, generator=g)[:E]):
                router[e, d - code + c] = 2.0
            # logits stay apart: every other expert is lifted by about a third of the distance between two neighbours
            t.update({p + "mlp.router": router, p + "mlp.router.b": 0.37 * step * (torch.arange(E) % 2)})
            for e in range(E):
                t.update({p + f"mlp.e{e}.up": lin(n, d, 2.0), p + f"mlp.e{e}.down": out(d, n, gain=1.5)})
            if "shared" in f:
                t.update({p + "mlp.shared.up": lin(f["shared"]["ff"], d, 2.0), p + "mlp.shared.down": out(d, f["shared"]["ff"])})
    return {n: x.to(torch.bfloat16) for n, x in t.items()}


def config(layers, width=80, vocab=200, eps=1e-5):
    return {"architecture": "Bekopel", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def tensors(cfg, seed=0, decay_rank=12):
    """name -> bf16 tensor, as a checkpoint of the design holds them."""
    if cfg["architecture"] == "Lerazen":
        return parallel_tensors(cfg, seed)
    if cfg["architecture"] == "Merulorn":
        return side_tensors(cfg, seed)
    if cfg["architecture"] == "Vosolorn":
        return output_norm_tensors(cfg, seed)
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s, std=1.0, mean=0.0: (torch.randn(*s, generator=g) * std + mean).to(torch.bfloat16)
    d, V = cfg["width"], cfg["vocab"]
    lin = lambda n, k, gain=1.0: rnd(n, k, std=gain * k ** -0.5)
    t = {"embed": rnd(V, d), "final.norm": rnd(d, std=0.1, mean=1.0), "head": lin(V, d)}
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if l["mlp"] else ()):
            t[p + n] = rnd(d, std=0.1, mean=1.0)
        p += "mix."
        if l["type"] == "latent_attention":
            H, qk = m["heads"], m["dim"] + m["rot_dim"]
            t.update({p + "q": lin(H * qk, d), p + "uk": lin(H * m["dim"], m["kv_rank"]),
                      p + "uv": lin(H * m["vdim"], m["kv_rank"]), p + "o": lin(d, H * m["vdim"]), p + "sink": rnd(H, mean=1.0)})
            if "kv_from" not in m:
                t.update({p + "dkv": lin(m["kv_rank"] + m["rot_dim"], d), p + "dkv.norm": rnd(m["kv_rank"], std=0.1, mean=1.0)})
        else:
            n = m["heads"] * m["dim"]
            t.update({p + x: lin(n, d) for x in ("r", "k", "v", "g", "a")})
            t.update({p + "a.b": rnd(n, mean=-1.0), p + "w1": lin(decay_rank, d, 2.0), p + "w2": lin(n, decay_rank, 2.0),
                      p + "w0": rnd(n, std=2.0, mean=-3.0), p + "norm": rnd(n, std=0.1, mean=1.0), p + "o": lin(d, n)})
        if l["mlp"]:
            ff = l["mlp"]["ff"]
            q = f"l{i}.mlp."
            t.update({q + "up": lin(ff, d), q + "down": lin(d, ff), q + "act": torch.tensor([0.8, 0.6, -0.4, 0.3]).to(torch.bfloat16)})
    return t


def save(cfg, t, path):
    from safetensors.torch import save_file
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    save_file(t, str(path / "model.safetensors"))
    return path


def stack_config(cfg, t, dtype="bfloat16", name="tiny-stack"):
    import dataclasses

    from byzantine_consensus_llm_agents_b200 import stack
    c = stack.DESIGNS[cfg["architecture"]](cfg, lambda n: tuple(t[n].shape), name)
    return dataclasses.replace(c, act_dtype=dtype)


def engine(cfg, t, dtype="bfloat16", tokens=512, rows=4, tokenizer=None, **kw):
    """Engine over a tiny model; its pages hold `tokens` tokens."""
    from byzantine_consensus_llm_agents_b200.engine import Engine
    from byzantine_consensus_llm_agents_b200.stack import StackWeights
    c = stack_config(cfg, t, dtype)
    w = StackWeights.from_tensors(c, t.__getitem__, torch.device("cuda:0"))
    kw = {"max_model_len": tokens, "max_rows": rows, "prefill_tokens": tokens, "kv_pages": tokens // 16, **kw}
    return Engine(c, w, tokenizer, **kw)
