"""ORACLE (test infrastructure only — never imported by the product path).

Plain, slow restatement of the mechanisms that layer-stack designs are made of (Bekopel: latent
attention with a sliding window and a sink, generalized delta rule, PolyNorm feed-forward, norms on
both sides of each sublayer; Lerazen: grouped-query attention with a linear distance bias, a query
temperature and values mixed with an earlier layer's, squared-relu and mixture-of-experts
feed-forwards, parallel sublayers, learned positions; Merulorn: attention with whole-projection query and key
norms and a gate per head beside a selective state-space mixer, clamped gated units, sinusoidal positions;
Vosolorn: attention with rotated values over a window and means of the blocks in front of it, a matrix memory with
exponential gates, gelu units, a mixture of plain experts with a shared one, norms and scales on the sublayers'
outputs only).  One function per mechanism; torch on the CPU, in the dtype of its
inputs (the tests use float64, rounding weights only).  A whole sequence is computed at once, token by
token where there is a recurrence, with no cache: what a cache, a batch or a cut of the prompt could get
wrong is absent here by construction.

Every function works on one sequence; x is [tokens, width].
"""
from __future__ import annotations

import math

import torch


def rms_norm(x, eps, weight=None):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if weight is None else y * weight


def poly_norm(z, coef, eps):
    a, b, c, e = coef
    return a * rms_norm(z, eps) + b * rms_norm(z ** 2, eps) + c * rms_norm(z ** 3, eps) + e


def rotate(x, positions, dims, base):
    """Rotate-half over the first `dims` entries of the last axis; x is [tokens, ..., n]."""
    half = dims // 2
    f = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    ang = positions.to(torch.float64)[:, None] * f[None, :]
    cos, sin = ang.cos().to(x.dtype), ang.sin().to(x.dtype)
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (half,)
    cos, sin = cos.view(shape), sin.view(shape)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], dim=-1)


def window_visible(n, size):
    """[query, key] boolean: 0 <= i - j < size (size 0: plain causal)."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    ok = j <= i
    return ok & (i - j < size) if size else ok


def softmax_with_sink(scores, visible, sink=None):
    """Weights over the visible keys; exp(sink) joins the denominator.  scores [heads, q, k], sink [heads]."""
    s = scores.masked_fill(~visible, -math.inf)
    top = s.max(-1, keepdim=True).values
    if sink is not None:
        top = torch.maximum(top, sink[:, None, None])
    p = torch.exp(s - top)
    den = p.sum(-1, keepdim=True)
    if sink is not None:
        den = den + torch.exp(sink[:, None, None] - top)
    return p / den


def latent_kv(h, w_dkv, norm_w, kv_rank, rot_dims, base, eps, positions):
    """(latent [t, kv_rank], rotated key part [t, rot_dim]) of a layer with its own down-projection."""
    down = h @ w_dkv.T
    return rms_norm(down[:, :kv_rank], eps, norm_w), rotate(down[:, kv_rank:], positions, rot_dims, base)


def latent_attention(h, latent, k_rot, w, m, positions):
    """m: dict(heads, dim, rot_dim, vdim, scale, window, rot_dims, base); w: dict(q, uk, uv, o, sink)."""
    t, H = h.shape[0], m["heads"]
    q = (h @ w["q"].T).view(t, H, m["dim"] + m["rot_dim"])
    qn, qr = q[..., :m["dim"]], rotate(q[..., m["dim"]:], positions, m["rot_dims"], m["base"])
    kn = (latent @ w["uk"].T).view(t, H, m["dim"])
    v = (latent @ w["uv"].T).view(t, H, m["vdim"])
    s = (torch.einsum("ihd,jhd->hij", qn, kn) + torch.einsum("ihd,jd->hij", qr, k_rot)) * m["scale"]
    p = softmax_with_sink(s, window_visible(t, m["window"]), w.get("sink"))
    o = torch.einsum("hij,jhd->ihd", p, v).reshape(t, H * m["vdim"])
    return o @ w["o"].T


def delta_gates(h, w):
    """(decay, removal rate), both [t, heads * dim]."""
    decay = torch.exp(-math.exp(-0.5) * torch.sigmoid(torch.tanh(h @ w["w1"].T) @ w["w2"].T + w["w0"]))
    return decay, torch.sigmoid(h @ w["a"].T + w["a.b"])


def delta_scan(r, k, v, decay, rate, state=None):
    """Token-by-token recurrence; all inputs [t, heads, dim].  Returns (o [t, heads, dim], state)."""
    t, H, D = r.shape
    S = torch.zeros(H, D, D, dtype=r.dtype) if state is None else state.clone()
    out = []
    for i in range(t):
        u = k[i] / torch.sqrt((k[i] ** 2).sum(-1, keepdim=True) + 1e-6)
        seen = torch.einsum("hd,hde->he", u, S)
        S = decay[i][:, :, None] * S - (rate[i] * u)[:, :, None] * seen[:, None, :] + k[i][:, :, None] * v[i][:, None, :]
        out.append(torch.einsum("hde,hd->he", S, r[i]))
    return torch.stack(out), S


def general_delta(h, w, heads, dim, eps):
    t = h.shape[0]
    split = lambda x: x.reshape(t, heads, dim)
    decay, rate = delta_gates(h, w)
    o, _ = delta_scan(split(h @ w["r"].T), split(h @ w["k"].T), split(h @ w["v"].T), split(decay), split(rate))
    o = rms_norm(o, eps).reshape(t, heads * dim) * w["norm"]
    return (o * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def feed_forward(h, w, eps):
    return poly_norm(h @ w["up"].T, [float(c) for c in w["act"]], eps) @ w["down"].T


def squared_relu(z):
    return torch.clamp(z, min=0) ** 2


def dense_ff(h, w):
    return squared_relu(h @ w["up"].T) @ w["down"].T


def head_slopes(heads):
    """Distance slope of every head: 2^-8 for the last one, a geometric series from 2^(-8 / heads)."""
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], dtype=torch.float64)


def query_temperature(positions, coef, every):
    return 1 + coef * torch.log(torch.floor((positions.to(torch.float64) + 1) / every) + 1)


def mix_values(v, v_first, weight):
    return (1 - weight) * v + weight * v_first


def grouped_values(h, w):
    return h @ w["v"].T + w["v.b"]


def grouped_attention(h, v, w, m, positions):
    """m: dict(heads, kv_heads, dim, vdim, scale, window, coef, every); v: the layer's (mixed) values
    [t, kv_heads * vdim]; w: dict(q, q.b, k, k.b, o, o.b)."""
    t, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = (h @ w["q"].T + w["q.b"]).view(t, H, m["dim"])
    q = q * query_temperature(positions, m["coef"], m["every"]).to(q.dtype)[:, None, None]
    k = (h @ w["k"].T + w["k.b"]).view(t, G, m["dim"])
    v = v.view(t, G, m["vdim"])
    mine = torch.arange(H) // (H // G)                      # the key/value head of each query head
    s = torch.einsum("ihd,jhd->hij", q, k[:, mine]) * m["scale"]
    away = (positions[:, None] - positions[None, :]).to(s.dtype)
    s = s - head_slopes(H).to(s.dtype)[:, None, None] * away
    p = softmax_with_sink(s, window_visible(t, m["window"]))
    o = torch.einsum("hij,jhd->ihd", p, v[:, mine]).reshape(t, H * m["vdim"])
    return o @ w["o"].T + w["o.b"]


def route(h, router, top):
    """(experts [t, top], weights [t, top]): the experts with the largest sigmoid scores and those scores."""
    s = torch.sigmoid(h @ router.T)
    best = torch.topk(s, top, dim=-1)
    return best.indices, best.values


def clamped_glu(g, u, limit):
    g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


def mixture(h, w, top, limit):
    """The routing weight scales an expert's input."""
    experts, weights = route(h, w["router"], top)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(experts[t].tolist(), weights[t]):
            x = s * h[t]
            y = clamped_glu(w[f"e{e}.gate"] @ x, w[f"e{e}.up"] @ x, limit)
            out[t] += w[f"e{e}.down"] @ y
    return out


def _lerazen(config, T, tokens, collect):
    eps, pos = float(config["norm"]["eps"]), torch.arange(len(tokens))
    x = T["embed"][torch.as_tensor(tokens, dtype=torch.long)] + T["pos"][pos]
    v_first = None
    for i, layer in enumerate(config["layers"]):
        p, mix, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        sub = lambda kind: {n[len(p + kind) + 1:]: t for n, t in T.items() if n.startswith(p + kind + ".")}
        w = sub("mix")
        h = rms_norm(x, eps, T[p + "norm1"])
        v = grouped_values(h, w)
        if mix.get("v_mix"):
            if v_first is None:
                v_first = v
            else:
                v = mix_values(v, v_first, w["vmix"])
        m = dict(heads=mix["heads"], kv_heads=mix["kv_heads"], dim=mix["dim"], vdim=mix["vdim"], scale=mix["scale"],
                 window=mix["mask"]["size"], coef=mix["q_temp"]["coef"], every=mix["q_temp"]["every"])
        y = grouped_attention(h, v, w, m, pos)
        if mlp and mlp["kind"] == "moe":
            y = y + mixture(h, sub("mlp"), mlp["router"]["top"], mlp["expert"]["limit"])
        elif mlp:
            y = y + dense_ff(h, sub("mlp"))
        x = x + y
        if collect is not None:
            collect.append(x.clone())
    return rms_norm(x, eps, T["final.norm"]) @ T["head"].T


def sinusoid(positions, width):
    """[t, width]: sine and cosine of position * 10000^(-2i / width) in turn."""
    i = torch.arange(width)
    f = torch.tensor([10000.0 ** (-2.0 * (k // 2) / width) for k in i.tolist()], dtype=torch.float64)
    ang = positions.to(torch.float64)[:, None] * f[None, :]
    return torch.where(i % 2 == 0, ang.sin(), ang.cos())


def zero_norm(x, eps, w):
    """RMS norm whose weight is stored around zero."""
    return rms_norm(x, eps, 1 + w)


def gated_attention(h, w, m, positions, eps):
    """m: dict(heads, kv_heads, dim, vdim, scale, coef, every).  Biased projections; query and key norms span all heads;
    one output gate per head."""
    t, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = rms_norm(h @ w["q"].T + w["q.b"], eps, w["q.norm"]).view(t, H, m["dim"])
    k = rms_norm(h @ w["k"].T + w["k.b"], eps, w["k.norm"]).view(t, G, m["dim"])
    v = (h @ w["v"].T + w["v.b"]).view(t, G, m["vdim"])
    q = q * query_temperature(positions, m["coef"], m["every"]).to(q.dtype)[:, None, None]
    mine = torch.arange(H) // (H // G)
    s = torch.einsum("ihd,jhd->hij", q, k[:, mine]) * m["scale"]
    p = softmax_with_sink(s, window_visible(t, 0))
    o = torch.einsum("hij,jhd->ihd", p, v[:, mine]) * torch.sigmoid(h @ w["g"].T)[:, :, None]
    return o.reshape(t, H * m["vdim"]) @ w["o"].T


def causal_conv(x, w, b, before=None):
    """Per channel: y_t = b + sum over taps k of w[:, k] * x_(t - taps + 1 + k); x [t, channels].  `before`: the taps - 1
    inputs ahead of x (zeros at the start of a sequence)."""
    taps = w.shape[1]
    full = torch.cat([x.new_zeros(taps - 1, x.shape[1]) if before is None else before, x])
    y = torch.zeros_like(x)
    for t in range(x.shape[0]):
        y[t] = b
        for k in range(taps):
            y[t] = y[t] + w[:, k] * full[t + k]
    return y


def silu(x):
    return x * torch.sigmoid(x)


def ssm_scan(x, B, C, dt, A_log, D, state=None):
    """x [t, heads, vdim], B and C [t, groups, n], dt [t, heads] (already positive).  Token by token
    S = exp(-exp(A_log) dt) S + dt B x^T,  y = S^T C + D x.  Returns (y, S [heads, n, vdim])."""
    t, H, P = x.shape
    mine = torch.arange(H) // (H // B.shape[1])
    S = torch.zeros(H, B.shape[2], P, dtype=x.dtype) if state is None else state.clone()
    y = []
    for i in range(t):
        keep = torch.exp(-torch.exp(A_log) * dt[i])
        S = keep[:, None, None] * S + dt[i][:, None, None] * B[i][mine][:, :, None] * x[i][:, None, :]
        y.append(torch.einsum("hnp,hn->hp", S, C[i][mine]) + D[:, None] * x[i])
    return torch.stack(y), S


def part_norm(x, parts, eps, w):
    """RMS norm of `parts` equal pieces of the last axis, each by its own root mean square."""
    return rms_norm(x.view(x.shape[0], parts, -1), eps).reshape(x.shape) * w


def mamba2(h, w, m, eps):
    """m: dict(heads, vdim, state, groups, norm_groups); taps from the weight's shape."""
    t, H, P, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    z, xbc, dt = torch.split(h @ w["in"].T, [inner, inner + 2 * G * N, H], dim=-1)
    xbc = silu(causal_conv(xbc, w["conv"], w["conv.b"]))
    x, B, C = torch.split(xbc, [inner, G * N, G * N], dim=-1)
    dt = torch.nn.functional.softplus(dt + w["dt_bias"], threshold=1e9)
    y, _ = ssm_scan(x.view(t, H, P), B.view(t, G, N), C.view(t, G, N), dt, w["A_log"], w["D"])
    return part_norm(y.reshape(t, inner) * silu(z), m["norm_groups"], eps, w["norm"]) @ w["o"].T


def _merulorn(config, T, tokens, collect):
    eps, pos, d = float(config["norm"]["eps"]), torch.arange(len(tokens)), config["width"]
    x = T["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    x = x * config["embedding"]["scale"] + sinusoid(pos, d).to(x.dtype)
    for i, layer in enumerate(config["layers"]):
        p, mix = f"l{i}.", layer["mixer"]
        sub = lambda kind: {n[len(p + kind) + 1:]: t for n, t in T.items() if n.startswith(p + kind + ".")}
        h = zero_norm(x, eps, T[p + "norm1"])
        if layer["type"] == "parallel":
            a = mix["left"]
            m = {**a, "coef": a["q_temp"]["coef"], "every": a["q_temp"]["every"]}
            y = mix["left_scale"] * gated_attention(h, sub("mix.left"), m, pos, eps) \
                + mix["right_scale"] * mamba2(h, sub("mix.right"), mix["right"], eps)
        elif layer["type"] == "mamba2":
            y = mamba2(h, sub("mix"), mix, eps)
        else:
            raise ValueError(f"unknown mixer {layer['type']!r}")
        x = x + y
        if layer.get("mlp"):
            h, w = zero_norm(x, eps, T[p + "norm2"]), sub("mlp")
            x = x + clamped_glu(h @ w["gate"].T, h @ w["up"].T, layer["mlp"]["limit"]) @ w["down"].T
        if collect is not None:
            collect.append(x.clone())
    return zero_norm(x, eps, T["final.norm"]) @ T["head"].T


def rotate_pairs(x, positions, dims, base, back=False):
    """Pairs (2i, 2i + 1) of the first `dims` entries of the last axis turn by position * base^(-2i / dims), or back."""
    y = x.clone()
    for i in range(dims // 2):
        a = positions.to(torch.float64) * float(base) ** (-2.0 * i / dims)
        if back:
            a = -a
        shape = (x.shape[0],) + (1,) * (x.dim() - 2)
        cos, sin = a.cos().to(x.dtype).view(shape), a.sin().to(x.dtype).view(shape)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i], y[..., 2 * i + 1] = u * cos - v * sin, v * cos + u * sin
    return y


def block_means(x, pool):
    """[t // pool, ...]: means of whole blocks of `pool` tokens."""
    n = x.shape[0] // pool
    return x[:n * pool].reshape(n, pool, *x.shape[1:]).mean(1)


def blocks_visible(n, n_blocks, size, pool):
    """[query, block] boolean: the whole block has left the window of `size` tokens."""
    i, b = torch.arange(n)[:, None], torch.arange(n_blocks)[None, :]
    return b * pool + pool - 1 <= i - size


def pooled_attention(h, w, m, positions, eps):
    """m: dict(heads, kv_heads, dim, vdim, scale, size, pool, dims, base).  Query and key norms per head, rotated queries,
    keys and values; tokens of a window and means of the blocks in front of it share one softmax."""
    t, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = rotate_pairs(rms_norm((h @ w["q"].T).view(t, H, m["dim"]), eps, w["q.norm"]), positions, m["dims"], m["base"])
    k = rotate_pairs(rms_norm((h @ w["k"].T).view(t, G, m["dim"]), eps, w["k.norm"]), positions, m["dims"], m["base"])
    v = rotate_pairs((h @ w["v"].T).view(t, G, m["vdim"]), positions, m["vdim"], m["base"])
    ok = window_visible(t, m["size"])
    if m["pool"]:
        kb, vb = block_means(k, m["pool"]), block_means(v, m["pool"])
        ok = torch.cat([ok, blocks_visible(t, kb.shape[0], m["size"], m["pool"])], dim=1)
        k, v = torch.cat([k, kb]), torch.cat([v, vb])
    mine = torch.arange(H) // (H // G)
    s = torch.einsum("ihd,jhd->hij", q, k[:, mine]) * m["scale"]
    o = torch.einsum("hij,jhd->ihd", softmax_with_sink(s, ok), v[:, mine])
    return rotate_pairs(o, positions, m["vdim"], m["base"], back=True).reshape(t, H * m["vdim"]) @ w["o"].T


def memory_gates(h, w, cap):
    """(log input gate, log forget gate), both [t, heads]."""
    soft = lambda z: cap * torch.tanh(z / cap)
    return soft(h @ w["i"].T + w["i.b"]), torch.nn.functional.logsigmoid(soft(h @ w["f"].T + w["f.b"]))


def memory_scan(q, k, v, log_i, log_f, state=None):
    """q (scaled) and k [t, heads, dim], v [t, heads, vdim], gates [t, heads].  Token by token with a running maximum m of
    the gates, which starts at 0.  Returns (o [t, heads, vdim], (S [heads, dim, vdim], n [heads, dim], m [heads]))."""
    t, H, D = k.shape
    S, n, m = (torch.zeros(H, D, v.shape[2], dtype=q.dtype), torch.zeros(H, D, dtype=q.dtype),
               torch.zeros(H, dtype=q.dtype)) if state is None else state
    out = []
    for i in range(t):
        top = torch.maximum(log_f[i] + m, log_i[i])
        keep, add, m = torch.exp(log_f[i] + m - top), torch.exp(log_i[i] - top), top
        S = keep[:, None, None] * S + add[:, None, None] * k[i][:, :, None] * v[i][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[i]
        den = torch.maximum((n * q[i]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append(torch.einsum("hde,hd->he", S, q[i]) / den[:, None])
    return torch.stack(out), (S, n, m)


def matrix_memory(h, w, m, eps):
    """m: dict(heads, dim, vdim, cap)."""
    t, H = h.shape[0], m["heads"]
    q, k = (h @ w["q"].T).view(t, H, -1) * m["dim"] ** -0.5, (h @ w["k"].T).view(t, H, -1)
    log_i, log_f = memory_gates(h, w, m["cap"])
    o, _ = memory_scan(q, k, (h @ w["v"].T).view(t, H, -1), log_i, log_f)
    o = rms_norm(o, eps).reshape(t, H * m["vdim"]) * w["norm"]
    return (o * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def gelu_erf(z):
    return 0.5 * z * (1 + torch.erf(z / math.sqrt(2)))


def route_softmax(h, router, bias, top):
    """(experts [t, top], weights [t, top]): the largest logits and the softmax over just them."""
    best = torch.topk(h @ router.T + bias, top, dim=-1)
    e = torch.exp(best.values - best.values.max(-1, keepdim=True).values)
    return best.indices, e / e.sum(-1, keepdim=True)


def plain_mixture(h, w, top):
    """Experts without gates, weighted outputs, and a shared expert where there is one."""
    experts, weights = route_softmax(h, w["router"], w["router.b"], top)
    unit = lambda x, p: w[p + "down"] @ gelu_erf(w[p + "up"] @ x)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(experts[t].tolist(), weights[t]):
            out[t] += s * unit(h[t], f"e{e}.")
        if "shared.up" in w:
            out[t] += unit(h[t], "shared.")
    return out


def _vosolorn(config, T, tokens, collect):
    eps, pos = float(config["norm"]["eps"]), torch.arange(len(tokens))
    x = rms_norm(T["embed"][torch.as_tensor(tokens, dtype=torch.long)], eps, T["embed.norm"])
    for i, layer in enumerate(config["layers"]):
        p, mix, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        sub = lambda kind: {n[len(p + kind) + 1:]: t for n, t in T.items() if n.startswith(p + kind + ".")}
        if layer["type"] == "attention":
            mask, rot = mix.get("mask") or {"size": 0}, mix["rot"]
            m = {**mix, "size": mask["size"], "pool": mask.get("pool", 0), "dims": rot["dims"], "base": rot["base"]}
            y = pooled_attention(x, sub("mix"), m, pos, eps)
        elif layer["type"] == "mlstm":
            y = matrix_memory(x, sub("mix"), {**mix, "cap": mix["gate_cap"]}, eps)
        else:
            raise ValueError(f"unknown mixer {layer['type']!r}")
        x = x + rms_norm(y, eps, T[p + "norm1"]) * T[p + "ls1"]
        if mlp:
            w = sub("mlp")
            y = plain_mixture(x, w, mlp["router"]["top"]) if mlp["kind"] == "moe" \
                else (gelu_tanh(x @ w["gate"].T) * (x @ w["up"].T)) @ w["down"].T
            x = x + rms_norm(y, eps, T[p + "norm2"]) * T[p + "ls2"]
        if collect is not None:
            collect.append(x.clone())
    return rms_norm(x, eps, T["final.norm"]) @ T["embed"].T * config["logit_scale"]


def forward(config, tensors, tokens, collect=None, dtype=torch.float64):
    """Logits [tokens, vocab] of one sequence.  `config` is the parsed config.json, `tensors` name -> tensor.
    `collect`: a list that receives the residual stream after every layer."""
    eps = float(config["norm"]["eps"])
    T = {n: x.to(dtype) if x.is_floating_point() else x for n, x in tensors.items()}
    if config["architecture"] == "Lerazen":
        return _lerazen(config, T, tokens, collect)
    if config["architecture"] == "Merulorn":
        return _merulorn(config, T, tokens, collect)
    if config["architecture"] == "Vosolorn":
        return _vosolorn(config, T, tokens, collect)
    pos = torch.arange(len(tokens))
    x = T["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    kv = {}
    for i, layer in enumerate(config["layers"]):
        p, mix = f"l{i}.", layer["mixer"]
        sub = lambda kind: {n[len(p + kind) + 1:]: t for n, t in T.items() if n.startswith(p + kind + ".")}
        w = sub("mix")
        h = rms_norm(x, eps, T[p + "norm1"])
        if layer["type"] == "latent_attention":
            rot, src = mix["rot"], mix.get("kv_from")
            if src is None:
                kv[i] = latent_kv(h, w["dkv"], w["dkv.norm"], mix["kv_rank"], rot["dims"], rot["base"], eps, pos)
            c, kr = kv[i if src is None else src]
            m = dict(heads=mix["heads"], dim=mix["dim"], rot_dim=mix["rot_dim"], vdim=mix["vdim"], scale=mix["scale"],
                     window=mix["mask"]["size"], rot_dims=rot["dims"], base=rot["base"])
            y = latent_attention(h, c, kr, w, m, pos)
        elif layer["type"] == "general_delta":
            y = general_delta(h, w, mix["heads"], mix["dim"], eps)
        else:
            raise ValueError(f"unknown mixer {layer['type']!r}")
        x = x + rms_norm(y, eps, T[p + "norm1b"])
        if layer.get("mlp"):
            y = feed_forward(rms_norm(x, eps, T[p + "norm2"]), sub("mlp"), eps)
            x = x + rms_norm(y, eps, T[p + "norm2b"])
        if collect is not None:
            collect.append(x.clone())
    return rms_norm(x, eps, T["final.norm"]) @ T["head"].T
