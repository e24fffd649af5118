"""Plain, slow statements of the mechanisms of heterogeneous-layer models (softmax attention with a sink beside a
state-space mixer, gated delta rule, Mamba-2), one function per mechanism, token by token, in the dtype of their inputs
(tests use float64). Nothing here is shared with the package."""

import math

import torch


def layer_norm(x, w, eps):
    mu = x.mean(-1, keepdim=True)
    var = ((x - mu) ** 2).mean(-1, keepdim=True)
    return (x - mu) / torch.sqrt(var + eps) * w


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(x):
    return x / (1 + torch.exp(-x))


def softplus(x):
    return torch.where(x > 0, x + torch.log1p(torch.exp(-x.abs())), torch.log1p(torch.exp(-x.abs())))


def sigmoid(x):
    return 1 / (1 + torch.exp(-x))


def causal_conv(u, w, bias=None):
    """u [T, C], w [C, taps]; the last column multiplies the current token; silu follows."""
    T, C = u.shape
    taps = w.shape[1]
    out = torch.zeros_like(u)
    for t in range(T):
        acc = torch.zeros(C, dtype=u.dtype) if bias is None else bias.clone()
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                acc = acc + w[:, j] * u[s]
        out[t] = acc
    return silu(out)


def rotate_interleaved(x, pos, dims, base):
    """x [T, H, D]; pairs (2i, 2i+1) of the first ``dims`` dimensions turn by pos * base^(-2i/dims)."""
    out = x.clone()
    for i in range(dims // 2):
        a = pos.to(x.dtype) * base ** (-2.0 * i / dims)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def sink_attention(q, k, v, scale, sink):
    """q [T, H, D], k [T, G, D], v [T, G, E]; every query's denominator also holds exp(sink_h)."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        for t in range(T):
            s = (k[: t + 1, g] @ q[t, h]) * scale
            m = torch.maximum(s.max(), sink[h])
            p = torch.exp(s - m)
            out[t, h] = (p @ v[: t + 1, g]) / (p.sum() + torch.exp(sink[h] - m))
    return out


def mamba2_scan(x, B, C, dt, A_log, D):
    """x [T, H, P], B, C [T, G, N], dt [T, H] (after softplus)."""
    T, H, P = x.shape
    G, N = B.shape[1:]
    S = torch.zeros(H, N, P, dtype=x.dtype)
    gi = torch.arange(H) // (H // G)
    y = torch.zeros_like(x)
    for t in range(T):
        a = torch.exp(-torch.exp(A_log) * dt[t])
        S = a[:, None, None] * S + dt[t][:, None, None] * B[t, gi][:, :, None] * x[t][:, None, :]
        y[t] = (S * C[t, gi][:, :, None]).sum(1) + D[:, None] * x[t]
    return y, S


def delta_scan(q, k, v, g, beta):
    """q, k [T, K, D] unit vectors (q already scaled), v [T, H, E], g (decay in (0, 1]), beta [T, H]."""
    T, H, E = v.shape
    K, D = q.shape[1:]
    ki = torch.arange(H) // (H // K)
    S = torch.zeros(H, D, E, dtype=v.dtype)
    o = torch.zeros_like(v)
    for t in range(T):
        S = g[t][:, None, None] * S
        kt, qt = k[t, ki], q[t, ki]
        u = beta[t][:, None] * (v[t] - (S * kt[:, :, None]).sum(1))
        S = S + kt[:, :, None] * u[:, None, :]
        o[t] = (S * qt[:, :, None]).sum(1)
    return o, S


def attention_mixer(h, W, c, eps):
    T = h.shape[0]
    H, G, D, E = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q = (h @ W["q"].T).view(T, H, D)
    k = (h @ W["k"].T).view(T, G, D)
    v = (h @ W["v"].T).view(T, G, E)
    q, k = unit_rms(q, eps) * W["q.norm"], unit_rms(k, eps) * W["k.norm"]
    pos = torch.arange(T)
    q = rotate_interleaved(q, pos, c["rot"]["dims"], c["rot"]["base"])
    k = rotate_interleaved(k, pos, c["rot"]["dims"], c["rot"]["base"])
    return sink_attention(q, k, v, c["scale"], W["sink"]).reshape(T, H * E) @ W["o"].T


def mamba2_mixer(h, W, c, eps):
    T = h.shape[0]
    H, P, N, G = c["heads"], c["vdim"], c["state"], c["groups"]
    inner = H * P
    z, xbc, dt = (h @ W["in"].T).split([inner, inner + 2 * G * N, H], dim=-1)
    xbc = causal_conv(xbc, W["conv"], W["conv.b"])
    x, B, C = xbc.split([inner, G * N, G * N], dim=-1)
    dt = softplus(dt + W["dt_bias"])
    y, _ = mamba2_scan(x.reshape(T, H, P), B.reshape(T, G, N), C.reshape(T, G, N), dt, W["A_log"], W["D"])
    y = y.reshape(T, inner) * silu(z)
    y = unit_rms(y.view(T, c["norm_groups"], -1), eps).reshape(T, inner) * W["norm"]
    return y @ W["o"].T


def delta_mixer(h, W, c, eps):
    T = h.shape[0]
    H, K, D, E = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q = causal_conv(h @ W["q"].T, W["q.conv"]).view(T, K, D)
    k = causal_conv(h @ W["k"].T, W["k.conv"]).view(T, K, D)
    v = causal_conv(h @ W["v"].T, W["v.conv"]).view(T, H, E)
    q = q / torch.sqrt((q * q).sum(-1, keepdim=True) + 1e-6) * D ** -0.5
    k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    beta = sigmoid(h @ W["b"].T)
    g = torch.exp(-torch.exp(W["A_log"]) * softplus(h @ W["a"].T + W["dt_bias"]))
    o, _ = delta_scan(q, k, v, g, beta)
    o = unit_rms(o, eps) * W["norm"] * silu(h @ W["g"].T).view(T, H, E)
    return o.reshape(T, H * E) @ W["o"].T


def parallel_mixer(h, W, c, eps):
    left = attention_mixer(h, sub(W, "left."), c["left"], eps)
    right = mamba2_mixer(h, sub(W, "right."), c["right"], eps)
    return c["left_scale"] * left + c["right_scale"] * right


MIXERS = {"parallel": parallel_mixer, "delta": delta_mixer, "mamba2": mamba2_mixer}


def sub(W, prefix):
    return {k[len(prefix):]: v for k, v in W.items() if k.startswith(prefix)}


def gated_mlp(h, W):
    return (torch.clamp(h @ W["gate"].T, min=0) * (h @ W["up"].T)) @ W["down"].T


def forward(cfg, W, tokens, dtype=torch.float64, want_layers=False):
    """Logits [T, vocab] of one sequence; ``cfg`` and ``W`` as stored in a model folder."""
    W = {k: v.to(dtype) for k, v in W.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens)]
    layers = []
    for i, spec in enumerate(cfg["layers"]):
        L = sub(W, f"l{i}.")
        x = x + MIXERS[spec["type"]](layer_norm(x, L["norm1"], eps), sub(L, "mix."), spec["mixer"], eps)
        if spec["mlp"] is not None:
            x = x + gated_mlp(layer_norm(x, L["norm2"], eps), sub(L, "mlp."))
        layers.append(x)
    logits = layer_norm(x, W["final.norm"], eps) @ W["head"].T
    return (logits, torch.stack(layers)) if want_layers else logits


def make_config(layers, vocab=70, width=40, eps=1e-5):
    return {"architecture": "Famalorn", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def make_weights(cfg, seed=0, dtype=torch.bfloat16):
    """Random weights of the shapes ``cfg`` implies, rounded to ``dtype``."""
    g = torch.Generator().manual_seed(seed)
    W, d = {}, cfg["width"]

    def lin(name, o, i, gain=1.0):
        W[name] = torch.randn(o, i, generator=g) * gain / math.sqrt(i)

    def vec(name, n, lo, hi):
        W[name] = lo + (hi - lo) * torch.rand(n, generator=g)

    def attn(p, c):
        lin(p + "q", c["heads"] * c["dim"], d)
        lin(p + "k", c["kv_heads"] * c["dim"], d)
        lin(p + "v", c["kv_heads"] * c["vdim"], d)
        vec(p + "q.norm", c["dim"], 0.6, 1.6)
        vec(p + "k.norm", c["dim"], 0.6, 1.6)
        vec(p + "sink", c["heads"], -1.0, 2.0)
        lin(p + "o", d, c["heads"] * c["vdim"])

    def mamba(p, c):
        inner, gn = c["heads"] * c["vdim"], c["groups"] * c["state"]
        lin(p + "in", 2 * inner + 2 * gn + c["heads"], d)
        lin(p + "conv", inner + 2 * gn, c["conv"])
        vec(p + "conv.b", inner + 2 * gn, -0.3, 0.3)
        vec(p + "dt_bias", c["heads"], -3.0, 0.5)
        vec(p + "A_log", c["heads"], -1.0, 1.5)
        vec(p + "D", c["heads"], 0.3, 1.2)
        vec(p + "norm", inner, 0.5, 1.5)
        lin(p + "o", d, inner)

    def delta(p, c):
        for n, r in (("q", c["kv_heads"] * c["dim"]), ("k", c["kv_heads"] * c["dim"]), ("v", c["heads"] * c["vdim"])):
            lin(p + n, r, d)
            lin(p + n + ".conv", r, c["conv"])
        lin(p + "b", c["heads"], d)
        lin(p + "a", c["heads"], d)
        vec(p + "A_log", c["heads"], -2.0, 1.0)
        vec(p + "dt_bias", c["heads"], -3.0, 0.0)
        vec(p + "norm", c["vdim"], 0.5, 1.5)
        lin(p + "g", c["heads"] * c["vdim"], d)
        lin(p + "o", d, c["heads"] * c["vdim"])

    lin("embed", cfg["vocab"], d, math.sqrt(d))
    for i, s in enumerate(cfg["layers"]):
        p = f"l{i}."
        vec(p + "norm1", d, 0.5, 1.5)
        c = s["mixer"]
        if s["type"] == "parallel":
            attn(p + "mix.left.", c["left"])
            mamba(p + "mix.right.", c["right"])
        else:
            {"mamba2": mamba, "delta": delta}[s["type"]](p + "mix.", c)
        if s["mlp"] is not None:
            vec(p + "norm2", d, 0.5, 1.5)
            lin(p + "mlp.gate", s["mlp"]["ff"], d)
            lin(p + "mlp.up", s["mlp"]["ff"], d)
            lin(p + "mlp.down", d, s["mlp"]["ff"])
    vec("final.norm", d, 0.5, 1.5)
    lin("head", cfg["vocab"], d)
    return {k: v.to(dtype) for k, v in W.items()}
