"""Plain, slow statements of the mechanisms of Bubitar models (multi-head latent attention with a sink, a gate and shared
latents; retention; clamped gated feed-forward with biases; a token table read by every layer; norms around every
sublayer), one function per mechanism, token by token, in the dtype of their inputs (tests use float64). Nothing here is
shared with the package."""

import math

import torch

from hybrid_oracle import sigmoid, silu, sub, unit_rms


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def rotation_table(rot):
    """-> (turn per position of every pair, factor of sine and cosine)."""
    n, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    s = rot.get("scaling")
    if s is None:
        return f, 1.0
    border = lambda turns: n * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(border(s["fast"])), 0), min(math.ceil(border(s["slow"])), n - 1)
    out = []
    for i, x in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(x / s["factor"] * r + x * (1 - r))
    return out, 0.1 * math.log(s["factor"]) + 1


def rotate_halves(x, pos, rot):
    """x [T, heads, D]: dimension i of the first rot dims turns with dimension i + dims / 2."""
    out, half = x.clone(), rot["dims"] // 2
    f, amp = rotation_table(rot)
    for i in range(half):
        a = pos.to(x.dtype) * f[i]
        c, s = (torch.cos(a) * amp)[:, None], (torch.sin(a) * amp)[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * c - v * s
        out[..., i + half] = v * c + u * s
    return out


def latent_rows(h, W, c, eps):
    """What a position leaves behind: the normed latent [T, kv_rank] and the turned key part [T, rot_dim]."""
    r = c["kv_rank"]
    z = h @ W["dkv"].T
    lat = rms_norm(z[:, :r], W["dkv.norm"], eps)
    return lat, rotate_halves(z[:, None, r:], torch.arange(h.shape[0]), {**c["rot"], "dims": c["rot_dim"]})[:, 0]


def latent_core(q, qr, lat, krot, uk, uv, gate, sink, scale):
    """q [T, H, D], qr [T, H, R] turned, lat [T, rank], krot [T, R] turned, uk [H, D, rank], uv [H, E, rank], gate [T, H] or
    None, sink [H] or None -> [T, H, E]"""
    T, H, _ = q.shape
    out = torch.zeros(T, H, uv.shape[1], dtype=q.dtype)
    for n in range(H):
        k, v = lat @ uk[n].T, lat @ uv[n].T
        for t in range(T):
            s = (k[: t + 1] @ q[t, n] + krot[: t + 1] @ qr[t, n]) * scale
            m = s.max() if sink is None else torch.maximum(s.max(), sink[n])
            p = torch.exp(s - m)
            total = p.sum() if sink is None else p.sum() + torch.exp(sink[n] - m)
            out[t, n] = (p @ v[: t + 1]) / total * (1 if gate is None else gate[t, n])
    return out


def latent_attention(h, W, c, lat, krot):
    T = h.shape[0]
    H, D, R, E, rank = c["heads"], c["dim"], c["rot_dim"], c["vdim"], c["kv_rank"]
    q = (h @ W["q"].T).view(T, H, D + R)
    qr = rotate_halves(q[..., D:], torch.arange(T), {**c["rot"], "dims": R})
    out = latent_core(q[..., :D], qr, lat, krot, W["uk"].view(H, D, rank), W["uv"].view(H, E, rank), sigmoid(h @ W["g"].T), W["sink"], c["scale"])
    return out.reshape(T, H * E) @ W["o"].T


def retention_scan(q, k, v, decay):
    """q, k [T, H, D] turned and scaled, v [T, H, E], decay [H]."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=v.dtype)
    o = torch.zeros_like(v)
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = (S * q[t][:, :, None]).sum(1)
    return o, S


def retention(h, W, c, eps):
    T = h.shape[0]
    H, D, E = c["heads"], c["dim"], c["vdim"]
    pos = torch.arange(T)
    q = rotate_halves((h @ W["q"].T).view(T, H, D), pos, c["rot"])
    k = rotate_halves((h @ W["k"].T).view(T, H, D), pos, c["rot"]) * D ** -0.5
    o, _ = retention_scan(q, k, (h @ W["v"].T).view(T, H, E), torch.tensor(c["decay"], dtype=h.dtype))
    return (unit_rms(o, eps).reshape(T, H * E) * silu(h @ W["g"].T)) @ W["o"].T


def clamped_mlp(h, W, limit):
    g = torch.clamp(h @ W["gate"].T + W["gate.b"], max=limit)
    u = torch.clamp(h @ W["up"].T + W["up.b"], min=-limit, max=limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ W["down"].T + W["down.b"]


def token_side(x, e, W, eps):
    y = (gelu_tanh(x @ W["gate"].T) * e) @ W["proj"].T
    return unit_rms(y, eps) * W["norm"]


def forward(cfg, W, tokens, dtype=torch.float64, want_layers=False):
    """Logits [T, vocab] of one sequence; ``cfg`` and ``W`` as stored in a model folder."""
    W = {k: v.to(dtype) for k, v in W.items()}
    eps, dim = cfg["norm"]["eps"], cfg["token_side"]["dim"]
    toks = torch.as_tensor(tokens)
    x = W["embed"][toks]
    layers, kept = [], {}
    for i, spec in enumerate(cfg["layers"]):
        L, c = sub(W, f"l{i}."), spec["mixer"]
        h, M = rms_norm(x, L["norm1"], eps), sub(L, "mix.")
        if spec["type"] == "retention":
            y = retention(h, M, c, eps)
        else:
            if c.get("kv_from") is None:
                kept[i] = latent_rows(h, M, c, eps)
            y = latent_attention(h, M, c, *kept[i if c.get("kv_from") is None else c["kv_from"]])
        x = x + rms_norm(y, L["norm1b"], eps)
        if spec["mlp"] is not None:
            y = clamped_mlp(rms_norm(x, L["norm2"], eps), sub(L, "mlp."), spec["mlp"]["limit"])
            x = x + rms_norm(y, L["norm2b"], eps)
        x = x + token_side(x, W["side.embed"][toks][:, i * dim : (i + 1) * dim], sub(L, "side."), eps)
        layers.append(x)
    logits = rms_norm(x, W["final.norm"], eps) @ W["head"].T
    return (logits, torch.stack(layers)) if want_layers else logits


def make_config(layers, vocab=70, width=40, eps=1e-5, side=6):
    return {"architecture": "Bubitar", "layers": layers, "norm": {"eps": eps}, "token_side": {"dim": side}, "vocab": vocab, "width": width}


def make_weights(cfg, seed=0, dtype=torch.bfloat16):
    """Random weights of the shapes ``cfg`` implies, rounded to ``dtype``."""
    g = torch.Generator().manual_seed(seed)
    W, d, dim = {}, cfg["width"], cfg["token_side"]["dim"]

    def lin(name, o, i, gain=1.0):
        W[name] = torch.randn(o, i, generator=g) * gain / math.sqrt(i)

    def vec(name, n, lo, hi):
        W[name] = lo + (hi - lo) * torch.rand(n, generator=g)

    lin("embed", cfg["vocab"], d, math.sqrt(d))
    lin("side.embed", cfg["vocab"], dim * len(cfg["layers"]), math.sqrt(dim * len(cfg["layers"])))
    for i, s in enumerate(cfg["layers"]):
        p, c, m = f"l{i}.", s["mixer"], f"l{i}.mix."
        H, D, E = c["heads"], c["dim"], c["vdim"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if s["mlp"] is not None else ()):
            vec(p + n, d, 0.5, 1.5)
        lin(m + "o", d, H * E)
        if s["type"] == "retention":
            for n, rows in (("q", H * D), ("k", H * D), ("v", H * E), ("g", H * E)):
                lin(m + n, rows, d)
        else:
            lin(m + "q", H * (D + c["rot_dim"]), d, 1.5)
            if c.get("kv_from") is None:
                lin(m + "dkv", c["kv_rank"] + c["rot_dim"], d, 1.5)
                vec(m + "dkv.norm", c["kv_rank"], 0.6, 1.6)
            lin(m + "uk", H * D, c["kv_rank"], 1.5)
            lin(m + "uv", H * E, c["kv_rank"])
            vec(m + "sink", H, -1.0, 2.0)
            lin(m + "g", H, d)
        if s["mlp"] is not None:
            F = s["mlp"]["ff"]
            for n, rows, cols in (("gate", F, d), ("up", F, d), ("down", d, F)):
                lin(p + "mlp." + n, rows, cols, 1.5)
                vec(f"{p}mlp.{n}.b", rows, -0.5, 0.5)
        lin(p + "side.gate", dim, d)
        lin(p + "side.proj", d, dim)
        vec(p + "side.norm", d, 0.3, 1.0)
    vec("final.norm", d, 0.5, 1.5)
    lin("head", cfg["vocab"], d)
    return {k: v.to(dtype) for k, v in W.items()}
