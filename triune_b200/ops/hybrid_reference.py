"""PyTorch statements of the heterogeneous-layer operators (:mod:`triune_b200.ops.hybrid`): the executor for CPU tensors.

Same argument conventions as the kernels: sequence rows ``[B * T, ...]``, recurrent states and convolution rings updated
in place or returned, everything that the kernels compute in 32-bit computed in fp32 here (fp64 tensors stay fp64)."""

from __future__ import annotations

from typing import Optional

import torch
import torch.nn.functional as F


def _wide(t: torch.Tensor) -> torch.Tensor:
    return t if t.dtype == torch.float64 else t.float()


def norm_rows(x, w, eps: float, kind: str, out_dtype):
    xf = _wide(x)
    if kind == "layer":
        xf = xf - xf.mean(-1, keepdim=True)
    return (xf * torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps) * w).to(out_dtype)


def activation(x, act: str):
    if act == "relu":
        return F.relu(x)
    if act == "silu":
        return F.silu(x)
    if act == "gelu_tanh":
        return F.gelu(x, approximate="tanh")
    raise ValueError(f"unknown activation {act!r}")


def gated_activation(gate, up, act: str, limit: float, alpha: float):
    """act(gate) * up; ``clamped``: g sigmoid(alpha g) (u + 1) with g at most ``limit`` and u within +-``limit``."""
    if act != "clamped":
        return activation(gate, act) * up
    g = gate.clamp(max=limit)
    return g * torch.sigmoid(alpha * g) * (up.clamp(-limit, limit) + 1)


def add_norm(x, y, bias, post, pre, out_dtype):
    """x += norm(y + bias) in place; -> norm(x), x itself (``pre`` is "rows") or None. Norms are (weight, eps, kind)."""
    yf = _wide(y)
    x += norm_rows(yf if bias is None else yf + bias, *post, x.dtype)
    if pre is None:
        return None
    return x.to(out_dtype) if pre == "rows" else norm_rows(x, *pre, out_dtype)


def gated_norm(y, gate, w, groups: int, eps: float, gate_first: bool, scale: float):
    yf, z = _wide(y), F.silu(_wide(gate))
    if gate_first:
        yf = yf * z
    parts = yf.unflatten(-1, (groups, -1))
    n = parts * torch.rsqrt(parts.pow(2).mean(-1, keepdim=True) + eps)
    if w is not None:
        n = n * (w.view(groups, -1) if w.numel() == yf.shape[-1] else w)
    n = n.flatten(-2)
    return ((n if gate_first else n * z) * scale).to(y.dtype)


def causal_conv(u, w, bias, ring, B: int, T: int, pos: int):
    """-> (silu(conv(u)) [B * T, C], new ring [B, taps, C])."""
    C, taps = w.shape
    x = _wide(u[:, :C]).view(B, T, C)
    past = [ring[:, (pos - j) % taps] if pos - j >= 0 else torch.zeros_like(ring[:, 0]) for j in range(taps - 1, 0, -1)]
    full = torch.cat([torch.stack(past, 1).to(x.dtype), x], 1) if past else x
    y = sum(full[:, j : j + T] * w[:, j] for j in range(taps))
    if bias is not None:
        y = y + bias
    new = ring.clone()
    for t in range(max(0, T - taps), T):
        new[:, (pos + t) % taps] = x[:, t].to(ring.dtype)
    return F.silu(y).reshape(B * T, C).to(u.dtype), new


def recurrent(q, k, v, a, b, A_log, dt_bias, D, state, B: int, T: int, kind: str, unit_eps: float, key_groups: int):
    """S <- g S + k u^T, out = S^T q (+ D v); advances ``state`` in place and returns [B * T, H * Dv]."""
    H, Dk, Dv = state.shape[1:]
    rep = H // key_groups
    q = _wide(q).reshape(B, T, key_groups, Dk)
    k = _wide(k).reshape(B, T, key_groups, Dk)
    vf = _wide(v).reshape(B, T, H, Dv)
    dt = F.softplus(_wide(a).reshape(B, T, H) + dt_bias)
    g = torch.exp(-torch.exp(A_log) * dt)
    if kind == "delta":
        q = q * torch.rsqrt(q.pow(2).sum(-1, keepdim=True) + unit_eps) * Dk ** -0.5
        k = k * torch.rsqrt(k.pow(2).sum(-1, keepdim=True) + unit_eps)
        beta = torch.sigmoid(_wide(b).reshape(B, T, H))
    q, k = q.repeat_interleave(rep, 2), k.repeat_interleave(rep, 2)
    S = state.to(vf.dtype)
    out = torch.empty_like(vf)
    for t in range(T):
        S = g[:, t, :, None, None] * S
        if kind == "delta":
            u = beta[:, t, :, None] * (vf[:, t] - torch.einsum("bhkv,bhk->bhv", S, k[:, t]))
        else:
            u = dt[:, t, :, None] * vf[:, t]
        S = S + k[:, t].unsqueeze(-1) * u.unsqueeze(-2)
        out[:, t] = torch.einsum("bhkv,bhk->bhv", S, q[:, t])
    if kind == "mamba2":
        out = out + D[:, None] * vf
    state.copy_(S)
    return out.reshape(B * T, H * Dv).to(v.dtype)


def head_norm_rotate(x, w: Optional[torch.Tensor], eps: float, freqs: torch.Tensor, pos: int):
    """x [B, T, heads, D] -> per-head RMS norm, then the first 2 * len(freqs) dimensions turned in neighbouring pairs."""
    xf = _wide(x)
    if w is not None:
        xf = xf * torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps) * w
    n = freqs.numel()
    if n:
        ang = (torch.arange(pos, pos + x.shape[1], dtype=torch.float64)[:, None] * freqs).to(freqs.device)
        c, s = torch.cos(ang).to(xf.dtype)[:, None], torch.sin(ang).to(xf.dtype)[:, None]
        r = xf[..., : 2 * n].unflatten(-1, (n, 2))
        u, v = r[..., 0], r[..., 1]
        xf = torch.cat((torch.stack((u * c - v * s, v * c + u * s), -1).flatten(-2), xf[..., 2 * n :]), -1)
    return xf.to(x.dtype)


def sink_attention(q, kc, vc, sink, scale: float, out_scale: float, pos: int, T: int):
    """q [B, T, H, D]; caches [B, G, cap, *] holding pos + T keys -> [B, T, H, E]."""
    H, G, n = q.shape[2], kc.shape[1], pos + T
    k = _wide(kc[:, :, :n, : q.shape[-1]]).repeat_interleave(H // G, 1)
    v = _wide(vc[:, :, :n]).repeat_interleave(H // G, 1)
    s = torch.einsum("bthd,bhnd->bhtn", _wide(q), k) * scale
    mask = torch.arange(n)[None, :] > torch.arange(pos, n)[:, None]
    s = s.masked_fill(mask.to(s.device), float("-inf"))
    if sink is not None:
        s = torch.cat((s, sink.to(s.dtype).view(1, H, 1, 1).expand(s.shape[0], H, T, 1)), -1)
    p = torch.softmax(s, -1)[..., :n]
    return (torch.einsum("bhtn,bhne->bthe", p, v) * out_scale).to(q.dtype)


def rotation_rows(freqs: torch.Tensor, amplitude: float, pos: int, T: int, dtype):
    """[T, 2 * len(freqs)]: cosines, then sines of positions pos .. pos + T - 1."""
    ang = torch.arange(pos, pos + T, dtype=torch.float64, device=freqs.device)[:, None] * freqs
    return (torch.cat((torch.cos(ang), torch.sin(ang)), -1) * amplitude).to(dtype)


def rotate_halves(x, table):
    """x [B, T, heads, D]: dimension i turns with dimension i + n, n = half of the table's columns."""
    xf, n = _wide(x), table.shape[1] // 2
    c, s = table[:, None, :n].to(xf.dtype), table[:, None, n:].to(xf.dtype)
    u, v = xf[..., :n], xf[..., n : 2 * n]
    return torch.cat((u * c - v * s, v * c + u * s, xf[..., 2 * n :]), -1)


def retention(q, k, v, table, decay, state, B: int, T: int):
    """Rotated q, k / sqrt(Dk); S <- decay S + k v^T, out = S^T q; advances ``state`` and returns [B * T, H * Dv]."""
    H, Dk, Dv = state.shape[1:]
    q = rotate_halves(q.reshape(B, T, H, Dk), table)
    k = rotate_halves(k.reshape(B, T, H, Dk), table) * Dk ** -0.5
    vf = _wide(v).reshape(B, T, H, Dv)
    S, g = state.to(vf.dtype), decay.to(vf.dtype)[:, None, None]
    out = torch.empty_like(vf)
    for t in range(T):
        S = g * S + k[:, t].unsqueeze(-1) * vf[:, t].unsqueeze(-2)
        out[:, t] = torch.einsum("bhkv,bhk->bhv", S, q[:, t])
    state.copy_(S)
    return out.reshape(B * T, H * Dv).to(v.dtype)


def latent_rows(rows, w, eps: float, table, rank: int, rank_p: int, B: int, T: int):
    """Projected rows [B * T, rank_p + rot] -> the normed latent and the rotated key part, as the cache holds them."""
    rows = rows.view(B, T, -1)
    out = torch.zeros_like(rows)
    out[..., :rank] = norm_rows(rows[..., :rank], w, eps, "rms", rows.dtype)
    out[..., rank_p:] = rotate_halves(rows[..., None, rank_p:], table)[:, :, 0].to(rows.dtype)
    return out


def latent_attention(q, up, cache, rank_p: int, D: int, Dp: int, E: int, R: int, table, gate, sink, scale: float, pos: int, T: int):
    """q [B, T, H, Dp + Rp]; up [H, Dp + Ep, rank_p]; cache [B, cap, rank_p + Rp] holding pos + T rows -> [B, T, H, E]."""
    n = pos + T
    lat, kr = _wide(cache[:, :n, :rank_p]), _wide(cache[:, :n, rank_p : rank_p + R])
    kv = torch.einsum("bnr,hdr->bhnd", lat.to(up.dtype), up)
    qf, qr = _wide(q[..., :D]), rotate_halves(q[..., Dp : Dp + R], table).to(q.dtype)
    s = (torch.einsum("bthd,bhnd->bhtn", qf, _wide(kv[..., :D])) + torch.einsum("bthr,bnr->bhtn", _wide(qr), kr)) * scale
    mask = torch.arange(n)[None, :] > torch.arange(pos, n)[:, None]
    s = s.masked_fill(mask.to(s.device), float("-inf"))
    H = q.shape[2]
    if sink is not None:
        s = torch.cat((s, sink.to(s.dtype).view(1, H, 1, 1).expand(s.shape[0], H, T, 1)), -1)
    p = torch.softmax(s, -1)[..., :n]
    o = torch.einsum("bhtn,bhne->bthe", p, _wide(kv[..., Dp : Dp + E]))
    if gate is not None:
        o = o * torch.sigmoid(_wide(gate))[..., None]
    return o.to(q.dtype)
