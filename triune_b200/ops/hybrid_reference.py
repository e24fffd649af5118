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


def gated_norm(y, gate, w, groups: int, eps: float, gate_first: bool, scale: float):
    yf, z = _wide(y), F.silu(_wide(gate))
    if gate_first:
        yf = yf * z
    parts = yf.unflatten(-1, (groups, -1))
    n = parts * torch.rsqrt(parts.pow(2).mean(-1, keepdim=True) + eps)
    wp = w.view(groups, -1) if w.numel() == yf.shape[-1] else w
    n = (n * wp).flatten(-2)
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
