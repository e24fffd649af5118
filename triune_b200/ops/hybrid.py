"""Operators of heterogeneous-layer models: layer norm of a 32-bit residual stream, gated activations, short causal
convolutions, the matrix-state recurrences (Mamba-2, gated delta rule), softmax attention with head norms, partial
rotation and a sink, and the fused one-token step.

CUDA tensors (bf16 or fp32) run the kernels of ``csrc/hybrid``; CPU tensors run :mod:`triune_b200.ops.hybrid_reference`.
Positions are an ``int`` or, for graph-replayed decoding, a CUDA int64 tensor. No gradients: these operators serve."""

from __future__ import annotations

from typing import Any, Dict, List, Optional, Tuple

import torch
import torch.nn.functional as F

from .. import _ext
from . import _tick, _tma_ok, gemm
from . import hybrid_reference as ref

NORM_KINDS = {"layer": 0, "rms": 1}
ACTS = {"relu": 0, "silu": 1, "gelu_tanh": 2, "identity": 3}
KINDS = {"mamba2": 0, "delta": 1}


def _pos(pos) -> Tuple[int, Optional[torch.Tensor]]:
    return (0, pos) if torch.is_tensor(pos) else (int(pos), None)


def _host_pos(pos) -> int:
    return int(pos.reshape(-1)[0]) if torch.is_tensor(pos) else int(pos)


_STATUS: Dict[Any, torch.Tensor] = {}


def status_word(device) -> torch.Tensor:
    """The device's int32 word that a kernel sets when one of its bounded waits expires (0 = none did)."""
    key = torch.device(device)
    if key not in _STATUS:
        _STATUS[key] = torch.zeros(1, dtype=torch.int32, device=key)
    return _STATUS[key]


def check_status(device) -> None:
    """Raise if a bounded wait of a kernel on ``device`` has expired (reads the word: waits for the device)."""
    word = _STATUS.get(torch.device(device))
    if word is not None and int(word.item()):
        raise RuntimeError(f"a kernel's bounded wait expired (status {int(word.item())}): its results are not valid")


def embed_rows(ids: torch.Tensor, table: torch.Tensor) -> torch.Tensor:
    """Embedding rows as the fp32 residual stream [tokens, width]."""
    ids = ids.reshape(-1)
    if _ext.use_kernels(table):
        _tick()
        return _ext.serving().hybrid_embed_rows(table, ids.long().contiguous())
    e = F.embedding(ids, table)
    return e if e.dtype == torch.float64 else e.float()


def norm_rows(x: torch.Tensor, w: torch.Tensor, eps: float, kind: str, out_dtype: torch.dtype) -> torch.Tensor:
    if _ext.use_kernels(x, w):
        _tick()
        return _ext.serving().hybrid_norm_rows(x, w, eps, NORM_KINDS[kind], out_dtype == torch.float32)
    return ref.norm_rows(x, w, eps, kind, out_dtype)


def linear(x: torch.Tensor, w: torch.Tensor, out_dtype: Optional[torch.dtype] = None) -> torch.Tensor:
    """x @ w^T; bf16 operands go to the tcgen05 GEMM where its alignment rules allow. fp32 operands are exact fp32
    products (never TF32)."""
    if (_ext.use_kernels(x, w) and x.dtype == torch.bfloat16 and w.shape[0] % 8 == 0 and w.shape[1] % 8 == 0
            and _tma_ok(x) and _tma_ok(w)):
        return gemm(x, w, out_dtype=out_dtype or torch.bfloat16)
    if x.is_cuda and x.dtype == torch.bfloat16 and out_dtype == torch.float32:
        return torch.mm(x, w.t(), out_dtype=torch.float32)  # unaligned sizes: library product, fp32 accumulator kept
    y = F.linear(x, w)
    return y if out_dtype is None or y.dtype == torch.float64 else y.to(out_dtype)


def linear_accumulate(x: torch.Tensor, y: torch.Tensor, w: torch.Tensor) -> None:
    """x += y @ w^T on the fp32 residual rows, inside the GEMM's reduce-add epilogue for bf16 operands."""
    if (_ext.use_kernels(y, w) and y.dtype == torch.bfloat16 and w.shape[0] % 8 == 0 and w.shape[1] % 8 == 0
            and _tma_ok(y) and _tma_ok(w)):
        gemm(y, w, x, accumulate=True)
    elif y.dtype == x.dtype:
        x.addmm_(y, w.t())
    elif y.is_cuda and y.dtype == torch.bfloat16:
        x.add_(torch.mm(y, w.t(), out_dtype=torch.float32))
    else:
        x.add_(F.linear(y, w))


def gated_mlp_hidden(h: torch.Tensor, gate_up: torch.Tensor, act: str) -> torch.Tensor:
    """act(h Wg^T) * (h Wu^T) with gate and up as one weight [2F, width]."""
    Fh = gate_up.shape[0] // 2
    if (_ext.use_kernels(h, gate_up) and h.dtype == torch.bfloat16 and act in ("silu", "relu") and Fh % 32 == 0
            and gate_up.shape[1] % 8 == 0 and _tma_ok(h) and _tma_ok(gate_up)):
        out = torch.empty(h.shape[0], Fh, device=h.device, dtype=h.dtype)
        _ext.serving().tc_gemm_swiglu(h, gate_up, out, None, 0 if act == "silu" else 1)  # activation in the GEMM's epilogue
        _tick()
        return out
    gu = linear(h, gate_up)
    if _ext.use_kernels(gu):
        _tick()
        return _ext.serving().hybrid_glu_rows(gu, Fh, ACTS[act])
    return ref.activation(gu[:, :Fh], act) * gu[:, Fh:]


def gated_norm(y, gate, w, out, inner: int, groups: int, eps: float, gate_first: bool, scale: float = 1.0) -> None:
    """RMS norm of ``inner / groups`` wide parts with a silu gate before or after it, times ``scale``, into ``out``."""
    if _ext.use_kernels(y, gate, out):
        _tick()
        _ext.serving().hybrid_gated_norm(y, gate, w, out, inner, groups, eps, 0 if gate_first else 1, scale)
    else:
        out[:, :inner] = ref.gated_norm(y[:, :inner], gate[:, :inner], w, groups, eps, gate_first, scale)


def causal_conv(u, w, bias, ring, B: int, T: int, pos):
    """-> (silu(conv(u)) [B * T, >= C], ring after the last token)."""
    if _ext.use_kernels(u, w):
        h, d = _pos(pos)
        new = torch.empty_like(ring)
        _tick(2)
        return _ext.serving().hybrid_causal_conv(u, w, bias, ring, new, B, T, h, d), new
    return ref.causal_conv(u, w, bias, ring, B, T, _host_pos(pos))


def recurrent(q, k, v, a, b, A_log, dt_bias, D, state, out, B: int, T: int, kind: str, key_groups: int,
              unit_eps: float = 1e-6) -> None:
    """Advances ``state`` [B, H, Dk, Dv] over T tokens in place; outputs into ``out``'s first H * Dv columns."""
    if _ext.use_kernels(q, state, out):
        _tick()
        _ext.serving().hybrid_recurrent(q, k, v, a, b, A_log, dt_bias, D, state, out, B, T, key_groups, KINDS[kind], unit_eps,
                                       True, status_word(out.device))
    else:
        H, Dk, Dv = state.shape[1:]
        n = B * T
        out[:, : H * Dv] = ref.recurrent(q[:n, : key_groups * Dk], k[:n, : key_groups * Dk], v[:n, : H * Dv], a[:n, :H],
                                         None if b is None else b[:n, :H], A_log, dt_bias, D, state, B, T, kind, unit_eps,
                                         key_groups)


def attention(proj, cols, q_w, k_w, eps: float, freqs, sink, kc, vc, out, B: int, T: int, heads: int, dim: int,
              vdim: int, scale: float, out_scale: float, pos) -> None:
    """Head norm, rotation, cache append and causal sink attention of T tokens after ``pos`` earlier ones. ``cols`` are
    the columns of q, k and v in ``proj``; ``kc`` / ``vc`` are [B, groups, capacity, padded head] and receive the new
    keys and values; ``out``'s first heads * vdim columns receive ``out_scale`` times the result."""
    if _ext.use_kernels(proj, kc, out):
        h, d = _pos(pos)
        e = _ext.serving()
        q = e.hybrid_attn_prep(proj, cols[0], cols[1], cols[2], q_w, k_w, eps, freqs, kc, vc, B, T, heads, dim, vdim, h, d)
        e.hybrid_attention(q, kc, vc, sink, out, dim, vdim, scale, out_scale, h, d, status_word(out.device))
        _tick(2)
        return
    p, G = _host_pos(pos), kc.shape[1]
    n = B * T
    q = proj[:n, cols[0] : cols[0] + heads * dim].view(B, T, heads, dim)
    k = proj[:n, cols[1] : cols[1] + G * dim].view(B, T, G, dim)
    v = proj[:n, cols[2] : cols[2] + G * vdim].view(B, T, G, vdim)
    q, k = ref.head_norm_rotate(q, q_w, eps, freqs, p), ref.head_norm_rotate(k, k_w, eps, freqs, p)
    kc[:, :, p : p + T, :dim] = k.transpose(1, 2)
    vc[:, :, p : p + T, :vdim] = v.transpose(1, 2)
    out[:, : heads * vdim] = ref.sink_attention(q, kc, vc[..., :vdim], sink, scale, out_scale, p, T).reshape(n, heads * vdim)


# ---- one-token step --------------------------------------------------------------------------------------------
STEP_MAX_ROWS = 8
STEP_SMEM = 200 * 1024


def step_supported(rows: int, widest_input: int) -> bool:
    """The matrix-vector kernels keep their input rows in shared memory."""
    return rows <= STEP_MAX_ROWS and rows * widest_input * 4 <= STEP_SMEM


def seg_norm(x, w, eps: float, kind: str) -> Dict[str, Any]:
    return {"x": x, "kind": 1, "norm": NORM_KINDS[kind], "w": w, "eps": eps}


def seg_plain(x, scale: float = 1.0) -> Dict[str, Any]:
    return {"x": x, "kind": 0, "scale": scale}


def seg_gated(x, gate, w, groups: int, eps: float, gate_first: bool, scale: float) -> Dict[str, Any]:
    return {"x": x, "kind": 2, "norm": 0 if gate_first else 1, "w": w, "eps": eps, "gate": gate, "groups": groups, "scale": scale}


def gemv(segments: List[Dict[str, Any]], w: torch.Tensor, y: torch.Tensor, epilogue: str = "store", act: str = "relu") -> torch.Tensor:
    """y [B, N] (store / add / gated) from W and input segments formed in the kernel's prologue; fp32 in and out."""
    _ext.serving().hybrid_gemv(segments, w, y, {"store": 0, "add": 1, "glu": 2}[epilogue], ACTS[act])
    _tick()
    return y


def mixer_step(proj: torch.Tensor, recurrent: Optional[Dict[str, Any]], attention: Optional[Dict[str, Any]], pos) -> None:
    """The recurrence and / or attention of one token per sequence as one launch (see ``csrc/hybrid/step.cu``)."""
    h, d = _pos(pos)
    _ext.serving().hybrid_mixer_step(proj, recurrent, attention, h, d)
    _tick()


def step_part_stride(vdim: int) -> int:
    return _ext.serving().hybrid_step_part_stride(vdim)


def step_head_chunk(heads_per_group: int) -> int:
    return _ext.serving().hybrid_step_head_chunk(heads_per_group)
