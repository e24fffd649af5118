"""Operators of heterogeneous-layer models: layer norm of a 32-bit residual stream, gated activations, short causal
convolutions, the matrix-state recurrences (Mamba-2, gated delta rule, retention), softmax attention with head norms,
partial rotation and a sink, multi-head latent attention, and the fused one-token step.

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
ACTS = {"relu": 0, "silu": 1, "gelu_tanh": 2, "identity": 3, "clamped": 4}
KINDS = {"mamba2": 0, "delta": 1, "retention": 2}
GLU_EPILOGUES = {"silu": 0, "relu": 1, "clamped": 2}  # gated activations that the GEMM epilogue has


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


def gated_mlp_hidden(h: torch.Tensor, gate_up: torch.Tensor, act: str, bias: Optional[torch.Tensor] = None, limit: float = 0.0,
                     alpha: float = 0.0) -> torch.Tensor:
    """act(h Wg^T) * (h Wu^T) with gate and up as one weight [2F, width] and one fp32 ``bias`` [2F]; ``clamped`` is
    g sigmoid(alpha g) (u + 1) with g at most ``limit`` and u within +-``limit``."""
    Fh = gate_up.shape[0] // 2
    if (_ext.use_kernels(h, gate_up) and h.dtype == torch.bfloat16 and act in GLU_EPILOGUES and Fh % 32 == 0
            and gate_up.shape[1] % 8 == 0 and _tma_ok(h) and _tma_ok(gate_up)):
        out = torch.empty(h.shape[0], Fh, device=h.device, dtype=h.dtype)
        # activation in the GEMM's epilogue
        _ext.serving().tc_gemm_swiglu(h, gate_up, out, None, GLU_EPILOGUES[act], bias, limit, alpha)
        _tick()
        return out
    gu = linear(h, gate_up)
    if _ext.use_kernels(gu):
        _tick()
        return _ext.serving().hybrid_glu_rows(gu, Fh, ACTS[act], bias, limit, alpha)
    if bias is not None:
        gu = gu + bias.to(gu.dtype)
    return ref.gated_activation(gu[:, :Fh], gu[:, Fh:], act, limit, alpha)


def token_side_hidden(gate: torch.Tensor, table: torch.Tensor, ids: torch.Tensor, col0: int, act: str = "gelu_tanh") -> torch.Tensor:
    """act(gate) [rows, dim] times columns col0 .. col0 + dim of each row's token in ``table``."""
    if _ext.use_kernels(gate, table):
        _tick()
        return _ext.serving().hybrid_side_rows(gate, table, ids, col0, ACTS[act])
    return ref.activation(gate, act) * F.embedding(ids.reshape(-1), table)[:, col0 : col0 + gate.shape[1]]


def add_norm(x: torch.Tensor, y: torch.Tensor, bias, post, pre, out_dtype: torch.dtype):
    """x += norm(y + bias) on the fp32 residual rows and, in the same pass, the next sublayer's input: -> norm(x), x itself
    (``pre`` is "rows") or None. Norms are (weight, eps, kind)."""
    if _ext.use_kernels(x, y):
        _tick()
        w, eps, kind = pre if isinstance(pre, tuple) else (None, 0.0, "rms")
        out = None if pre is None else torch.empty(x.shape, device=x.device, dtype=out_dtype)
        _ext.serving().hybrid_add_norm(x, y, bias, post[0], post[1], NORM_KINDS[post[2]], out, w, eps, NORM_KINDS[kind])
        return out
    return ref.add_norm(x, y, bias, post, pre, out_dtype)


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


def rotation_rows(freqs: torch.Tensor, amplitude: float, pos, T: int, dtype=torch.float32) -> torch.Tensor:
    """Cosines, then sines (times ``amplitude``) of the turns of positions pos .. pos + T - 1: [T, 2 * len(freqs)]."""
    if freqs.is_cuda and _ext.use_kernels(freqs):
        h, d = _pos(pos)
        _tick()
        return _ext.serving().hybrid_rotation_rows(freqs, amplitude, T, h, d)
    return ref.rotation_rows(freqs, amplitude, _host_pos(pos), T, torch.float64 if dtype == torch.float64 else torch.float32)


def retention(q, k, v, table, decay, state, out, B: int, T: int) -> None:
    """Linear attention with a fixed ``decay`` per head (fp64 [H]) on rotated queries and keys; advances ``state``
    [B, H, Dk, Dv] over T tokens in place; outputs into ``out``'s first H * Dv columns."""
    H, Dk, Dv = state.shape[1:]
    if _ext.use_kernels(q, state, out):
        _tick()
        _ext.serving().hybrid_retention(q, k, v, table, decay, state, out, B, T, True, status_word(out.device))
    else:
        n = B * T
        out[:, : H * Dv] = ref.retention(q[:n, : H * Dk], k[:n, : H * Dk], v[:n, : H * Dv], table, decay, state, B, T)


LATENT_BYTES = 2 << 30  # keys and values that a prompt expands at a time; longer contexts go in groups of heads


def latent_attention(proj, col_q: int, col_g: Optional[int], own: Optional[Tuple[int, torch.Tensor, float]], cache, up, table, sink, out,
                     B: int, T: int, rank: int, D: int, R: int, E: int, scale: float, out_scale: float, pos) -> None:
    """Causal attention over latents, keys and values expanded per head. ``proj`` holds queries at ``col_q`` (heads of
    [pad8(D) | pad8(R)], the second part rotated here, in place) and gate logits at ``col_g`` (or None); ``up``
    [H, pad8(D) + pad8(E), pad8(rank)] expands a latent into a head's key and value. ``own`` = (column, norm weight, eps)
    of this layer's latents, which are normed, rotated and appended to ``cache`` [B, 1, capacity, pad8(rank) + pad8(R)];
    None reads what another layer has appended."""
    H, rank_p = up.shape[0], up.shape[2]
    Dp = -(-D // 8) * 8
    Rp = cache.shape[3] - rank_p
    if _ext.use_kernels(proj, cache, out):
        h, d = _pos(pos)
        e = _ext.serving()
        ocol, ow, oeps = own if own is not None else (-1, None, 0.0)
        e.hybrid_latent_prep(proj, col_q, H, Dp, Rp, ocol, ow, oeps, cache, rank, rank_p, R, table, B, T, h, d)
        n = cache.shape[2] if d is not None else h + T  # a position on the device: every row of the cache, masked
        per = max(1, min(H, LATENT_BYTES // (B * n * up.shape[1] * up.element_size())))
        rows = cache[:, 0, :n, :rank_p]
        for g in range(0, H, per):
            w = up[g : g + per]
            kv = linear(rows, w.reshape(-1, rank_p))
            e.hybrid_latent_attention(proj, col_q, -1 if col_g is None else col_g, cache, kv, sink, out, g, w.shape[0], B, T, Dp, Rp,
                                      rank_p, D, R, E, scale, out_scale, h, d, status_word(out.device))
        _tick(1 + -(-H // per))
        return
    p, n = _host_pos(pos), B * T
    if own is not None:
        c, w, eps = own
        cache[:, 0, p : p + T] = ref.latent_rows(proj[:n, c : c + rank_p + Rp], w, eps, table, rank, rank_p, B, T)
    q = proj[:n, col_q : col_q + H * (Dp + Rp)].view(B, T, H, Dp + Rp)
    gate = None if col_g is None else proj[:n, col_g : col_g + H].view(B, T, H)
    o = ref.latent_attention(q, up, cache[:, 0], rank_p, D, Dp, E, R, table, gate, sink, scale, p, T)
    out[:, : H * E] = (o * out_scale).reshape(n, H * E)


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


def seg_added(x, y, bias, post, pre, x_out) -> Dict[str, Any]:
    """norm(x + post_norm(y + bias)), or the sum itself without ``pre``; the sum also goes to ``x_out`` (or nowhere)."""
    w, eps, kind = pre if pre is not None else (None, 0.0, "rms")
    return {"x": x, "kind": 3, "y": y, "bias": bias, "post_w": post[0], "post_eps": post[1], "post_norm": NORM_KINDS[post[2]], "w": w,
            "eps": eps, "norm": NORM_KINDS[kind], "x_out": x_out}


def gemv(segments: List[Dict[str, Any]], w: torch.Tensor, y: torch.Tensor, epilogue: str = "store", act: str = "relu",
         bias: Optional[torch.Tensor] = None, limit: float = 0.0, alpha: float = 0.0, side=None) -> torch.Tensor:
    """y [B, N] (store / add / gated / act times a token's table row) from W and input segments formed in the kernel's
    prologue; fp32 in and out. ``side`` = (table, ids, first column) of the last kind."""
    table, ids, col = side if side is not None else (None, None, 0)
    _ext.serving().hybrid_gemv(segments, w, y, {"store": 0, "add": 1, "glu": 2, "side": 3}[epilogue], ACTS[act], bias, limit, alpha,
                               table, ids, col)
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


def latent_step_splits(B: int, heads: int) -> int:
    return _ext.serving().hybrid_latent_step_splits(B, heads)


def latent_step(proj, col_q: int, col_g: Optional[int], own: Optional[Tuple[int, torch.Tensor, float]], cache, up, freqs, amplitude: float,
                sink, qa, part, out, rank: int, D: int, R: int, E: int, scale: float, out_scale: float, pos) -> None:
    """One token per sequence in the latent space: the queries take up the key expansion (``qa`` [B, H, rank + rot]), attend
    to the cached rows themselves in split ranges (``part``), and the value expansion runs on the combined result. The
    columns and ``own`` are those of :func:`latent_attention`, ``proj`` and ``out`` fp32."""
    h, d = _pos(pos)
    ocol, ow, oeps = own if own is not None else (-1, None, 0.0)
    _ext.serving().hybrid_latent_step(proj, col_q, -1 if col_g is None else col_g, ocol, ow, oeps, cache, up, freqs, amplitude, sink, qa,
                                      part, out, rank, D, R, E, scale, out_scale, h, d)
    _tick(3)
