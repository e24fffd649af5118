"""Sequence mixers of heterogeneous-layer models: softmax attention with head norms, partial rotation and a sink;
Mamba-2; the gated delta rule. A layer's mixer is one or several of these *cores* side by side on the same input, their
scaled outputs summed.

Layout: the input projections of all cores are ONE weight ``in_weight`` and the output projections ONE weight
``out_weight``, so a layer's mixer is two GEMMs around its cores however many cores it has; every named segment of the
projection starts at a multiple of eight columns (rows of zeros fill the gaps), which keeps the kernels' vector and TMA
accesses aligned for any head size. The output scales are applied to the cores' outputs before they are rounded, and the
output GEMM adds straight into the 32-bit residual stream. Small vectors that only enter 32-bit arithmetic are buffers:
they stay fp32 when the weights are cast."""

from __future__ import annotations

from typing import Any, Dict, List, Optional, Tuple

import torch
import torch.nn as nn

from ..ops import hybrid as hops
from .layer_state import KV_GRAIN, LayerState

UNIT_EPS = 1e-6  # under the root of the delta rule's unit vectors


def pad8(n: int) -> int:
    return -(-n // 8) * 8


class Segments:
    """Named column ranges, each starting at a multiple of eight."""

    def __init__(self, parts: List[Tuple[str, int]]):
        self.at: Dict[str, int] = {}
        self.width: Dict[str, int] = {}
        col = 0
        for name, n in parts:
            self.at[name], self.width[name] = col, n
            col += pad8(n)
        self.total = col


class Core(nn.Module):
    """One mixer: ``inputs`` are its segments of the fused input projection, ``out_width`` its share of the output."""

    inputs: Segments
    out_width: int

    def __init__(self, spec: Dict[str, Any], eps: float):
        super().__init__()
        self.eps, self.out_scale = float(eps), float(spec.get("out_scale", 1.0))

    def vector(self, name: str, *shape: int, fill: float = 0.0) -> None:
        self.register_buffer(name, torch.full(shape, fill))

    def new_state(self, B: int, device, dtype) -> Dict[str, torch.Tensor]:
        raise NotImplementedError

    growable: Tuple[str, ...] = ()


class AttentionCore(Core):
    growable = ("k", "v")

    def __init__(self, spec: Dict[str, Any], eps: float):
        super().__init__(spec, eps)
        self.heads, self.kv_heads = int(spec["heads"]), int(spec["kv_heads"])
        self.dim, self.vdim, self.scale = int(spec["dim"]), int(spec["vdim"]), float(spec["scale"])
        self.inputs = Segments([("q", self.heads * self.dim), ("k", self.kv_heads * self.dim), ("v", self.kv_heads * self.vdim)])
        self.out_width = self.heads * self.vdim
        self.qk_norm, self.has_sink = bool(spec.get("qk_norm", True)), bool(spec.get("sink", True))
        if self.qk_norm:
            self.vector("q_norm", self.dim, fill=1.0)
            self.vector("k_norm", self.dim, fill=1.0)
        if self.has_sink:
            self.vector("sink", self.heads)
        n = int(spec.get("rot_dims", 0)) // 2
        i = torch.arange(n, dtype=torch.float64)
        self.register_buffer("freqs", float(spec.get("rot_base", 1e4)) ** (-2.0 * i / max(1, 2 * n)), persistent=False)

    def new_state(self, B, device, dtype):
        shape = (B, self.kv_heads, 4 * KV_GRAIN)
        return {"k": torch.zeros(*shape, pad8(self.dim), device=device, dtype=dtype),
                "v": torch.zeros(*shape, pad8(self.vdim), device=device, dtype=dtype)}

    def _vec(self, name):
        return getattr(self, name, None)

    def forward(self, proj, col0: int, st: LayerState, pre: str, B: int, T: int, pos, out) -> None:
        cols = [col0 + self.inputs.at[n] for n in ("q", "k", "v")]
        hops.attention(proj, cols, self._vec("q_norm"), self._vec("k_norm"), self.eps, self.freqs, self._vec("sink"),
                       st[pre + "k"], st[pre + "v"], out, B, T, self.heads, self.dim, self.vdim, self.scale, self.out_scale, pos)

    def step(self, proj, col0: int, st: LayerState, pre: str, B: int):
        """-> (arguments of the step kernel, its output, input segment of the output projection)."""
        rep = self.heads // self.kv_heads
        groups = B * self.kv_heads * -(-rep // hops.step_head_chunk(rep))
        splits = max(1, min(64, 2 * 148 // groups))
        s = st.scratch
        if pre + "part" not in s or s[pre + "part"].shape[:2] != (B, self.heads):
            s[pre + "part"] = torch.empty(B, self.heads, splits, hops.step_part_stride(self.vdim), device=proj.device)
            s[pre + "counters"] = torch.zeros(groups, dtype=torch.int32, device=proj.device)
        out = torch.empty(B, self.out_width, device=proj.device)
        at = self.inputs.at
        args = {"k": st[pre + "k"], "v": st[pre + "v"], "part": s[pre + "part"], "counters": s[pre + "counters"], "out": out,
                "freqs": self.freqs, "heads": self.heads, "dim": self.dim, "vdim": self.vdim, "col_q": col0 + at["q"],
                "col_k": col0 + at["k"], "col_v": col0 + at["v"], "q_w": self._vec("q_norm"), "k_w": self._vec("k_norm"),
                "eps": self.eps, "sink": self._vec("sink"), "splits": splits, "scale": self.scale, "out_scale": self.out_scale}
        return args, hops.seg_plain(out)


class RecurrentCore(Core):
    """What Mamba-2 and the delta rule share: short convolution, matrix state, gated norm."""

    kind = ""
    gate_first = True

    def _setup(self, heads: int, key_groups: int, dk: int, dv: int, taps: int, conv: Segments, gate: str, norm_groups: int):
        self.heads, self.key_groups, self.dk, self.dv, self.taps = heads, key_groups, dk, dv, taps
        self.conv_at, self.gate_name, self.norm_groups = conv, gate, norm_groups
        self.out_width = heads * dv
        self.vector("conv_w", conv.total, taps)
        self.vector("A_log", heads)
        self.vector("dt_bias", heads)

    def new_state(self, B, device, dtype):
        wide = torch.float64 if dtype == torch.float64 else torch.float32
        return {"S": torch.zeros(B, self.heads, self.dk, self.dv, device=device, dtype=wide),
                "conv": torch.zeros(B, self.taps, self.conv_at.total, device=device, dtype=wide)}

    def forward(self, proj, col0: int, st: LayerState, pre: str, B: int, T: int, pos, out) -> None:
        at, ca = self.inputs.at, self.conv_at.at
        u, ring = hops.causal_conv(proj[:, col0 + at["u"] :], self.conv_w, getattr(self, "conv_b", None), st[pre + "conv"],
                                   B, T, pos)
        if torch.is_tensor(pos):  # inside a capture: the state keeps its address
            st[pre + "conv"].copy_(ring)
        else:
            st[pre + "conv"] = ring
        y = torch.empty(B * T, pad8(self.out_width), device=proj.device, dtype=proj.dtype)
        hops.recurrent(u[:, ca["q"] :], u[:, ca["k"] :], u[:, ca["v"] :], proj[:, col0 + at["a"] :],
                       proj[:, col0 + at["b"] :] if "b" in at else None, self.A_log, self.dt_bias, getattr(self, "D", None),
                       st[pre + "S"], y, B, T, self.kind, self.key_groups, UNIT_EPS)
        hops.gated_norm(y, proj[:, col0 + at[self.gate_name] :], self.norm, out, self.out_width, self.norm_groups, self.eps,
                        self.gate_first, self.out_scale)

    def step(self, proj, col0: int, st: LayerState, pre: str, B: int):
        at, ca = self.inputs.at, self.conv_at.at
        out = torch.empty(B, self.out_width, device=proj.device)
        args = {"state": st[pre + "S"], "ring": st[pre + "conv"], "conv_w": self.conv_w, "conv_b": getattr(self, "conv_b", None),
                "out": out, "key_groups": self.key_groups, "kind": hops.KINDS[self.kind], "col_u": col0 + at["u"],
                "col_a": col0 + at["a"], "col_b": col0 + at.get("b", 0), "off_q": ca["q"], "off_k": ca["k"], "off_v": ca["v"],
                "A_log": self.A_log, "dt_bias": self.dt_bias, "D": getattr(self, "D", None), "unit_eps": UNIT_EPS}
        gate = proj[:, col0 + at[self.gate_name] :]
        return args, hops.seg_gated(out, gate, self.norm, self.norm_groups, self.eps, self.gate_first, self.out_scale)


class Mamba2Core(RecurrentCore):
    kind, gate_first = "mamba2", True

    def __init__(self, spec, eps):
        super().__init__(spec, eps)
        H, P, N, G = int(spec["heads"]), int(spec["vdim"]), int(spec["state"]), int(spec["groups"])
        conv = Segments([("v", H * P), ("k", G * N), ("q", G * N)])  # x, B, C of the usual notation
        self.inputs = Segments([("z", H * P), ("u", conv.total), ("a", H)])
        self._setup(H, G, N, P, int(spec["conv"]), conv, "z", int(spec["norm_groups"]))
        self.vector("conv_b", conv.total)
        self.vector("D", H, fill=1.0)
        self.vector("norm", H * P, fill=1.0)


class DeltaCore(RecurrentCore):
    kind, gate_first = "delta", False

    def __init__(self, spec, eps):
        super().__init__(spec, eps)
        H, K, D, E = int(spec["heads"]), int(spec["kv_heads"]), int(spec["dim"]), int(spec["vdim"])
        conv = Segments([("q", K * D), ("k", K * D), ("v", H * E)])
        self.inputs = Segments([("u", conv.total), ("g", H * E), ("b", H), ("a", H)])
        self._setup(H, K, D, E, int(spec["conv"]), conv, "g", H)
        self.vector("norm", E, fill=1.0)


CORES = {"attention": AttentionCore, "mamba2": Mamba2Core, "delta": DeltaCore}


class Mixer(nn.Module):
    """One or several cores on the same input: ``sum_i out_scale_i * W_o,i core_i(W_in,i h)`` added to the residual."""

    def __init__(self, width: int, specs: List[Dict[str, Any]], eps: float):
        super().__init__()
        self.cores = nn.ModuleList([CORES[s["kind"]](s, eps) for s in specs])
        self.cols, self.outs, col, out = [], [], 0, 0
        for c in self.cores:
            self.cols.append(col)
            self.outs.append(out)
            col += c.inputs.total
            out += c.out_width
        self.in_width, self.out_width = col, out
        # large projections are whole 256-row tiles, so that the GEMM runs on CTA pairs
        rows = -(-col // 256) * 256 if col >= 1024 else col
        self.in_weight = nn.Parameter(torch.zeros(rows, width))
        self.out_weight = nn.Parameter(torch.zeros(width, pad8(out)))

    def new_state(self, B: int, device, dtype) -> LayerState:
        tensors, grow = {}, []
        for i, c in enumerate(self.cores):
            for n, t in c.new_state(B, device, dtype).items():
                tensors[f"{i}.{n}"] = t
            grow += [f"{i}.{n}" for n in c.growable]
        return LayerState(tensors, tuple(grow))

    def forward(self, h, x, st: LayerState, B: int, T: int, pos) -> None:
        """x += mixer(h) over T tokens per sequence; ``st`` advances."""
        proj = hops.linear(h, self.in_weight)
        kp = self.out_weight.shape[1]
        y = torch.empty(B * T, kp, device=h.device, dtype=h.dtype)
        if kp > self.out_width:
            y[:, self.out_width :] = 0
        for i, c in enumerate(self.cores):
            c(proj, self.cols[i], st, f"{i}.", B, T, pos, y[:, self.outs[i] :])
        hops.linear_accumulate(x, y, self.out_weight)

    def step(self, x, norm_segment, st: LayerState, B: int, pos) -> None:
        """The same for one token per sequence: input projection with the norm in its prologue, one launch for a
        recurrence and an attention together, output projection with the gated norm in its prologue."""
        proj = torch.empty(B, self.in_width, device=x.device)
        hops.gemv([norm_segment], self.in_weight[: self.in_width], proj)
        segments, recs, atts = [], [], []
        for i, c in enumerate(self.cores):
            args, seg = c.step(proj, self.cols[i], st, f"{i}.", B)
            (atts if isinstance(c, AttentionCore) else recs).append(args)
            segments.append(seg)
        for j in range(max(len(recs), len(atts))):
            hops.mixer_step(proj, recs[j] if j < len(recs) else None, atts[j] if j < len(atts) else None, pos)
        hops.gemv(segments, self.out_weight[:, : self.out_width], x, "add")

    def step_widths(self) -> List[int]:
        return [self.out_width]

    def supports_step(self) -> bool:
        """The step kernels take one or two cores with heads of at most 256 (attention keys: 512)."""
        if len(self.cores) > 2:
            return False
        for c in self.cores:
            if isinstance(c, AttentionCore) and (c.dim > 512 or c.vdim > 256):
                return False
            if isinstance(c, RecurrentCore) and c.dk > 256:
                return False
        return True
