"""Sequence mixers of heterogeneous-layer models: softmax attention with head norms, partial rotation and a sink;
multi-head latent attention with a sink, an output gate and latents that layers may share; Mamba-2; the gated delta rule;
retention. A layer's mixer is one or several of these *cores* side by side on the same input, their
scaled outputs summed.

Layout: the input projections of all cores are ONE weight ``in_weight`` and the output projections ONE weight
``out_weight``, so a layer's mixer is two GEMMs around its cores however many cores it has; every named segment of the
projection starts at a multiple of eight columns (rows of zeros fill the gaps), which keeps the kernels' vector and TMA
accesses aligned for any head size. The output scales are applied to the cores' outputs before they are rounded, and the
output GEMM adds straight into the 32-bit residual stream. Small vectors that only enter 32-bit arithmetic are buffers:
they stay fp32 when the weights are cast."""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Tuple

import torch
import torch.nn as nn

from ..ops import hybrid as hops
from .layer_state import KV_GRAIN, LayerState
from .rotary import rotary_frequencies

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


@dataclass
class Portion:
    """One call of the model: ``T`` tokens of each of ``B`` sequences after ``pos`` earlier ones, the states of every layer,
    and the rotation tables that its layers share."""

    B: int
    T: int
    pos: Any
    dtype: torch.dtype
    ids: torch.Tensor
    states: List[LayerState]
    tables: Dict[Any, torch.Tensor] = field(default_factory=dict)

    def rotation(self, core: "Core") -> torch.Tensor:
        key = core.rot_key
        if key not in self.tables:
            self.tables[key] = hops.rotation_rows(core.freqs, core.amplitude, self.pos, self.T, self.dtype)
        return self.tables[key]


class Core(nn.Module):
    """One mixer: ``inputs`` are its segments of the fused input projection, ``out_width`` its share of the output."""

    inputs: Segments
    out_width: int

    def __init__(self, spec: Dict[str, Any], eps: float):
        super().__init__()
        self.eps, self.out_scale = float(eps), float(spec.get("out_scale", 1.0))

    def vector(self, name: str, *shape: int, fill: float = 0.0) -> None:
        self.register_buffer(name, torch.full(shape, fill))

    def rotary(self, spec: Dict[str, Any]) -> None:
        dims, base, scaling = int(spec.get("rot_dims", 0)), float(spec.get("rot_base", 1e4)), spec.get("rot_scaling")
        freqs, self.amplitude = rotary_frequencies(dims, base, scaling)
        self.register_buffer("freqs", freqs, persistent=False)
        self.rot_key = (dims, base, tuple(sorted(scaling.items())) if scaling else None)

    def new_state(self, B: int, device, dtype) -> Dict[str, torch.Tensor]:
        raise NotImplementedError

    def supports_step(self) -> bool:
        return True

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
        self.rotary(spec)  # neighbouring dimensions are pairs

    def supports_step(self) -> bool:
        return self.dim <= 512 and self.vdim <= 256

    def new_state(self, B, device, dtype):
        shape = (B, self.kv_heads, 4 * KV_GRAIN)
        return {"k": torch.zeros(*shape, pad8(self.dim), device=device, dtype=dtype),
                "v": torch.zeros(*shape, pad8(self.vdim), device=device, dtype=dtype)}

    def _vec(self, name):
        return getattr(self, name, None)

    def forward(self, proj, col0: int, st: LayerState, pre: str, p: Portion, out) -> None:
        cols = [col0 + self.inputs.at[n] for n in ("q", "k", "v")]
        hops.attention(proj, cols, self._vec("q_norm"), self._vec("k_norm"), self.eps, self.freqs, self._vec("sink"),
                       st[pre + "k"], st[pre + "v"], out, p.B, p.T, self.heads, self.dim, self.vdim, self.scale, self.out_scale, p.pos)

    def step(self, proj, col0: int, st: LayerState, pre: str, p: Portion):
        """-> (arguments of the step kernel, input segment of the output projection)."""
        B = p.B
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

    def supports_step(self) -> bool:
        return self.dk <= 256

    def forward(self, proj, col0: int, st: LayerState, pre: str, p: Portion, out) -> None:
        at, ca = self.inputs.at, self.conv_at.at
        B, T, pos = p.B, p.T, p.pos
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

    def step(self, proj, col0: int, st: LayerState, pre: str, p: Portion):
        at, ca = self.inputs.at, self.conv_at.at
        out = torch.empty(p.B, self.out_width, device=proj.device)
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


class RetentionCore(Core):
    """Linear attention with a fixed decay per head on rotated queries and keys (dimension i is paired with dimension
    i + rot_dims / 2), every head's output divided by its root mean square and gated by silu."""

    def __init__(self, spec, eps):
        super().__init__(spec, eps)
        H, D, E = self.heads, self.dim, self.vdim = int(spec["heads"]), int(spec["dim"]), int(spec["vdim"])
        self.inputs = Segments([("q", H * D), ("k", H * D), ("v", H * E), ("g", H * E)])
        self.out_width = H * E
        self.register_buffer("decay", torch.tensor(spec["decay"], dtype=torch.float64), persistent=False)
        self.rotary(spec)

    def supports_step(self) -> bool:
        return self.dim <= 256

    def new_state(self, B, device, dtype):
        wide = torch.float64 if dtype == torch.float64 else torch.float32
        return {"S": torch.zeros(B, self.heads, self.dim, self.vdim, device=device, dtype=wide)}

    def forward(self, proj, col0: int, st: LayerState, pre: str, p: Portion, out) -> None:
        q, k, v, g = (proj[:, col0 + self.inputs.at[n] :] for n in ("q", "k", "v", "g"))
        y = torch.empty(p.B * p.T, pad8(self.out_width), device=proj.device, dtype=proj.dtype)
        hops.retention(q, k, v, p.rotation(self), self.decay, st[pre + "S"], y, p.B, p.T)
        hops.gated_norm(y, g, None, out, self.out_width, self.heads, self.eps, False, self.out_scale)

    def step(self, proj, col0: int, st: LayerState, pre: str, p: Portion):
        at = self.inputs.at
        out = torch.empty(p.B, self.out_width, device=proj.device)
        args = {"state": st[pre + "S"], "out": out, "kind": hops.KINDS["retention"], "col_q": col0 + at["q"], "col_k": col0 + at["k"],
                "col_v": col0 + at["v"], "decay": self.decay, "freqs": self.freqs, "amplitude": self.amplitude}
        return args, hops.seg_gated(out, proj[:, col0 + at["g"] :], None, self.heads, self.eps, False, self.out_scale)


class LatentCore(Core):
    """Multi-head latent attention: keys and values are expansions of one normed latent per position, beside one rotated key
    part that all heads share; the cache holds only these. Prompts expand keys and values per head; a step folds the key
    expansion into the query and runs the value expansion on the attended latent. With ``kv_from`` the layer reads the
    latents of an earlier layer. Heads are padded to multiples of eight inside the weights, never in what they mean."""

    def __init__(self, spec, eps):
        super().__init__(spec, eps)
        H = self.heads = int(spec["heads"])
        self.dim, self.rot, self.vdim, self.rank = (int(spec[n]) for n in ("dim", "rot_dims", "vdim", "kv_rank"))
        self.scale, self.kv_from = float(spec["scale"]), spec.get("kv_from")
        self.dim_p, self.rot_p, self.vdim_p, self.rank_p = pad8(self.dim), pad8(self.rot), pad8(self.vdim), pad8(self.rank)
        self.has_gate, self.has_sink = bool(spec.get("gate", True)), bool(spec.get("sink", True))
        parts = [("q", H * (self.dim_p + self.rot_p))]
        if self.kv_from is None:
            parts.append(("c", self.rank_p + self.rot_p))
            self.vector("c_norm", self.rank, fill=1.0)
            self.growable = ("c",)
        if self.has_gate:
            parts.append(("g", H))
        if self.has_sink:
            self.vector("sink", H)
        self.inputs = Segments(parts)
        self.out_width = H * self.vdim
        self.up = nn.Parameter(torch.zeros(H, self.dim_p + self.vdim_p, self.rank_p))  # per head: key rows, value rows
        self.rotary(spec)

    def supports_step(self) -> bool:
        return self.rank_p + self.rot_p <= 2048 and self.vdim <= 1024

    def new_state(self, B, device, dtype):
        if self.kv_from is not None:
            return {}
        return {"c": torch.zeros(B, 1, 4 * KV_GRAIN, self.rank_p + self.rot_p, device=device, dtype=dtype)}

    def _rows(self, col0: int, st: LayerState, pre: str, p: Portion):
        """-> (cached rows, (column, norm weight, eps) of this layer's own latents)"""
        if self.kv_from is not None:
            return p.states[self.kv_from]["0.c"], None
        return st[pre + "c"], (col0 + self.inputs.at["c"], self.c_norm, self.eps)

    def _gate(self, col0: int):
        return col0 + self.inputs.at["g"] if self.has_gate else None

    def forward(self, proj, col0: int, st: LayerState, pre: str, p: Portion, out) -> None:
        cache, own = self._rows(col0, st, pre, p)
        hops.latent_attention(proj, col0 + self.inputs.at["q"], self._gate(col0), own, cache, self.up, p.rotation(self),
                              getattr(self, "sink", None), out, p.B, p.T, self.rank, self.dim, self.rot, self.vdim, self.scale,
                              self.out_scale, p.pos)

    def step(self, proj, col0: int, st: LayerState, pre: str, p: Portion):
        cache, own = self._rows(col0, st, pre, p)
        s, B = st.scratch, p.B
        if pre + "part" not in s or s[pre + "part"].shape[0] != B:
            s[pre + "qa"] = torch.empty(B, self.heads, self.rank_p + self.rot_p, device=proj.device)
            s[pre + "part"] = torch.empty(B, self.heads, hops.latent_step_splits(B, self.heads), hops.step_part_stride(self.rank_p),
                                          device=proj.device)
        out = torch.empty(B, self.out_width, device=proj.device)
        hops.latent_step(proj, col0 + self.inputs.at["q"], self._gate(col0), own, cache, self.up, self.freqs, self.amplitude,
                         getattr(self, "sink", None), s[pre + "qa"], s[pre + "part"], out, self.rank, self.dim, self.rot, self.vdim,
                         self.scale, self.out_scale, p.pos)
        return None, hops.seg_plain(out)


CORES = {"attention": AttentionCore, "latent": LatentCore, "mamba2": Mamba2Core, "delta": DeltaCore, "retention": RetentionCore}


class Mixer(nn.Module):
    """One or several cores on the same input: ``sum_i out_scale_i * W_o,i core_i(W_in,i h)``; the layer applies the output
    projection, whose result it norms or adds."""

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

    def forward(self, h, st: LayerState, p: Portion):
        """Rows of the output projection's input for T tokens per sequence; ``st`` advances."""
        proj = hops.linear(h, self.in_weight)
        kp = self.out_weight.shape[1]
        y = torch.empty(p.B * p.T, kp, device=h.device, dtype=h.dtype)
        if kp > self.out_width:
            y[:, self.out_width :] = 0
        for i, c in enumerate(self.cores):
            c(proj, self.cols[i], st, f"{i}.", p, y[:, self.outs[i] :])
        return y

    def step(self, norm_segment, st: LayerState, p: Portion):
        """The same for one token per sequence: input projection with the norm in its prologue, then one launch for a
        recurrence and an attention together. -> input segments of the output projection (gated norms in its prologue)."""
        proj = torch.empty(p.B, self.in_width, device=self.in_weight.device)
        hops.gemv([norm_segment], self.in_weight[: self.in_width], proj)
        segments, recs, atts = [], [], []
        for i, c in enumerate(self.cores):
            args, seg = c.step(proj, self.cols[i], st, f"{i}.", p)
            if args is not None:
                (atts if isinstance(c, AttentionCore) else recs).append(args)
            segments.append(seg)
        for j in range(max(len(recs), len(atts))):
            hops.mixer_step(proj, recs[j] if j < len(recs) else None, atts[j] if j < len(atts) else None, p.pos)
        return segments

    def supports_step(self) -> bool:
        """The output projection's prologue takes one or two cores."""
        return len(self.cores) <= 2 and all(c.supports_step() for c in self.cores)
