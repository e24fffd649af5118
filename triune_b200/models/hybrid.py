"""HybridTransformer: decoder-only models whose layers differ in their mixers (attention, Mamba-2, gated delta rule, or
several of them side by side) and may or may not have a feed-forward sublayer, over a 32-bit residual stream.

It serves through the same interface as the other families: ``init_cache`` / ``forward(input_ids, cache=...)`` with the
framework's list of ``(state, position)`` per layer (the states are :class:`LayerState`), so the generation loop, the
graph-replayed decoder, the session manager and the HTTP layer work on it unchanged. Prompts (any number of tokens, in
any portions) run GEMMs plus the sequence kernels; one token per sequence runs the fused step kernels: three launches for
a mixer (five for latent attention), two for a feed-forward, two for a token side."""

from __future__ import annotations

from typing import Any, List, Optional

import torch
import torch.nn as nn

from .. import _ext
from ..config import ModelConfig
from ..ops import hybrid as hops
from .hybrid_mixers import Mixer, Portion
from .layer_state import LayerState


class RowNorm(nn.Module):
    """Layer or RMS norm of fp32 rows; the weight is a buffer and stays fp32."""

    def __init__(self, width: int, kind: str, eps: float):
        super().__init__()
        self.kind, self.eps = kind, float(eps)
        self.register_buffer("weight", torch.ones(width))

    @property
    def args(self):
        return self.weight, self.eps, self.kind

    def forward(self, x, out_dtype):
        return hops.norm_rows(x, self.weight, self.eps, self.kind, out_dtype)

    def segment(self, x):
        return hops.seg_norm(x, self.weight, self.eps, self.kind)


class Residual:
    """The fp32 residual rows, with at most one addition ``norm(y + bias)`` not yet made: the kernel that forms the next
    sublayer's input makes it on the way (a row pass for prompts, the prologue of the next projection in a step)."""

    def __init__(self, x: torch.Tensor):
        self.x, self.waiting = x, None

    def add(self, y, bias, norm: RowNorm) -> None:
        self.waiting = (y, bias, norm.args)

    def _made(self, pre, dtype):
        y, bias, post = self.waiting
        self.waiting = None
        return hops.add_norm(self.x, y, bias, post, pre, dtype)

    def rows(self) -> torch.Tensor:
        if self.waiting is not None:
            self._made(None, None)
        return self.x

    def normed(self, norm: RowNorm, dtype) -> torch.Tensor:
        return norm(self.x, dtype) if self.waiting is None else self._made(norm.args, dtype)

    def cast(self, dtype) -> torch.Tensor:
        """The rows themselves as an operand of a product."""
        if self.waiting is not None:
            return self._made("rows", dtype)
        return self.x if self.x.dtype == dtype else self.x.to(dtype)

    def segment(self, norm: Optional[RowNorm], keep: bool = True):
        """Input segment of a step's projection: the normed rows, or the rows."""
        if self.waiting is None:
            return hops.seg_plain(self.x) if norm is None else norm.segment(self.x)
        (y, bias, post), self.waiting = self.waiting, None
        old = self.x
        if keep:  # other blocks still read the old rows
            self.x = torch.empty_like(old)
        return hops.seg_added(old, y.float(), bias, post, None if norm is None else norm.args, self.x if keep else None)

    def select(self, view) -> "Residual":
        """The rows that ``view`` picks, as a stream of their own."""
        out = Residual(view(self.x))
        if self.waiting is not None:
            out.waiting = (view(self.waiting[0]), *self.waiting[1:])
        return out


class GatedFFN(nn.Module):
    """down(act(gate h) * (up h)), gate and up as one weight; optional biases (fp32 buffers)."""

    def __init__(self, width: int, hidden: int, act: str, bias: bool = False, limit: float = 0.0, alpha: float = 0.0):
        super().__init__()
        self.hidden, self.act, self.limit, self.alpha = hidden, act, float(limit), float(alpha)
        self.gate_up = nn.Parameter(torch.zeros(2 * hidden, width))
        self.down = nn.Parameter(torch.zeros(width, hidden))
        self.register_buffer("gate_up_b", torch.zeros(2 * hidden) if bias else None)
        self.register_buffer("down_b", torch.zeros(width) if bias else None)

    def forward(self, h):
        return hops.gated_mlp_hidden(h, self.gate_up, self.act, self.gate_up_b, self.limit, self.alpha)

    def step(self, segment, B: int):
        h = torch.empty(B, self.hidden, device=self.down.device)
        return hops.gemv([segment], self.gate_up, h, "glu", self.act, self.gate_up_b, self.limit, self.alpha)


class TokenSide(nn.Module):
    """A layer's own part of a token table, gated by the residual: norm(proj(gelu_tanh(gate x) * e))."""

    def __init__(self, width: int, dim: int, layer: int, eps: float):
        super().__init__()
        self.dim, self.col0 = dim, layer * dim
        self.gate = nn.Parameter(torch.zeros(dim, width))
        self.proj = nn.Parameter(torch.zeros(width, dim))
        self.norm = RowNorm(width, "rms", eps)

    def forward(self, s: Residual, table, p: Portion) -> None:
        g = hops.token_side_hidden(hops.linear(s.cast(p.dtype), self.gate), table, p.ids, self.col0)
        s.add(hops.linear(g, self.proj), None, self.norm)

    def step(self, s: Residual, table, p: Portion) -> None:
        g = torch.empty(p.B, self.dim, device=table.device)
        hops.gemv([s.segment(None)], self.gate, g, "side", "gelu_tanh", side=(table, p.ids, self.col0))
        y = torch.empty_like(s.x)
        s.add(hops.gemv([hops.seg_plain(g)], self.proj, y), None, self.norm)


class HybridLayer(nn.Module):
    """A mixer, a feed-forward where the layer has one, a token side where the model has one; a norm before every sublayer
    and, with ``post_norm``, one behind it."""

    def __init__(self, cfg: ModelConfig, spec, index: int = 0):
        super().__init__()
        d = cfg.hidden_dim
        norm = lambda: RowNorm(d, cfg.norm, cfg.norm_eps)
        self.norm1, self.mixer = norm(), Mixer(d, spec["mixers"], cfg.norm_eps)
        self.norm1b = norm() if cfg.post_norm else None
        self.ffn = self.norm2 = self.norm2b = self.side = None
        if spec.get("ff"):
            self.norm2 = norm()
            self.ffn = GatedFFN(d, int(spec["ff"]), spec.get("act", "silu"), bool(spec.get("ff_bias")), spec.get("limit", 0.0),
                                spec.get("alpha", 0.0))
            self.norm2b = norm() if cfg.post_norm else None
        if cfg.token_side:
            self.side = TokenSide(d, cfg.token_side, index, cfg.norm_eps)

    @staticmethod
    def _project(s: Residual, y, weight, bias, post: Optional[RowNorm]) -> None:
        if post is not None:
            s.add(hops.linear(y, weight), bias, post)
            return
        hops.linear_accumulate(s.rows(), y, weight)
        if bias is not None:
            s.x += bias

    @staticmethod
    def _project_step(s: Residual, segments, weight, bias, post: Optional[RowNorm]) -> None:
        if post is not None:
            s.add(hops.gemv(segments, weight, torch.empty_like(s.x)), bias, post)
        else:
            hops.gemv(segments, weight, s.x, "add", bias=bias)

    def forward(self, s: Residual, st: LayerState, p: Portion, table=None) -> None:
        y = self.mixer(s.normed(self.norm1, p.dtype), st, p)
        self._project(s, y, self.mixer.out_weight, None, self.norm1b)
        if self.ffn is not None:
            y = self.ffn(s.normed(self.norm2, p.dtype))
            self._project(s, y, self.ffn.down, self.ffn.down_b, self.norm2b)
        if self.side is not None:
            self.side(s, table, p)

    def step(self, s: Residual, st: LayerState, p: Portion, table=None) -> None:
        segments = self.mixer.step(s.segment(self.norm1), st, p)
        self._project_step(s, segments, self.mixer.out_weight[:, : self.mixer.out_width], None, self.norm1b)
        if self.ffn is not None:
            h = self.ffn.step(s.segment(self.norm2), p.B)
            self._project_step(s, [hops.seg_plain(h)], self.ffn.down, self.ffn.down_b, self.norm2b)
        if self.side is not None:
            self.side.step(s, table, p)


class HybridTransformer(nn.Module):
    def __init__(self, cfg: ModelConfig):
        super().__init__()
        self.cfg = self.model_config = cfg
        self.vocab_size, self.hidden_dim, self.num_layers = cfg.vocab_size, cfg.hidden_dim, len(cfg.layers)
        self.embed = nn.Parameter(torch.zeros(cfg.vocab_size, cfg.hidden_dim))
        self.side_embed = nn.Parameter(torch.zeros(cfg.vocab_size, len(cfg.layers) * cfg.token_side)) if cfg.token_side else None
        self.layers = nn.ModuleList([HybridLayer(cfg, s, i) for i, s in enumerate(cfg.layers)])
        self.final_norm = RowNorm(cfg.hidden_dim, cfg.norm, cfg.norm_eps)
        self.head = nn.Parameter(torch.zeros(cfg.vocab_size, cfg.hidden_dim))
        widths = [cfg.hidden_dim] + [l.mixer.out_width for l in self.layers] + [l.ffn.hidden for l in self.layers if l.ffn is not None]
        self._widest = max(widths)
        self._stepable = all(l.mixer.supports_step() for l in self.layers)

    @classmethod
    def from_config(cls, cfg: ModelConfig) -> "HybridTransformer":
        return cls(cfg.validate())

    @torch.no_grad()
    def init_weights(self, seed: int = 0) -> "HybridTransformer":
        """Random weights of a sensible scale (benchmarks, tests); a model of this family is otherwise loaded."""
        g = torch.Generator(device=self.embed.device).manual_seed(seed)
        for n, p in self.named_parameters():
            p.normal_(0.0, 1.0 if n in ("embed", "side_embed") else p.shape[-1] ** -0.5, generator=g)
        for n, b in self.named_buffers():
            leaf = n.rsplit(".", 1)[-1]
            if leaf == "conv_w":
                b.normal_(0.0, b.shape[-1] ** -0.5, generator=g)
            elif leaf in ("A_log", "dt_bias"):
                b.uniform_(-2.0, 0.5, generator=g)
        return self

    # ------------------------------------------------------------------ cache
    def init_cache(self, batch_size: int = 1) -> List[Any]:
        return [(l.mixer.new_state(batch_size, self.embed.device, self.embed.dtype), 0) for l in self.layers]

    def num_parameters(self) -> int:
        return sum(t.numel() for t in self.state_dict().values())  # parameters and the small vectors that are buffers

    # ------------------------------------------------------------------ forward
    @torch.no_grad()
    def forward(self, input_ids=None, cache=None, last_token_only: bool = False, force_depth=None, positions=None,
                on_layer=None, **_):
        """Logits [B, n, vocab] of the last token, of the given ``positions`` (indices into this call's tokens; an empty
        list runs the layers and returns no rows) or of every token. With a cache, runs only the tokens it brings, after
        those the cache holds, and returns the advanced cache. ``on_layer(index, x)`` sees the residual rows."""
        B, T = input_ids.shape
        states = cache if cache is not None else self.init_cache(B)
        pos = states[0][1]
        dtype = self.embed.dtype
        s = Residual(hops.embed_rows(input_ids, self.embed))
        own = [st if st is not None else l.mixer.new_state(B, s.x.device, dtype) for l, (st, _) in zip(self.layers, states)]
        p = Portion(B, T, pos, dtype, input_ids.reshape(-1).long().contiguous(), own)
        step = T == 1 and self._stepable and _ext.use_kernels(s.x) and hops.step_supported(B, self._widest)
        for i, layer in enumerate(self.layers):
            if not torch.is_tensor(pos):  # a position on the device: the caller has reserved
                own[i].reserve(pos + T)
            (layer.step if step else layer)(s, own[i], p, self.side_embed)
            if on_layer is not None:
                on_layer(i, s.rows())
        return self._logits(s, B, T, last_token_only, positions), ([(st, pos + T) for st in own] if cache is not None else None)

    def _logits(self, s: Residual, B: int, T: int, last_token_only: bool, positions):
        if last_token_only:
            pick = lambda t: t.view(B, T, -1)[:, -1:]
        elif positions is not None:
            at = torch.as_tensor(positions, dtype=torch.long, device=s.x.device)
            pick = lambda t: t.view(B, T, -1)[:, at]
        else:
            pick = lambda t: t.view(B, T, -1)
        n = pick(s.x).shape[1]
        if n == 0:
            return s.x.new_zeros(B, 0, self.vocab_size)
        r = s.select(lambda t: pick(t).reshape(B * n, -1).contiguous())
        if _ext.use_kernels(r.x) and hops.step_supported(B * n, self.hidden_dim):
            out = torch.empty(B * n, self.vocab_size, device=r.x.device)
            hops.gemv([r.segment(self.final_norm, keep=False)], self.head, out)
        else:
            out = hops.linear(r.normed(self.final_norm, self.embed.dtype), self.head, torch.float32)
        return out.view(B, n, self.vocab_size)
