"""HybridTransformer: decoder-only models whose layers differ in their mixers (attention, Mamba-2, gated delta rule, or
several of them side by side) and may or may not have a feed-forward sublayer, over a 32-bit residual stream.

It serves through the same interface as the other families: ``init_cache`` / ``forward(input_ids, cache=...)`` with the
framework's list of ``(state, position)`` per layer (the states are :class:`LayerState`), so the generation loop, the
graph-replayed decoder, the session manager and the HTTP layer work on it unchanged. Prompts (any number of tokens, in
any portions) run GEMMs plus the sequence kernels; one token per sequence runs the fused step kernels: five launches per
layer with a feed-forward, three without."""

from __future__ import annotations

from typing import Any, List, Optional

import torch
import torch.nn as nn

from .. import _ext
from ..config import ModelConfig
from ..ops import hybrid as hops
from .hybrid_mixers import Mixer
from .layer_state import LayerState


class RowNorm(nn.Module):
    """Layer or RMS norm of fp32 rows; the weight is a buffer and stays fp32."""

    def __init__(self, width: int, kind: str, eps: float):
        super().__init__()
        self.kind, self.eps = kind, float(eps)
        self.register_buffer("weight", torch.ones(width))

    def forward(self, x, out_dtype):
        return hops.norm_rows(x, self.weight, self.eps, self.kind, out_dtype)

    def segment(self, x):
        return hops.seg_norm(x, self.weight, self.eps, self.kind)


class GatedFFN(nn.Module):
    """down(act(gate h) * (up h)), gate and up as one weight."""

    def __init__(self, width: int, hidden: int, act: str):
        super().__init__()
        self.hidden, self.act = hidden, act
        self.gate_up = nn.Parameter(torch.zeros(2 * hidden, width))
        self.down = nn.Parameter(torch.zeros(width, hidden))

    def forward(self, h, x) -> None:
        hops.linear_accumulate(x, hops.gated_mlp_hidden(h, self.gate_up, self.act), self.down)

    def step(self, x, norm_segment) -> None:
        h = torch.empty(x.shape[0], self.hidden, device=x.device)
        hops.gemv([norm_segment], self.gate_up, h, "glu", self.act)
        hops.gemv([hops.seg_plain(h)], self.down, x, "add")


class HybridLayer(nn.Module):
    def __init__(self, cfg: ModelConfig, spec):
        super().__init__()
        d = cfg.hidden_dim
        self.norm1 = RowNorm(d, cfg.norm, cfg.norm_eps)
        self.mixer = Mixer(d, spec["mixers"], cfg.norm_eps)
        self.ffn = None
        if spec.get("ff"):
            self.norm2 = RowNorm(d, cfg.norm, cfg.norm_eps)
            self.ffn = GatedFFN(d, int(spec["ff"]), spec.get("act", "silu"))

    def forward(self, x, st: LayerState, B: int, T: int, pos, dtype) -> None:
        self.mixer(self.norm1(x, dtype), x, st, B, T, pos)
        if self.ffn is not None:
            self.ffn(self.norm2(x, dtype), x)

    def step(self, x, st: LayerState, B: int, pos) -> None:
        self.mixer.step(x, self.norm1.segment(x), st, B, pos)
        if self.ffn is not None:
            self.ffn.step(x, self.norm2.segment(x))


class HybridTransformer(nn.Module):
    def __init__(self, cfg: ModelConfig):
        super().__init__()
        self.cfg = self.model_config = cfg
        self.vocab_size, self.hidden_dim, self.num_layers = cfg.vocab_size, cfg.hidden_dim, len(cfg.layers)
        self.embed = nn.Parameter(torch.zeros(cfg.vocab_size, cfg.hidden_dim))
        self.layers = nn.ModuleList([HybridLayer(cfg, s) for s in cfg.layers])
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
            p.normal_(0.0, 1.0 if n == "embed" else p.shape[-1] ** -0.5, generator=g)
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
        return sum(t.numel() for t in list(self.parameters()) + [b for n, b in self.named_buffers() if not n.endswith("freqs")])

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
        new_cache = []
        x = hops.embed_rows(input_ids, self.embed)
        dtype = self.embed.dtype
        step = T == 1 and self._stepable and _ext.use_kernels(x) and hops.step_supported(B, self._widest)
        for i, layer in enumerate(self.layers):
            st = states[i][0]
            if st is None:
                st = layer.mixer.new_state(B, x.device, dtype)
            if not torch.is_tensor(pos):  # a position on the device: the caller has reserved
                st.reserve(pos + T)
            if step:
                layer.step(x, st, B, pos)
            else:
                layer(x, st, B, T, pos, dtype)
            if on_layer is not None:
                on_layer(i, x)
            new_cache.append((st, pos + T))
        return self._logits(x, B, T, last_token_only, positions), (new_cache if cache is not None else None)

    def _logits(self, x, B: int, T: int, last_token_only: bool, positions):
        rows = x.view(B, T, -1)
        if last_token_only:
            rows = rows[:, -1:]
        elif positions is not None:
            rows = rows[:, torch.as_tensor(positions, dtype=torch.long, device=x.device)]
        n = rows.shape[1]
        if n == 0:
            return x.new_zeros(B, 0, self.vocab_size)
        rows = rows.reshape(B * n, -1).contiguous()
        if _ext.use_kernels(rows) and hops.step_supported(B * n, self.hidden_dim):
            out = torch.empty(B * n, self.vocab_size, device=x.device)
            hops.gemv([self.final_norm.segment(rows)], self.head, out)
        else:
            h = self.final_norm(rows, self.embed.dtype)
            out = hops.linear(h, self.head, torch.float32)
        return out.view(B, n, self.vocab_size)
