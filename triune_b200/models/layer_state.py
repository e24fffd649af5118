"""Per-layer sequence state of mixers that carry more than one tensor.

The framework's cache is a list of ``(state, position)`` per layer. A GLA layer's state is one tensor; a layer of a
heterogeneous model carries any of a key/value cache, a recurrent matrix state and a convolution ring. ``LayerState``
holds them by name and offers what the cache's users do with a state: ``clone`` / ``copy_`` (graph-replayed decoding),
``reserve`` (room for more positions before a capture), ``pack`` / ``unpack`` (sessions parked in one flat buffer)."""

from __future__ import annotations

from typing import Any, Dict, List, Optional, Tuple

import torch

KV_GRAIN = 64  # capacities are multiples of this many positions


class LayerState:
    """``tensors``: the state proper. Names in ``growable`` are [B, groups, capacity, head] and hold ``position`` valid
    entries along dimension 2. ``scratch``: work space of the step kernels, not part of the state."""

    def __init__(self, tensors: Dict[str, torch.Tensor], growable: Tuple[str, ...] = ()):
        self.tensors, self.growable = tensors, tuple(growable)
        self.scratch: Dict[str, torch.Tensor] = {}

    def __getitem__(self, name: str) -> torch.Tensor:
        return self.tensors[name]

    def __setitem__(self, name: str, t: torch.Tensor) -> None:
        self.tensors[name] = t

    @property
    def capacity(self) -> Optional[int]:
        return self.tensors[self.growable[0]].shape[2] if self.growable else None

    def reserve(self, positions: int) -> bool:
        """Make room for ``positions`` in all; doubles, so that appending costs amortised constant time. True when the
        tensors moved."""
        cap = self.capacity
        if cap is None or positions <= cap:
            return False
        new = -(-max(positions, 2 * cap) // KV_GRAIN) * KV_GRAIN
        for n in self.growable:
            old = self.tensors[n]
            t = torch.zeros(*old.shape[:2], new, old.shape[3], dtype=old.dtype, device=old.device)
            t[:, :, :cap].copy_(old)
            self.tensors[n] = t
        return True

    def clone(self) -> "LayerState":
        return LayerState({k: t.clone() for k, t in self.tensors.items()}, self.growable)

    def copy_(self, other: "LayerState") -> "LayerState":
        """Take over ``other``'s values in place. A growable tensor keeps its own, larger capacity."""
        if other is self:
            return self
        for n, src in other.tensors.items():
            dst = self.tensors[n]
            if n in self.growable and dst.shape[2] != src.shape[2]:
                m = min(dst.shape[2], src.shape[2])
                dst[:, :, :m].copy_(src[:, :, :m])
            else:
                dst.copy_(src)
        return self

    def nbytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in self.tensors.values())

    def pack(self, position: int) -> Tuple[List[torch.Tensor], List[Any]]:
        """-> (flat tensors, layout); key/value caches are cut to their valid positions."""
        flats, layout = [], []
        for n, t in self.tensors.items():
            cut = t[:, :, :position] if n in self.growable else t
            flats.append(cut.detach().reshape(-1))
            layout.append((n, tuple(cut.shape), t.dtype, n in self.growable))
        return flats, layout

    @classmethod
    def unpack(cls, flats: List[torch.Tensor], layout: List[Any]) -> "LayerState":
        tensors = {n: f.view(shape).to(dt).contiguous() for f, (n, shape, dt, _) in zip(flats, layout)}
        return cls(tensors, tuple(n for n, _, _, g in layout if g))
