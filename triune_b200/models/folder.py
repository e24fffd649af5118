"""Models that live in a folder (``config.json`` + ``model.safetensors``) under the names of their design.

A design is a reader of its configuration and a map from every stored tensor to a view of the fused weights, so loading and
saving are the same loop for all of them. A view is a tensor, or one of the composite views below."""

from __future__ import annotations

import json
from pathlib import Path
from typing import Any, Dict, List, Optional

import torch

from ..config import ModelConfig
from ..export.safetensors_io import load_file, save_file
from .hybrid import HybridTransformer


class Stacked:
    """Several row blocks of the model that are one tensor in the file."""

    def __init__(self, parts: List[torch.Tensor]):
        self.parts = parts

    @property
    def shape(self):
        return torch.Size([sum(t.shape[0] for t in self.parts), *self.parts[0].shape[1:]])

    def copy_(self, src: torch.Tensor) -> None:
        for t, s in zip(self.parts, src.split([t.shape[0] for t in self.parts])):
            t.copy_(s)

    def detach(self) -> torch.Tensor:
        return torch.cat([t.detach() for t in self.parts])


class PerHead:
    """Row blocks [heads, rows, columns] that are stored head by head, each head's blocks behind one another."""

    def __init__(self, parts: List[torch.Tensor]):
        self.parts = parts

    @property
    def shape(self):
        H, _, n = self.parts[0].shape
        return torch.Size([H * sum(t.shape[1] for t in self.parts), n])

    def copy_(self, src: torch.Tensor) -> None:
        rows = [t.shape[1] for t in self.parts]
        for t, s in zip(self.parts, src.view(self.parts[0].shape[0], sum(rows), -1).split(rows, 1)):
            t.copy_(s)

    def detach(self) -> torch.Tensor:
        return torch.cat([t.detach() for t in self.parts], 1).flatten(0, 1)


class FolderModel(HybridTransformer):
    """Base of the designs: ``Design(config=<dict or path>)`` builds one with zero weights, ``from_pretrained(folder)``
    loads one. Subclasses give ``read_config`` and ``named_views``."""

    @staticmethod
    def read_config(raw: Dict[str, Any]) -> ModelConfig:
        raise NotImplementedError

    def named_views(self) -> Dict[str, Any]:
        raise NotImplementedError

    def __init__(self, config=None, cfg: Optional[ModelConfig] = None):
        if cfg is None:
            raw = config if isinstance(config, dict) else json.loads(Path(config).read_text(encoding="utf-8"))
            super().__init__(self.read_config(raw))
            self.raw_config = raw
        else:
            super().__init__(cfg)

    @classmethod
    def from_pretrained(cls, folder, device="cpu", dtype: Optional[torch.dtype] = None) -> "FolderModel":
        from ..utils import place_model

        folder = Path(folder)
        model = cls(config=folder / "config.json")
        model.load_named(load_file(str(folder / "model.safetensors")))
        return place_model(model, device, dtype).eval()

    @torch.no_grad()
    def load_named(self, tensors: Dict[str, torch.Tensor]) -> None:
        views = self.named_views()
        missing, extra = sorted(set(views) - set(tensors)), sorted(set(tensors) - set(views))
        if missing or extra:
            raise ValueError(f"tensors do not fit the configuration: missing {missing[:4]}, unknown {extra[:4]}")
        for n, v in views.items():
            t = tensors[n]
            if tuple(t.shape) != tuple(v.shape):
                raise ValueError(f"{n}: stored {tuple(t.shape)}, the configuration implies {tuple(v.shape)}")
            v.copy_(t.to(torch.float32) if t.dtype == torch.bfloat16 else t)

    def save_pretrained(self, folder, dtype: torch.dtype = torch.bfloat16) -> None:
        folder = Path(folder)
        folder.mkdir(parents=True, exist_ok=True)
        (folder / "config.json").write_text(json.dumps(self.raw_config, indent=1), encoding="utf-8")
        save_file({n: v.detach().to(dtype).contiguous().cpu() for n, v in self.named_views().items()}, str(folder / "model.safetensors"))
