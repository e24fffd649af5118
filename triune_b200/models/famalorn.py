"""Famalorn: the reader of its model folders (``config.json`` + ``model.safetensors``).

A Famalorn is a :class:`HybridTransformer` with layer norms and ReLU-gated feed-forwards whose layers are ``mamba2``,
``delta`` (gated delta rule) or ``parallel`` (sink attention beside Mamba-2). This module maps its configuration to a
:class:`ModelConfig` and its tensor names to the fused weights, both ways."""

from __future__ import annotations

from typing import Any, Dict, Iterator, Tuple

import torch

from ..config import ModelConfig
from .folder import FolderModel, Stacked
from .hybrid import HybridTransformer
from .hybrid_mixers import AttentionCore, Core, DeltaCore
from .zoo import register_model

FF_ACT = "relu"


def _attention(m: Dict[str, Any], scale: float) -> Dict[str, Any]:
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    return {"kind": "attention", "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"],
            "rot_dims": rot["dims"], "rot_base": rot["base"], "scale": m["scale"], "out_scale": scale}


def _mamba2(m: Dict[str, Any], scale: float = 1.0) -> Dict[str, Any]:
    return {"kind": "mamba2", "out_scale": scale, **{k: m[k] for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups")}}


def _delta(m: Dict[str, Any]) -> Dict[str, Any]:
    return {"kind": "delta", **{k: m[k] for k in ("heads", "kv_heads", "dim", "vdim", "conv")}}


def layer_spec(entry: Dict[str, Any]) -> Dict[str, Any]:
    m = entry["mixer"]
    if entry["type"] == "parallel":
        mixers = [_attention(m["left"], m["left_scale"]), _mamba2(m["right"], m["right_scale"])]
    elif entry["type"] == "mamba2":
        mixers = [_mamba2(m)]
    elif entry["type"] == "delta":
        mixers = [_delta(m)]
    else:
        raise ValueError(f"unknown layer type {entry['type']!r}")
    mlp = entry.get("mlp")
    if mlp is not None and mlp["kind"] != "dense":
        raise ValueError(f"unknown feed-forward {mlp['kind']!r}")
    return {"mixers": mixers, "ff": mlp["ff"] if mlp is not None else None, "act": FF_ACT}


def read_config(raw: Dict[str, Any]) -> ModelConfig:
    return ModelConfig(family="hybrid", vocab_size=raw["vocab"], hidden_dim=raw["width"], num_layers=len(raw["layers"]),
                       num_heads=1, head_dim=raw["width"], norm="layer", norm_eps=raw["norm"]["eps"], tie_embeddings=False,
                       layers=[layer_spec(e) for e in raw["layers"]]).validate()


# ---- tensor names ----------------------------------------------------------------------------------------------
# Every stored tensor is a view (or several stacked views) of a parameter or buffer of the model.
View = Tuple[str, Any]


def _rows(w: torch.Tensor, col0: int, core: Core, seg: str) -> torch.Tensor:
    a = col0 + core.inputs.at[seg]
    return w[a : a + core.inputs.width[seg]]


def _core_views(core: Core, w_in: torch.Tensor, col0: int, w_out: torch.Tensor, out0: int, p: str) -> Iterator[View]:
    yield p + "o", w_out[:, out0 : out0 + core.out_width]
    if isinstance(core, AttentionCore):
        for n in ("q", "k", "v"):
            yield p + n, _rows(w_in, col0, core, n)
        yield p + "q.norm", core.q_norm
        yield p + "k.norm", core.k_norm
        yield p + "sink", core.sink
        return
    yield p + "A_log", core.A_log
    yield p + "dt_bias", core.dt_bias
    yield p + "norm", core.norm
    ca, cw, u0 = core.conv_at.at, core.conv_at.width, col0 + core.inputs.at["u"]
    if isinstance(core, DeltaCore):
        for n in ("q", "k", "v"):
            yield p + n, w_in[u0 + ca[n] : u0 + ca[n] + cw[n]]
            yield f"{p}{n}.conv", core.conv_w[ca[n] : ca[n] + cw[n]]
        for n in ("b", "a", "g"):
            yield p + n, _rows(w_in, col0, core, n)
        return
    yield p + "D", core.D
    # one stored matrix [z | x | B | C | dt] and one stored convolution over [x | B | C]
    parts = [_rows(w_in, col0, core, "z")] + [w_in[u0 + ca[n] : u0 + ca[n] + cw[n]] for n in ("v", "k", "q")]
    yield p + "in", Stacked(parts + [_rows(w_in, col0, core, "a")])
    yield p + "conv", Stacked([core.conv_w[ca[n] : ca[n] + cw[n]] for n in ("v", "k", "q")])
    yield p + "conv.b", Stacked([core.conv_b[ca[n] : ca[n] + cw[n]] for n in ("v", "k", "q")])


def named_views(model: HybridTransformer) -> Dict[str, Any]:
    out: Dict[str, Any] = {"embed": model.embed.data, "head": model.head.data, "final.norm": model.final_norm.weight}
    for i, l in enumerate(model.layers):
        p = f"l{i}."
        out[p + "norm1"] = l.norm1.weight
        prefixes = [p + "mix."] if len(l.mixer.cores) == 1 else [p + "mix.left.", p + "mix.right."]
        for core, col, o, pre in zip(l.mixer.cores, l.mixer.cols, l.mixer.outs, prefixes):
            out.update(_core_views(core, l.mixer.in_weight.data, col, l.mixer.out_weight.data, o, pre))
        if l.ffn is not None:
            out[p + "norm2"] = l.norm2.weight
            out[p + "mlp.gate"], out[p + "mlp.up"] = l.ffn.gate_up.data[: l.ffn.hidden], l.ffn.gate_up.data[l.ffn.hidden :]
            out[p + "mlp.down"] = l.ffn.down.data
    return out


@register_model("famalorn")
class Famalorn(FolderModel):
    """``Famalorn(config=<dict or path>)`` builds one with zero weights; ``from_pretrained(folder)`` loads one."""

    read_config = staticmethod(read_config)
    named_views = named_views
