"""Bubitar: the reader of its model folders (``config.json`` + ``model.safetensors``).

A Bubitar is a :class:`HybridTransformer` with RMS norms before and behind every sublayer whose layers are ``retention`` or
``latent_attention`` (multi-head latent attention with a sink and an output gate; ``kv_from`` names an earlier layer whose
latents are read), with clamped gated feed-forwards that have biases, and a token table of which every layer reads its own
part. This module maps its configuration to a :class:`ModelConfig` and its tensor names to the fused weights, both ways."""

from __future__ import annotations

from typing import Any, Dict, Iterator, Optional, Tuple

import torch

from ..config import ModelConfig
from .folder import FolderModel, PerHead, Stacked
from .hybrid import HybridTransformer
from .hybrid_mixers import Mixer, RetentionCore
from .zoo import register_model

FF_ALPHA = 1.702  # slope of the feed-forward's sigmoid


def _rotation(rot: Optional[Dict[str, Any]], dims: Optional[int] = None) -> Dict[str, Any]:
    rot = rot or {"dims": 0, "base": 1.0}
    return {"rot_dims": rot["dims"] if dims is None else dims, "rot_base": rot["base"], "rot_scaling": rot.get("scaling")}


def layer_spec(entry: Dict[str, Any]) -> Dict[str, Any]:
    m, mlp = entry["mixer"], entry.get("mlp")
    if entry["type"] == "retention":
        mixer = {"kind": "retention", **{k: m[k] for k in ("heads", "dim", "vdim", "decay")}, **_rotation(m.get("rot"))}
    elif entry["type"] == "latent_attention":
        mixer = {"kind": "latent", **{k: m[k] for k in ("heads", "dim", "vdim", "kv_rank", "scale")}, **_rotation(m["rot"], m["rot_dim"]),
                 "kv_from": m.get("kv_from")}
    else:
        raise ValueError(f"unknown layer type {entry['type']!r}")
    spec = {"mixers": [mixer], "ff": None}
    if mlp is not None:
        if mlp["kind"] != "dense":
            raise ValueError(f"unknown feed-forward {mlp['kind']!r}")
        spec.update(ff=mlp["ff"], act="clamped", limit=mlp["limit"], alpha=FF_ALPHA, ff_bias=True)
    return spec


def read_config(raw: Dict[str, Any]) -> ModelConfig:
    return ModelConfig(family="hybrid", vocab_size=raw["vocab"], hidden_dim=raw["width"], num_layers=len(raw["layers"]),
                       num_heads=1, head_dim=raw["width"], norm="rms", norm_eps=raw["norm"]["eps"], tie_embeddings=False, post_norm=True,
                       token_side=(raw.get("token_side") or {"dim": 0})["dim"], layers=[layer_spec(e) for e in raw["layers"]]).validate()


def _mixer_views(mixer: Mixer, p: str) -> Iterator[Tuple[str, Any]]:
    core, w = mixer.cores[0], mixer.in_weight.data
    at, width = core.inputs.at, core.inputs.width
    yield p + "o", mixer.out_weight.data[:, : core.out_width]
    yield p + "g", w[at["g"] : at["g"] + width["g"]]
    if isinstance(core, RetentionCore):
        for n in ("q", "k", "v"):
            yield p + n, w[at[n] : at[n] + width[n]]
        return
    D, Dp, R, E, n = core.dim, core.dim_p, core.rot, core.vdim, core.rank
    q = w[at["q"] : at["q"] + width["q"]].view(core.heads, Dp + core.rot_p, -1)
    yield p + "q", PerHead([q[:, :D], q[:, Dp : Dp + R]])
    yield p + "uk", PerHead([core.up.data[:, :D, :n]])
    yield p + "uv", PerHead([core.up.data[:, Dp : Dp + E, :n]])
    yield p + "sink", core.sink
    if core.kv_from is None:
        c = at["c"]
        yield p + "dkv", Stacked([w[c : c + n], w[c + core.rank_p : c + core.rank_p + R]])
        yield p + "dkv.norm", core.c_norm


def named_views(model: HybridTransformer) -> Dict[str, Any]:
    out: Dict[str, Any] = {"embed": model.embed.data, "head": model.head.data, "final.norm": model.final_norm.weight}
    if model.side_embed is not None:
        out["side.embed"] = model.side_embed.data
    for i, l in enumerate(model.layers):
        p = f"l{i}."
        out[p + "norm1"], out[p + "norm1b"] = l.norm1.weight, l.norm1b.weight
        out.update(_mixer_views(l.mixer, p + "mix."))
        if l.ffn is not None:
            F = l.ffn.hidden
            out[p + "norm2"], out[p + "norm2b"] = l.norm2.weight, l.norm2b.weight
            for n, rows in (("gate", slice(0, F)), ("up", slice(F, 2 * F))):
                out[f"{p}mlp.{n}"], out[f"{p}mlp.{n}.b"] = l.ffn.gate_up.data[rows], l.ffn.gate_up_b[rows]
            out[p + "mlp.down"], out[p + "mlp.down.b"] = l.ffn.down.data, l.ffn.down_b
        if l.side is not None:
            out[p + "side.gate"], out[p + "side.proj"], out[p + "side.norm"] = l.side.gate.data, l.side.proj.data, l.side.norm.weight
    return out


@register_model("bubitar")
class Bubitar(FolderModel):
    """``Bubitar(config=<dict or path>)`` builds one with zero weights; ``from_pretrained(folder)`` loads one."""

    read_config = staticmethod(read_config)
    named_views = named_views
