"""Configurations and helpers shared by the CPU and GPU tests of heterogeneous-layer models."""

import torch

import hybrid_oracle as oracle


def attn(heads, kv, dim, vdim, rot, base=1e4, scale=None):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "rot": {"dims": rot, "base": base},
            "scale": dim ** -0.5 if scale is None else scale}


def mamba(heads, vdim, state, groups, conv, norm_groups):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def delta(heads, kv, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}


def layer(kind, mixer, ff=None):
    return {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def parallel(left, right, ls=1.0, rs=1.0):
    return {"left": left, "right": right, "left_scale": ls, "right_scale": rs}


CONFIGS = {
    # grouped heads everywhere, key and value sizes that differ, a feed-forward on some layers only
    "grouped": oracle.make_config([
        layer("delta", delta(4, 2, 24, 16, 2)),
        layer("parallel", parallel(attn(4, 2, 16, 24, 8, 1e3, 0.3), mamba(4, 16, 24, 2, 3, 4), 1.3, 0.5), 56),
        layer("mamba2", mamba(6, 8, 16, 3, 4, 2), 32),
    ], vocab=72, width=40),
    # nothing is a multiple of eight; one key head; whole heads rotate; five taps and one tap
    "odd": oracle.make_config([
        layer("parallel", parallel(attn(3, 1, 20, 10, 20, 5e5), mamba(3, 10, 12, 1, 5, 1), 0.7, 1.1), 30),
        layer("delta", delta(3, 3, 12, 20, 1), 18),
        layer("mamba2", mamba(5, 6, 9, 5, 2, 5)),
    ], vocab=51, width=36, eps=1e-4),
    # heads of serving size
    "wide": oracle.make_config([
        layer("mamba2", mamba(4, 64, 128, 1, 4, 2)),
        layer("delta", delta(4, 2, 128, 96, 4), 128),
        layer("parallel", parallel(attn(8, 2, 128, 64, 64), mamba(2, 64, 64, 2, 4, 1), 0.8, 0.6)),
    ], vocab=128, width=96),
    # no rotation at all, every group its own head, ungrouped
    "plain": oracle.make_config([
        layer("parallel", parallel(attn(2, 2, 64, 64, 0), mamba(2, 32, 64, 2, 4, 2)), 64),
        layer("delta", delta(2, 2, 64, 64, 4), 64),
    ], vocab=64, width=64),
}


def build(cfg, W, device="cpu", dtype=torch.float32):
    from triune_b200.models.zoo import MODEL_REGISTRY
    from triune_b200.utils import place_model

    m = MODEL_REGISTRY[cfg["architecture"].lower()](config=cfg)
    m.load_named(W)
    return place_model(m, device, dtype).eval()


def tokens(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def run_portions(model, toks, portions):
    """Logits [len(toks), vocab] of one sequence fed in the given portions (the rest in one)."""
    from triune_b200.inference import advance

    dev = next(model.parameters()).device
    cache, at, out = model.init_cache(1), 0, []
    for n in list(portions) + [len(toks)]:
        part = toks[at : at + n]
        if not part:
            break
        lg, cache = advance(model, torch.tensor([part], device=dev), cache)
        out.append(lg[0].double().cpu())
        at += len(part)
    return torch.cat(out)


def rel(a, b):
    """Largest per-position rms difference over the reference's rms, means taken off."""
    a, b = a.double().cpu(), b.double().cpu()
    d = a - b
    d = d - d.mean(-1, keepdim=True)
    return float(d.pow(2).mean(-1).sqrt().max() / (b - b.mean(-1, keepdim=True)).pow(2).mean().sqrt())
