"""Configurations shared by the CPU and GPU tests of Bubitar models."""

import bubitar_oracle as oracle


def retention(heads, dim, vdim, decay, rot=None, base=1e4):
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay,
                                           "rot": {"dims": dim if rot is None else rot, "base": base}}}


def latent(heads, dim, rot_dim, vdim, rank, scale, base=1e4, scaling=None, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale,
         "rot": {"dims": rot_dim, "base": base, **({"scaling": scaling} if scaling else {})}}
    return {"type": "latent_attention", "mixer": m if kv_from is None else {**m, "kv_from": kv_from}}


def with_mlp(layer, ff=None, limit=1.0):
    return {**layer, "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


YARN = {"factor": 8.0, "original": 64, "fast": 8.0, "slow": 1.0}

CONFIGS = {
    # an own latent first, then read by layers with other heads and value sizes; a feed-forward on some layers only
    "shared": oracle.make_config([
        with_mlp(latent(4, 16, 8, 24, 32, 0.3, 1e3, YARN), 64, 0.7),
        with_mlp(retention(4, 16, 24, [0.5, 0.9, 0.99, 1.0], 8), 32, 2.0),
        with_mlp(latent(2, 24, 8, 16, 32, 0.2, 1e3, YARN, kv_from=0), 48, 1.2),
        with_mlp(latent(6, 8, 4, 8, 16, 0.4)),
        with_mlp(latent(3, 16, 4, 40, 16, 0.25, kv_from=3), 32, 0.4),
    ], vocab=72, width=40),
    # nothing is a multiple of eight
    "odd": oracle.make_config([
        with_mlp(retention(3, 20, 10, [0.25, 0.875, 0.999], 12, 5e5), 30, 0.9),
        with_mlp(latent(3, 10, 6, 14, 20, 0.35, 1e3, {"factor": 2.5, "original": 40, "fast": 4.0, "slow": 0.5}), 18, 1.5),
        with_mlp(retention(1, 6, 5, [0.95])),
        with_mlp(latent(5, 7, 6, 9, 20, 0.3, 1e3, {"factor": 2.5, "original": 40, "fast": 4.0, "slow": 0.5}, kv_from=1), 21, 0.8),
    ], vocab=51, width=36, eps=1e-4, side=5),
    # heads of serving size
    "wide": oracle.make_config([
        with_mlp(retention(2, 128, 128, [0.95, 0.9975]), 128, 1.3),
        with_mlp(latent(4, 128, 64, 128, 256, 0.07, 1e5, {"factor": 6.0, "original": 128, "fast": 24.0, "slow": 1.0}), 64, 2.0),
        with_mlp(retention(3, 64, 192, [0.9375, 0.99, 0.999], 32)),
        with_mlp(latent(20, 64, 32, 64, 256, 0.1)),
    ], vocab=128, width=96, side=16),
    # one head of everything, no rotation in the retention
    "single": oracle.make_config([
        with_mlp(latent(1, 32, 16, 32, 64, 0.14), 64),
        with_mlp(retention(1, 32, 32, [0.985], 0), 32),
    ], vocab=64, width=64, side=8),
}
