"""Small Filasun models for the tests: configurations with unlike sizes and a writer of checkpoint directories."""
import json
import os

import torch

import filasun_oracle as oracle


def mamba2(heads, vdim, state, groups=1, conv=4, norm_groups=1, ff=0, limit=2.0):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups},
            "mlp": {"kind": "dense", "ff": ff, "limit": limit} if ff else None}


def parallel(heads, kv_heads, dim, vdim, window, r_heads, r_dim, r_vdim, decay=None, ff=0, softcap=20.0, scale=None, scales=(0.8, 0.4), limit=1.2):
    decay = decay or [1.0 - 0.5 ** (1 + 2 * h) for h in range(r_heads)]
    return {"type": "parallel", "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or 1.7 * dim ** -0.5, "softcap": softcap, "mask": {"size": window}},
        "right": {"heads": r_heads, "dim": r_dim, "vdim": r_vdim, "decay": decay}, "left_scale": scales[0], "right_scale": scales[1]},
        "mlp": {"kind": "dense", "ff": ff, "limit": limit} if ff else None}


CONFIGS = {
    # nothing is a multiple of 8; groups of heads everywhere, norm in parts, three streams
    "odd": {"vocab": 97, "width": 76, "norm": {"eps": 1e-5}, "streams": 3, "logit_softcap": 9.0, "max_positions": 400, "layers": [
        parallel(6, 2, 12, 20, 33, 3, 10, 14, ff=50), mamba2(6, 10, 14, groups=3, conv=3, norm_groups=4), parallel(5, 5, 9, 7, 90, 2, 17, 5, ff=30),
        mamba2(3, 18, 36, groups=1, conv=2, norm_groups=1, ff=44)]},
    # sizes the tensor-core paths take; windows of a page, less and more; grouped and single key / value heads
    "aligned": {"vocab": 192, "width": 128, "norm": {"eps": 1e-6}, "streams": 2, "logit_softcap": 30.0, "max_positions": 600, "layers": [
        parallel(8, 2, 32, 48, 64, 4, 64, 24, ff=160, softcap=8.0), mamba2(8, 32, 64, groups=2, conv=4, norm_groups=2), parallel(6, 2, 80, 24, 21, 2, 128, 128),
        parallel(4, 4, 64, 64, 130, 8, 16, 64, ff=96, softcap=50.0, scales=(1.0, 1.0))]},
    # Mamba-2 first and last, long convolution, one stream, eps that matters, a window of one token, decays of zero and one
    "mamba_first": {"vocab": 130, "width": 96, "norm": {"eps": 1e-2}, "streams": 1, "logit_softcap": 12.0, "max_positions": 520, "layers": [
        mamba2(3, 24, 144, groups=1, conv=5, norm_groups=3, ff=40), parallel(1, 1, 40, 56, 1, 4, 24, 8, decay=[0.0, 0.5, 0.99, 1.0], scales=(0.5, 1.5)),
        mamba2(4, 88, 16, groups=4, conv=1), mamba2(8, 16, 128, groups=8, conv=9, norm_groups=8)]},
    # no Mamba-2 layer, five streams, windows longer than the sequence
    "parallel_only": {"vocab": 64, "width": 64, "norm": {"eps": 1e-6}, "streams": 5, "logit_softcap": 15.0, "max_positions": 300, "layers": [
        parallel(4, 1, 16, 16, 1000, 4, 16, 16, ff=64), parallel(2, 2, 16, 40, 128, 1, 72, 16, ff=64)]},
    # no attention at all
    "mamba_only": {"vocab": 72, "width": 64, "norm": {"eps": 1e-6}, "streams": 2, "logit_softcap": 15.0, "max_positions": 300, "layers": [
        mamba2(4, 16, 32, groups=1, conv=4, ff=48), mamba2(2, 32, 16, groups=2, conv=3, norm_groups=2)]},
}
for _c in CONFIGS.values():
    _c["architecture"] = "Filasun"


def write_checkpoint(path, cfg, weights):
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in weights.items()}, os.path.join(path, "model.safetensors"))
    return str(path)


def build(name, tmp_path, sharp=1.5, seed=3):
    cfg = CONFIGS[name]
    W = oracle.random_weights(cfg, seed, sharp)
    return cfg, W, write_checkpoint(os.path.join(str(tmp_path), name), cfg, W)
