"""Small Sapanex models for the tests: configurations with unlike sizes and a writer of checkpoint directories."""
import json
import os

import sapanex_oracle as oracle

YARN = {"factor": 8.0, "original": 64, "fast": 16.0, "slow": 1.0}


def attention(heads, kv_heads, dim, vdim, window, pool, rot_dims, ff=0, scale=None, base=10000.0, scaling=YARN):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or 1.3 * dim ** -0.5,
                                           "mask": {"size": window, "pool": pool}, "rot": {"base": base, "dims": rot_dims, "scaling": scaling}},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def general_delta(heads, dim, rank, ff=0):
    """`rank` is kept beside the config (a checkpoint gives it by the shape of a tensor)."""
    return {"type": "general_delta", "mixer": {"heads": heads, "dim": dim}, "mlp": {"kind": "dense", "ff": ff} if ff else None, "rank": rank}


CONFIGS = {
    # nothing is a multiple of 8; windows and pools that do not divide a page, one longer than the other
    "odd": {"vocab": 101, "width": 76, "norm": {"eps": 1e-5}, "embedding": {"scale": 3.0}, "postln_alpha": 1.7, "layers": [
        attention(6, 2, 12, 10, 19, 7, 6, ff=50), general_delta(3, 10, 5), attention(5, 5, 9, 14, 5, 23, 8, ff=30, scaling=None), general_delta(2, 18, 11, ff=44)]},
    # sizes the tensor-core paths take; pools of a few tokens, one that equals a page and one that exceeds it
    "aligned": {"vocab": 192, "width": 128, "norm": {"eps": 1e-6}, "embedding": {"scale": 0.5}, "postln_alpha": 1.0, "layers": [
        general_delta(4, 64, 16, ff=160), attention(8, 2, 32, 48, 30, 4, 16), general_delta(2, 128, 24), attention(6, 2, 80, 24, 64, 64, 80, ff=96, base=500.0),
        attention(4, 4, 64, 64, 21, 70, 32, ff=64)]},
    # pools of one to three tokens (many pooled rows per page), a window of one token, one key / value head, eps that matters
    "fine": {"vocab": 130, "width": 96, "norm": {"eps": 1e-2}, "embedding": {"scale": 7.0}, "postln_alpha": 3.1, "layers": [
        attention(4, 1, 16, 24, 1, 1, 16, ff=40), general_delta(3, 24, 9, ff=56), attention(8, 8, 40, 56, 12, 3, 24), attention(2, 1, 24, 8, 3, 2, 2, ff=24)]},
    # no attention at all, heads past the one-kernel step
    "delta_only": {"vocab": 72, "width": 64, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0}, "postln_alpha": 2.0, "layers": [
        general_delta(2, 32, 8, ff=48), general_delta(1, 144, 6), general_delta(4, 8, 40)]},
    # no recurrent state at all; a window longer than the sequence
    "attention_only": {"vocab": 64, "width": 64, "norm": {"eps": 1e-6}, "embedding": {"scale": 2.0}, "postln_alpha": 1.4, "layers": [
        attention(4, 2, 16, 16, 40, 16, 8, ff=64), attention(2, 2, 16, 40, 1000, 8, 16)]},
}
for _c in CONFIGS.values():
    _c["architecture"] = "Sapanex"
    _c["ranks"] = [s.pop("rank", None) for s in _c["layers"]]


def write_checkpoint(path, cfg, weights):
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump({k: v for k, v in cfg.items() if k != "ranks"}, f)
    save_file({k: v.contiguous() for k, v in weights.items()}, os.path.join(path, "model.safetensors"))
    return str(path)


def build(name, tmp_path, sharp=1.5, seed=3):
    cfg = CONFIGS[name]
    W = oracle.random_weights(cfg, seed, sharp)
    return cfg, W, write_checkpoint(os.path.join(str(tmp_path), name), cfg, W)
