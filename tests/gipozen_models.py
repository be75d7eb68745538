"""Small Gipozen models for the tests: configurations with unlike sizes and a writer of checkpoint directories."""
import os

import gipozen_oracle as oracle
from tuvutar_models import write_checkpoint

__all__ = ["CONFIGS", "attention", "build", "dense", "moe", "write_checkpoint"]


def attention(heads, kv_heads, dim, vdim, size, keep, conv, diff, mlp=None, src=None, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or 1.3 * dim ** -0.5, "conv": conv, "diff": diff,
         "mask": {"size": size, "keep_first": keep}}
    if src is not None:
        m["kv_from"] = src
    return {"type": "attention", "mixer": m, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, identity, top, ff, shared, limit, shared_limit=None):
    out = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "identity": identity, "top": top}}
    if shared:
        out["shared"] = {"ff": shared, "limit": shared_limit or limit}
    return out


def model(vocab, width, eps, logit_scale, layers):
    return {"architecture": "Gipozen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale, "layers": layers}


CONFIGS = {
    # nothing is a multiple of 8; windows that do not divide a page, kept tokens across a page's edge, two readers of one layer with masks of their own
    "odd": model(101, 76, 1e-5, 0.7, [attention(6, 2, 11, 10, 19, 3, 4, 0.3, dense(50)), attention(6, 2, 11, 10, 7, 70, 3, 0.8, moe(5, 3, 2, 30, 44, 0.6, 1.1), src=0),
                                      attention(3, 3, 9, 14, 33, 0, 2, 0.1), attention(8, 2, 11, 10, 100, 1, 5, 0.45, moe(7, 1, 4, 18, 26, 3.0), src=0)]),
    # sizes the tensor-core paths take
    "aligned": model(192, 128, 1e-6, 3.0, [attention(8, 2, 32, 48, 40, 5, 4, 0.25, dense(160)), attention(4, 4, 64, 64, 21, 70, 2, 0.6, moe(12, 4, 5, 64, 96, 0.8, 0.5)),
                                           attention(8, 2, 32, 48, 90, 9, 3, 0.5, moe(6, 2, 3, 128, 40, 2.0), src=0), attention(6, 1, 80, 72, 64, 64, 4, 0.35, dense(96))]),
    # a window of one token, one key / value head, one tap, no identity experts, a single choice, no shared expert, eps that matters
    "fine": model(130, 96, 1e-2, 1.0, [attention(4, 1, 16, 24, 1, 1, 1, 0.2, moe(4, 0, 1, 40, 0, 1.5)), attention(8, 8, 40, 56, 12, 0, 7, 0.9, dense(56)),
                                       attention(2, 1, 24, 8, 3, 2, 2, 0.4, moe(3, 1, 4, 24, 16, 0.4)), attention(4, 1, 16, 24, 30, 12, 1, 0.7, src=0)]),
    # no convolution anywhere: no state; a window longer than the sequence
    "stateless": model(64, 64, 1e-6, 0.4, [attention(4, 2, 16, 16, 30, 6, 1, 0.3, dense(64)), attention(4, 2, 16, 16, 1000, 0, 1, 0.3, moe(4, 2, 2, 32, 32, 2.0), src=0),
                                           attention(2, 2, 16, 40, 50, 3, 1, 0.55)]),
}


def build(name, tmp_path, sharp=1.5, seed=3):
    cfg = CONFIGS[name]
    W = oracle.random_weights(cfg, seed, sharp)
    return cfg, W, write_checkpoint(os.path.join(str(tmp_path), name), cfg, W)
