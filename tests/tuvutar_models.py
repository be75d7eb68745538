"""Small Tuvutar models for the tests: configurations with unlike sizes and a writer of checkpoint directories."""
import json
import os

import torch

import tuvutar_oracle as oracle


def latent(heads, dim, rot, vdim, rank, ff=0, src=None, base=1000.0, scaling=None, scale=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale or (dim + rot) ** -0.5,
         "rot": {"base": base, "dims": rot}}
    if scaling:
        m["rot"]["scaling"] = scaling
    if src is not None:
        m["kv_from"] = src
    return {"type": "latent_attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def delta(heads, kv_heads, dim, vdim, conv, ff=0):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


YARN_A = {"factor": 3.0, "original": 96, "fast": 4.0, "slow": 1.0}
YARN_B = {"factor": 8.0, "original": 512, "fast": 32.0, "slow": 1.0}

CONFIGS = {
    # nothing is a multiple of 8; grouped key heads, unequal head sizes, a layer that reads another's rows with its own heads
    "odd": {"vocab": 97, "width": 76, "norm": {"eps": 1e-5}, "layers": [
        latent(3, 12, 4, 20, 28, ff=50, scaling=YARN_A, scale=0.31), delta(6, 2, 10, 14, 3), delta(4, 4, 36, 18, 2, ff=30),
        latent(5, 8, 4, 12, 28, src=0, scaling=YARN_A, scale=0.4)]},
    # sizes the tensor-core paths take; two rotations, rows of two widths, no scaling in the second
    "aligned": {"vocab": 192, "width": 128, "norm": {"eps": 1e-6}, "layers": [
        latent(8, 32, 16, 24, 64, ff=160, base=500.0, scaling=YARN_B), delta(8, 4, 64, 32, 4),
        latent(4, 16, 32, 40, 96, base=20000.0), delta(2, 1, 128, 128, 4, ff=96), latent(16, 24, 32, 16, 96, ff=64, src=2, base=20000.0)]},
    # delta first and last, one head, long convolution, a wide key, eps that matters
    "delta_first": {"vocab": 130, "width": 96, "norm": {"eps": 1e-2}, "layers": [
        delta(3, 1, 144, 24, 5, ff=40), latent(1, 40, 8, 56, 72, base=100.0), delta(1, 1, 16, 88, 4), delta(5, 5, 24, 8, 6)]},
    # no recurrent layer at all
    "latent_only": {"vocab": 64, "width": 64, "norm": {"eps": 1e-6}, "layers": [
        latent(4, 16, 8, 16, 128, ff=64, scaling=YARN_A), latent(2, 16, 8, 16, 128, ff=64, src=0, scaling=YARN_A)]},
}
for _c in CONFIGS.values():
    _c["architecture"] = "Tuvutar"


def write_checkpoint(path, cfg, weights):
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in weights.items()}, os.path.join(path, "model.safetensors"))
    return str(path)


def tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def make_llm(path, dtype, device, pages=12, slots=4, **kw):
    from nanoengine_b200 import LLM, Config
    kw.setdefault("max_num_batched_tokens", pages * 64)
    return LLM(Config(model=path, dtype=dtype, device=device, max_num_seqs=slots, num_kvcache_blocks=pages, max_model_len=pages * 64,
                      enable_prefix_caching=False, executor_backend="inproc", status_log_interval_s=0, **kw))


def feed_all(llm, seq, toks, cuts, seq_id=1, end=True):
    """Feed `toks` cut into portions of the given sizes (the last size repeats); all logits."""
    out, at, k = [], 0, 0
    while at < len(toks):
        n = min(cuts[min(k, len(cuts) - 1)], len(toks) - at)
        out.append(torch.from_numpy(llm.feed([(seq_id, toks[at: at + n])], [list(range(n))])))
        at, k = at + n, k + 1
    if end:
        assert llm.end_feed([seq_id]) == 1
    return torch.cat(out)


def error(got, want):
    """Largest root-mean-square difference of a row of logits, mean taken off, in units of the logits' own spread."""
    want = want.float()
    d = got.float() - want
    d = d - d.mean(-1, keepdim=True)
    return float(d.pow(2).mean(-1).sqrt().max() / (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt())


def build(name, tmp_path, sharp=1.5, seed=3):
    cfg = CONFIGS[name]
    W = oracle.random_weights(cfg, seed, sharp)
    return cfg, W, write_checkpoint(os.path.join(str(tmp_path), name), cfg, W)
