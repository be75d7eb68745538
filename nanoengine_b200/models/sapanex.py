"""Sapanex: a decoder whose config lists every layer - attention over a window and pooled blocks, or a generalised delta rule, each with its own
sizes, and a feed-forward with squared relu or none - around a 32-bit residual stream with the norm behind the sum:

    x <- norm1(alpha x + mixer(x));  x <- norm2(alpha x + ff(x))

Sublayers read the stream itself; one kernel does the sum, the norm and the copy in the activation dtype.  Token embeddings enter scaled; the
same table, unscaled, gives the logits.

The paged cache holds tokens and pooled blocks of the attention layers, the state pools the delta layers; both are indexed by a layer's rank
among its kind."""
from __future__ import annotations

import re
from typing import Dict, Iterable, Tuple

import torch
import torch.nn as nn

from .. import ops
from ..ops import reference as ref
from ..parallel.dist import get_dist_context
from ..runtime.context import ForwardContext
from .config import ModelConfig, _yarn_of
from .layers import DenseMLP, QLinear, RMSNorm
from .mixers import GeneralDeltaMixer, PooledAttentionMixer


class SapanexLayer(nn.Module):
    def __init__(self, cfg: ModelConfig, layer_idx: int, dtype, device):
        super().__init__()
        spec = cfg.layer_specs[layer_idx]
        m, D, eps = spec["mixer"], cfg.hidden_size, cfg.rms_norm_eps
        self.kind = spec["type"]
        if self.kind == "attention":
            self.mixer = PooledAttentionMixer(D, int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]), int(m["mask"]["size"]),
                                              int(m["mask"]["pool"]), eps, cfg.cache_rank(layer_idx), dtype, device)
            sc = _yarn_of(m["rot"].get("scaling"))
            base = float(m["rot"]["base"])
            # the rotations of keys and of values: (dims, base, scaling)
            self.rope_keys = ((int(m["rot"]["dims"]), base, None if sc is None else tuple(sorted(sc.items()))), (int(m["vdim"]), base, None))
        else:
            self.mixer = GeneralDeltaMixer(D, int(m["heads"]), int(m["dim"]), int(m["decay_rank"]), eps, cfg.state_rank(layer_idx), dtype, device)
        self.norm1 = RMSNorm(D, eps, dtype, device)
        self.mlp = None
        if spec["mlp"] is not None:
            self.norm2 = RMSNorm(D, eps, dtype, device)
            self.mlp = DenseMLP(D, int(spec["mlp"]["ff"]), dtype, device, act="relu2")


class SapanexForCausalLM(nn.Module):
    def __init__(self, cfg: ModelConfig, dtype=torch.bfloat16, device="cpu", layer_range=None):
        super().__init__()
        assert layer_range is None and get_dist_context().attn_tp_size == 1, "this family runs with attention_tp = pp = 1"
        self.cfg, self.dtype = cfg, dtype
        self.layers = nn.ModuleList([SapanexLayer(cfg, i, dtype, device) for i in range(cfg.num_hidden_layers)])
        self.norm = RMSNorm(cfg.hidden_size, cfg.rms_norm_eps, dtype, device)
        self.embed_tokens = QLinear(cfg.hidden_size, cfg.vocab_size, dtype, device)      # the table, and the head's weight
        # one rotary table per distinct rotation among the layers
        self._rope: Dict[Tuple, str] = {}
        for layer in self.layers:
            for key in layer.rope_keys if layer.kind == "attention" else ():
                if key not in self._rope:
                    dims, base, sc = key
                    self._rope[key] = f"rope_{len(self._rope)}"
                    table = ref.rope_cos_sin_cache(dims, cfg.max_position_embeddings, base, None if sc is None else dict(sc), exact=True)
                    self.register_buffer(self._rope[key], table.to(device), persistent=False)
        self.trace_residual = None        # a list: receives the residual stream after every layer (debugging, eager runs only)
        for p in self.parameters():
            p.requires_grad_(False)

    @property
    def num_cache_layers(self) -> int:
        return sum(1 for i in range(self.cfg.num_hidden_layers) if self.cfg.keeps_rows(i))

    def _mix(self, layer: SapanexLayer, h, positions, ctx: ForwardContext):
        if layer.kind != "attention":
            return layer.mixer(h, ctx)
        return layer.mixer(h, positions, ctx, *(getattr(self, self._rope[k]) for k in layer.rope_keys))

    def forward(self, input_ids, positions, ctx: ForwardContext, inputs_embeds=None):
        assert inputs_embeds is None, "this family takes token ids"
        alpha, eps = self.cfg.postnorm_alpha, self.cfg.rms_norm_eps
        h, x = ops.embed_scaled(input_ids, self.embed_tokens.weight[: self.cfg.vocab_size], self.cfg.embedding_scale)
        for i, layer in enumerate(self.layers):
            w_last = self.norm.weight if i + 1 == len(self.layers) else None
            h, x = ops.postnorm(self._mix(layer, h, positions, ctx), x, alpha, layer.norm1.weight, eps, w_last if layer.mlp is None else None)
            if layer.mlp is not None:
                h, x = ops.postnorm(layer.mlp(h), x, alpha, layer.norm2.weight, eps, w_last)
            if self.trace_residual is not None:
                self.trace_residual.append(x.clone())
        return h

    def compute_logits(self, hidden):
        return ops.lm_head(hidden, self.embed_tokens.weight)[:, : self.cfg.vocab_size]

    # ---- weights ---------------------------------------------------------------------------
    def load_weights(self, weights: Iterable[Tuple[str, torch.Tensor]]) -> int:
        """Tensors under the design's own names: embed, final.norm, l<i>.norm1 / norm2, l<i>.mix.<part>, l<i>.mlp.up / down."""
        expected = set(sapanex_param_shapes(self.cfg))
        seen, mixers = set(), {}
        with torch.no_grad():
            for name, t in weights:
                if name not in expected:
                    raise ValueError(f"{name}: no such tensor in this model")
                seen.add(name)
                w = t.float()
                if name == "embed":
                    self.embed_tokens.set_weight(w); continue
                if name == "final.norm":
                    self.norm.weight.copy_(w); continue
                li, rest = re.match(r"l(\d+)\.(.+)$", name).groups()
                L = self.layers[int(li)]
                if rest in ("norm1", "norm2"):
                    getattr(L, rest).weight.copy_(w)
                elif rest in ("mlp.up", "mlp.down"):
                    (L.mlp.up_proj if rest == "mlp.up" else L.mlp.down_proj).set_weight(w)
                else:
                    g = mixers.setdefault(li, {})
                    g[rest[4:]] = w
                    if len(g) == len(L.mixer.parts()):
                        L.mixer.load(mixers.pop(li))
        missing = expected - seen
        if missing:
            raise ValueError(f"incomplete checkpoint: {sorted(missing)[:4]}")
        return len(seen)


def sapanex_param_shapes(cfg: ModelConfig) -> Dict[str, Tuple[int, ...]]:
    """Every tensor name of a checkpoint with its shape."""
    D = cfg.hidden_size
    out: Dict[str, Tuple[int, ...]] = {"embed": (cfg.vocab_size, D)}
    for i in range(cfg.num_hidden_layers):
        p, layer = f"l{i}.", SapanexLayer(cfg, i, torch.bfloat16, "meta")
        out[p + "norm1"] = (D,)
        for n, shape in layer.mixer.parts().items():
            out[p + "mix." + n] = shape
        if layer.mlp is not None:
            F = layer.mlp.down_proj.in_features
            out[p + "norm2"], out[p + "mlp.up"], out[p + "mlp.down"] = (D,), (F, D), (D, F)
    out["final.norm"] = (D,)
    return out


def sapanex_random_tensor(name: str, shape, g: torch.Generator, dev) -> torch.Tensor:
    """A random tensor of a sensible size for its role: matrices scaled by their fan-in, norms around one, slow decays."""
    t = torch.randn(shape, generator=g, device=dev, dtype=torch.float32)
    leaf = name.rsplit(".", 1)[-1]
    if leaf.startswith("norm"):
        return 1.0 + 0.1 * t
    if leaf == "w0":
        return t - 2.0
    return t * (1.0 if name == "embed" or name.endswith("a.b") else shape[-1] ** -0.5)
