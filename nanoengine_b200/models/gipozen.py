"""Gipozen: a decoder whose config lists every layer - differential attention over a window and the first tokens, with its own sizes and keys and
values of its own or of an earlier layer, and a feed-forward with normed powers, a mixture of clamped gated experts, or none - around a 32-bit
residual stream whose layers are averaged over the depth:

    x <- x + mixer(norm1(x));  X_{i+1} = x + ff(norm2(x));  x <- sum_{j <= i+1} dwa[j] X_j        (X_0: the embeddings)

The results X_j of a step's tokens are kept until the step ends.  One kernel does what lies between two sublayers: the sum, behind a layer the
average, the next sublayer's norm.  Norm weights are single numbers; the factor of the logits is part of the last one.

The paged cache holds the keys of both maps and the values of the layers that have their own, the state pools the windows of every layer's short
convolutions; rows and states are numbered separately."""
from __future__ import annotations

import re
from typing import Dict, Iterable, Tuple

import torch
import torch.nn as nn

from .. import ops
from ..parallel.dist import get_dist_context
from ..runtime.context import ForwardContext
from .config import ModelConfig
from .layers import GatedSharedMoE, PolyNormMLP, QLinear
from .mixers import DifferentialAttentionMixer, _const

GATE_SLOPE = 1.702        # of the sigmoid in the experts


class GipozenLayer(nn.Module):
    def __init__(self, cfg: ModelConfig, layer_idx: int, dtype, device):
        super().__init__()
        spec = cfg.layer_specs[layer_idx]
        m, f, D, eps = spec["mixer"], spec["mlp"], cfg.hidden_size, cfg.rms_norm_eps
        src = cfg.kv_source_layer(layer_idx)
        self.mixer = DifferentialAttentionMixer(D, int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]), int(m["mask"].get("size") or 0),
                                                int(m["mask"].get("keep_first") or 0), float(m["diff"]), int(m["conv"]), eps, cfg.cache_rank(src), src != layer_idx,
                                                cfg.state_rank(layer_idx) if cfg.keeps_state(layer_idx) else None, dtype, device)
        self.norm1, self.norm2 = _const(1, device=device, fill=1.0), _const(1, device=device, fill=1.0)
        self.dwa = _const(layer_idx + 2, device=device)
        self.mlp, self.kind = None, None if f is None else f["kind"]
        if self.kind == "dense":
            self.mlp = PolyNormMLP(D, int(f["ff"]), eps, dtype, device)
        elif self.kind == "moe":
            act = lambda e: ("clamp_linear", float(e["limit"]), GATE_SLOPE)
            r, shared = f["router"], f.get("shared")
            self.mlp = GatedSharedMoE(D, int(r["experts"]), int(r["identity"]), int(r["top"]), int(f["expert"]["ff"]), act(f["expert"]),
                                      int(shared["ff"]) if shared else 0, act(shared) if shared else None, dtype, device)

    def mlp_parts(self) -> Dict[str, Tuple[int, ...]]:
        """Tensor name below the feed-forward -> shape."""
        if self.kind == "dense":
            D, F = self.mlp.up_proj.in_features, self.mlp.up_proj.out_features
            return {"up": (F, D), "down": (D, F), "act": (4,)}
        M, out = self.mlp, {}
        D = M.router_weight.shape[1]
        blocks = [(f"e{e}", M.experts.inter) for e in range(M.num_experts)] + ([("shared", M.shared.down_proj.in_features)] if M.shared is not None else [])
        for n, F in blocks:
            out[n + ".gate"], out[n + ".up"], out[n + ".down"] = (F, D), (F, D), (D, F)
        out["router"], out["correction"] = (M.num_scores, D), (M.num_scores,)
        if M.shared is not None:
            out["shared.sg"] = (1, D)
        return out

    def load_mlp(self, leaf: str, w: torch.Tensor, pending: Dict[str, torch.Tensor]) -> None:
        M = self.mlp
        if self.kind == "dense":
            M.coef.copy_(w) if leaf == "act" else getattr(M, leaf + "_proj").set_weight(w)
        elif leaf == "router":
            M.router_weight[: M.num_scores].copy_(w)
        elif leaf == "correction":
            M.correction.copy_(w)
        elif leaf == "shared.sg":
            M.router_weight[M.num_scores:].copy_(w)
        elif leaf == "shared.down":
            M.shared.down_proj.set_weight(w)
        elif leaf.startswith("shared."):
            pending[leaf] = w
            if len(pending) == 2:
                M.shared.gate_up_proj.set_weight(torch.cat([pending.pop("shared.gate"), pending.pop("shared.up")], 0))
        else:
            e, which = leaf.split(".")
            M.experts.load_expert(int(e[1:]), which, w)


class GipozenForCausalLM(nn.Module):
    def __init__(self, cfg: ModelConfig, dtype=torch.bfloat16, device="cpu", layer_range=None):
        super().__init__()
        assert layer_range is None and get_dist_context().attn_tp_size == 1, "this family runs with attention_tp = pp = 1"
        self.cfg, self.dtype = cfg, dtype
        self.embed_tokens = nn.Embedding(cfg.vocab_size, cfg.hidden_size, dtype=dtype, device=device)
        self.layers = nn.ModuleList([GipozenLayer(cfg, i, dtype, device) for i in range(cfg.num_hidden_layers)])
        self.norm = _const(1, device=device, fill=cfg.logit_scale)          # the last norm's weight times the factor of the logits
        self.lm_head = QLinear(cfg.hidden_size, cfg.vocab_size, dtype, device, None)
        self.trace_residual = None        # a list: receives the stream after every layer (debugging, eager runs only)
        for p in self.parameters():
            p.requires_grad_(False)

    @property
    def num_cache_layers(self) -> int:
        return sum(1 for i in range(self.cfg.num_hidden_layers) if self.cfg.keeps_rows(i))

    def forward(self, input_ids, positions, ctx: ForwardContext, inputs_embeds=None):
        assert inputs_embeds is None, "this family takes token ids"
        eps, n = self.cfg.rms_norm_eps, len(self.layers)
        firsts = [layer.norm1 for layer in self.layers] + [self.norm]
        h, x, bank = ops.depth_embed(input_ids, self.embed_tokens.weight, firsts[0], eps, n + 1)
        for i, layer in enumerate(self.layers):
            y = layer.mixer(h, ctx)
            if layer.mlp is not None:
                h, x = ops.depth_mix(y, x, layer.norm2, eps)
                y = layer.mlp(h)
            h, x = ops.depth_mix(y, x, firsts[i + 1], eps, bank, i + 1, layer.dwa, last=i + 1 == n and self.trace_residual is None)
            if self.trace_residual is not None:
                self.trace_residual.append(x.clone())
        return h

    def compute_logits(self, hidden):
        return ops.lm_head(hidden, self.lm_head.weight)[:, : self.cfg.vocab_size]

    # ---- weights ---------------------------------------------------------------------------
    def load_weights(self, weights: Iterable[Tuple[str, torch.Tensor]]) -> int:
        """Tensors under the design's own names: embed, head, final.norm, l<i>.norm1 / norm2 / dwa, l<i>.mix.<part>, l<i>.mlp.<part>."""
        expected = set(gipozen_param_shapes(self.cfg))
        seen, mixers, pending = set(), {}, {}
        with torch.no_grad():
            for name, t in weights:
                if name not in expected:
                    raise ValueError(f"{name}: no such tensor in this model")
                seen.add(name)
                w = t.float()
                if name == "embed":
                    self.embed_tokens.weight.copy_(w); continue
                if name == "head":
                    self.lm_head.set_weight(w); continue
                if name == "final.norm":
                    self.norm.copy_(w * self.cfg.logit_scale); continue
                li, rest = re.match(r"l(\d+)\.(.+)$", name).groups()
                L = self.layers[int(li)]
                if rest in ("norm1", "norm2", "dwa"):
                    getattr(L, rest).copy_(w)
                elif rest.startswith("mlp."):
                    L.load_mlp(rest[4:], w, pending.setdefault(li, {}))
                else:
                    g = mixers.setdefault(li, {})
                    g[rest[4:]] = w
                    if len(g) == len(L.mixer.parts()):
                        L.mixer.load(mixers.pop(li))
        missing = expected - seen
        if missing:
            raise ValueError(f"incomplete checkpoint: {sorted(missing)[:4]}")
        return len(seen)


def gipozen_param_shapes(cfg: ModelConfig) -> Dict[str, Tuple[int, ...]]:
    """Every tensor name of a checkpoint with its shape."""
    D, V = cfg.hidden_size, cfg.vocab_size
    out: Dict[str, Tuple[int, ...]] = {"embed": (V, D)}
    for i in range(cfg.num_hidden_layers):
        p, layer = f"l{i}.", GipozenLayer(cfg, i, torch.bfloat16, "meta")
        out[p + "norm1"], out[p + "dwa"] = (), (i + 2,)
        out.update({p + "mix." + n: shape for n, shape in layer.mixer.parts().items()})
        if layer.mlp is not None:
            out[p + "norm2"] = ()
            out.update({p + "mlp." + n: shape for n, shape in layer.mlp_parts().items()})
    out["final.norm"], out["head"] = (), (V, D)
    return out


def gipozen_random_tensor(name: str, shape, g: torch.Generator, dev) -> torch.Tensor:
    """A random tensor of a sensible size for its role: matrices scaled by their fan-in, norms around one, averages that keep the newest layer."""
    t = torch.randn(shape, generator=g, device=dev, dtype=torch.float32)
    leaf = name.rsplit(".", 1)[-1]
    if leaf.startswith("norm"):
        return 1.0 + 0.1 * t
    if leaf == "dwa":
        t = 0.1 * t
        t[-1] += 1.0
        return t
    if leaf == "act":
        return 0.3 + 0.1 * t
    if leaf in ("lq1", "lk1", "lq2", "lk2"):
        return t * (0.3 * shape[0] ** -0.25)
    if leaf == "correction":
        return 0.01 * t
    return t * (1.0 if name == "embed" else 0.5 if leaf == "conv" else shape[-1] ** -0.5)
