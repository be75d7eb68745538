"""Filasun: a decoder whose config lists every layer - a Mamba-2 mixer, or windowed attention and decayed linear attention side by side, each
with its own sizes, and a clamped gated feed-forward or none - around several residual streams with constant hyper-connections.

    u = sum_s in_s x_s;   y = sublayer(rmsnorm(u));   x_t <- sum_s mix[s, t] x_s + out_t y       (32-bit; per sublayer)

The streams start as token embedding + learned position vector and are summed in front of the last norm; the logits are soft-capped.
One kernel does what lies between two sublayers: the mix of the streams, the next sublayer's read of them and its norm.

The paged cache holds the keys and values of the parallel layers, the state pools their linear attention's states and the Mamba-2 layers'
states and convolution windows; a parallel layer is counted in both."""
from __future__ import annotations

import re
from typing import Dict, Iterable, Tuple

import torch
import torch.nn as nn

from .. import ops
from ..parallel.dist import get_dist_context
from ..runtime.context import ForwardContext
from .config import ModelConfig
from .layers import QLinear, RMSNorm, SwiGLUMLP
from .mixers import Mamba2Mixer, ParallelMixer

GATE_SLOPE = 1.702        # of the sigmoid in the feed-forward


class StreamWeights(nn.Module):
    """Constant hyper-connection of one sublayer: how it reads the streams, how its output enters them, how they mix ([from, to])."""

    def __init__(self, streams: int, device):
        super().__init__()
        self.w_in = nn.Parameter(torch.ones(streams, dtype=torch.float32, device=device), requires_grad=False)
        self.w_out = nn.Parameter(torch.ones(streams, dtype=torch.float32, device=device), requires_grad=False)
        self.mix = nn.Parameter(torch.eye(streams, dtype=torch.float32, device=device), requires_grad=False)


class FilasunLayer(nn.Module):
    def __init__(self, cfg: ModelConfig, layer_idx: int, dtype, device):
        super().__init__()
        spec = cfg.layer_specs[layer_idx]
        m, D, eps = spec["mixer"], cfg.hidden_size, cfg.rms_norm_eps
        norm = lambda: RMSNorm(D, eps, dtype, device)
        if spec["type"] == "mamba2":
            self.mixer = Mamba2Mixer(D, int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"]), int(m["conv"]), int(m["norm_groups"]), eps,
                                     cfg.state_rank(layer_idx), dtype, device)
        else:
            l, r = m["left"], m["right"]
            self.mixer = ParallelMixer(D, int(l["heads"]), int(l["kv_heads"]), int(l["dim"]), int(l["vdim"]), float(l["scale"]), float(l["softcap"]),
                                       int(l["mask"]["size"]), int(r["heads"]), int(r["dim"]), int(r["vdim"]), r["decay"], float(m["left_scale"]),
                                       float(m["right_scale"]), eps, cfg.cache_rank(layer_idx), cfg.state_rank(layer_idx), dtype, device)
        self.norm1, self.hc1 = norm(), StreamWeights(cfg.hc_mult, device)
        self.mlp = None
        if spec["mlp"] is not None:
            self.norm2, self.hc2 = norm(), StreamWeights(cfg.hc_mult, device)
            self.mlp = SwiGLUMLP(D, int(spec["mlp"]["ff"]), dtype, device, None, act=("clamp_linear", float(spec["mlp"]["limit"]), GATE_SLOPE))


class FilasunForCausalLM(nn.Module):
    def __init__(self, cfg: ModelConfig, dtype=torch.bfloat16, device="cpu", layer_range=None):
        super().__init__()
        assert layer_range is None and get_dist_context().attn_tp_size == 1, "this family runs with attention_tp = pp = 1"
        self.cfg, self.dtype = cfg, dtype
        self.embed_tokens = nn.Embedding(cfg.vocab_size, cfg.hidden_size, dtype=dtype, device=device)
        self.embed_positions = nn.Embedding(cfg.max_position_embeddings, cfg.hidden_size, dtype=dtype, device=device)
        self.layers = nn.ModuleList([FilasunLayer(cfg, i, dtype, device) for i in range(cfg.num_hidden_layers)])
        self.norm = RMSNorm(cfg.hidden_size, cfg.rms_norm_eps, dtype, device)
        self.lm_head = QLinear(cfg.hidden_size, cfg.vocab_size, dtype, device, None)
        self.register_buffer("stream_sum", torch.ones(cfg.hc_mult, dtype=torch.float32, device=device), persistent=False)
        self.trace_residual = None        # a list: receives the sum of the streams after every layer (debugging, eager runs only)
        for p in self.parameters():
            p.requires_grad_(False)

    @property
    def num_cache_layers(self) -> int:
        return sum(1 for i in range(self.cfg.num_hidden_layers) if self.cfg.keeps_rows(i))

    def forward(self, input_ids, positions, ctx: ForwardContext, inputs_embeds=None):
        assert inputs_embeds is None, "this family takes token ids"
        eps, subs = self.cfg.rms_norm_eps, []
        for layer in self.layers:
            subs.append((layer.norm1, layer.hc1, lambda h, m=layer.mixer: m(h, ctx)))
            if layer.mlp is not None:
                subs.append((layer.norm2, layer.hc2, layer.mlp))
        reads = [(hc.w_in, norm.weight) for norm, hc, _ in subs] + [(self.stream_sum, self.norm.weight)]
        h, x = ops.stream_embed(input_ids, positions, self.embed_tokens.weight, self.embed_positions.weight, *reads[0], eps)
        for i, (_, hc, fn) in enumerate(subs):
            last = i + 1 == len(subs) and self.trace_residual is None
            h, x = ops.stream_mix(fn(h), x, hc.w_out, hc.mix, *reads[i + 1], eps, last)
            if self.trace_residual is not None and (i + 1 == len(subs) or subs[i + 1][0] in self._firsts()):
                self.trace_residual.append(x.sum(1))
        return h

    def _firsts(self):
        return [layer.norm1 for layer in self.layers]

    def compute_logits(self, hidden):
        return ops.cap_logits(ops.lm_head(hidden, self.lm_head.weight), self.cfg.final_logit_softcapping)[:, : self.cfg.vocab_size]

    # ---- weights ---------------------------------------------------------------------------
    def load_weights(self, weights: Iterable[Tuple[str, torch.Tensor]]) -> int:
        """Tensors under the design's own names: embed, pos, head, final.norm, l<i>.norm1 / norm2, l<i>.hc1 / hc2.in / out / mix, l<i>.mix.<part>,
        l<i>.mlp.gate / up / down."""
        expected = set(filasun_param_shapes(self.cfg))
        seen, mixers, gu = set(), {}, {}
        with torch.no_grad():
            for name, t in weights:
                if name not in expected:
                    raise ValueError(f"{name}: no such tensor in this model")
                seen.add(name)
                w = t.float()
                if name == "embed":
                    self.embed_tokens.weight.copy_(w); continue
                if name == "pos":
                    self.embed_positions.weight.copy_(w); continue
                if name == "head":
                    self.lm_head.set_weight(w); continue
                if name == "final.norm":
                    self.norm.weight.copy_(w); continue
                li, rest = re.match(r"l(\d+)\.(.+)$", name).groups()
                L = self.layers[int(li)]
                if rest in ("norm1", "norm2"):
                    getattr(L, rest).weight.copy_(w)
                elif rest.startswith("hc"):
                    hc, leaf = rest.split(".")
                    getattr(getattr(L, hc), {"in": "w_in", "out": "w_out", "mix": "mix"}[leaf]).copy_(w)
                elif rest == "mlp.down":
                    L.mlp.down_proj.set_weight(w)
                elif rest.startswith("mlp."):
                    g = gu.setdefault(li, {})
                    g[rest[4:]] = w
                    if len(g) == 2:
                        L.mlp.gate_up_proj.set_weight(torch.cat([g["gate"], g["up"]], 0))
                        gu.pop(li)
                else:
                    g = mixers.setdefault(li, {})
                    g[rest[4:]] = w
                    if len(g) == len(L.mixer.parts()):
                        L.mixer.load(g)
                        mixers.pop(li)
        missing = expected - seen
        if missing:
            raise ValueError(f"incomplete checkpoint: {sorted(missing)[:4]}")
        return len(seen)


def filasun_param_shapes(cfg: ModelConfig) -> Dict[str, Tuple[int, ...]]:
    """Every tensor name of a checkpoint with its shape."""
    D, V, S = cfg.hidden_size, cfg.vocab_size, cfg.hc_mult
    out: Dict[str, Tuple[int, ...]] = {"embed": (V, D), "pos": (cfg.max_position_embeddings, D)}
    for i in range(cfg.num_hidden_layers):
        p, layer = f"l{i}.", FilasunLayer(cfg, i, torch.bfloat16, "meta")
        for q in (1, 2) if layer.mlp is not None else (1,):
            out[f"{p}norm{q}"], out[f"{p}hc{q}.in"], out[f"{p}hc{q}.out"], out[f"{p}hc{q}.mix"] = (D,), (S,), (S,), (S, S)
        for n, shape in layer.mixer.parts().items():
            out[p + "mix." + n] = shape
        if layer.mlp is not None:
            F = layer.mlp.down_proj.in_features
            out[p + "mlp.gate"], out[p + "mlp.up"], out[p + "mlp.down"] = (F, D), (F, D), (D, F)
    out["final.norm"], out["head"] = (D,), (V, D)
    return out


def filasun_random_tensor(name: str, shape, g: torch.Generator, dev) -> torch.Tensor:
    """A random tensor of a sensible size for its role: matrices scaled by their fan-in, norms around one, streams that keep their size."""
    t = torch.randn(shape, generator=g, device=dev, dtype=torch.float32)
    leaf = name.rsplit(".", 1)[-1]
    if ".hc" in name:
        S = shape[0]
        return 0.1 * t + (torch.eye(S, device=dev) * 0.9 if leaf == "mix" else 1.0 / S if leaf == "in" else 1.0)
    if leaf.startswith("norm"):
        return 1.0 + 0.1 * t
    if leaf in ("A_log", "D", "b"):
        return (0.5 if leaf == "A_log" else 0.1) * t
    if leaf == "dt_bias":
        return 0.5 * t - 2.0
    return t * (1.0 if name == "embed" else 0.3 if name == "pos" else 0.5 if leaf == "conv" else shape[-1] ** -0.5)
