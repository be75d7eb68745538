"""Tuvutar: a decoder whose config lists every layer - a latent-attention or a gated delta-rule mixer with its own sizes, and a
dense GELU feed-forward or none - inside a 32-bit residual stream with a norm before and after every sublayer.

    x <- x + norm1b(mixer(norm1(x)));  x <- x + norm2b(ff(norm2(x)))      (norm weights stored as the deviation from one)

Latent attention   the MLA layer of this package (`deepseek.MLAAttention`) without a query bottleneck: [q | latent | rotary key] from
                   one GEMM, pages of [normed latent | rotated key part], the absorbed form for every step (prompts without a
                   prefix take the expanded form where the tensor-core kernel covers the head sizes).  A layer with `kv_from` has no
                   latent projection and reads the rows an earlier layer stored.
Delta              the gated delta-net of this package (`qwen3_5.GatedDeltaNet`) with everything between its projections in 32-bit.

The paged cache holds the latent layers that keep rows, the state pools the delta layers; both are indexed by a layer's rank
among its kind.  The residual add, the norm after a sublayer and the norm before the next one are one kernel.
"""
from __future__ import annotations

import re
from typing import Dict, Iterable, Tuple

import torch
import torch.nn as nn

from .. import ops
from ..ops import reference as ref
from ..parallel.dist import get_dist_context
from ..runtime.context import ForwardContext
from .config import ModelConfig
from .deepseek import MLAAttention
from .layers import QLinear, RMSNorm, SwiGLUMLP
from .qwen3_5 import GatedDeltaNet


class TuvutarLayer(nn.Module):
    def __init__(self, cfg: ModelConfig, layer_idx: int, dtype, device):
        super().__init__()
        lc = cfg.layer_config(layer_idx)
        self.kind = cfg.layer_type(layer_idx)
        if self.kind == "full_attention":
            src = cfg.kv_source_layer(layer_idx)
            rank = sum(1 for j in range(src) if cfg.layer_type(j) == "full_attention" and cfg.kv_source_layer(j) == j)
            self.mixer = MLAAttention(lc, layer_idx, dtype, device, cache_idx=rank, merged_kv=True, reads_only=src != layer_idx)
            self.rope_key = rope_key(lc)
        else:
            self.mixer = GatedDeltaNet(lc, cfg.num_layers_of("linear_attention", layer_idx), dtype, device, exact=True)
        norm = lambda: RMSNorm(cfg.hidden_size, cfg.rms_norm_eps, dtype, device, unit_offset=cfg.norm_unit_offset)
        self.norm1, self.norm1b = norm(), norm()
        self.mlp = None
        if cfg.layer_specs[layer_idx]["mlp"] is not None:
            self.norm2, self.norm2b = norm(), norm()
            self.mlp = SwiGLUMLP(cfg.hidden_size, lc.intermediate_size, dtype, device, None, act=lc.glu_act)

    def forward(self, h, x, next_norm: RMSNorm, positions, ctx: ForwardContext, rope: Dict):
        """h: this layer's normed input, x: the residual stream.  Returns the next sublayer's input and the stream."""
        y = self.mixer(h, ctx) if self.kind == "linear_attention" else self.mixer(h, positions, ctx, rope[self.rope_key])
        if self.mlp is None:
            return ops.residual_norm(y, x, self.norm1b.weight, next_norm.weight, next_norm.eps, next_norm.unit_offset)
        h, x = ops.residual_norm(y, x, self.norm1b.weight, self.norm2.weight, self.norm2.eps, self.norm2.unit_offset)
        return ops.residual_norm(self.mlp(h), x, self.norm2b.weight, next_norm.weight, next_norm.eps, next_norm.unit_offset)


def rope_key(lc: ModelConfig) -> Tuple:
    sc = lc.rope_scaling
    return (lc.qk_rope_head_dim, lc.rope_theta, None if sc is None else tuple(sorted(sc.items())))


class TuvutarForCausalLM(nn.Module):
    def __init__(self, cfg: ModelConfig, dtype=torch.bfloat16, device="cpu", layer_range=None):
        super().__init__()
        assert layer_range is None and get_dist_context().attn_tp_size == 1, "this family runs with attention_tp = pp = 1"
        self.cfg, self.dtype = cfg, dtype
        self.embed_tokens = nn.Embedding(cfg.vocab_size, cfg.hidden_size, dtype=dtype, device=device)
        self.layers = nn.ModuleList([TuvutarLayer(cfg, i, dtype, device) for i in range(cfg.num_hidden_layers)])
        self.norm = RMSNorm(cfg.hidden_size, cfg.rms_norm_eps, dtype, device, unit_offset=cfg.norm_unit_offset)
        self.lm_head = QLinear(cfg.hidden_size, cfg.vocab_size, dtype, device, None)
        # one rotary table per distinct rotation among the layers
        self._rope: Dict[Tuple, str] = {}
        for i, layer in enumerate(self.layers):
            if layer.kind == "full_attention" and layer.rope_key not in self._rope:
                lc = cfg.layer_config(i)
                name = f"rope_{len(self._rope)}"
                rc = ref.rope_cos_sin_cache(lc.qk_rope_head_dim, cfg.max_position_embeddings, lc.rope_theta, lc.rope_scaling)
                self.register_buffer(name, rc.to(device), persistent=False)
                self._rope[layer.rope_key] = name
        self.trace_residual = None        # a list: receives the residual stream after every layer (debugging, eager runs only)
        for p in self.parameters():
            p.requires_grad_(False)

    @property
    def num_cache_layers(self) -> int:
        c = self.cfg
        return sum(1 for i in range(c.num_hidden_layers) if c.layer_type(i) == "full_attention" and c.kv_source_layer(i) == i)

    def forward(self, input_ids, positions, ctx: ForwardContext, inputs_embeds=None):
        assert inputs_embeds is None, "this family takes token ids"
        rope = {k: getattr(self, n) for k, n in self._rope.items()}
        norms = [layer.norm1 for layer in self.layers] + [self.norm]
        h, x = ops.embed_norm(input_ids, self.embed_tokens.weight, norms[0].weight, norms[0].eps, norms[0].unit_offset)
        for i, layer in enumerate(self.layers):
            h, x = layer(h, x, norms[i + 1], positions, ctx, rope)
            if self.trace_residual is not None:
                self.trace_residual.append(x.clone())
        return h

    def compute_logits(self, hidden):
        return ops.lm_head(hidden, self.lm_head.weight)[:, : self.cfg.vocab_size]

    # ---- weights ---------------------------------------------------------------------------
    def load_weights(self, weights: Iterable[Tuple[str, torch.Tensor]]) -> int:
        """Tensors under the design's own names: embed, head, final.norm, l<i>.norm1 / norm1b / norm2 / norm2b, l<i>.mix.<part>,
        l<i>.mlp.gate / up / down."""
        expected = set(tuvutar_param_shapes(self.cfg))
        seen, parts = set(), {}

        def group(key, part, order, w, setter):
            g = parts.setdefault(key, {})
            g[part] = w
            if len(g) == len(order):
                setter(torch.cat([g[o] for o in order], 0))
                parts.pop(key)

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
                    self.norm.weight.copy_(w); continue
                li, rest = re.match(r"l(\d+)\.(.+)$", name).groups()
                L = self.layers[int(li)]
                if rest in ("norm1", "norm1b", "norm2", "norm2b"):
                    getattr(L, rest).weight.copy_(w)
                elif rest == "mlp.down":
                    L.mlp.down_proj.set_weight(w)
                elif rest.startswith("mlp."):
                    group(li + ".gu", rest[4:], ("gate", "up"), w, L.mlp.gate_up_proj.set_weight)
                elif L.kind == "full_attention":
                    self._load_latent(L.mixer, li, rest[4:], w, group)
                else:
                    self._load_delta(L.mixer, li, rest[4:], w, group)
        missing = expected - seen
        if missing:
            raise ValueError(f"incomplete checkpoint: {sorted(missing)[:4]}")
        return len(seen)

    @staticmethod
    def _load_latent(A: MLAAttention, li: str, leaf: str, w, group):
        if leaf in ("q", "dkv"):
            group(li + ".qkv", leaf, ("q",) if A.reads_only else ("q", "dkv"), w, A.q_kv_proj.set_weight)
        elif leaf == "dkv.norm":
            A.kv_a_layernorm.weight.copy_(w)
        elif leaf == "uk":
            A.set_uk_uv(uk=w)
        elif leaf == "uv":
            A.set_uk_uv(uv=w)
        else:
            A.o_proj.set_weight(w)

    @staticmethod
    def _load_delta(G: GatedDeltaNet, li: str, leaf: str, w, group):
        if leaf in ("q", "k", "v", "g"):
            group(li + ".in", leaf, ("q", "k", "v", "g"), w, G.in_proj.set_weight)
        elif leaf in ("a", "b"):
            group(li + ".ab", leaf, ("a", "b"), w, G.in_proj_ab.set_weight)
        elif leaf.endswith(".conv"):
            group(li + ".conv", leaf, ("q.conv", "k.conv", "v.conv"), w, G.conv_weight.copy_)
        elif leaf == "A_log":
            G.A_log.copy_(w)
        elif leaf == "dt_bias":
            G.dt_bias.copy_(w)
        elif leaf == "norm":
            G.norm_weight.copy_(w)
        else:
            G.out_proj.set_weight(w)


def tuvutar_param_shapes(cfg: ModelConfig) -> Dict[str, Tuple[int, ...]]:
    """Every tensor name of a checkpoint with its shape."""
    D, V = cfg.hidden_size, cfg.vocab_size
    out: Dict[str, Tuple[int, ...]] = {"embed": (V, D)}
    for i in range(cfg.num_hidden_layers):
        c, p = cfg.layer_config(i), f"l{i}."
        for n in ("norm1", "norm1b"):
            out[p + n] = (D,)
        m = p + "mix."
        if cfg.layer_type(i) == "full_attention":
            H, nope, rope, v, R = c.num_attention_heads, c.qk_nope_head_dim, c.qk_rope_head_dim, c.v_head_dim, c.kv_lora_rank
            out[m + "q"] = (H * (nope + rope), D)
            if cfg.kv_source_layer(i) == i:
                out[m + "dkv"], out[m + "dkv.norm"] = (R + rope, D), (R,)
            out[m + "uk"], out[m + "uv"], out[m + "o"] = (H * nope, R), (H * v, R), (D, H * v)
        else:
            Hk, H, dk, dv, K = (c.linear_num_key_heads, c.linear_num_value_heads, c.linear_key_head_dim, c.linear_value_head_dim,
                                c.linear_conv_kernel_dim)
            for n, rows in (("q", Hk * dk), ("k", Hk * dk), ("v", H * dv)):
                out[m + n], out[m + n + ".conv"] = (rows, D), (rows, K)
            out[m + "g"], out[m + "a"], out[m + "b"] = (H * dv, D), (H, D), (H, D)
            out[m + "A_log"], out[m + "dt_bias"], out[m + "norm"], out[m + "o"] = (H,), (H,), (dv,), (D, H * dv)
        if cfg.layer_specs[i]["mlp"] is not None:
            F = c.intermediate_size
            out[p + "norm2"] = out[p + "norm2b"] = (D,)
            out[p + "mlp.gate"], out[p + "mlp.up"], out[p + "mlp.down"] = (F, D), (F, D), (D, F)
    out["final.norm"], out["head"] = (D,), (V, D)
    return out
