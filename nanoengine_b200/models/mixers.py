"""Sequence mixers with explicit sizes and constants, for families that list their layers one by one.

Mamba2Mixer     z | x | B | C from one GEMM, the step sizes from a second one with an fp32 result; short convolution, state-space recurrence
                and gated norm are `ops.mamba2_mix`.
ParallelMixer   two mixers over the same input, summed with constant weights: windowed grouped-query attention with capped scores, a
                distance bias and an output gate per head (`ops.gqa_attention_biased`), and linear attention with a constant decay per head
                (`ops.lightning_mix`).  Both read one merged projection and write into one row, so the pair costs two GEMMs; the weights of
                the sum are applied to the fp32 results before they are rounded.  The layer owns rows of the paged cache and a state.
PooledAttentionMixer   grouped-query attention over a window of tokens and the means of the blocks of tokens in front of it, with q and k
                normed over all heads at once, partly rotated, and values that are cached rotated and whose sums are turned back
                (`ops.pooled_attention_prepare`, `ops.gqa_attention_biased`).
GeneralDeltaMixer   delta rule with a decay and a removal rate per key channel; everything from one GEMM, the decay's second, low-rank
                factor from another one with an fp32 result; recurrence, norm and gate are `ops.general_delta`.
DifferentialAttentionMixer   two softmax maps per head over the same values, their difference normed and gated, over a window and the first tokens,
                with a short convolution behind the projections (`ops.conv_rows`, `ops.differential_attention`); a layer may read the rows
                of an earlier one."""
from __future__ import annotations

from typing import Dict, Optional, Sequence

import torch
import torch.nn as nn

from .. import ops
from ..runtime.context import ForwardContext
from .layers import QLinear


def _const(*shape, dtype=torch.float32, device=None, fill=0.0):
    return nn.Parameter(torch.full(shape, fill, dtype=dtype, device=device), requires_grad=False)


def distance_slopes(heads: int) -> torch.Tensor:
    """Geometric slopes 2^(-8 (h + 1) / heads) of the distance bias."""
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], dtype=torch.float32)


class Mamba2Mixer(nn.Module):
    def __init__(self, hidden: int, heads: int, vdim: int, state: int, groups: int, conv: int, norm_groups: int, eps: float, state_idx: int, dtype, device):
        super().__init__()
        self.heads, self.vdim, self.state, self.groups, self.norm_groups = heads, vdim, state, groups, norm_groups
        self.eps, self.state_idx = eps, state_idx
        self.inner = heads * vdim
        self.conv_dim = self.inner + 2 * groups * state
        self.in_proj = QLinear(hidden, self.inner + self.conv_dim, dtype, device, None)
        self.dt_proj = QLinear(hidden, heads, dtype, device, None)
        self.out_proj = QLinear(self.inner, hidden, dtype, device, None)
        self.conv_weight, self.conv_bias = _const(self.conv_dim, conv, dtype=dtype, device=device), _const(self.conv_dim, dtype=dtype, device=device)
        self.A_log, self.dt_bias, self.D = (_const(heads, device=device) for _ in range(3))
        self.norm_weight = _const(self.inner, dtype=dtype, device=device, fill=1.0)

    def forward(self, h, ctx: ForwardContext):
        proj = self.in_proj(h)
        dt = ops.linear_fp32(h, self.dt_proj.weight)[:, : self.heads]
        y = ops.mamba2_mix(proj, dt, self.conv_weight, self.conv_bias, self.A_log, self.dt_bias, self.D, self.norm_weight, self.norm_groups,
                           ctx.conv_states[self.state_idx], ctx.rec_states[self.state_idx], ctx.state_slots, ctx.cu_seqlens_q, ctx.seq_fresh,
                           self.heads, self.groups, self.vdim, self.state, self.eps, ctx.max_seqlen_q)
        return self.out_proj(y)

    def parts(self):
        """Tensor name below the mixer -> shape."""
        D = self.in_proj.in_features
        return {"in": (self.inner + self.conv_dim + self.heads, D), "conv": tuple(self.conv_weight.shape), "conv.b": (self.conv_dim,),
                "dt_bias": (self.heads,), "A_log": (self.heads,), "D": (self.heads,), "norm": (self.inner,), "o": (D, self.inner)}

    def load(self, w: Dict[str, torch.Tensor]) -> None:
        rows = self.inner + self.conv_dim
        self.in_proj.set_weight(w["in"][:rows])
        self.dt_proj.set_weight(w["in"][rows:])
        self.out_proj.set_weight(w["o"])
        for p, n in ((self.conv_weight, "conv"), (self.conv_bias, "conv.b"), (self.A_log, "A_log"), (self.dt_bias, "dt_bias"), (self.D, "D"), (self.norm_weight, "norm")):
            p.copy_(w[n])


class ParallelMixer(nn.Module):
    # rows of the merged projection; the gate of the attention heads, a few odd rows, comes last
    ORDER = ("left.q", "left.k", "left.v", "right.q", "right.k", "right.v", "right.g", "left.g")

    def __init__(self, hidden: int, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, softcap: float, window: int, lin_heads: int, lin_dim: int,
                 lin_vdim: int, decay: Sequence[float], left_scale: float, right_scale: float, eps: float, cache_idx: int, state_idx: int, dtype, device):
        super().__init__()
        self.hidden, self.heads, self.kv_heads, self.dim, self.vdim = hidden, heads, kv_heads, dim, vdim
        self.scale, self.softcap, self.window = scale, softcap, window
        self.lin_heads, self.lin_dim, self.lin_vdim = lin_heads, lin_dim, lin_vdim
        self.left_scale, self.right_scale, self.eps, self.cache_idx, self.state_idx = left_scale, right_scale, eps, cache_idx, state_idx
        rows = {n: self.parts()[n][0] for n in self.ORDER}
        self.rows = [rows[n] for n in self.ORDER]
        self.left_width, self.right_width = heads * vdim, lin_heads * lin_vdim
        self.in_proj = QLinear(hidden, sum(self.rows), dtype, device, None, bias_fp32=True)
        self.out_proj = QLinear(self.left_width + self.right_width, hidden, dtype, device, None, bias_fp32=True)
        self.norm_weight = _const(self.right_width, dtype=dtype, device=device, fill=1.0)
        self.register_buffer("slopes", distance_slopes(heads).to(device), persistent=False)
        self.register_buffer("decay", torch.tensor(list(decay), dtype=torch.float64).float().to(device), persistent=False)

    def forward(self, h, ctx: ForwardContext):
        T = h.shape[0]
        q, k, v, lq, lk, lv, lg, gate = self.in_proj(h).split(self.rows, -1)
        kc, vc = ctx.kv_caches[self.cache_idx]
        ops.kv_rows(kc, vc, ctx.slot_mapping, k, v)
        y = torch.empty(T, self.left_width + self.right_width, dtype=h.dtype, device=h.device)
        ops.gqa_attention_biased(q.unflatten(-1, (self.heads, self.dim)), kc, vc, ctx.block_tables, ctx.cu_seqlens_q, ctx.context_lens, self.scale, self.window,
                                 self.softcap, self.slopes, gate, self.left_scale, y[:, : self.left_width], ctx.max_seqlen_q)
        ops.lightning_mix(lq, lk, lv, lg, self.decay, self.norm_weight, ctx.rec_states[self.state_idx], ctx.state_slots, ctx.cu_seqlens_q, ctx.seq_fresh,
                          self.lin_heads, self.lin_dim, self.lin_vdim, self.eps, self.right_scale, y[:, self.left_width:], ctx.max_seqlen_q)
        return self.out_proj(y)

    def parts(self):
        D, H, G = self.hidden, self.heads, self.kv_heads
        out = {}
        for n, r in (("q", H * self.dim), ("k", G * self.dim), ("v", G * self.vdim)):
            out["left." + n], out[f"left.{n}.b"] = (r, D), (r,)
        out["left.g"], out["left.o"], out["left.o.b"] = (H, D), (D, H * self.vdim), (D,)
        lq, lv = self.lin_heads * self.lin_dim, self.lin_heads * self.lin_vdim
        for n, r in (("q", lq), ("k", lq), ("v", lv), ("g", lv)):
            out["right." + n] = (r, D)
        out["right.norm"], out["right.o"] = (lv,), (D, lv)
        return out

    def load(self, w: Dict[str, torch.Tensor]) -> None:
        self.in_proj.set_weight(torch.cat([w[n] for n in self.ORDER], 0))
        b = torch.cat([w["left.q.b"], w["left.k.b"], w["left.v.b"]])
        self.in_proj.bias.zero_()
        self.in_proj.bias[: b.numel()].copy_(b)
        self.out_proj.set_weight(torch.cat([w["left.o"], w["right.o"]], 1))
        self.out_proj.bias.zero_()
        self.out_proj.bias[: self.hidden].copy_(self.left_scale * w["left.o.b"])
        self.norm_weight.copy_(w["right.norm"])


class PooledAttentionMixer(nn.Module):
    ORDER = ("q", "k", "v")

    def __init__(self, hidden: int, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, window: int, pool: int, eps: float, cache_idx: int, dtype, device):
        super().__init__()
        self.hidden, self.heads, self.kv_heads, self.dim, self.vdim = hidden, heads, kv_heads, dim, vdim
        self.scale, self.window, self.pool, self.eps, self.cache_idx = scale, window, pool, eps, cache_idx
        self.in_proj = QLinear(hidden, heads * dim + kv_heads * (dim + vdim), dtype, device)
        self.out_proj = QLinear(heads * vdim, hidden, dtype, device)
        self.q_norm, self.k_norm = _const(heads * dim, dtype=dtype, device=device, fill=1.0), _const(kv_heads * dim, dtype=dtype, device=device, fill=1.0)

    def forward(self, h, positions, ctx: ForwardContext, key_table, value_table):
        """The tables [positions, dims] (cos | sin): of the rotated part of queries and keys, and of whole values."""
        kc, vc, kp, vp = ctx.kv_caches[self.cache_idx]
        q = ops.pooled_attention_prepare(self.in_proj(h), self.heads, self.kv_heads, self.dim, self.vdim, self.q_norm, self.k_norm, self.eps, positions, key_table,
                                         value_table, kc, vc, kp, vp, self.pool, ctx.slot_mapping, ctx.block_tables, ctx.cu_seqlens_q, ctx.max_seqlen_q)
        return self.out_proj(ops.gqa_attention_biased(q, kc, vc, ctx.block_tables, ctx.cu_seqlens_q, ctx.context_lens, self.scale, self.window,
                                                      max_q_len=ctx.max_seqlen_q, pooled=(kp, vp), pool=self.pool, turn_back=value_table))

    def parts(self):
        D, q, k, v = self.hidden, self.heads * self.dim, self.kv_heads * self.dim, self.kv_heads * self.vdim
        return {"q": (q, D), "k": (k, D), "v": (v, D), "q.norm": (q,), "k.norm": (k,), "o": (D, self.heads * self.vdim)}

    def load(self, w: Dict[str, torch.Tensor]) -> None:
        self.in_proj.set_weight(torch.cat([w[n] for n in self.ORDER], 0))
        self.out_proj.set_weight(w["o"])
        self.q_norm.copy_(w["q.norm"])
        self.k_norm.copy_(w["k.norm"])


class GeneralDeltaMixer(nn.Module):
    # rows of the merged projection; the first factor of the decay's projection comes last: its tanh is part of the GEMM's epilogue
    ORDER = ("r", "k", "a", "v", "g", "w1")

    def __init__(self, hidden: int, heads: int, dim: int, rank: int, eps: float, state_idx: int, dtype, device):
        super().__init__()
        self.hidden, self.heads, self.dim, self.rank, self.eps, self.state_idx = hidden, heads, dim, rank, eps, state_idx
        self.width = w = heads * dim
        self.in_proj = QLinear(hidden, 5 * w + rank, dtype, device)
        self.decay_proj = QLinear(rank, w, dtype, device)
        self.out_proj = QLinear(w, hidden, dtype, device)
        self.w0, self.a_bias = _const(w, device=device), _const(w, device=device)
        self.norm_weight = _const(w, dtype=dtype, device=device, fill=1.0)

    def forward(self, h, ctx: ForwardContext):
        proj = self.in_proj(h, act="tanh", act_from=5 * self.width)
        decay = ops.linear_fp32(proj[:, 5 * self.width: 5 * self.width + self.rank], self.decay_proj.weight)
        return self.out_proj(ops.general_delta(proj, decay, self.w0, self.a_bias, self.norm_weight, ctx.rec_states[self.state_idx], ctx.state_slots, ctx.cu_seqlens_q,
                                               ctx.seq_fresh, self.heads, self.dim, self.dim, self.eps, ctx.max_seqlen_q))

    def parts(self):
        D, w = self.hidden, self.width
        out = {n: (w, D) for n in ("r", "k", "v", "g", "a")}
        out.update({"a.b": (w,), "w1": (self.rank, D), "w2": (w, self.rank), "w0": (w,), "norm": (w,), "o": (D, w)})
        return out

    def load(self, w: Dict[str, torch.Tensor]) -> None:
        self.in_proj.set_weight(torch.cat([w[n] for n in self.ORDER], 0))
        self.decay_proj.set_weight(w["w2"])
        self.out_proj.set_weight(w["o"])
        for p, n in ((self.w0, "w0"), (self.a_bias, "a.b"), (self.norm_weight, "norm")):
            p.copy_(w[n])


class DifferentialAttentionMixer(nn.Module):
    """`reads_only`: the layer has no keys and values of its own and reads cache layer `cache_idx` as an earlier layer left it.  `window` 0: all
    earlier tokens.  `diff`: the constant part of the weight of the second map."""

    def __init__(self, hidden: int, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, window: int, keep_first: int, diff: float, conv: int, eps: float,
                 cache_idx: int, reads_only: bool, state_idx: Optional[int], dtype, device):
        super().__init__()
        self.hidden, self.heads, self.kv_heads, self.dim, self.vdim = hidden, heads, kv_heads, dim, vdim
        self.scale, self.window, self.keep_first, self.diff, self.eps = scale, window, keep_first, diff, eps
        self.cache_idx, self.reads_only, self.state_idx = cache_idx, reads_only, state_idx
        self.rows = {"q": heads * 2 * dim} if reads_only else {"q": heads * 2 * dim, "k": kv_heads * 2 * dim, "v": kv_heads * vdim}
        self.channels = sum(self.rows.values())
        self.in_proj = QLinear(hidden, self.channels + heads * vdim, dtype, device)          # rows: q, k, v, output gate
        self.out_proj = QLinear(heads * vdim, hidden, dtype, device)
        self.conv_weight = _const(conv, self.channels, dtype=dtype, device=device)           # newest token's weights last
        self.mixing = _const(1, device=device)                                               # weight of the second map

    def forward(self, h, ctx: ForwardContext):
        T = h.shape[0]
        proj = self.in_proj(h)
        kc, vc = ctx.kv_caches[self.cache_idx]
        own = (None, None) if self.reads_only else (kc, vc)
        q = ops.conv_rows(proj, self.conv_weight, self.rows["q"], *own, ctx.slot_mapping, None if self.state_idx is None else ctx.conv_states[self.state_idx],
                          ctx.state_slots, ctx.cu_seqlens_q, ctx.seq_fresh, ctx.max_seqlen_q)
        o = ops.differential_attention(q.view(T, self.heads, 2, self.dim), kc, vc, ctx.block_tables, ctx.cu_seqlens_q, ctx.context_lens, self.scale, self.window,
                                       self.keep_first, self.mixing, 1.0 - self.diff, self.eps, proj[:, self.channels:], ctx.max_seqlen_q)
        return self.out_proj(o)

    def parts(self):
        D, inner = self.hidden, self.heads * self.vdim
        out = {}
        for n, r in self.rows.items():
            out[n], out[n + ".conv"] = (r, D), (r, self.conv_weight.shape[0])
        out.update({n: (self.dim,) for n in ("lq1", "lk1", "lq2", "lk2")})
        out["g"], out["o"] = (inner, D), (D, inner)
        return out

    def load(self, w: Dict[str, torch.Tensor]) -> None:
        self.in_proj.set_weight(torch.cat([w[n] for n in (*self.rows, "g")], 0))
        self.out_proj.set_weight(w["o"])
        self.conv_weight.copy_(torch.cat([w[n + ".conv"] for n in self.rows], 0).t())
        e = lambda i: (w["lq" + i].double() * w["lk" + i].double()).sum().exp()
        self.mixing.fill_(float(e("1") - e("2")) + self.diff)
