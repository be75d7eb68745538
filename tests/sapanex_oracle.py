"""Plain statement of the Sapanex design, one function per mechanism, token by token where the mechanism is sequential.

Works on the raw config dictionary and a name -> tensor dictionary, shares nothing with the package, and is slow on purpose.
Everything runs in the dtype of the weights (float64 by default), one sequence at a time, without any cache: a prompt of n tokens is
always computed from its first token."""
import math

import torch


# ---- small pieces --------------------------------------------------------------------------------------------------
def sigmoid(x):
    return 1 / (1 + torch.exp(-x))


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def squared_relu(x):
    return torch.where(x > 0, x * x, torch.zeros_like(x))


# ---- rotation --------------------------------------------------------------------------------------------------------
def plain_frequencies(dims, base):
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def yarn_frequencies(dims, base, scaling):
    """Frequencies and the factor of cos and sin."""
    freq = plain_frequencies(dims, base)
    if scaling is None:
        return freq, 1.0

    def dim_of(turns):
        return dims * math.log(scaling["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(dim_of(scaling["fast"])), 0)
    hi = min(math.ceil(dim_of(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freq):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / scaling["factor"] * ramp + f * (1 - ramp))
    return out, 0.1 * math.log(scaling["factor"]) + 1


def rotate(x, freq, factor=1.0, back=False):
    """x [n, heads, width], row = position: the first 2 len(freq) columns turn (column i with column i + len(freq)), the rest pass."""
    half = len(freq)
    out = x.clone()
    for p in range(x.shape[0]):
        a = torch.tensor([(-p if back else p) * f for f in freq], dtype=torch.float64)
        c, s = (a.cos() * factor).to(x.dtype), (a.sin() * factor).to(x.dtype)
        u, v = x[p, :, :half], x[p, :, half: 2 * half]
        out[p, :, :half], out[p, :, half: 2 * half] = u * c - v * s, v * c + u * s
    return out


# ---- attention -------------------------------------------------------------------------------------------------------
def pool_blocks(x, pool):
    """x [n, heads, width] -> the means of all whole blocks of `pool` rows."""
    whole = x.shape[0] // pool
    return [x[b * pool: (b + 1) * pool].mean(0) for b in range(whole)]


def visible(i, size, pool):
    """What position i sees: the tokens of its window and the pooled blocks that lie wholly in front of it."""
    tokens = [j for j in range(i + 1) if i - j < size]
    blocks = [b for b in range(i // pool + 1) if b * pool + pool - 1 <= i - size]
    return tokens, blocks


def window_attention(q, k, v, scale, size, pool, hide=None):
    """q [n, H, d], k [n, G, d], v [n, G, dv] -> [n, H, dv].  `hide` plants a mistake: hide(i) gives the tokens and the blocks query i leaves out."""
    n, H, _ = q.shape
    rep = H // k.shape[1]
    kb, vb = pool_blocks(k, pool), pool_blocks(v, pool)
    out = torch.zeros(n, H, v.shape[2], dtype=q.dtype)
    for i in range(n):
        tokens, blocks = visible(i, size, pool)
        if hide is not None:
            no_tokens, no_blocks = hide(i)
            tokens, blocks = [j for j in tokens if j not in no_tokens or j == i], [b for b in blocks if b not in no_blocks]
        keys = torch.cat([k[tokens]] + [kb[b][None] for b in blocks])
        values = torch.cat([v[tokens]] + [vb[b][None] for b in blocks])
        for h in range(H):
            s = keys[:, h // rep] @ q[i, h] * scale
            e = torch.exp(s - s.max())
            out[i, h] = (e / e.sum()) @ values[:, h // rep]
    return out


def attention(h, W, m, eps, hide=None):
    n, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(h @ W["q"].T, W["q.norm"], eps).view(n, H, d)
    k = rms_norm(h @ W["k"].T, W["k.norm"], eps).view(n, G, d)
    v = (h @ W["v"].T).view(n, G, dv)
    freq, factor = yarn_frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
    vfreq = plain_frequencies(dv, m["rot"]["base"])
    q, k, v = rotate(q, freq, factor), rotate(k, freq, factor), rotate(v, vfreq)
    o = window_attention(q, k, v, m["scale"], m["mask"]["size"], m["mask"]["pool"], hide)
    return rotate(o, vfreq, back=True).reshape(n, H * dv) @ W["o"].T


# ---- generalised delta rule --------------------------------------------------------------------------------------------
def delta_step(S, r, k, v, w, a):
    """One token: S [heads, dim of keys, dim of values], the rest [heads, dim]."""
    u = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    seen = (u[:, :, None] * S).sum(1)                                        # u^T S
    new = w[:, :, None] * S - (a * u)[:, :, None] * seen[:, None, :] + k[:, :, None] * v[:, None, :]
    return new, (new * r[:, :, None]).sum(1)


def recurrence(r, k, v, w, a):
    """[n, heads, dim] each -> o [n, heads, dim of values] and the state after the last token."""
    S = torch.zeros(r.shape[1], r.shape[2], v.shape[2], dtype=r.dtype)
    o = torch.zeros(r.shape[0], r.shape[1], v.shape[2], dtype=r.dtype)
    for t in range(r.shape[0]):
        S, o[t] = delta_step(S, r[t], k[t], v[t], w[t], a[t])
    return o, S


def general_delta(h, W, m, eps):
    n, H, d = h.shape[0], m["heads"], m["dim"]
    r, k, v = ((h @ W[x].T).view(n, H, d) for x in ("r", "k", "v"))
    w = torch.exp(-math.exp(-0.5) * sigmoid(torch.tanh(h @ W["w1"].T) @ W["w2"].T + W["w0"])).view(n, H, d)
    a = sigmoid(h @ W["a"].T + W["a.b"]).view(n, H, d)
    o, _ = recurrence(r, k, v, w, a)
    o = unit_rms(o, eps).reshape(n, H * d) * W["norm"] * sigmoid(h @ W["g"].T)
    return o @ W["o"].T


# ---- the model ---------------------------------------------------------------------------------------------------------
def part(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(cfg, weights, tokens, layers_out=None, hide=None):
    """Logits [n, vocab] of one sequence; `layers_out` (a list) receives the residual stream after every layer; hide: see window_attention."""
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = weights["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        args = (x, part(weights, p + "mix."), layer["mixer"], eps)
        y = attention(*args, hide) if layer["type"] == "attention" else general_delta(*args)
        x = rms_norm(alpha * x + y, weights[p + "norm1"], eps)
        if layer["mlp"] is not None:
            y = squared_relu(x @ weights[p + "mlp.up"].T) @ weights[p + "mlp.down"].T
            x = rms_norm(alpha * x + y, weights[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms_norm(x, weights["final.norm"], eps) @ weights["embed"].T


def greedy(cfg, weights, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(cfg, weights, toks)[-1].argmax()))
    return toks[len(prompt):]


def shapes(cfg):
    """Every tensor name with its shape; cfg["ranks"]: the rank of every layer's decay projection (None for attention)."""
    D = cfg["width"]
    out = {"embed": (cfg["vocab"], D), "final.norm": (D,)}
    for i, s in enumerate(cfg["layers"]):
        m, p = s["mixer"], f"l{i}."
        out[p + "norm1"] = (D,)
        if s["type"] == "attention":
            hq, hk, hv = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
            out.update({p + "mix.q": (hq, D), p + "mix.k": (hk, D), p + "mix.v": (hv, D), p + "mix.q.norm": (hq,), p + "mix.k.norm": (hk,),
                        p + "mix.o": (D, m["heads"] * m["vdim"])})
        else:
            w, rank = m["heads"] * m["dim"], cfg["ranks"][i]
            for n in ("r", "k", "v", "g", "a"):
                out[p + "mix." + n] = (w, D)
            out.update({p + "mix.a.b": (w,), p + "mix.w1": (rank, D), p + "mix.w2": (w, rank), p + "mix.w0": (w,), p + "mix.norm": (w,), p + "mix.o": (D, w)})
        if s["mlp"] is not None:
            out.update({p + "norm2": (D,), p + "mlp.up": (s["mlp"]["ff"], D), p + "mlp.down": (D, s["mlp"]["ff"])})
    return out


def random_weights(cfg, seed=0, sharp=1.0):
    """bf16-representable float64 weights.  `sharp` scales the query and key norms: larger scores, so that single keys matter."""
    g = torch.Generator().manual_seed(seed)
    W = {}
    for name, shape in shapes(cfg).items():
        t, leaf = torch.randn(shape, generator=g, dtype=torch.float64), name.rsplit(".", 1)[-1]
        if leaf in ("norm", "norm1", "norm2"):
            t = (1 + 0.2 * t) * (sharp if name.endswith((".q.norm", ".k.norm")) else 1.0)
        elif leaf == "w0":
            t = 1.5 * t - 2.0
        elif name.endswith(".a.b"):
            t = t - 0.5
        elif name != "embed":
            t = t * shape[-1] ** -0.5
        W[name] = t.to(torch.bfloat16).double()
    return W
