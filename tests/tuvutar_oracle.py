"""Plain statement of the Tuvutar design, one function per mechanism, token by token where the mechanism is sequential.

Works on the raw config dictionary and a name -> tensor dictionary, shares nothing with the package, and is slow on purpose.
Everything runs in the dtype of `x` (float64 by default), one sequence at a time, without any cache: a prompt of n tokens is
always computed from its first token."""
import math

import torch


# ---- norms ---------------------------------------------------------------------------------------------------------
def over_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def offset_norm(x, w, eps):
    """RMS norm whose weight is stored around zero."""
    return over_rms(x, eps) * (1 + w)


# ---- rotary positions ------------------------------------------------------------------------------------------------
def rotary_frequencies(rot, dtype=torch.float64):
    """(frequency of every pair, magnitude of cos and sin)."""
    dims, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    mag = 1.0
    if sc:
        def turn_dim(t):
            return dims * math.log(sc["original"] / (2 * math.pi * t)) / (2 * math.log(base))
        lo = max(math.floor(turn_dim(sc["fast"])), 0)
        hi = min(math.ceil(turn_dim(sc["slow"])), dims - 1)
        out = []
        for i, fi in enumerate(f):
            ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            out.append(fi / sc["factor"] * ramp + fi * (1 - ramp))
        f, mag = out, 0.1 * math.log(sc["factor"]) + 1.0
    return torch.tensor(f, dtype=dtype), mag


def rotate(x, positions, rot):
    """x [n, ..., dims]: pairs (2i, 2i + 1) turned by position * frequency_i."""
    f, mag = rotary_frequencies(rot, x.dtype)
    ang = positions.to(x.dtype)[:, None] * f[None]
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (f.numel(),)
    c, s = (ang.cos() * mag).view(shape), (ang.sin() * mag).view(shape)
    out = torch.empty_like(x)
    u, v = x[..., 0::2], x[..., 1::2]
    out[..., 0::2] = u * c - v * s
    out[..., 1::2] = v * c + u * s
    return out


# ---- latent attention ----------------------------------------------------------------------------------------------
def latent_rows(h, W, p, m, eps):
    """The two cached parts of every token: normed latent c [n, kv_rank], rotated shared key part [n, rot_dim]."""
    kv = h @ W[p + "dkv"].T
    R = m["kv_rank"]
    c = over_rms(kv[:, :R], eps) * W[p + "dkv.norm"]
    pos = torch.arange(h.shape[0])
    return c, rotate(kv[:, R:], pos, m["rot"])


def latent_attention(h, W, p, m, rows, hide=None):
    """Causal attention over the latent rows, keys and values expanded per head.  `hide`: plant a mistake - hide(i, n) returns the
    keys query i leaves out."""
    n, H, d, r, vd = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, kr = rows
    q = (h @ W[p + "q"].T).view(n, H, d + r)
    qr = rotate(q[..., d:], torch.arange(n), m["rot"])
    k = (c @ W[p + "uk"].T).view(n, H, d)
    v = (c @ W[p + "uv"].T).view(n, H, vd)
    out = torch.zeros(n, H, vd, dtype=h.dtype)
    for i in range(n):
        s = (torch.einsum("hd,jhd->hj", q[i, :, :d], k[: i + 1]) + qr[i] @ kr[: i + 1].T) * m["scale"]
        if hide is not None:
            s[:, [j for j in hide(i, n) if j <= i and i > 0]] = -1e30
        out[i] = torch.einsum("hj,jhv->hv", torch.softmax(s, -1), v[: i + 1])
    return out.reshape(n, H * vd) @ W[p + "o"].T


# ---- gated delta rule ------------------------------------------------------------------------------------------------
def silu(x):
    return x / (1 + torch.exp(-x))


def short_conv(x, w):
    """Causal convolution per channel (last tap = the current token), then silu."""
    n, taps = x.shape[0], w.shape[1]
    out = torch.zeros_like(x)
    for t in range(n):
        for j in range(taps):
            src = t - (taps - 1) + j
            if src >= 0:
                out[t] += x[src] * w[:, j]
    return silu(out)


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def softplus(x):
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


def delta_rule(q, k, v, g, beta):
    """q, k [n, kv_heads, dim], v [n, heads, vdim], g and beta [n, heads]; the state [dim, vdim] of every head starts at zero."""
    n, H, vd = v.shape
    rep = H // q.shape[1]
    out = torch.zeros_like(v)
    for h in range(H):
        S = torch.zeros(q.shape[2], vd, dtype=v.dtype)
        for t in range(n):
            kt, qt = k[t, h // rep], q[t, h // rep]
            S = g[t, h] * S
            u = beta[t, h] * (v[t, h] - S.T @ kt)
            S = S + kt[:, None] * u[None, :]
            out[t, h] = S.T @ qt
    return out


def delta_mixer(h, W, p, m, eps):
    n, H, Hk, d, vd = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = short_conv(h @ W[p + "q"].T, W[p + "q.conv"]).view(n, Hk, d)
    k = short_conv(h @ W[p + "k"].T, W[p + "k.conv"]).view(n, Hk, d)
    v = short_conv(h @ W[p + "v"].T, W[p + "v.conv"]).view(n, H, vd)
    beta = 1 / (1 + torch.exp(-(h @ W[p + "b"].T)))
    g = torch.exp(-torch.exp(W[p + "A_log"]) * softplus(h @ W[p + "a"].T + W[p + "dt_bias"]))
    o = delta_rule(unit(q) * d ** -0.5, unit(k), v, g, beta)
    o = over_rms(o, eps) * W[p + "norm"] * silu(h @ W[p + "g"].T).view(n, H, vd)
    return o.reshape(n, H * vd) @ W[p + "o"].T


# ---- feed-forward ----------------------------------------------------------------------------------------------------
def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def dense_ff(h, W, p):
    return (gelu_tanh(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


# ---- the stack -------------------------------------------------------------------------------------------------------
def forward(cfg, weights, tokens, dtype=torch.float64, trace=None, hide=None):
    """Logits [n, vocab] of one sequence.  `trace` (a list) receives the residual stream after every layer; `hide`: see
    latent_attention."""
    W = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.tensor(list(tokens))]
    rows = {}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        h = offset_norm(x, W[p + "norm1"], eps)
        if L["type"] == "latent_attention":
            rows[i] = rows[m["kv_from"]] if m.get("kv_from") is not None else latent_rows(h, W, p + "mix.", m, eps)
            y = latent_attention(h, W, p + "mix.", m, rows[i], hide)
        else:
            y = delta_mixer(h, W, p + "mix.", m, eps)
        x = x + offset_norm(y, W[p + "norm1b"], eps)
        if L["mlp"] is not None:
            x = x + offset_norm(dense_ff(offset_norm(x, W[p + "norm2"], eps), W, p + "mlp."), W[p + "norm2b"], eps)
        if trace is not None:
            trace.append(x.clone())
    return offset_norm(x, W["final.norm"], eps) @ W["head"].T


# ---- random models ---------------------------------------------------------------------------------------------------
def random_weights(cfg, seed=0, sharp=1.5):
    """Weights of every tensor of the design, bf16-representable, scaled so that no mechanism vanishes.  `sharp` scales the queries:
    with a large value single keys stand out of hundreds."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, s=1.0):
        return (torch.randn(*shape, generator=g) * s).to(torch.bfloat16)

    D, V = cfg["width"], cfg["vocab"]
    W = {"embed": rnd(V, D), "head": rnd(V, D, s=D ** -0.5), "final.norm": rnd(D, s=0.2)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        for nm in ["norm1", "norm1b"] + (["norm2", "norm2b"] if L["mlp"] else []):
            W[p + nm] = rnd(D, s=0.2)
        q = p + "mix."
        if L["type"] == "latent_attention":
            H, d, r, vd, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            W[q + "q"] = rnd(H * (d + r), D, s=sharp * D ** -0.5)
            if m.get("kv_from") is None:
                W[q + "dkv"] = rnd(R + r, D, s=D ** -0.5)
                W[q + "dkv.norm"] = (1 + 0.2 * torch.randn(R, generator=g)).to(torch.bfloat16)
            W[q + "uk"], W[q + "uv"] = rnd(H * d, R, s=R ** -0.5), rnd(H * vd, R, s=R ** -0.5)
            W[q + "o"] = rnd(D, H * vd, s=(H * vd) ** -0.5)
        else:
            H, Hk, d, vd, K = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            for nm, rows in (("q", Hk * d), ("k", Hk * d), ("v", H * vd), ("g", H * vd), ("b", H), ("a", H)):
                W[q + nm] = rnd(rows, D, s=D ** -0.5)
                if nm in "qkv":
                    W[q + nm + ".conv"] = rnd(rows, K, s=0.6)
            W[q + "A_log"], W[q + "dt_bias"] = rnd(H, s=0.5), (rnd(H, s=0.5) - 3).to(torch.bfloat16)
            W[q + "norm"] = (1 + 0.2 * torch.randn(vd, generator=g)).to(torch.bfloat16)
            W[q + "o"] = rnd(D, H * vd, s=(H * vd) ** -0.5)
        if L["mlp"]:
            F = L["mlp"]["ff"]
            W[p + "mlp.gate"], W[p + "mlp.up"], W[p + "mlp.down"] = rnd(F, D, s=D ** -0.5), rnd(F, D, s=D ** -0.5), rnd(D, F, s=F ** -0.5)
    return W


def greedy(cfg, weights, prompt, n):
    """n greedily chosen tokens after `prompt`."""
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(cfg, weights, toks)[-1].argmax()))
    return toks[len(prompt):]
