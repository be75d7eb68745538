"""Plain statement of the Filasun design, one function per mechanism, token by token where the mechanism is sequential.

Works on the raw config dictionary and a name -> tensor dictionary, shares nothing with the package, and is slow on purpose.
Everything runs in the dtype of the weights (float64 by default), one sequence at a time, without any cache: a prompt of n tokens is
always computed from its first token."""
import torch


# ---- small pieces --------------------------------------------------------------------------------------------------
def sigmoid(x):
    return 1 / (1 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def cap(x, limit):
    return limit * torch.tanh(x / limit)


# ---- hyper-connections ------------------------------------------------------------------------------------------------
def streams_read(x, w_in):
    """x [n, streams, width] -> the sublayer's input before its norm."""
    return sum(w_in[s] * x[:, s] for s in range(x.shape[1]))


def streams_write(x, y, w_out, mix):
    """mix [from, to]."""
    new = torch.empty_like(x)
    for t in range(x.shape[1]):
        new[:, t] = sum(mix[s, t] * x[:, s] for s in range(x.shape[1])) + w_out[t] * y
    return new


# ---- Mamba-2 ----------------------------------------------------------------------------------------------------------
def short_conv(x, w, b):
    """Causal convolution per channel (last tap = the current token) with a bias, then silu."""
    n, taps = x.shape[0], w.shape[1]
    out = torch.zeros_like(x) + b
    for t in range(n):
        for j in range(taps):
            src = t - (taps - 1) + j
            if src >= 0:
                out[t] += x[src] * w[:, j]
    return silu(out)


def state_space(x, B, C, dt, A_log, D):
    """x [n, heads, vdim], B and C [n, groups, state], dt [n, heads] after softplus; every head's [state, vdim] starts at zero."""
    n, H, vd = x.shape
    rep = H // B.shape[1]
    y = torch.zeros_like(x)
    for h in range(H):
        S = torch.zeros(B.shape[2], vd, dtype=x.dtype)
        for t in range(n):
            S = torch.exp(-torch.exp(A_log[h]) * dt[t, h]) * S + dt[t, h] * B[t, h // rep][:, None] * x[t, h][None, :]
            y[t, h] = S.T @ C[t, h // rep] + D[h] * x[t, h]
    return y


def part_norm(y, parts, eps):
    n, W = y.shape
    y = y.reshape(n, parts, W // parts)
    return (y / torch.sqrt((y * y).mean(-1, keepdim=True) + eps)).reshape(n, W)


def mamba2(h, W, p, m, eps):
    n, H, vd, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * vd
    a = h @ W[p + "in"].T
    z, xbc, dt = a[:, :inner], a[:, inner: 2 * inner + 2 * G * N], a[:, 2 * inner + 2 * G * N:]
    assert dt.shape[1] == H
    xbc = short_conv(xbc, W[p + "conv"], W[p + "conv.b"])
    x, B, C = xbc[:, :inner].reshape(n, H, vd), xbc[:, inner: inner + G * N].reshape(n, G, N), xbc[:, inner + G * N:].reshape(n, G, N)
    y = state_space(x, B, C, softplus(dt + W[p + "dt_bias"]), W[p + "A_log"], W[p + "D"]).reshape(n, inner)
    return (part_norm(y * silu(z), m["norm_groups"], eps) * W[p + "norm"]) @ W[p + "o"].T


# ---- windowed attention with a capped score and a distance bias -----------------------------------------------------------
def slopes(H, dtype=torch.float64):
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / H) for h in range(H)], dtype=dtype)


def window_attention(q, k, v, scale, softcap, window, hide=None):
    """q [n, H, dim], k [n, G, dim], v [n, G, vdim].  `hide` plants a mistake: hide(i, n) returns the keys query i leaves out."""
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    sl = slopes(H, q.dtype)
    out = torch.zeros(n, H, v.shape[2], dtype=q.dtype)
    for i in range(n):
        lo = max(0, i - window + 1)
        dist = (i - torch.arange(lo, i + 1)).to(q.dtype)
        for h in range(H):
            g = h // (H // G)
            s = cap((k[lo: i + 1, g] @ q[i, h]) * scale, softcap) - sl[h] * dist
            if hide is not None:
                for j in hide(i, n):
                    if lo <= j < i:
                        s[j - lo] = -1e30
            out[i, h] = torch.softmax(s, 0) @ v[lo: i + 1, g]
    return out


def left_mixer(h, W, p, m, hide=None):
    n, H, G, d, vd = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ W[p + "q"].T + W[p + "q.b"]).reshape(n, H, d)
    k = (h @ W[p + "k"].T + W[p + "k.b"]).reshape(n, G, d)
    v = (h @ W[p + "v"].T + W[p + "v.b"]).reshape(n, G, vd)
    o = window_attention(q, k, v, m["scale"], m["softcap"], m["mask"]["size"], hide)
    o = o * sigmoid(h @ W[p + "g"].T)[:, :, None]
    return o.reshape(n, H * vd) @ W[p + "o"].T + W[p + "o.b"]


# ---- linear attention with a constant decay per head -----------------------------------------------------------------------
def decayed_attention(q, k, v, decay):
    n, H, vd = v.shape
    out = torch.zeros_like(v)
    for h in range(H):
        S = torch.zeros(q.shape[2], vd, dtype=v.dtype)
        for t in range(n):
            S = decay[h] * S + k[t, h][:, None] * v[t, h][None, :]
            out[t, h] = S.T @ q[t, h]
    return out


def right_mixer(h, W, p, m, eps):
    n, H, d, vd = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k = (silu(h @ W[p + c].T).reshape(n, H, d) for c in "qk")
    v = silu(h @ W[p + "v"].T).reshape(n, H, vd)
    o = decayed_attention(q, k, v, m["decay"]).reshape(n, H * vd)
    return (rms_norm(o, W[p + "norm"], eps) * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def parallel_mixer(h, W, p, m, eps, hide=None):
    return m["left_scale"] * left_mixer(h, W, p + "left.", m["left"], hide) + m["right_scale"] * right_mixer(h, W, p + "right.", m["right"], eps)


# ---- feed-forward ----------------------------------------------------------------------------------------------------
def clamped_ff(h, W, p, limit):
    g = torch.clamp(h @ W[p + "gate"].T, max=limit)
    u = torch.clamp(h @ W[p + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ W[p + "down"].T


# ---- the stack -------------------------------------------------------------------------------------------------------
def forward(cfg, weights, tokens, dtype=torch.float64, trace=None, hide=None):
    """Logits [n, vocab] of one sequence.  `trace` (a list) receives the sum of the streams after every layer; `hide`: see
    window_attention."""
    W = {k: v.to(dtype) for k, v in weights.items()}
    eps, n = cfg["norm"]["eps"], len(tokens)
    e = W["embed"][torch.tensor(list(tokens))] + W["pos"][:n]
    x = e[:, None, :].repeat(1, cfg["streams"], 1)

    def sublayer(x, p, q, fn):
        u = streams_read(x, W[f"{p}hc{q}.in"])
        return streams_write(x, fn(rms_norm(u, W[f"{p}norm{q}"], eps)), W[f"{p}hc{q}.out"], W[f"{p}hc{q}.mix"])

    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        if L["type"] == "mamba2":
            x = sublayer(x, p, 1, lambda h: mamba2(h, W, p + "mix.", m, eps))
        else:
            x = sublayer(x, p, 1, lambda h: parallel_mixer(h, W, p + "mix.", m, eps, hide))
        if L["mlp"] is not None:
            x = sublayer(x, p, 2, lambda h: clamped_ff(h, W, p + "mlp.", L["mlp"]["limit"]))
        if trace is not None:
            trace.append(x.sum(1))
    return cap(rms_norm(x.sum(1), W["final.norm"], eps) @ W["head"].T, cfg["logit_softcap"])


# ---- random models ---------------------------------------------------------------------------------------------------
def random_weights(cfg, seed=0, sharp=1.5):
    """Weights of every tensor of the design, bf16-representable, scaled so that no mechanism vanishes.  `sharp` scales the queries of
    the attention: with a large value single keys stand out."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, s=1.0, mean=0.0):
        return (torch.randn(*shape, generator=g) * s + mean).to(torch.bfloat16)

    D, V, S = cfg["width"], cfg["vocab"], cfg["streams"]
    W = {"embed": rnd(V, D), "pos": rnd(cfg["max_positions"], D, s=0.5), "head": rnd(V, D, s=D ** -0.5), "final.norm": rnd(D, s=0.2, mean=1.0)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        for q in (1, 2) if L["mlp"] else (1,):
            W[f"{p}norm{q}"] = rnd(D, s=0.2, mean=1.0)
            W[f"{p}hc{q}.in"], W[f"{p}hc{q}.out"] = rnd(S, s=0.4, mean=0.8), rnd(S, s=0.4, mean=0.8)
            W[f"{p}hc{q}.mix"] = (torch.eye(S) * 0.8 + torch.randn(S, S, generator=g) * 0.3 / S ** 0.5).to(torch.bfloat16)
        a = p + "mix."
        if L["type"] == "mamba2":
            H, vd, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
            inner, C = H * vd, H * vd + 2 * G * N
            W[a + "in"] = rnd(inner + C + H, D, s=D ** -0.5)
            W[a + "conv"], W[a + "conv.b"] = rnd(C, m["conv"], s=0.6), rnd(C, s=0.3)
            W[a + "dt_bias"], W[a + "A_log"], W[a + "D"] = rnd(H, s=0.5, mean=-1.5), rnd(H, s=0.7), rnd(H, s=0.5, mean=0.5)
            W[a + "norm"], W[a + "o"] = rnd(inner, s=0.2, mean=1.0), rnd(D, inner, s=inner ** -0.5)
        else:
            l, r = m["left"], m["right"]
            for nm, rows, s in (("q", l["heads"] * l["dim"], sharp), ("k", l["kv_heads"] * l["dim"], 1.0), ("v", l["kv_heads"] * l["vdim"], 1.0)):
                W[f"{a}left.{nm}"], W[f"{a}left.{nm}.b"] = rnd(rows, D, s=s * D ** -0.5), rnd(rows, s=0.3)
            W[a + "left.g"] = rnd(l["heads"], D, s=D ** -0.5)
            W[a + "left.o"], W[a + "left.o.b"] = rnd(D, l["heads"] * l["vdim"], s=(l["heads"] * l["vdim"]) ** -0.5), rnd(D, s=0.3)
            for nm, rows in (("q", r["heads"] * r["dim"]), ("k", r["heads"] * r["dim"]), ("v", r["heads"] * r["vdim"]), ("g", r["heads"] * r["vdim"])):
                W[f"{a}right.{nm}"] = rnd(rows, D, s=D ** -0.5)
            W[a + "right.norm"] = rnd(r["heads"] * r["vdim"], s=0.2, mean=1.0)
            W[a + "right.o"] = rnd(D, r["heads"] * r["vdim"], s=(r["heads"] * r["vdim"]) ** -0.5)
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
