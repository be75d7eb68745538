"""Plain statement of the Gipozen design, one function per mechanism.

Works on the raw config dictionary and a name -> tensor dictionary, shares nothing with the package, and is slow on purpose.
Everything runs in the dtype of the weights (float64 by default), one sequence at a time, without any cache: a prompt of n tokens is
always computed from its first token."""
import math

import torch

SLOPE = 1.702


# ---- small pieces --------------------------------------------------------------------------------------------------
def sigmoid(x):
    return 1 / (1 + torch.exp(-x))


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, g, eps):
    """g: one number."""
    return unit_rms(x, eps) * g


def poly_norm(z, coef, eps):
    """z [n, ff]; coef = (a, b, c, e)."""
    a, b, c, e = (float(v) for v in coef)
    return a * unit_rms(z, eps) + b * unit_rms(z * z, eps) + c * unit_rms(z * z * z, eps) + e


def short_conv(u, w):
    """u [n, channels], w [channels, taps]: every channel over its own last `taps` values, the newest with the last weight."""
    n, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for t in range(n):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                y[t] += w[:, j] * u[s]
    return y


# ---- attention -------------------------------------------------------------------------------------------------------
def visible(i, size, keep_first):
    """The positions that position i sees."""
    return [j for j in range(i + 1) if i - j < size or j < keep_first]


def one_map(q, k, v, scale, size, keep_first, hide=None):
    """q [n, d], k [n, d], v [n, dv] of one head -> [n, dv].  `hide` plants a mistake: hide(i) gives the positions query i leaves out."""
    s = torch.full((q.shape[0], q.shape[0]), float("-inf"), dtype=q.dtype)
    scores = q @ k.T * scale
    for i in range(q.shape[0]):
        at = visible(i, size, keep_first)
        if hide is not None:
            no = hide(i)
            at = [j for j in at if j not in no or j == i]
        s[i, at] = scores[i, at]
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return (e / e.sum(-1, keepdim=True)) @ v


def mixing_factor(W, diff):
    return float(torch.exp((W["lq1"] * W["lk1"]).sum()) - torch.exp((W["lq2"] * W["lk2"]).sum())) + diff


def combine(a1, a2, lam, diff, eps):
    """One head's two maps [n, dv] -> [n, dv]."""
    return unit_rms(a1 - lam * a2, eps) * (1 - diff)


def keys_and_values(h, W):
    return short_conv(h @ W["k"].T, W["k.conv"]), short_conv(h @ W["v"].T, W["v.conv"])


def attention(h, W, m, eps, kv=None, hide=None):
    """h [n, width]; kv: keys and values of an earlier layer, or None for the layer's own.  Returns the output and the keys and values used."""
    n, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = short_conv(h @ W["q"].T, W["q.conv"]).view(n, H, 2, d)
    if kv is None:
        kv = keys_and_values(h, W)
    k, v = kv[0].view(n, G, 2, d), kv[1].view(n, G, dv)
    lam = mixing_factor(W, m["diff"])
    heads = []
    for x in range(H):
        y = x // (H // G)
        a1, a2 = (one_map(q[:, x, i], k[:, y, i], v[:, y], m["scale"], m["mask"]["size"], m["mask"]["keep_first"], hide) for i in (0, 1))
        heads.append(combine(a1, a2, lam, m["diff"], eps))
    o = torch.cat(heads, -1) * sigmoid(h @ W["g"].T)
    return o @ W["o"].T, kv


# ---- feed-forwards ------------------------------------------------------------------------------------------------------
def dense(h, W, eps):
    return poly_norm(h @ W["up"].T, W["act"], eps) @ W["down"].T


def expert(h, gate, up, down, limit):
    g = torch.clamp(h @ gate.T, max=limit)
    u = torch.clamp(h @ up.T, -limit, limit)
    return (g * sigmoid(SLOPE * g) * (u + 1)) @ down.T


def route(z, correction, top):
    """z [E] logits of one token -> chosen experts and their weights."""
    e = torch.exp(z - z.max())
    s = e / e.sum()
    order = sorted(range(z.numel()), key=lambda i: -float(s[i] + correction[i]))[:top]
    return order, [s[i] for i in order]


def experts(h, W, spec):
    router = spec["router"]
    z = h @ W["router"].T
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for i, w in zip(*route(z[t], W["correction"], router["top"])):
            if i >= router["experts"]:
                out[t] += w * h[t]
            else:
                out[t] += w * expert(h[t], *(W[f"e{i}.{n}"] for n in ("gate", "up", "down")), spec["expert"]["limit"])
    if spec.get("shared"):
        out = out + sigmoid(h @ W["shared.sg"].T) * expert(h, *(W["shared." + n] for n in ("gate", "up", "down")), spec["shared"]["limit"])
    return out


# ---- the model ---------------------------------------------------------------------------------------------------------
def part(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def depth_average(history, w):
    return sum(w[j] * x for j, x in enumerate(history))


def forward(cfg, weights, tokens, layers_out=None, hide=None):
    """Logits [n, vocab] of one sequence; `layers_out` (a list) receives the stream after every layer, averaged over the depth; hide: see one_map."""
    eps = cfg["norm"]["eps"]
    x = weights["embed"][torch.tensor(tokens)]
    history, kvs = [x], []
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        src = m.get("kv_from")
        y, kv = attention(rms_norm(x, weights[p + "norm1"], eps), part(weights, p + "mix."), m, eps, None if src is None else kvs[src], hide)
        kvs.append(kv)
        x = x + y
        if layer["mlp"] is not None:
            h, W = rms_norm(x, weights[p + "norm2"], eps), part(weights, p + "mlp.")
            x = x + (dense(h, W, eps) if layer["mlp"]["kind"] == "dense" else experts(h, W, layer["mlp"]))
        history.append(x)
        x = depth_average(history, weights[p + "dwa"])
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms_norm(x, weights["final.norm"], eps) @ weights["head"].T * cfg["logit_scale"]


def greedy(cfg, weights, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(cfg, weights, toks)[-1].argmax()))
    return toks[len(prompt):]


def shapes(cfg):
    """Every tensor name with its shape."""
    D = cfg["width"]
    out = {"embed": (cfg["vocab"], D), "final.norm": (), "head": (cfg["vocab"], D)}
    for i, s in enumerate(cfg["layers"]):
        m, f, p = s["mixer"], s["mlp"], f"l{i}."
        d, inner = m["dim"], m["heads"] * m["vdim"]
        out[p + "norm1"], out[p + "dwa"] = (), (i + 2,)
        rows = {"q": m["heads"] * 2 * d}
        if m.get("kv_from") is None:
            rows.update(k=m["kv_heads"] * 2 * d, v=m["kv_heads"] * m["vdim"])
        for n, r in rows.items():
            out[p + "mix." + n], out[p + f"mix.{n}.conv"] = (r, D), (r, m["conv"])
        for n in ("lq1", "lk1", "lq2", "lk2"):
            out[p + "mix." + n] = (d,)
        out[p + "mix.g"], out[p + "mix.o"] = (inner, D), (D, inner)
        if f is None:
            continue
        out[p + "norm2"] = ()
        if f["kind"] == "dense":
            out.update({p + "mlp.up": (f["ff"], D), p + "mlp.down": (D, f["ff"]), p + "mlp.act": (4,)})
            continue
        r = f["router"]
        blocks = [(f"e{e}", f["expert"]["ff"]) for e in range(r["experts"])] + ([("shared", f["shared"]["ff"])] if f.get("shared") else [])
        for n, ff in blocks:
            out.update({p + f"mlp.{n}.gate": (ff, D), p + f"mlp.{n}.up": (ff, D), p + f"mlp.{n}.down": (D, ff)})
        total = r["experts"] + r["identity"]
        out[p + "mlp.router"], out[p + "mlp.correction"] = (total, D), (total,)
        if f.get("shared"):
            out[p + "mlp.shared.sg"] = (1, D)
    return out


def random_weights(cfg, seed=0, sharp=1.0):
    """bf16-representable float64 weights.  `sharp` scales the queries and keys: larger scores, so that single keys matter."""
    g = torch.Generator().manual_seed(seed)
    W = {}
    for name, shape in shapes(cfg).items():
        t, leaf = torch.randn(shape, generator=g, dtype=torch.float64), name.rsplit(".", 1)[-1]
        if leaf in ("norm", "norm1", "norm2"):
            t = 1 + 0.2 * t
        elif leaf == "dwa":
            t = 0.3 * t + torch.tensor([0.0] * (shape[0] - 1) + [1.0], dtype=torch.float64)
        elif leaf == "conv":
            t = 0.5 * t * (sharp if name.endswith((".q.conv", ".k.conv")) else 1.0)
            t[:, -1] += 0.7 * (sharp if name.endswith((".q.conv", ".k.conv")) else 1.0)
        elif leaf in ("lq1", "lk1", "lq2", "lk2"):
            t = t * (0.5 * shape[0] ** -0.25)
        elif leaf == "act":
            t = 0.3 * t + torch.tensor([1.0, 0.5, 0.3, 0.0], dtype=torch.float64)
        elif leaf == "correction":
            t = 0.05 * t
        elif leaf == "router":
            t = t * (1.5 * shape[-1] ** -0.5)
        elif name != "embed":
            t = t * shape[-1] ** -0.5
        W[name] = t.to(torch.bfloat16).double()
    return W
