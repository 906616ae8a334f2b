"""A plain, slow Debisun in float64 on the CPU: one function per mechanism, written from the
design's equations and sharing nothing with the package.  A model is the config.json dictionary
plus a dict of tensors by name.  Sequences are independent, so there is no batch anywhere.
"""
from __future__ import annotations

import math

import torch

F = torch.float64


def layer_norm(x, w, b, eps):
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * w + b


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def squared_relu(z):
    return torch.clamp(z, min=0.0) ** 2


def short_conv(u, w):
    """y_t = sum_j w[:, j] u_(t - taps + 1 + j) for u [T, channels], zeros before the start."""
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=F), u])
    return sum(w[:, j] * padded[j:j + u.shape[0]] for j in range(taps))


def bucket(n, rows, most):
    """Which row of the bias table a key n positions back reads: its own row while n is below half the
    rows, then rows that widen logarithmically up to distance `most`, then the last."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(most / half) * (rows - half)))


def distance_bias(T, rel, most):
    """[T, T, heads]: rel[bucket(i - j)] where j <= i, zero elsewhere."""
    rows = torch.tensor([bucket(n, rel.shape[0], most) for n in range(T)])
    back = torch.arange(T).view(T, 1) - torch.arange(T).view(1, T)
    return rel[rows[back.clamp(min=0)]] * (back >= 0).unsqueeze(-1)


def chunk_mask(T, size):
    """[T, T] bool: key j is seen from i when j <= i and both lie in the same stretch of `size`
    positions counted from the sequence's start (size 0: every earlier key)."""
    i, j = torch.arange(T).view(T, 1), torch.arange(T).view(1, T)
    vis = j <= i
    return vis & (i // size == j // size) if size else vis


def softmax_plus_one(scores, visible):
    """exp(s_j) / (1 + sum exp(s_j)) over the visible keys of every row."""
    s = scores.masked_fill(~visible, -math.inf)
    m = torch.clamp(s.max(-1, keepdim=True).values, min=0.0)
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(-m))


def attention(h, get, m):
    """Grouped-query attention: convolved q, k and v, capped scores plus a learned distance bias,
    chunked, one added to the softmax's denominator."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    proj = {n: h @ get(n).T for n in ("q", "k", "v")}
    if m.get("conv"):
        proj = {n: short_conv(u, get(n + ".conv")) for n, u in proj.items()}
    q, k, v = proj["q"].view(T, H, d), proj["k"].view(T, G, d), proj["v"].view(T, G, dv)
    bias = distance_bias(T, get("rel"), m["bias_max"])
    vis = chunk_mask(T, m["mask"]["size"] if m.get("mask") else 0)
    cap = m.get("softcap") or 0.0
    out = torch.zeros(T, H, dv, dtype=F)
    for hh in range(H):
        g = hh // (H // G)
        s = (q[:, hh] @ k[:, g].T) * m["scale"]
        if cap:
            s = cap * torch.tanh(s / cap)
        out[:, hh] = softmax_plus_one(s + bias[:, :, hh], vis) @ v[:, g]
    return out.reshape(T, H * dv) @ get("o").T


def squared_relu_ff(h, get):
    return squared_relu(h @ get("up").T) @ get("down").T


def route(z, correction, r):
    """z [experts + identity] router logits of one token -> (chosen, their weights, margin): softmax
    scores, the choice by score + correction, the chosen ones' scores over their sum times the scale.
    The margin is how far the last choice is from the best output left out."""
    s = torch.softmax(z, -1)
    choice = s + correction
    order = sorted(range(z.numel()), key=lambda e: (-float(choice[e]), e))
    chosen = order[:r["top"]]
    total = sum(float(s[e]) for e in chosen) + 1e-20
    gap = float(choice[order[r["top"] - 1]] - choice[order[r["top"]]]) if len(order) > r["top"] else math.inf
    return chosen, [float(s[e]) / total * r.get("scale", 1.0) for e in chosen], gap


def moe_ff(h, get, mlp, gaps=None):
    """Experts and identity outputs (which hand the input on) by the router, plus a shared expert that
    a number per token gates."""
    r = mlp["router"]
    z = h @ get("router").T
    out = torch.zeros_like(h)
    sent = {}                                   # router output -> [(token, weight)]
    for t in range(h.shape[0]):
        chosen, weights, gap = route(z[t], get("correction"), r)
        if gaps is not None:
            gaps.append(gap)
        for e, w in zip(chosen, weights):
            sent.setdefault(e, []).append((t, w))
    for e, pairs in sent.items():
        rows = torch.tensor([t for t, _ in pairs])
        y = squared_relu_ff(h[rows], lambda n: get(f"e{e}.{n}")) if e < r["experts"] else h[rows]
        out[rows] += torch.tensor([w for _, w in pairs], dtype=F).view(-1, 1) * y
    if mlp.get("shared") is not None:
        out = out + torch.sigmoid(h @ get("shared.sg").T) * squared_relu_ff(h, lambda n: get("shared." + n))
    return out


def side_input(x, e, get, eps):
    """What the layer's own part of a token's second embedding adds to the stream."""
    y = (gelu_tanh(x @ get("gate").T) * e) @ get("proj").T
    return rms(y, eps) * get("norm")


def forward(cfg, tensors, tokens, layers_out=None, gaps=None):
    """Logits [T, vocab] of one sequence; `layers_out` (a list) receives the stream after every
    layer, `gaps` (a list) one list per mixture layer of every token's routing margin."""
    W = {n: t.to(F) for n, t in tensors.items()}
    eps = cfg["norm"]["eps"]
    idx = torch.tensor(list(tokens), dtype=torch.long)
    x = W["embed"][idx]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = layer_norm(x, W[p + "norm1"], W[p + "norm1.b"], eps)
        x = x + attention(h, lambda n: W[p + "mix." + n], L["mixer"]) * W[p + "ls1"]
        mlp = L.get("mlp")
        if mlp is not None:
            h = layer_norm(x, W[p + "norm2"], W[p + "norm2.b"], eps)
            get = lambda n: W[p + "mlp." + n]
            if mlp["kind"] == "dense":
                y = squared_relu_ff(h, get)
            else:
                g = [] if gaps is not None else None
                y = moe_ff(h, get, mlp, g)
                if gaps is not None:
                    gaps.append(g)
            x = x + y * W[p + "ls2"]
        if cfg.get("token_side"):
            n = cfg["token_side"]["dim"]
            e = W["side.embed"][idx][:, i * n:(i + 1) * n]
            x = x + side_input(x, e, lambda name: W[p + "side." + name], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return layer_norm(x, W["final.norm"], W["final.norm.b"], eps) @ W["head"].T


def greedy_generate(cfg, tensors, prompt, n_new):
    seq, out = list(prompt), []
    for _ in range(n_new):
        out.append(int(torch.argmax(forward(cfg, tensors, seq)[-1])))
        seq.append(out[-1])
    return out
