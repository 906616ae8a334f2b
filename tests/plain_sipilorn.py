"""Plain, slow implementation of the Sipilorn decoder, used only as the test oracle.

Whole sequences, no cache, no state carried between calls, one function per mechanism, CPU torch in
float64.  It shares no code with the package under test: it reads config.json as a dictionary and takes
the tensors as a dictionary of torch tensors by name.

Notation.  T tokens, width D, positions 0 .. T-1.  rms(x) = x / sqrt(mean(x^2) + eps) along the last
axis.  A linear weight W is [out, in] and acts as h @ W.T.
"""
from __future__ import annotations

import torch
import torch.nn.functional as nnf

F = torch.float64
UNIT_EPS = 1e-6


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rotate_halves(x, base, dims):
    """x [T, heads, d]: the first `dims` values of a head turn by t * base^(-2i/dims), value i with
    value i + dims/2; the rest pass."""
    if dims == 0:
        return x.clone()
    half = dims // 2
    i = torch.arange(half, dtype=F)
    a = torch.arange(x.shape[0], dtype=F)[:, None] * float(base) ** (-2.0 * i / dims)
    c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def window_mask(T, size):
    """[T, T]: whether row i sees column j; `size` None: every earlier position."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & (i - j < (size if size is not None else T))


def window_attention(h, W, p, m, eps):
    """Gated softmax attention over a window: normed and rotated q and k heads, and a logistic gate for
    every value of the concatenated heads.  Returns the gated heads [T, heads * vdim], before `o`."""
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms((h @ W[p + "q"].T).view(T, H, d), eps) * W[p + "q.norm"]
    k = rms((h @ W[p + "k"].T).view(T, G, d), eps) * W[p + "k.norm"]
    v = (h @ W[p + "v"].T).view(T, G, dv)
    q, k = (rotate_halves(x, m["rot"]["base"], m["rot"]["dims"]) for x in (q, k))
    see = window_mask(T, m["mask"]["size"] if m.get("mask") is not None else None)
    out = torch.zeros(T, H, dv, dtype=F)
    for hh in range(H):
        g = hh // (H // G)
        s = (q[:, hh] @ k[:, g].T) * m["scale"]
        out[:, hh] = torch.softmax(s.masked_fill(~see, -torch.inf), -1) @ v[:, g]
    return out.reshape(T, H * dv) * torch.sigmoid(h @ W[p + "g"].T)


def short_conv(x, w):
    """y_t = sum_j w[:, j] x_(t - taps + 1 + j), zeros before the start; x [T, C], w [C, taps]."""
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=F), x])
    return sum(w[:, j] * padded[j:j + x.shape[0]] for j in range(taps))


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + UNIT_EPS)


def gated_delta_rule(q, k, v, decay, beta):
    """Per head, from S = 0: S <- decay_t S; u = beta_t (v_t - S^T k_t); S <- S + k_t u^T; o_t = S^T q_t.
    q, k [T, G, d], v [T, H, dv], decay and beta [T, H]; head h reads q and k of head h // (H / G)."""
    T, H, dv = v.shape
    G, d = q.shape[1], q.shape[2]
    q, k = (x.repeat_interleave(H // G, dim=1) for x in (q, k))
    S = torch.zeros(H, d, dv, dtype=F)
    out = torch.zeros(T, H, dv, dtype=F)
    for t in range(T):
        S = S * decay[t][:, None, None]
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out


def delta_inputs(h, W, p, m):
    """(q, k, v, decay, beta) of the recurrence from the mixer's input."""
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (nnf.silu(short_conv(h @ W[p + n].T, W[p + n + ".conv"])) for n in ("q", "k", "v"))
    q, k = unit(q.view(T, G, d)) * d ** -0.5, unit(k.view(T, G, d))
    beta = torch.sigmoid(h @ W[p + "b"].T)
    decay = torch.exp(-torch.exp(W[p + "A_log"]) * nnf.softplus(h @ W[p + "a"].T + W[p + "dt_bias"], threshold=200.0))
    return q, k, v.view(T, H, dv), decay, beta


def delta_mixer(h, W, p, m, eps):
    """The gated delta rule with its short convolutions, output norm and gate.  Returns [T, heads * vdim],
    before `o`."""
    T, H, dv = h.shape[0], m["heads"], m["vdim"]
    o = gated_delta_rule(*delta_inputs(h, W, p, m))
    o = rms(o, eps) * W[p + "norm"] * nnf.silu(h @ W[p + "g"].T).view(T, H, dv)
    return o.reshape(T, H * dv)


def mixer(h, W, p, L, eps):
    m = L["mixer"]
    if L["type"] == "delta":
        return delta_mixer(h, W, p, m, eps) @ W[p + "o"].T
    left = window_attention(h, W, p + "left.", m["left"], eps) @ W[p + "left.o"].T
    right = delta_mixer(h, W, p + "right.", m["right"], eps) @ W[p + "right.o"].T
    return m["left_scale"] * left + m["right_scale"] * right


def dense(h, W, p):
    return (nnf.silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def expert(h, W, p):
    return torch.relu(h @ W[p + "up"].T) ** 2 @ W[p + "down"].T


def experts_by_token(h, W, p, tokens):
    """Every token id has its experts in a table; each counts one over their number."""
    table = W[p + "table"].long()[tokens]
    top = table.shape[1]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in table[t].tolist():
            out[t] += expert(h[t:t + 1], W, f"{p}e{j}.")[0] / top
    return out


def feed_forward(h, W, p, mlp, tokens):
    return dense(h, W, p) if mlp["kind"] == "dense" else experts_by_token(h, W, p, tokens)


def run_order(cfg):
    """(layer, number of the pass it starts or None) in the order layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop or loop["start"] == loop["stop"]:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return [(i, None) for i in range(a)] + \
        [(i, t if i == a else None) for t in range(loop["times"]) for i in range(a, b)] + \
        [(i, None) for i in range(b, n)]


def forward(cfg, tensors, tokens, streams=None):
    """float64 logits [T, vocab]; `streams`, a list, receives the residual stream after every layer run."""
    W = {n: (t if n.endswith(".table") else t.to(F)) for n, t in tensors.items()}
    eps = cfg["norm"]["eps"]
    toks = torch.tensor(list(tokens), dtype=torch.long)
    x = rms(W["embed"][toks], eps) * W["embed.norm"]
    for i, t in run_order(cfg):
        L, p = cfg["layers"][i], f"l{i}."
        if t is not None:
            x = x + W["loop.step"][t]
        y = mixer(rms(x, eps) * W[p + "norm1"], W, p + "mix.", L, eps)
        if L["mlp"] is not None:
            y = y + feed_forward(rms(x, eps) * W[p + "norm2"], W, p + "mlp.", L["mlp"], toks)
        x = x + y
        if streams is not None:
            streams.append(x.clone())
    logits = (rms(x, eps) * W["final.norm"]) @ W["head"].T
    cap = cfg.get("logit_softcap")
    return cap * torch.tanh(logits / cap) if cap else logits
