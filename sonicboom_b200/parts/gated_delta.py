"""The gated delta rule: a recurrence over a matrix state with one decay per token and head, whose update replaces
what the state holds under the unit key,

    S <- g_t S;   u = beta_t (v_t - S^T k_t);   S <- S + k_t u^T;   o_t = S^T q_t            per head, S_0 = 0,

so that the read-out sees the token's own write.  q and k have `n_kv_heads` heads of `head_dim` values, v `n_heads`
heads of `vdim`; head h reads key head h // (n_heads / n_kv_heads).  Every channel of q, k and v passes a short causal
convolution over time (`conv` taps) and silu; q and k are divided by sqrt(sum of squares over the head +
`unit_eps`), and q is multiplied by `q_scale`.  beta = sigmoid(B h) and g = exp(-exp(A_log) * softplus(A h + dt_bias)),
one number per head.  Output: an RMS norm within each head (`eps`, one weight vector for all heads), the gate
silu(G h), then the product with O.

q, k, v, g, beta's and the decay's logits are one product; everything from its float32 rows to the gated result is
float32 (`ops.gated_delta`: one kernel for a step of one token a sequence, a chunked scan for prompts and
portions).  State of a sequence: "memory" (float32 [heads, vdim, head_dim]) and, with more than one tap, "ring" (the
convolution's last inputs, float32 [taps, channels], the input of position p in row p mod taps).

Tensors after the prefix: q, k [n_kv_heads * head_dim, width]; v, g [n_heads * vdim, width]; q.conv, k.conv, v.conv
[channels, taps]; b, a [n_heads, width]; A_log, dt_bias [n_heads]; norm [vdim]; o [width, n_heads * vdim]."""
from __future__ import annotations

import torch

from .. import ops
from ..cache.kv import StateNeed
from ..weights.loader import TensorRequest
from .attention import _cat
from .base import Mixer, register_mixer


@register_mixer("gated_delta_rule")
class GatedDeltaRule(Mixer):
    def __init__(self, spec, dtype, device):
        from ..config.specs import ConfigError
        self.spec, self.dtype, self.device = spec, dtype, device
        p = dict(spec.params)
        self.h, self.g, self.dim = spec.n_heads, spec.n_kv_heads, spec.head_dim
        self.vd, self.taps = int(p.get("vdim", self.dim)), int(p.get("conv", 1))
        self.eps, self.unit_eps = float(p.get("eps", 1e-6)), float(p.get("unit_eps", 1e-6))
        self.q_scale = float(p.get("q_scale", 1.0))
        if self.h % self.g:
            raise ConfigError(f"{self.h} heads are not a multiple of {self.g} key heads")
        if self.taps < 1:
            raise ConfigError(f"a convolution of {self.taps} taps")
        self.kw, self.vw = self.g * self.dim, self.h * self.vd
        # columns of the input product: the convolved channels [q | k | v], the gate, beta's and the decay's logits
        self.channels = 2 * self.kw + self.vw
        self.g_off = self.channels
        self.b_off = self.g_off + self.vw
        self.a_off = self.b_off + self.h
        self.w_in = self.w_o = self.conv_w = self.a_log = self.dt_bias = self.norm_w = None

    def state_need(self):
        need = {"memory": StateNeed((self.h, self.vd, self.dim), torch.float32)}
        if self.taps > 1:
            need["ring"] = StateNeed((self.taps, self.channels), torch.float32)
        return need

    def tensor_requests(self):
        p, d = self.spec.prefix, self.spec.width
        req = []
        for n, w in (("q", self.kw), ("k", self.kw), ("v", self.vw)):
            req += [TensorRequest(p + n, (w, d)), TensorRequest(p + n + ".conv", (w, self.taps))]
        return req + [TensorRequest(p + "g", (self.vw, d)), TensorRequest(p + "b", (self.h, d)), TensorRequest(p + "a", (self.h, d)),
                      TensorRequest(p + "A_log", (self.h,), "bias"), TensorRequest(p + "dt_bias", (self.h,), "bias"),
                      TensorRequest(p + "norm", (self.vd,), "norm"), TensorRequest(p + "o", (d, self.vw))]

    def bind(self, get):
        p = self.spec.prefix
        rows = [get(p + n) for n in ("q", "k", "v", "g", "b", "a")]
        pad = -(self.a_off + self.h) % 4             # rows of a multiple of four values: 16-byte copies of them
        if pad:
            rows.append(torch.zeros((pad, self.spec.width), dtype=rows[0].dtype, device=rows[0].device))
        self.w_in = _cat(rows)
        self.w_o = get(p + "o")
        self.conv_w = torch.cat([get(p + n + ".conv").float() for n in ("q", "k", "v")]).contiguous()
        self.a_log, self.dt_bias, self.norm_w = (get(p + n).float().contiguous() for n in ("A_log", "dt_bias", "norm"))

    def first_weights(self, rows):
        n, k = self.w_in.shape
        late = self.w_in.dtype == torch.bfloat16 and ops.requests_weights_late(rows, n, k, self.w_in.device)
        return self.w_in if late else None

    def input_matrix(self):
        return self.w_in

    def output_matrix(self):
        return self.w_o

    def release_matrices(self):
        self.w_in = self.w_o = None

    def mix_rows(self, proj, at, ctx, out, col=0, scale=1.0):
        return ops.gated_delta(proj, at, at + self.a_off, at + self.b_off, at + self.g_off, ctx.plan, self.h, self.g, self.dim,
                               self.vd, self.conv_w, self.a_log, self.dt_bias, self.q_scale, self.unit_eps, self.norm_w,
                               self.eps, ctx.state("ring") if self.taps > 1 else None, ctx.state("memory"), out, col, scale)

    def forward(self, h, ctx, residual=None):
        rows = h.shape[0]
        proj = torch.empty((rows, self.w_in.shape[0]), dtype=torch.float32, device=h.device)
        ops.linear(h, self.w_in, proj)
        mixed = torch.empty((rows, self.vw), dtype=self.dtype, device=h.device)
        self.mix_rows(proj, 0, ctx, mixed)
        out = residual if residual is not None else \
            torch.empty((rows, self.spec.width), dtype=torch.float32, device=h.device)
        return ctx.linear(mixed, self.w_o, out, ops.EPI_RESIDUAL if residual is not None else ops.EPI_NONE,
                          residual=residual, act_dtype=self.dtype)
