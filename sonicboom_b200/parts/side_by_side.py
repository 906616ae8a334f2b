"""Two mixers on the same input, joined by their mean after a norm each, or by a weighted sum.

`join` "mean" (the default): with L and R the two results,

    y = (rms(L) * w_left + rms(R) * w_right) / 2,      rms(u) = u / sqrt(mean(u^2) + eps)

over the model width, with plain weights.  `params`: `left`, `right` (the two `MixerSpec`s, of
any registered kinds), `left_out`, `right_out` (tensor names of the two weights after the
prefix), `eps`.  The halves of the weights are made at bind (halving is exact), so each side joins the stream
with the kernel that norms a sublayer's result and adds it (`ops.norm_add`).

`join` "sum":  y = left_scale * L + right_scale * R (`params`: `left`, `right`, `left_scale`, `right_scale`).  Two mixers that
open themselves (`Mixer.input_matrix`) share their products: one over both input matrices' rows, and one over
both output matrices' columns, whose operand's columns each side writes times its scale in float32 before they
are rounded; the norm after the mixer can ride on that product.  Others run one after the other and join
by `ops.stream_join`.

At most one of the two may keep paged keys and values, and at most one
fixed-size state: a schedule entry owns one cache entry and one state row."""
from __future__ import annotations

import torch

from .. import ops
from ..weights.loader import TensorRequest
from .attention import _cat
from .base import MIXERS, Mixer, make, register_mixer


@register_mixer("side_by_side")
class SideBySide(Mixer):
    def __init__(self, spec, dtype, device):
        from ..config.specs import ConfigError
        self.spec, self.dtype, self.device = spec, dtype, device
        p = dict(spec.params)
        self.join = p.get("join", "mean")
        if self.join not in ("mean", "sum"):
            raise ConfigError(f"side_by_side join {self.join!r} (mean or sum)")
        try:
            self.sides = [make(MIXERS, "mixer", p[k], dtype, device) for k in ("left", "right")]
            self.names = (p["left_out"], p["right_out"]) if self.join == "mean" else ()
            self.scales = (float(p["left_scale"]), float(p["right_scale"])) if self.join == "sum" else ()
        except KeyError as e:
            raise ConfigError(f"side_by_side needs the parameter {e.args[0]}") from None
        self.eps = float(p.get("eps", 1e-6))
        if sum(s.kv_need() is not None for s in self.sides) > 1 or \
                sum(s.state_need() is not None for s in self.sides) > 1:
            raise ConfigError("side_by_side: both sides ask for the same kind of cache")
        self.half_weights = self.w_in = self.w_o = self.scale_rows = None
        self.right_at = self.right_col = 0          # where the right side's columns start in the shared products' operands

    def kv_need(self):
        return next((n for n in (s.kv_need() for s in self.sides) if n is not None), None)

    def state_need(self):
        return next((n for n in (s.state_need() for s in self.sides) if n is not None), None)

    def tensor_requests(self):
        p, d = self.spec.prefix, self.spec.width
        return [r for s in self.sides for r in s.tensor_requests()] + \
            [TensorRequest(p + n, (d,), "norm") for n in self.names]

    def bind(self, get):
        for s in self.sides:
            s.bind(get)
        if self.join == "mean":
            self.half_weights = [(get(self.spec.prefix + n) * 0.5).contiguous() for n in self.names]
            return
        ins, outs = [s.input_matrix() for s in self.sides], [s.output_matrix() for s in self.sides]
        if any(t is None for t in ins + outs):
            self.scale_rows = [torch.full((self.spec.width,), c, dtype=torch.float32, device=self.device) for c in self.scales]
            return
        d = self.spec.width
        pad = [torch.zeros((-t.shape[0] % 4, d), dtype=t.dtype, device=t.device) for t in ins]      # 16-byte starts
        self.w_in = _cat([ins[0], pad[0], ins[1], pad[1]])
        self.right_at, self.right_col = ins[0].shape[0] + pad[0].shape[0], outs[0].shape[1]
        self.w_o = torch.cat(outs if outs[0].dtype == outs[1].dtype else [t.float() for t in outs], dim=1).contiguous()
        for s in self.sides:
            s.release_matrices()

    def first_weights(self, rows):
        if self.w_in is None:
            return self.sides[0].first_weights(rows)
        n, k = self.w_in.shape
        late = self.w_in.dtype == torch.bfloat16 and ops.requests_weights_late(rows, n, k, self.w_in.device)
        return self.w_in if late else None

    def forward(self, h, ctx, residual=None):
        if self.w_in is not None:
            return self._shared(h, ctx, residual)
        x = residual if residual is not None else \
            torch.zeros((h.shape[0], self.spec.width), dtype=torch.float32, device=h.device)
        for i, side in enumerate(self.sides):
            ctx.next_norm = ctx.next_weights = None        # a row kernel follows a side's product
            y = side.forward(h, ctx)
            if self.join == "mean":
                ops.norm_add(y, x, self.half_weights[i], self.eps, x)
            else:
                ops.stream_join(y, x, self.scale_rows[i], x)
        return x

    def _shared(self, h, ctx, residual):
        rows = h.shape[0]
        proj = torch.empty((rows, self.w_in.shape[0]), dtype=torch.float32, device=h.device)
        ops.linear(h, self.w_in, proj)
        mixed = torch.empty((rows, self.w_o.shape[1]), dtype=self.dtype, device=h.device)
        for side, at, col, scale in zip(self.sides, (0, self.right_at), (0, self.right_col), self.scales):
            side.mix_rows(proj, at, ctx, mixed, col, scale)
        out = residual if residual is not None else \
            torch.empty((rows, self.spec.width), dtype=torch.float32, device=h.device)
        return ctx.linear(mixed, self.w_o, out, ops.EPI_RESIDUAL if residual is not None else ops.EPI_NONE,
                          residual=residual, act_dtype=self.dtype)
