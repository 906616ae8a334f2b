"""RMSNorm: y = (x / sqrt(mean(x^2) + eps)) * w, plain weight
(core/src/nn/norm.cpp:25-42; the model's use: core/src/model/emit.cpp:170-176, 440, 449, 512-515)."""
from __future__ import annotations

import torch

from .. import ops
from ..weights.loader import TensorRequest
from .base import Norm, register_norm


@register_norm("rmsnorm")
class RMSNorm(Norm):
    def __init__(self, spec, dtype, device):
        self.width, self.eps, self.tensor = spec.width, float(spec.eps), spec.tensor
        self.weight = None

    def tensor_requests(self):
        return [TensorRequest(self.tensor, (self.width,), "norm")]

    def bind(self, get):
        self.weight = get(self.tensor)

    def as_rms(self):
        return self.weight, self.eps

    def forward(self, x, out_dtype, rows=None):
        n = x.shape[0] if rows is None else rows.numel()
        out = torch.empty((n, self.width), dtype=out_dtype, device=x.device)
        return ops.rmsnorm(x, self.weight, self.eps, out, rows)


@register_norm("rmsnorm_scalar")
class ScalarRMSNorm(RMSNorm):
    """RMS norm whose weight is one number for all coordinates: y = x / sqrt(mean(x^2) + eps) * g.
    The stored tensor has shape []; bound, it is spread over the width, so every kernel that
    takes an RMS norm's weight vector (the norm kernel itself, and the kernels that norm a row
    they have just finished) serves it unchanged."""

    def tensor_requests(self):
        return [TensorRequest(self.tensor, (), "norm")]

    def bind(self, get):
        self.weight = get(self.tensor).reshape(1).expand(self.width).contiguous()


@register_norm("rmsnorm_one_plus")
class OnePlusRMSNorm(RMSNorm):
    """RMS norm whose stored weight is an offset from one: y = x / sqrt(mean(x^2) + eps) * (1 + w).
    Bound, 1 + w is worked out once in float32 (a bfloat16 sum would lose the offset's low bits),
    so every kernel that takes an RMS norm's weight vector serves it unchanged."""

    def tensor_requests(self):
        return [TensorRequest(self.tensor, (self.width,), "bias")]

    def bind(self, get):
        self.weight = (get(self.tensor).float() + 1.0).contiguous()


@register_norm("layernorm")
class LayerNorm(Norm):
    """Layer norm with a weight and optionally a bias (the spec names its tensor): y = (x - mean) /
    sqrt(var + eps) * w [+ b], the variance being the mean of the squared deviations.  It is not an RMS
    norm, so no product kernel applies it to its own result (`as_rms` is None); `ops.stream_join` writes
    it along with the rows it finishes, else it runs as a kernel of its own."""

    def __init__(self, spec, dtype, device):
        self.width, self.eps, self.tensor, self.bias_tensor = spec.width, float(spec.eps), spec.tensor, spec.bias
        self.weight = self.bias = None

    def tensor_requests(self):
        return [TensorRequest(self.tensor, (self.width,), "norm")] + \
               ([TensorRequest(self.bias_tensor, (self.width,), "bias")] if self.bias_tensor else [])

    def bind(self, get):
        self.weight = get(self.tensor)
        if self.bias_tensor:
            self.bias = get(self.bias_tensor)
            if self.bias.dtype != self.weight.dtype:
                self.weight, self.bias = self.weight.float(), self.bias.float()

    def as_layer(self):
        return self.weight, self.bias, self.eps

    def forward(self, x, out_dtype, rows=None):
        n = x.shape[0] if rows is None else rows.numel()
        out = torch.empty((n, self.width), dtype=out_dtype, device=x.device)
        return ops.layernorm(x, self.weight, self.eps, out, rows, bias=self.bias)


class NormPair(Norm):
    """Two RMS norms of the same rows: what a block whose sublayers have norms of their own on one input names as its
    `input_norm()`.  `forward` returns both results; with one eps (and weights of one dtype) a kernel writes
    both from one reading of the row, here or where the rows are finished (`as_pair`)."""

    def __init__(self, first, second):
        self.first, self.second = first, second

    def as_pair(self):
        a, b = self.first.as_rms(), self.second.as_rms()
        if a is None or b is None or a[1] != b[1] or a[0].dtype != b[0].dtype:
            return None
        return a[0], b[0], a[1]

    def forward(self, x, out_dtype, rows=None):
        pair = self.as_pair() if rows is None else None
        if pair is None:
            return self.first.forward(x, out_dtype, rows), self.second.forward(x, out_dtype, rows)
        return ops.rmsnorm_pair(x, pair[0], pair[1], pair[2], torch.empty(x.shape, dtype=out_dtype, device=x.device),
                                torch.empty(x.shape, dtype=out_dtype, device=x.device))


class StreamCast(Norm):
    """Not a norm: the rows as they are, in the dtype asked for.  A block whose sublayers read the
    stream itself names this as its `input_norm()`, so that whatever finishes the stream's rows
    before it (`ops.norm_add` with a weight of None) can leave the copy behind."""

    def forward(self, x, out_dtype, rows=None):
        if rows is not None:
            raise NotImplementedError("a stream cast gathers no rows")
        return ops.cast(x, out_dtype)
