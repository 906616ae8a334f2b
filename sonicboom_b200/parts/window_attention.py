"""Grouped-query softmax attention over a sliding window of the paged cache, with the options
that attention layers of newer designs combine:

* query/key heads of size `head_dim` and value heads of size `vdim` (the cache entry's heads are
  as wide as the larger of the two, rounded up to what the tensor-core kernels take; the padding
  is zeros, so scores and sums are unchanged);
* rotation of a prefix of every q and k head in either layout of pairs (the spec's position
  encoding: "rope_halves" pairs i with i + n/2, "rope_interleaved" 2i with 2i + 1);
* `qk_norm` = (q name, k name): the whole q projection of a token (all heads at once) and the
  whole k projection are RMS-normed with a plain weight of that size before the rotation;
* `values` = "keys": there is no value matrix, the values are the key projection as it leaves
  the matrix (before norm and rotation);
* `rotate_values`: the value of position j is turned by j over all of vdim (same layout of
  pairs, frequencies base^(-2m/vdim)) before it is cached, and every head's result at position i
  is turned back by i: what a head sums depends on i - j only;
* `sink` = name: one learned number per query head whose exponential joins the softmax's
  denominator (it has no key, no value and is not scaled);
* `bias` = (q name, k name, v name): the three projections have biases;
* `head_norm` = ("before", q name, k name): every q and k head is RMS-normed by itself before the
  rotation, with one weight of head_dim values for all heads; ("after",): every head is divided by
  its root mean square after the rotation, without a weight;
* `softcap` = c: a score s becomes c tanh(s / c) before the softmax;
* `gate` = name: a matrix [heads, width]; head h's result is multiplied by the logistic function
  of its product with the mixer's input (it rides on the input product);
* `value_gate` = name: a matrix [heads*vdim, width]; every value of the concatenated heads is multiplied by the
  logistic function of its own product with the mixer's input (it rides on the input product too);
* `conv` = taps: every channel of q, k and v passes a short causal convolution over time right after the
  projection (tensors: the projection's name + ".conv", [channels, taps]); the last taps - 1 projected
  values of a sequence are state of the cache;
* `distance_bias` = (name, most[, rows]): a learned number is added to the capped score, row
  `distance_bucket(i - j)` of a table [rows, heads] whose rows beyond the first half widen logarithmically
  up to distance `most` (`rows` is the stored tensor's when not given);
* `chunk` = n: the query at position i sees key j <= i only when floor(i / n) = floor(j / n), positions
  counted from the sequence's start; the cache gives the pages of earlier chunks back;
* `sink` may also be a number: every head's sink has that score;
* a position encoding with a `magnitude` (stretched rotations) multiplies cosines and sines by it.

Tensors after the prefix: q [heads*head_dim, width], k [kv_heads*head_dim, width], v
[kv_heads*vdim, width] unless the values are the keys, o [width, heads*vdim], and what the options
name.  All input projections are one product; `ops.attn_prep` finishes its float32 rows into
queries and cache rows (`ops.conv_heads` with a convolution and nothing else to do to the heads), the
framework's attention kernels run on them unchanged, and
`ops.attn_unrotate` turns results back and drops the padding where either is needed (`ops.attn_gate` with a
`value_gate`, or as one side of a mixer that shares its products)."""
from __future__ import annotations

import math

import torch

from .. import ops
from ..cache.kv import KVNeed, StateNeed
from ..weights.loader import TensorRequest
from .attention import _cat
from .base import POSITION_ENCODINGS, Mixer, make, register_mixer
from .rotary import frequency_table

HEAD_STEP = 16          # the tensor-core attention kernels take head sizes in these steps


def distance_bucket(n: int, rows: int, most: int) -> int:
    """The table row for a key n positions back: its own for n below half the rows, then rows that widen
    logarithmically until distance `most`, then the last."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(most / half) * (rows - half)))


def bias_by_distance(table: torch.Tensor, most: int, longest: int = 0) -> torch.Tensor:
    """float32 [heads, n]: the bias of every distance 0 ... n - 1, the last entry standing for all larger
    ones (no more than `longest` entries when distances stay below it)."""
    from ..config.specs import ConfigError
    rows = table.shape[0]
    if rows < 2 or 2 * most <= rows:
        raise ConfigError(f"a distance bias of {rows} rows up to distance {most} (at least 2 rows, half of them below it)")
    n = most + 1 if longest <= 0 else min(most + 1, longest)
    index = torch.tensor([distance_bucket(d, rows, most) for d in range(n)], device=table.device)
    return table.float()[index].t().contiguous()


@register_mixer("window_attention")
class WindowAttention(Mixer):
    def __init__(self, spec, dtype, device):
        from ..config.specs import ConfigError
        self.spec, self.dtype, self.device = spec, dtype, device
        p = dict(spec.params)
        self.hq, self.hkv, self.dim = spec.n_heads, spec.n_kv_heads, spec.head_dim
        self.vdim = int(p.get("vdim", self.dim))
        self.eps = float(p.get("eps", 1e-6))
        self.values_are_keys = p.get("values", "own") == "keys"
        self.rotate_values = bool(p.get("rotate_values", False))
        self.qk_norm, self.sink_name = p.get("qk_norm"), p.get("sink")
        self.bias_names, self.gate_name = p.get("bias"), p.get("gate")
        self.value_gate = p.get("value_gate")
        if self.value_gate and (self.gate_name or self.rotate_values):
            raise ConfigError("a gate for every value goes with unrotated values and no gate per head")
        self.gate_name = self.value_gate or self.gate_name
        self.softcap = float(p.get("softcap", 0.0) or 0.0)
        self.taps, self.chunk = int(p.get("conv", 0) or 0), int(p.get("chunk", 0) or 0)
        self.distance_bias = p.get("distance_bias")
        self.sink_value = None
        if isinstance(self.sink_name, (int, float)):
            self.sink_value, self.sink_name = float(self.sink_name), None
        if self.chunk < 0 or self.taps < 0:
            raise ConfigError(f"a convolution of {self.taps} taps, chunks of {self.chunk} positions (0: none)")
        head_norm = p.get("head_norm")
        self.head_norm = head_norm[0] if head_norm else None
        if self.head_norm not in (None, "before", "after") or (self.head_norm and self.qk_norm):
            raise ConfigError(f"head_norm {head_norm!r}: ('before', q name, k name) or ('after',), and not "
                              "beside a norm of the whole projection")
        if self.head_norm == "before":
            self.qk_norm = tuple(head_norm[1:3])
        if self.softcap < 0.0:
            raise ConfigError(f"a score cap of {self.softcap} (0: none)")
        self.names = tuple(p.get("names", ("q", "k", "v", "o")))
        if self.hq % self.hkv:
            raise ConfigError(f"{self.hq} query heads are not a multiple of {self.hkv} key/value heads")
        if self.values_are_keys and self.vdim != self.dim:
            raise ConfigError(f"values that are the keys need vdim == head_dim, not {self.vdim} and {self.dim}")
        if self.rotate_values and self.vdim % 2:
            raise ConfigError(f"rotated values need an even vdim, not {self.vdim}")
        if self.rotate_values and spec.position is None:
            raise ConfigError("rotated values take their frequencies' base from the position encoding")
        self.hd = (max(self.dim, self.vdim) + HEAD_STEP - 1) // HEAD_STEP * HEAD_STEP
        self.rot, self.interleaved, self.inv_freq, self.v_inv_freq = 0, False, None, None
        self.rot_scale = 1.0
        if spec.position is not None:
            pe = make(POSITION_ENCODINGS, "position encoding", spec.position, dtype, device)
            self.rot_scale = float(getattr(pe, "magnitude", 1.0))
            self.interleaved = getattr(pe, "layout", "halves") == "interleaved"
            self.rot = spec.position.rotary_dim
            self.inv_freq = pe.inv_freq if self.rot > 0 else None
            if self.rotate_values:
                self.v_inv_freq = frequency_table(spec.position.theta, self.vdim, device)
        self.qw, self.kw = self.hq * self.dim, self.hkv * self.dim
        self.vw = 0 if self.values_are_keys else self.hkv * self.vdim
        self.gw = 0 if not self.gate_name else self.hq * self.vdim if self.value_gate else self.hq
        if self.bias_names and self.values_are_keys:
            raise ConfigError("biases of q, k and v need a value projection of its own")
        if self.taps and (self.values_are_keys or self.gate_name):
            raise ConfigError("a convolution of q, k and v needs a value projection and no gate beside them")
        # nothing but the convolution happens to a head: its kernel writes queries and cache rows
        self.conv_only = bool(self.taps) and self.rot == 0 and not self.rotate_values and not self.qk_norm and not self.head_norm
        self.w_in = self.w_o = self.q_norm = self.k_norm = self.sink = self.b_in = self.w_conv = self.bias = None

    def kv_need(self):
        return KVNeed(self.hkv, self.hd, self.spec.window, chunk=self.chunk)

    def state_need(self):
        return StateNeed((self.taps - 1, self.qw + self.kw + self.vw), torch.float32) if self.taps > 1 else None

    def tensor_requests(self):
        p, d = self.spec.prefix, self.spec.width
        q, k, v, o = self.names
        req = [TensorRequest(p + q, (self.qw, d)), TensorRequest(p + k, (self.kw, d)),
               TensorRequest(p + o, (d, self.hq * self.vdim))]
        if not self.values_are_keys:
            req.append(TensorRequest(p + v, (self.hkv * self.vdim, d)))
        if self.qk_norm:
            per_head = self.head_norm == "before"
            req += [TensorRequest(p + self.qk_norm[0], (self.dim if per_head else self.qw,), "norm"),
                    TensorRequest(p + self.qk_norm[1], (self.dim if per_head else self.kw,), "norm")]
        if self.bias_names:
            req += [TensorRequest(p + n, (w,), "bias") for n, w in zip(self.bias_names, (self.qw, self.kw, self.vw))]
        if self.gate_name:
            req.append(TensorRequest(p + self.gate_name, (self.gw, d)))
        if self.sink_name:
            req.append(TensorRequest(p + self.sink_name, (self.hq,), "bias"))
        if self.taps:
            req += [TensorRequest(p + n + ".conv", (w, self.taps)) for n, w in ((q, self.qw), (k, self.kw), (v, self.vw))]
        if self.distance_bias:
            name, _, rows = (tuple(self.distance_bias) + (None,))[:3]
            req.append(TensorRequest(p + name, (-1 if rows is None else int(rows), self.hq), "bias"))
        return req

    def bind(self, get):
        p = self.spec.prefix
        q, k, v, o = self.names
        # rows of the one input product: [q | gate | k | v]; an entry that reads another's cache stops after the gate
        names = [q] + ([self.gate_name] if self.gate_name else []) + ([k] if self.values_are_keys else [k, v])
        self.w_in = _cat([get(p + n) for n in names])
        if self.bias_names:
            bq, bk, bv = (get(p + n).float() for n in self.bias_names)
            zero = [torch.zeros(self.gw, dtype=torch.float32, device=bq.device)] if self.gw else []
            self.b_in = torch.cat([bq] + zero + [bk, bv]).contiguous()
        self.w_o = get(p + o)
        if self.qk_norm:
            self.q_norm, self.k_norm = get(p + self.qk_norm[0]), get(p + self.qk_norm[1])
            if self.q_norm.dtype != self.k_norm.dtype:
                self.q_norm, self.k_norm = self.q_norm.float(), self.k_norm.float()
        if self.sink_name:
            self.sink = get(p + self.sink_name).float().contiguous()
        elif self.sink_value is not None:
            self.sink = torch.full((self.hq,), self.sink_value, dtype=torch.float32, device=self.w_o.device)
        if self.taps:
            self.w_conv = _cat([get(p + n + ".conv") for n in (q, k, v)])
        if self.distance_bias:
            self.bias = ops.DistanceBias(bias_by_distance(get(p + self.distance_bias[0]), int(self.distance_bias[1]), self.chunk))

    def first_weights(self, rows):
        n, k = self.w_in.shape
        late = self.w_in.dtype == torch.bfloat16 and ops.requests_weights_late(rows, n, k, self.w_in.device)
        return self.w_in if late else None

    def input_matrix(self):
        """Opens only without what belongs to the whole product's rows (biases, convolutions)."""
        return None if self.taps or self.bias_names else self.w_in

    def output_matrix(self):
        return self.w_o

    def release_matrices(self):
        self.w_in = self.w_o = None

    def mix_rows(self, proj, at, ctx, out, col=0, scale=1.0):
        mixed = self._attend(proj, at, ctx)
        if self.rotate_values or (self.gw and not self.value_gate):
            mixed = self._finish(mixed, proj, at, ctx)
            return ops.attn_gate(mixed, out, self.hq, self.vdim, self.vdim, None, scale, col)
        return ops.attn_gate(mixed, out, self.hq, self.hd, self.vdim, (proj, at + self.qw) if self.value_gate else None,
                             scale, col)

    def forward(self, h, ctx, residual=None):
        rows = h.shape[0]
        width_in = self.qw + self.gw + ((self.kw + self.vw) if ctx.owns_cache else 0)
        proj = torch.empty((rows, width_in), dtype=torch.float32, device=h.device)
        if self.b_in is not None:
            ops.linear(h, self.w_in[:width_in], proj, ops.EPI_BIAS, bias=self.b_in[:width_in])
        else:
            ops.linear(h, self.w_in[:width_in], proj)
        mixed = self._attend(proj, 0, ctx)
        if self.value_gate:
            gated = torch.empty((rows, self.hq * self.vdim), dtype=self.dtype, device=h.device)
            mixed = ops.attn_gate(mixed, gated, self.hq, self.hd, self.vdim, (proj, self.qw))
        elif self.rotate_values or self.hd != self.vdim or self.gw:
            mixed = self._finish(mixed, proj, 0, ctx)
        out = residual if residual is not None else \
            torch.empty((rows, self.spec.width), dtype=torch.float32, device=h.device)
        return ctx.linear(mixed, self.w_o, out, ops.EPI_RESIDUAL if residual is not None else ops.EPI_NONE,
                          residual=residual, act_dtype=self.dtype)

    def _finish(self, mixed, proj, at, ctx):
        """The heads' results turned back, without padding, times their gates (one number per head)."""
        rows = proj.shape[0]
        turned = torch.empty((rows, self.hq * self.vdim), dtype=self.dtype, device=proj.device)
        return ops.attn_unrotate(mixed, turned, self.hq, self.hd, self.vdim, self.interleaved, self.v_inv_freq,
                                 ctx.plan.row_pos, gate=(proj, at + self.qw) if self.gw else None)

    def _attend(self, proj, at, ctx):
        """The heads' results [rows, heads * hd] from the input product's rows, which start at column `at`."""
        rows, plan = proj.shape[0], ctx.plan
        k_off, width_in = at + self.qw + self.gw, proj.shape[1]
        storage = ctx.kv_storage()
        g = plan.groups[ctx.kv_group()]
        q = torch.empty((rows, self.hq, self.hd), dtype=self.dtype, device=proj.device)
        if self.taps and not ctx.owns_cache:
            from ..config.specs import ConfigError
            raise ConfigError("attention with convolved projections has keys and values of its own")
        state = ctx.state() if self.taps > 1 else None
        if self.conv_only and self.taps <= ops.conv_heads_max_taps():
            ops.conv_heads(proj, self.w_conv, plan, g.page_off, g.page_ids, g.page_size, self.hq, self.hkv, self.dim,
                           self.vdim, state, storage, q)
        else:
            if self.taps:
                turned = torch.empty_like(proj)
                proj = ops.causal_conv(proj, 0, width_in, self.w_conv, None, plan, state, turned)
            ops.attn_prep(proj, at, k_off, -1 if self.values_are_keys else k_off + self.kw, self.hq, self.hkv,
                          self.dim, self.vdim, self.hd, self.rot, self.interleaved, self.inv_freq, self.v_inv_freq,
                          self.q_norm, self.k_norm, self.eps, plan.row_seq, plan.row_pos, g.page_off, g.page_ids,
                          g.page_size, storage if ctx.owns_cache else None, q, head_norm=self.head_norm,
                          rot_scale=self.rot_scale)
        mixed = torch.empty((rows, self.hq * self.hd), dtype=self.dtype, device=proj.device)
        return ops.attention(q, mixed, plan, ctx.kv_group(), storage, self.hq, self.hkv, self.hd, self.spec.window,
                             self.spec.scale, warm=self.w_o, sink=self.sink, softcap=self.softcap, chunk=self.chunk,
                             bias=self.bias)
