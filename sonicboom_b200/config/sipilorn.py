"""Typed configuration of the Sipilorn decoder, read from its own config.json keys.

A Sipilorn model norms its embedding rows and is a list of layers in which mixer and feed-forward read the same
stream through an RMS norm of their own and join it together, x <- x + (mix(n1(x)) + ffn(n2(x))).  A stretch of
the layers may run several times in a row with the same weights; every pass has its own cache and state and starts
with a learned vector added to the stream.  A layer's mixer is the gated delta rule, or a weighted sum of
windowed softmax attention and the gated delta rule on the same input; its feed-forward is a dense gated one, or
experts that a table names for every token id (no router).  The logits are capped.  config.json gives every size
and every constant that may differ between models:

    architecture            "Sipilorn"
    vocab, width            sizes of the embedding / head and of the residual stream
    norm.eps                eps of every RMS norm
    logit_softcap           c: logits = c tanh(logits / c) (absent: none)
    loop                    optional {start, stop, times}: layers start .. stop-1 run `times` times
    layers[i].type          "delta" | "parallel"
    layers[i].mixer         that mixer's sizes and constants (below)
    layers[i].mlp           null, {kind: "dense", ff}, or {kind: "moe", router {experts, top}, expert {ff}}

    delta:      heads, kv_heads (of q and k), dim (of q and k), vdim, conv (taps)
    parallel:   left  {heads, kv_heads, dim, vdim, scale, mask {size} (absent: every earlier key), rot {base, dims}}
                right {the keys of delta}, left_scale, right_scale

What the design fixes is written into the part records by `to_spec`: the unit vectors' eps and the scale dim^(-1/2) of
the delta rule's queries, per-head norms before the rotation in halves, a logistic gate for every value of the
attention's result, the experts' weights 1/top, and the tensor names (`embed.norm`, `l<i>.norm1`, `l<i>.mix.q.conv`,
`l<i>.mix.left.q.norm`, `l<i>.mix.right.A_log`, `l<i>.mlp.table`, `l<i>.mlp.e<j>.up`, `loop.step`, ...).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

from .mefupel import LoopConfig, _rot, loop_config, loop_order
from .specs import (ConfigError, FeedForwardSpec, LayerSpec, MixerSpec, ModelSpec, NormSpec, PositionSpec, ScheduleEntry,
                    StreamInjection)
from .zolulix import MAX_POSITIONS, _num, _sub

UNIT_EPS = 1e-6              # a unit vector is x / sqrt(sum(x^2) + eps)


@dataclass(frozen=True)
class GatedDeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclass(frozen=True)
class GatedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_base: float
    rot_dims: int
    window: int = 0            # mask.size; 0: every earlier key


@dataclass(frozen=True)
class WeightedSumConfig:
    left: GatedAttentionConfig
    right: GatedDeltaConfig
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class SipilornMlp:
    kind: str                  # "dense" | "moe"
    ff: int
    experts: int = 0
    top: int = 0


@dataclass(frozen=True)
class SipilornLayer:
    type: str
    mixer: object
    mlp: Optional[SipilornMlp]


def _heads(m: dict, w: str) -> dict:
    heads, kv_heads = _num(m, "heads", w), _num(m, "kv_heads", w)
    if heads % kv_heads:
        raise ConfigError(f"missing/invalid config key: {w}kv_heads ({heads} heads are not a multiple of {kv_heads})")
    return dict(heads=heads, kv_heads=kv_heads, dim=_num(m, "dim", w), vdim=_num(m, "vdim", w))


def _delta(m: dict, w: str) -> GatedDeltaConfig:
    return GatedDeltaConfig(**_heads(m, w), conv=_num(m, "conv", w))


def _mixer(kind, m: dict, w: str):
    if kind == "delta":
        return _delta(m, w)
    if kind != "parallel":
        raise ConfigError(f"unsupported config key: {w[:-6]}type = {kind!r} (delta or parallel)")
    a, aw = _sub(m, "left", w), w + "left."
    sizes = _heads(a, aw)
    base, dims = _rot(a, aw, sizes["dim"])
    left = GatedAttentionConfig(
        **sizes, scale=_num(a, "scale", aw, float), rot_base=base, rot_dims=dims,
        window=_num(_sub(a, "mask", aw), "size", aw + "mask.") if a.get("mask") is not None else 0)
    return WeightedSumConfig(left, _delta(_sub(m, "right", w), w + "right."), _num(m, "left_scale", w, float, positive=False),
                             _num(m, "right_scale", w, float, positive=False))


def _mlp(mlp, w: str) -> Optional[SipilornMlp]:
    if mlp is None:
        return None
    kind = mlp.get("kind") if isinstance(mlp, dict) else mlp
    if kind == "dense":
        return SipilornMlp(kind="dense", ff=_num(mlp, "ff", w))
    if kind != "moe":
        raise ConfigError(f"unsupported config key: {w}kind = {kind!r} (dense or moe)")
    r = _sub(mlp, "router", w)
    c = SipilornMlp(kind="moe", ff=_num(_sub(mlp, "expert", w), "ff", w + "expert."),
                    experts=_num(r, "experts", w + "router."), top=_num(r, "top", w + "router."))
    if c.top > c.experts:
        raise ConfigError(f"missing/invalid config key: {w}router.top ({c.top} of {c.experts} experts)")
    return c


@dataclass(frozen=True)
class SipilornConfig:
    vocab: int
    width: int
    eps: float
    layers: tuple
    loop: Optional[LoopConfig] = None
    logit_softcap: float = 0.0
    architecture: str = "Sipilorn"

    @classmethod
    def from_dict(cls, d: dict) -> "SipilornConfig":
        vocab, width = _num(d, "vocab", ""), _num(d, "width", "")
        eps = _num(_sub(d, "norm", ""), "eps", "norm.", float, positive=False)
        if eps < 0:
            raise ConfigError("missing/invalid config key: norm.eps (must be >= 0)")
        cap = _num(d, "logit_softcap", "", float, positive=False) if d.get("logit_softcap") is not None else 0.0
        if cap < 0:
            raise ConfigError("missing/invalid config key: logit_softcap (must be >= 0)")
        raw = d.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("missing/invalid config key: layers (a non-empty list)")
        layers = []
        for i, L in enumerate(raw):
            w = f"layers[{i}]."
            if not isinstance(L, dict):
                raise ConfigError(f"missing/invalid config key: layers[{i}] (expected an object)")
            layers.append(SipilornLayer(L.get("type"), _mixer(L.get("type"), _sub(L, "mixer", w), w + "mixer."),
                                        _mlp(L.get("mlp"), w + "mlp.")))
        return cls(vocab=vocab, width=width, eps=eps, layers=tuple(layers), loop=loop_config(d, len(layers)), logit_softcap=cap)

    def to_dict(self) -> dict:
        """config.json content that `from_dict` reads back to an equal configuration."""
        def delta(m):
            return {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "conv": m.conv}
        out = []
        for L in self.layers:
            m = L.mixer
            if L.type == "delta":
                mixer = delta(m)
            else:
                a = m.left
                left = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale,
                        "rot": {"base": a.rot_base, "dims": a.rot_dims}}
                if a.window:
                    left["mask"] = {"size": a.window}
                mixer = {"left": left, "right": delta(m.right), "left_scale": m.left_scale, "right_scale": m.right_scale}
            e = L.mlp
            mlp = None if e is None else {"kind": "dense", "ff": e.ff} if e.kind == "dense" else \
                {"kind": "moe", "router": {"experts": e.experts, "top": e.top}, "expert": {"ff": e.ff}}
            out.append({"type": L.type, "mixer": mixer, "mlp": mlp})
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
             "layers": out}
        if self.loop is not None:
            d["loop"] = {"start": self.loop.start, "stop": self.loop.stop, "times": self.loop.times}
        if self.logit_softcap:
            d["logit_softcap"] = self.logit_softcap
        return d

    def to_spec(self) -> ModelSpec:
        """The model as parts: one block per layer in which mixer and feed-forward join the stream together; a layer
        inside the loop appears once per pass in the schedule, each run with a cache entry and state of its own."""
        d, eps = self.width, self.eps

        def delta(m, prefix):
            return MixerSpec(
                kind="gated_delta_rule", width=d, n_heads=m.heads, n_kv_heads=m.kv_heads, head_dim=m.dim, prefix=prefix,
                params=(("vdim", m.vdim), ("conv", m.conv), ("q_scale", float(m.dim) ** -0.5), ("unit_eps", UNIT_EPS),
                        ("eps", eps)))

        layers, unused = [], []
        for i, L in enumerate(self.layers):
            p = f"l{i}."
            m = L.mixer
            if L.type == "delta":
                mixer = delta(m, p + "mix.")
            else:
                a = m.left
                left = MixerSpec(
                    kind="window_attention", width=d, n_heads=a.heads, n_kv_heads=a.kv_heads, head_dim=a.dim,
                    window=a.window, scale=a.scale, prefix=p + "mix.left.",
                    position=PositionSpec("rope_halves", a.dim, a.rot_base, a.rot_dims),
                    params=(("vdim", a.vdim), ("eps", eps), ("head_norm", ("before", "q.norm", "k.norm")), ("value_gate", "g")))
                mixer = MixerSpec(
                    kind="side_by_side", width=d, prefix=p + "mix.",
                    params=(("join", "sum"), ("left", left), ("right", delta(m.right, p + "mix.right.")),
                            ("left_scale", m.left_scale), ("right_scale", m.right_scale)))
            ff, e = None, L.mlp
            if e is not None and e.kind == "dense":
                ff = FeedForwardSpec(kind="swiglu", width=d, intermediate=e.ff, activation="silu", prefix=p + "mlp.",
                                     params=(("names", ("gate", "up", "down")),))
            elif e is not None:
                ff = FeedForwardSpec(kind="experts_relu2", width=d, intermediate=e.ff, activation="relu2", prefix=p + "mlp.",
                                     params=(("experts", e.experts), ("top", e.top), ("by_token", ("table", self.vocab))))
            else:
                unused.append((p + "norm2", (d,)))         # a file may hold it; nothing reads it
            layers.append(LayerSpec(
                arrangement="parallel_residual", mixer=mixer, mixer_norm=NormSpec("rmsnorm", d, eps, p + "norm1"),
                feed_forward=ff, feed_forward_norm=NormSpec("rmsnorm", d, eps, p + "norm2") if ff is not None else None))
        order = loop_order(len(self.layers), self.loop)
        times = self.loop.times if self.loop is not None else 0
        injections = tuple(StreamInjection(before_entry=e, tensor="loop.step", rows=times, row=t)
                           for e, (_, t) in enumerate(order) if t is not None)
        if self.loop is not None and not injections:
            unused.append(("loop.step", (times, d)))       # a loop over no layers leaves its vectors unused
        spec = ModelSpec(
            architecture=self.architecture, width=d, vocab=self.vocab, max_positions=MAX_POSITIONS,
            embedding_tensor="embed", embedding_norm=NormSpec("rmsnorm", d, eps, "embed.norm"), layers=tuple(layers),
            schedule=tuple(ScheduleEntry(i) for i, _ in order),
            final_norm=NormSpec("rmsnorm", d, eps, "final.norm"), head_tensor="head", logit_cap=self.logit_softcap,
            injections=injections, unused_tensors=tuple(unused))
        spec.validate()
        return spec
