"""Typed configuration of the Debisun decoder, read from its own config.json keys.

A Debisun model is a list of layers with a layer norm (weight and bias) before each sublayer and a
learned weight per channel on its result, x1 = x + s1 * mix(n1(x)); x2 = x1 + s2 * ffn(n2(x1)).  After its
feed-forward a layer adds a token input of its own: its part of the token's row in a second embedding
table, gated by the stream, projected back and RMS-normed.  The mixer is grouped-query attention within
chunks of positions, whose q, k and v pass short causal convolutions, whose capped scores get a learned
bias by distance, and whose softmax has one added to its denominator; positions enter no other way.  The
feed-forward is dense with the square of relu, or a mixture of such experts and identity outputs, chosen
by softmax scores, plus a shared expert gated by one number per token.  config.json gives every size and
every constant that may differ between models:

    architecture                "Debisun"
    vocab, width                sizes of the embedding / head and of the residual stream
    norm.eps                    eps of every norm
    token_side.dim              values of the second embedding table per layer (absent: no token inputs)
    layers[i].type              "attention"
    layers[i].mixer             heads, kv_heads, dim, vdim, scale, softcap (absent: none), conv (taps; absent:
                                no convolutions), bias_max (the distance the bias table's last row starts
                                at), mask {size} (chunk length; absent: every earlier key is seen)
    layers[i].mlp               null, {kind: "dense", ff}, or {kind: "moe", router {experts, top, identity,
                                scale}, expert {ff}, shared {ff} (optional)}

The number of rows of the bias table is the stored tensor's; `mixer.bias_rows` may state it, and must when
weights are made at random.

What the design fixes is written into the part records by `to_spec`: the sink's score of 0, that the
chosen experts' weights are renormalised, and the tensor names (`l<i>.norm1`, `l<i>.norm1.b`, `l<i>.ls1`,
`l<i>.mix.q.conv`, `l<i>.mix.rel`, `l<i>.mlp.e<j>.up`, `l<i>.mlp.shared.sg`, `l<i>.side.gate`, `side.embed`, ...).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

from .specs import (ConfigError, FeedForwardSpec, LayerSpec, MixerSpec, ModelSpec, NormSpec, ScheduleEntry,
                    SideInputSpec, SideTableSpec)
from .zolulix import MAX_POSITIONS, _num, _sub

SINK_SCORE = 0.0             # exp(0) = 1 joins every softmax's denominator


@dataclass(frozen=True)
class ChunkedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    bias_max: int
    softcap: float = 0.0
    conv: int = 0              # taps; 0: no convolutions
    chunk: int = 0             # mask.size; 0: every earlier key
    bias_rows: Optional[int] = None


@dataclass(frozen=True)
class DebisunMlp:
    kind: str                  # "dense" | "moe"
    ff: int
    experts: int = 0
    identity: int = 0
    top: int = 0
    route_scale: float = 1.0
    shared_ff: int = 0         # 0: no shared expert


@dataclass(frozen=True)
class DebisunLayer:
    type: str
    mixer: ChunkedAttentionConfig
    mlp: Optional[DebisunMlp]


def _mixer(kind, m: dict, w: str) -> ChunkedAttentionConfig:
    if kind != "attention":
        raise ConfigError(f"unsupported config key: {w[:-6]}type = {kind!r} (only 'attention')")
    c = ChunkedAttentionConfig(
        heads=_num(m, "heads", w), kv_heads=_num(m, "kv_heads", w), dim=_num(m, "dim", w), vdim=_num(m, "vdim", w),
        scale=_num(m, "scale", w, float), bias_max=_num(m, "bias_max", w),
        softcap=_num(m, "softcap", w, float, positive=False) if m.get("softcap") is not None else 0.0,
        conv=_num(m, "conv", w, positive=False) if m.get("conv") is not None else 0,
        chunk=_num(_sub(m, "mask", w), "size", w + "mask.") if m.get("mask") is not None else 0,
        bias_rows=_num(m, "bias_rows", w) if m.get("bias_rows") is not None else None)
    if c.heads % c.kv_heads:
        raise ConfigError(f"missing/invalid config key: {w}kv_heads ({c.heads} query heads are not a multiple of "
                          f"{c.kv_heads})")
    if c.softcap < 0 or c.conv < 0:
        raise ConfigError(f"missing/invalid config key: {w}softcap / {w}conv (must be >= 0)")
    if c.bias_rows is not None and (c.bias_rows < 2 or 2 * c.bias_max <= c.bias_rows):
        raise ConfigError(f"missing/invalid config key: {w}bias_max ({c.bias_max} for a table of {c.bias_rows} rows)")
    return c


def _mlp(mlp, w: str) -> Optional[DebisunMlp]:
    if mlp is None:
        return None
    kind = mlp.get("kind") if isinstance(mlp, dict) else mlp
    if kind == "dense":
        return DebisunMlp(kind="dense", ff=_num(mlp, "ff", w))
    if kind != "moe":
        raise ConfigError(f"unsupported config key: {w}kind = {kind!r} (dense or moe)")
    r, e = _sub(mlp, "router", w), _sub(mlp, "expert", w)
    c = DebisunMlp(
        kind="moe", ff=_num(e, "ff", w + "expert."), experts=_num(r, "experts", w + "router."),
        identity=_num(r, "identity", w + "router.", positive=False) if r.get("identity") is not None else 0,
        top=_num(r, "top", w + "router."),
        route_scale=_num(r, "scale", w + "router.", float) if r.get("scale") is not None else 1.0,
        shared_ff=_num(_sub(mlp, "shared", w), "ff", w + "shared.") if mlp.get("shared") is not None else 0)
    if c.identity < 0:
        raise ConfigError(f"missing/invalid config key: {w}router.identity (must be >= 0)")
    if c.top > c.experts + c.identity:
        raise ConfigError(f"missing/invalid config key: {w}router.top ({c.top} of {c.experts} experts and "
                          f"{c.identity} identities)")
    return c


@dataclass(frozen=True)
class DebisunConfig:
    vocab: int
    width: int
    eps: float
    layers: tuple
    side_dim: int = 0            # 0: no token inputs
    architecture: str = "Debisun"

    @classmethod
    def from_dict(cls, d: dict) -> "DebisunConfig":
        vocab, width = _num(d, "vocab", ""), _num(d, "width", "")
        eps = _num(_sub(d, "norm", ""), "eps", "norm.", float, positive=False)
        if eps < 0:
            raise ConfigError("missing/invalid config key: norm.eps (must be >= 0)")
        side = _num(_sub(d, "token_side", ""), "dim", "token_side.") if d.get("token_side") is not None else 0
        raw = d.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("missing/invalid config key: layers (a non-empty list)")
        layers = []
        for i, L in enumerate(raw):
            w = f"layers[{i}]."
            if not isinstance(L, dict):
                raise ConfigError(f"missing/invalid config key: layers[{i}] (expected an object)")
            layers.append(DebisunLayer(L.get("type"), _mixer(L.get("type"), _sub(L, "mixer", w), w + "mixer."),
                                       _mlp(L.get("mlp"), w + "mlp.")))
        return cls(vocab=vocab, width=width, eps=eps, layers=tuple(layers), side_dim=side)

    def to_dict(self) -> dict:
        """config.json content that `from_dict` reads back to an equal configuration."""
        out = []
        for L in self.layers:
            m = L.mixer
            mixer = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale,
                     "softcap": m.softcap, "conv": m.conv, "bias_max": m.bias_max}
            if m.chunk:
                mixer["mask"] = {"size": m.chunk}
            if m.bias_rows is not None:
                mixer["bias_rows"] = m.bias_rows
            mlp = None
            if L.mlp is not None and L.mlp.kind == "dense":
                mlp = {"kind": "dense", "ff": L.mlp.ff}
            elif L.mlp is not None:
                e = L.mlp
                mlp = {"kind": "moe", "router": {"experts": e.experts, "identity": e.identity, "top": e.top,
                                                 "scale": e.route_scale}, "expert": {"ff": e.ff}}
                if e.shared_ff:
                    mlp["shared"] = {"ff": e.shared_ff}
            out.append({"type": L.type, "mixer": mixer, "mlp": mlp})
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
             "layers": out}
        if self.side_dim:
            d["token_side"] = {"dim": self.side_dim}
        return d

    def to_spec(self) -> ModelSpec:
        """The model as parts: one scaled pre-norm block per layer."""
        d, eps = self.width, self.eps

        def norm(name):
            return NormSpec("layernorm", d, eps, name, name + ".b")
        layers, unused = [], []
        for i, L in enumerate(self.layers):
            p = f"l{i}."
            m = L.mixer
            mixer = MixerSpec(
                kind="window_attention", width=d, n_heads=m.heads, n_kv_heads=m.kv_heads, head_dim=m.dim, scale=m.scale,
                prefix=p + "mix.",
                params=(("vdim", m.vdim), ("conv", m.conv), ("softcap", m.softcap), ("chunk", m.chunk),
                        ("distance_bias", ("rel", m.bias_max, m.bias_rows)), ("sink", SINK_SCORE)))
            ff = None
            if L.mlp is not None and L.mlp.kind == "dense":
                ff = FeedForwardSpec(kind="relu2", width=d, intermediate=L.mlp.ff, activation="relu2", prefix=p + "mlp.")
            elif L.mlp is not None:
                e = L.mlp
                shared = None if not e.shared_ff else FeedForwardSpec(
                    kind="relu2", width=d, intermediate=e.shared_ff, activation="relu2", prefix=p + "mlp.shared.")
                ff = FeedForwardSpec(
                    kind="experts_relu2", width=d, intermediate=e.ff, activation="relu2", prefix=p + "mlp.",
                    params=(("experts", e.experts), ("identity", e.identity), ("top", e.top), ("scale", e.route_scale),
                            ("shared", shared), ("shared_gate", "shared.sg"), ("correction", "correction")))
            else:
                # a layer without a feed-forward may still store its second norm and scale
                unused += [(p + n, (d,)) for n in ("norm2", "norm2.b", "ls2")]
            side = SideInputSpec(p + "side.", d, self.side_dim, i, eps) if self.side_dim else None
            layers.append(LayerSpec(
                arrangement="pre_norm_scaled", mixer=mixer, mixer_norm=norm(p + "norm1"), mixer_scale=p + "ls1",
                feed_forward=ff, feed_forward_norm=norm(p + "norm2") if ff is not None else None,
                feed_forward_scale=p + "ls2" if ff is not None else None, side_input=side))
        spec = ModelSpec(
            architecture=self.architecture, width=d, vocab=self.vocab, max_positions=MAX_POSITIONS,
            embedding_tensor="embed", layers=tuple(layers),
            schedule=tuple(ScheduleEntry(i) for i in range(len(self.layers))),
            final_norm=norm("final.norm"), head_tensor="head", unused_tensors=tuple(unused),
            side_table=SideTableSpec("side.embed", self.side_dim, len(self.layers)) if self.side_dim else None)
        spec.validate()
        return spec
