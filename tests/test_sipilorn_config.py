"""Sipilorn without a device: configuration keys and their errors, the parts a configuration becomes, the tensor
list, random expert tables, and properties of the plain implementation's own mechanisms."""
import copy
import json

import pytest
import torch

import plain_sipilorn as ps
from sipilorn_util import CONFIGS, attention, delta, dense, layer, model, moe, parallel, write_model
from sonicboom_b200.config import ConfigError, SipilornConfig, spec_from_config_dict
from sonicboom_b200.models import tensor_requests

F = torch.float64


@pytest.mark.parametrize("name", list(CONFIGS))
def test_round_trip_and_parts(name):
    cfg = CONFIGS[name]
    c, spec = spec_from_config_dict(cfg)
    assert isinstance(c, SipilornConfig) and SipilornConfig.from_dict(json.loads(json.dumps(c.to_dict()))) == c
    assert spec.architecture == "Sipilorn" and spec.embedding_norm.tensor == "embed.norm" and spec.logit_cap == cfg.get("logit_softcap", 0.0)
    assert [e.layer for e in spec.schedule] == [i for i, _ in ps.run_order(cfg)]
    starts = [(e, t) for e, (_, t) in enumerate(ps.run_order(cfg)) if t is not None]
    assert [(i.before_entry, i.row) for i in spec.injections] == starts and not any(i.embedding for i in spec.injections)
    for L, raw in zip(spec.layers, cfg["layers"]):
        assert L.arrangement == "parallel_residual" and (L.feed_forward is None) == (raw["mlp"] is None) == (L.feed_forward_norm is None)
        m, right = raw["mixer"], L.mixer
        if raw["type"] == "parallel":
            p = dict(L.mixer.params)
            assert L.mixer.kind == "side_by_side" and p["join"] == "sum" and (p["left_scale"], p["right_scale"]) == (m["left_scale"], m["right_scale"])
            left, right, m = p["left"], p["right"], m["right"]
            a = raw["mixer"]["left"]
            assert left.kind == "window_attention" and left.window == a.get("mask", {}).get("size", 0) and left.scale == a["scale"]
            assert left.position.kind == "rope_halves" and left.position.rotary_dim == a["rot"]["dims"]
            assert dict(left.params)["value_gate"] == "g" and dict(left.params)["head_norm"] == ("before", "q.norm", "k.norm")
        p = dict(right.params)
        assert right.kind == "gated_delta_rule" and (right.n_heads, right.n_kv_heads, right.head_dim) == (m["heads"], m["kv_heads"], m["dim"])
        assert (p["vdim"], p["conv"], p["q_scale"], p["unit_eps"], p["eps"]) == (m["vdim"], m["conv"], m["dim"] ** -0.5, 1e-6, cfg["norm"]["eps"])
        if raw["mlp"] is not None:
            assert L.feed_forward.kind == ("swiglu" if raw["mlp"]["kind"] == "dense" else "experts_relu2")


def test_tensor_list():
    _, spec = spec_from_config_dict(CONFIGS["A"])
    req = {r.name: r for r in tensor_requests(spec)}
    names = {n: tuple(r.shape) for n, r in req.items() if not r.optional}
    assert names["embed"] == (211, 64) and names["embed.norm"] == names["final.norm"] == (64,) and names["loop.step"] == (3, 64)
    assert names["l0.mix.q"] == (32, 64) and names["l0.mix.v.conv"] == (144, 4) and names["l0.mix.o"] == (64, 144)
    assert names["l0.mix.A_log"] == names["l0.mix.dt_bias"] == (6,) and names["l0.mix.b"] == names["l0.mix.a"] == (6, 64)
    assert names["l0.mix.norm"] == (24,) and names["l0.mlp.table"] == (211, 2) and names["l0.mlp.e4.down"] == (64, 24)
    assert "l0.mlp.router" not in names and "l0.mlp.correction" not in names and req["l0.mlp.table"].role == "table"
    assert names["l1.mix.left.q.norm"] == (16,) and names["l1.mix.left.g"] == (96, 64) and names["l1.mix.left.o"] == (64, 96)
    assert names["l1.mix.right.k.conv"] == (24, 2) and names["l1.mlp.gate"] == (40, 64) and "l2.norm2" not in names
    assert req["l2.norm2"].optional and "l2.norm2" in req                  # a file may hold it; nothing reads it
    _, spec = spec_from_config_dict(CONFIGS["C"])
    assert not any(r.name == "loop.step" for r in tensor_requests(spec))
    empty = copy.deepcopy(CONFIGS["C"])
    empty["loop"] = {"start": 1, "stop": 1, "times": 4}                    # a loop over no layers
    _, spec = spec_from_config_dict(empty)
    assert not spec.injections and [r.optional for r in tensor_requests(spec) if r.name == "loop.step"] == [True]


@pytest.mark.parametrize("edit,key", [
    (lambda d: d.pop("vocab"), "vocab"),
    (lambda d: d["norm"].pop("eps"), "norm.eps"),
    (lambda d: d.update(logit_softcap=-1.0), "logit_softcap"),
    (lambda d: d["loop"].update(stop=9), "loop"),
    (lambda d: d["loop"].pop("times"), "loop.times"),
    (lambda d: d["layers"][0].update(type="gla"), "layers[0].type"),
    (lambda d: d["layers"][0]["mixer"].update(kv_heads=4), "layers[0].mixer.kv_heads"),
    (lambda d: d["layers"][0]["mixer"].pop("conv"), "layers[0].mixer.conv"),
    (lambda d: d["layers"][0]["mixer"].update(conv=0), "layers[0].mixer.conv"),
    (lambda d: d["layers"][1]["mixer"].pop("left"), "layers[1].mixer.left"),
    (lambda d: d["layers"][1]["mixer"]["left"].pop("scale"), "layers[1].mixer.left.scale"),
    (lambda d: d["layers"][1]["mixer"]["left"]["mask"].pop("size"), "layers[1].mixer.left.mask.size"),
    (lambda d: d["layers"][1]["mixer"]["left"]["rot"].update(dims=18), "layers[1].mixer.left.rot.dims"),
    (lambda d: d["layers"][1]["mixer"]["right"].update(heads=0), "layers[1].mixer.right.heads"),
    (lambda d: d["layers"][1]["mixer"].pop("right_scale"), "layers[1].mixer.right_scale"),
    (lambda d: d["layers"][0]["mlp"]["router"].update(top=6), "layers[0].mlp.router.top"),
    (lambda d: d["layers"][0]["mlp"]["expert"].pop("ff"), "layers[0].mlp.expert.ff"),
    (lambda d: d["layers"][1]["mlp"].update(kind="sparse"), "layers[1].mlp.kind"),
])
def test_errors_name_the_key(edit, key):
    d = copy.deepcopy(CONFIGS["A"])
    edit(d)
    with pytest.raises(ConfigError) as e:
        spec_from_config_dict(d)
    assert key in str(e.value)


def test_random_tables_name_different_experts(tmp_path):
    cfg = model(300, 16, [layer(delta(1, 1, 8, 8), moe(7, 3, 8)), layer(delta(1, 1, 8, 8), moe(4, 4, 8)),
                          layer(delta(1, 1, 8, 8), moe(1, 1, 8)), layer(delta(1, 1, 8, 8), dense(8))])
    _, tensors = write_model(tmp_path / "m", cfg, seed=5)
    t = tensors["l0.mlp.table"]
    assert t.dtype == torch.int32 and tuple(t.shape) == (300, 3) and sorted(set(t.flatten().tolist())) == list(range(7))
    assert all(len(set(r)) == 3 for r in t.tolist()) and len({tuple(r) for r in t.tolist()}) == 14
    assert all(sorted(r) == [0, 1, 2, 3] for r in tensors["l1.mlp.table"].tolist()) and not tensors["l2.mlp.table"].any()
    _, again = write_model(tmp_path / "n", cfg, seed=5)
    assert torch.equal(t, again["l0.mlp.table"])


def test_a_table_with_an_expert_that_does_not_exist_is_refused():
    from sonicboom_b200.parts.feedforward import ExpertsSquaredRelu
    _, spec = spec_from_config_dict(CONFIGS["A"])
    ff = ExpertsSquaredRelu(spec.layers[0].feed_forward, torch.float32, "cpu")
    for bad in (5, -1):
        made = {r.name: (torch.full(r.shape, bad, dtype=torch.int32) if r.role == "table" else torch.zeros(r.shape))
                for r in ff.tensor_requests()}
        with pytest.raises(ConfigError, match="table"):
            ff.bind(made.__getitem__)


def test_the_delta_rule_of_the_plain_implementation():
    g = torch.Generator().manual_seed(1)
    T, H, d, dv = 7, 2, 5, 3
    q, k, v = (torch.randn(T, n, m, generator=g, dtype=F) for n, m in ((1, d), (1, d), (H, dv)))
    k = ps.unit(k)
    one, zero = torch.ones(T, H, dtype=F), torch.zeros(T, H, dtype=F)
    # beta 1 and no decay: what is written under a key is read back under it
    o = ps.gated_delta_rule(k, k, v, one, one)
    assert torch.allclose(o, v, atol=1e-5)
    # beta 0: nothing is ever written; decay 0: only the token itself is seen
    assert not ps.gated_delta_rule(q, k, v, one, zero).any()
    o = ps.gated_delta_rule(q, k, v, zero, 0.5 * one)
    assert torch.allclose(o, 0.5 * v * (q * k).sum(-1, keepdim=True))
    x, w = torch.randn(6, 3, dtype=F, generator=g), torch.randn(3, 4, dtype=F, generator=g)
    y = ps.short_conv(x, w)
    assert torch.allclose(y[0], w[:, 3] * x[0]) and torch.allclose(y[5], sum(w[:, j] * x[2 + j] for j in range(4)))
    assert torch.allclose(ps.unit(x).norm(dim=-1), torch.ones(6, dtype=F), atol=1e-5)
    assert ps.window_mask(5, 2).sum(-1).tolist() == [1, 2, 2, 2, 2] and ps.window_mask(4, None).sum(-1).tolist() == [1, 2, 3, 4]


def test_a_pair_of_norms_is_one_only_when_eps_and_dtype_agree():
    from sonicboom_b200.config import NormSpec
    from sonicboom_b200.parts.norm import LayerNorm, NormPair, RMSNorm
    a, b, c = (RMSNorm(NormSpec("rmsnorm", 8, e, "x"), torch.float32, "cpu") for e in (1e-5, 1e-5, 1e-6))
    for n in (a, b, c):
        n.weight = torch.ones(8)
    assert NormPair(a, b).as_pair()[2] == 1e-5 and NormPair(a, c).as_pair() is None and NormPair(a, b).as_rms() is None
    b.weight = b.weight.bfloat16()
    assert NormPair(a, b).as_pair() is None
    assert NormPair(a, LayerNorm(NormSpec("layernorm", 8, 1e-5, "x"), torch.float32, "cpu")).as_pair() is None


def test_sides_ask_for_one_cache_and_one_state():
    from sonicboom_b200.models import DecoderModel
    _, spec = spec_from_config_dict(model(40, 16, [layer(parallel(attention(2, 1, 16, 8, 5), delta(2, 1, 8, 8, conv=1))),
                                                   layer(delta(2, 1, 8, 8, conv=3))], loop=(0, 2, 2)))
    m = DecoderModel(spec, torch.float32, "cpu")
    kv, st = m.kv_needs(), m.state_needs()
    assert [n is not None for n in kv] == [True, False, True, False] and kv[0].window == 5 and kv[0].head_dim == 16
    assert [sorted(s) for s in st] == [["memory"], ["memory", "ring"]] * 2
    assert st[0]["memory"].shape == (2, 8, 8) and st[1]["ring"].shape == (3, 32)
