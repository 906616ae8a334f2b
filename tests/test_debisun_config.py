"""Debisun without a device: configuration keys and their errors, the parts a configuration becomes, the
tensor list, the distance buckets, the cache's pages of past chunks, and properties of the plain
implementation's own mechanisms."""
import copy
import json
import math

import pytest
import torch

import plain_debisun as pd
from debisun_util import CONFIGS, attention, calm_tokens, dense, layer, model, moe, write_model
from sonicboom_b200.cache.kv import Cache, KVNeed
from sonicboom_b200.config import ConfigError, DebisunConfig, spec_from_config_dict
from sonicboom_b200.models import tensor_requests
from sonicboom_b200.parts.window_attention import bias_by_distance, distance_bucket

F = torch.float64


@pytest.mark.parametrize("name", list(CONFIGS))
def test_round_trip_and_parts(name):
    cfg = CONFIGS[name]
    c, spec = spec_from_config_dict(cfg)
    assert isinstance(c, DebisunConfig) and DebisunConfig.from_dict(c.to_dict()) == c
    assert DebisunConfig.from_dict(json.loads(json.dumps(c.to_dict()))) == c
    assert spec.architecture == "Debisun" and len(spec.layers) == len(cfg["layers"]) == len(spec.schedule)
    assert (spec.side_table is None) == ("token_side" not in cfg)
    for i, (L, raw) in enumerate(zip(spec.layers, cfg["layers"])):
        assert L.arrangement == "pre_norm_scaled" and L.mixer_norm.bias == f"l{i}.norm1.b" and L.mixer_scale == f"l{i}.ls1"
        assert (L.feed_forward is None) == (raw["mlp"] is None) == (L.feed_forward_norm is None) == (L.feed_forward_scale is None)
        m, p = raw["mixer"], dict(L.mixer.params)
        assert L.mixer.kind == "window_attention" and L.mixer.position is None and L.mixer.window == 0
        assert p["chunk"] == (m["mask"]["size"] if "mask" in m else 0) and p["conv"] == m.get("conv", 0)
        assert p["softcap"] == m.get("softcap", 0.0) and p["sink"] == 0.0 and L.mixer.scale == m["scale"]
        assert p["distance_bias"] == ("rel", m["bias_max"], m["bias_rows"])
        if raw["mlp"] is not None and raw["mlp"]["kind"] == "moe":
            f = dict(L.feed_forward.params)
            assert L.feed_forward.kind == "experts_relu2" and f["identity"] == raw["mlp"]["router"].get("identity", 0)
            assert f["scale"] == raw["mlp"]["router"].get("scale", 1.0) and (f["shared"] is None) == ("shared" not in raw["mlp"])
        elif raw["mlp"] is not None:
            assert L.feed_forward.kind == "relu2"
        if L.side_input is not None:
            assert (L.side_input.part, L.side_input.dim) == (i, cfg["token_side"]["dim"])


def test_tensor_list():
    _, spec = spec_from_config_dict(CONFIGS["A"])
    names = {r.name: tuple(r.shape) for r in tensor_requests(spec) if not r.optional}
    assert names["embed"] == (211, 64) and names["side.embed"] == (211, 48) and names["head"] == (211, 64)
    assert names["l0.norm1"] == names["l0.norm1.b"] == names["l0.norm2.b"] == names["l0.ls1"] == names["l0.ls2"] == (64,)
    assert names["l0.mix.q"] == (64, 64) and names["l0.mix.v"] == (48, 64) and names["l0.mix.o"] == (64, 96)
    assert names["l0.mix.q.conv"] == (64, 3) and names["l0.mix.v.conv"] == (48, 3) and names["l0.mix.rel"] == (8, 4)
    assert names["l0.mlp.router"] == (8, 64) and names["l0.mlp.correction"] == (8,) and names["l0.mlp.e4.down"] == (64, 24)
    assert "l0.mlp.e5.up" not in names and names["l0.mlp.shared.sg"] == (1, 64) and names["l0.mlp.shared.up"] == (40, 64)
    assert names["l0.side.gate"] == (12, 64) and names["l0.side.proj"] == (64, 12) and names["l0.side.norm"] == (64,)
    assert "l1.norm2" not in names and "l1.ls2" not in names and names["final.norm.b"] == (64,)
    optional = {r.name for r in tensor_requests(spec) if r.optional}
    assert {"l1.norm2", "l1.norm2.b", "l1.ls2"} <= optional          # a file may hold them; nothing reads them
    _, spec = spec_from_config_dict(CONFIGS["C"])
    assert not any("side" in r.name for r in tensor_requests(spec))
    stored = copy.deepcopy(CONFIGS["B"])                              # the table's rows are the stored tensor's
    del stored["layers"][0]["mixer"]["bias_rows"]
    _, spec = spec_from_config_dict(stored)
    assert {r.name: tuple(r.shape) for r in tensor_requests(spec)}["l0.mix.rel"] == (-1, 6)


@pytest.mark.parametrize("edit,key", [
    (lambda d: d.pop("vocab"), "vocab"),
    (lambda d: d["norm"].pop("eps"), "norm.eps"),
    (lambda d: d["token_side"].update(dim=0), "token_side.dim"),
    (lambda d: d["layers"][0].update(type="attention_2"), "layers[0].type"),
    (lambda d: d["layers"][0]["mixer"].update(kv_heads=3), "layers[0].mixer.kv_heads"),
    (lambda d: d["layers"][0]["mixer"]["mask"].pop("size"), "layers[0].mixer.mask.size"),
    (lambda d: d["layers"][0]["mixer"].pop("bias_max"), "layers[0].mixer.bias_max"),
    (lambda d: d["layers"][0]["mixer"].update(bias_max=4), "layers[0].mixer.bias_max"),
    (lambda d: d["layers"][0]["mixer"].update(softcap=-1.0), "layers[0].mixer.softcap"),
    (lambda d: d["layers"][0]["mixer"].update(conv=-1), "layers[0].mixer.conv"),
    (lambda d: d["layers"][0]["mixer"].pop("scale"), "layers[0].mixer.scale"),
    (lambda d: d["layers"][0]["mlp"]["router"].update(top=9), "layers[0].mlp.router.top"),
    (lambda d: d["layers"][0]["mlp"]["router"].update(identity=-1), "layers[0].mlp.router.identity"),
    (lambda d: d["layers"][2]["mlp"].update(kind="sparse"), "layers[2].mlp.kind"),
    (lambda d: d["layers"][0]["mlp"]["expert"].pop("ff"), "layers[0].mlp.expert.ff"),
    (lambda d: d["layers"][0]["mlp"]["shared"].pop("ff"), "layers[0].mlp.shared.ff"),
])
def test_errors_name_the_key(edit, key):
    d = copy.deepcopy(CONFIGS["A"])
    edit(d)
    with pytest.raises(ConfigError) as e:
        spec_from_config_dict(d)
    assert key in str(e.value)


@pytest.mark.parametrize("rows,most", [(32, 150), (8, 20), (2, 3), (4, 6), (16, 300), (6, 11), (64, 4096)])
def test_distance_buckets(rows, most):
    half = rows // 2
    got = [distance_bucket(n, rows, most) for n in range(2 * most)]
    assert got == [pd.bucket(n, rows, most) for n in range(2 * most)]
    assert got[:half] == list(range(half)) and got[half] == half
    assert all(b - a in (0, 1) or (b > a and rows > most) for a, b in zip(got, got[1:]))      # never back, one row at a time
    assert all(b == rows - 1 for b in got[most:]) and max(got) == rows - 1
    table = torch.randn(rows, 3)
    for longest in (0, 7, most + 50):
        by = bias_by_distance(table, most, longest)
        assert by.shape == (3, min(most + 1, longest) if longest else most + 1) and by.is_contiguous()
        for n in range(2 * most if not longest else min(longest, 2 * most)):
            assert torch.equal(by[:, min(n, by.shape[1] - 1)], table[got[n]])


def test_pages_of_past_chunks_are_given_back():
    need = KVNeed(1, 16, chunk=100)
    assert [need.first_read(p) for p in (0, 99, 100, 250)] == [0, 0, 100, 200]
    assert KVNeed(1, 16, 30, chunk=100).first_read(110) == 100 and KVNeed(1, 16, 30, chunk=100).first_read(180) == 151
    assert KVNeed(1, 16).first_read(500) == 0 and KVNeed(1, 16, 30).first_read(20) == 0
    c = Cache([need, KVNeed(1, 16)], [None, None], 640, torch.float32, "cpu")
    s = c.open()
    for upto, held in ((60, 1), (100, 1), (128, 1), (129, 2), (199, 3), (200, 1), (300, 1)):
        c.reserve(s, upto)
        c.advance(s, upto)
        pages = c.page_list(s, 0)
        assert sum(p >= 0 for p in pages) == held, (upto, pages)
        assert all(p >= 0 for p in pages[need.first_read(upto) // 64:]) and all(p >= 0 for p in c.page_list(s, 1))
    c.check()
    c.reserve(s, 310)
    c.advance(s, 310)
    assert not c.truncate(s, 299) and not c.truncate(s, 150)     # the chunks before have lost their pages
    assert c.truncate(s, 301) and c.length(s) == 301             # the same chunk has not
    c.close(s)
    c.check()
    assert all(g.pool.free_count == c.n_pages for g in c.groups)
    full = Cache([KVNeed(1, 16, chunk=64)], [None], 640, torch.float32, "cpu")
    s = full.open()
    full.reserve(s, 128)
    full.advance(s, 128)                                         # a chunk's edge on a page's edge: nothing is left
    assert all(p < 0 for p in full.page_list(s, 0)) and full.groups[0].pool.held_count == 0


def test_chunks_bias_sink_and_convolution_of_the_plain_implementation():
    vis = pd.chunk_mask(10, 4)
    assert vis.sum(-1).tolist() == [1, 2, 3, 4, 1, 2, 3, 4, 1, 2] and pd.chunk_mask(5, 0).sum(-1).tolist() == [1, 2, 3, 4, 5]
    assert not vis[4, 3] and vis[7, 4] and not vis[4, 5]
    s = torch.randn(10, 10, dtype=F)
    w = pd.softmax_plus_one(s, vis)
    e = torch.exp(s).masked_fill(~vis, 0.0)
    assert torch.allclose(w, e / (1.0 + e.sum(-1, keepdim=True))) and bool((w.sum(-1) < 1).all())
    assert torch.allclose(pd.softmax_plus_one(s + 700.0, vis).sum(-1), torch.ones(10, dtype=F))       # no overflow
    rel = torch.randn(4, 2, dtype=F)
    b = pd.distance_bias(9, rel, 6)
    assert torch.equal(b[8, 8], rel[0]) and torch.equal(b[8, 7], rel[1]) and torch.equal(b[8, 0], rel[3]) and bool((b[3, 4] == 0).all())
    u, cw = torch.randn(6, 3, dtype=F), torch.randn(3, 4, dtype=F)
    y = pd.short_conv(u, cw)
    assert torch.allclose(y[0], cw[:, 3] * u[0]) and torch.allclose(y[5], sum(cw[:, j] * u[2 + j] for j in range(4)))


def test_the_router_hands_tokens_to_experts_and_identities():
    r = {"experts": 3, "identity": 2, "top": 2, "scale": 2.0}
    z = torch.tensor([1.0, 0.5, -1.0, 2.0, 0.0], dtype=F)
    corr = torch.zeros(5, dtype=F)
    s = torch.softmax(z, -1)
    chosen, weights, gap = pd.route(z, corr, r)
    assert chosen == [3, 0] and sum(weights) == pytest.approx(2.0) and gap == pytest.approx(float(s[0] - s[1]))
    assert weights[0] / weights[1] == pytest.approx(float(s[3] / s[0]))
    corr[2] = 1.0                                                     # a correction moves the choice, not the weights
    chosen, weights, _ = pd.route(z, corr, r)
    assert chosen == [2, 3] and weights[0] / weights[1] == pytest.approx(float(s[2] / s[3]))


def test_calm_tokens_have_no_close_router_call(tmp_path):
    cfg, tensors = write_model(tmp_path / "m", model(60, 32, [layer(attention(2, 1, 16, 16, 8, (4, 6)), moe(4, 2, 16, 2)),
                                                              layer(attention(2, 1, 16, 16, 8, (4, 6)), dense(16))]), seed=3)
    toks, ref = calm_tokens(cfg, tensors, 40, 5)
    gaps = []
    again = pd.forward(cfg, tensors, toks, gaps=gaps)
    assert torch.equal(again, ref) and len(gaps) == 1 and min(gaps[0]) >= 0.01
    assert ref.shape == (40, cfg["vocab"]) and bool(torch.isfinite(ref).all())
    assert math.isfinite(float(ref.abs().max()))
