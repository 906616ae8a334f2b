"""Debisun on the device against the plain implementation: every mechanism alone (kernels, then
one-layer models), the stream after every layer, whole prompts, token-by-token decoding, portions,
unequal batches, reused slots and pages, chunk edges, the distance bias, the sink, far keys, long decoding,
greedy generation through the entry point, the command line and the trace replay program."""
import json
import math

import numpy as np
import pytest
import torch

import plain_debisun as pd
import sonicboom_b200 as sb
from sonicboom_b200 import llm, ops
from sonicboom_b200.cache.kv import Cache, KVNeed, StateNeed
from sonicboom_b200.engine.step import StepEntry, StepPlan
from sonicboom_b200.parts.window_attention import bias_by_distance
from test_gpu_generate import replay
from debisun_util import CONFIGS, attention, calm_tokens, dense, layer, model, moe, tokens, write_model

pytestmark = pytest.mark.gpu
# The largest root mean square of a row's difference, over the root mean square of the whole
# reference (a request's logits).  The plain implementation is float64; bfloat16 rounds to 2^-9.
TOL = {"float32": 3e-5, "bfloat16": 8e-2}
DTYPES = ["float32", "bfloat16"]
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
SEEN = {}
F = torch.float64


def rel_err(got, ref):
    ref = ref.to(F)
    ref = ref.reshape(-1, ref.shape[-1])
    d = got.to(F).cpu().reshape(ref.shape) - ref
    return float(d.pow(2).mean(-1).sqrt().max() / ref.pow(2).mean().sqrt().clamp_min(1e-30))


def model_err(got, ref, dtype):
    e = rel_err(got, ref)
    SEEN[dtype] = max(SEEN.get(dtype, 0.0), e)
    return e


def teardown_module(module):
    print("largest row errors of whole models:", {k: f"{v:.2e}" for k, v in SEEN.items()})


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    out = {}
    for name, cfg in CONFIGS.items():
        d = tmp_path_factory.mktemp(f"debisun{name}")
        out[name] = (d,) + write_model(d, cfg, seed=60 + ord(name))
    return out


@pytest.fixture(scope="module")
def engines(folders):
    made = {}

    def get(name, dtype, max_tokens=2048):
        key = (name, dtype)
        if key not in made:
            made[key] = sb.load_model(folders[name][0], dtype=dtype)
        return sb.Engine(made[key], max_tokens=max_tokens)
    return get


def run_cuts(engine, toks, cuts):
    """Logits at every position of one request fed in portions of the given sizes."""
    s = engine.open()
    outs, at = [], 0
    for n in cuts:
        outs.append(engine.step([(s, toks[at:at + n], list(range(n)))]).float().cpu())
        at += n
    assert at == len(toks)
    engine.close(s)
    return torch.cat(outs)


# ------------------------------------------------------------------ mechanisms alone: kernels
@pytest.mark.parametrize("rows,width", [(1, 8), (7, 44), (5, 63), (40, 1000), (3, 4096), (600, 2048), (300, 5000), (4, 8192), (9, 12288), (2, 17000)])
def test_a_result_joins_the_stream_and_the_next_norm_rides_along(rows, width):
    g = torch.Generator().manual_seed(rows + width)
    y, x = torch.randn(rows, width, generator=g) * 2, torch.randn(rows, width, generator=g) + 0.4
    w, nw, nb = (torch.randn(width, generator=g) for _ in range(3))
    for norm_eps in (None, 1e-3):
        for wd in (torch.float32, torch.bfloat16):
            s = w.to(wd).double()
            v = y.double() if norm_eps is None else pd.rms(y.double(), norm_eps)
            ref = x.double() + s * v
            plain = ops.stream_join(y.cuda(), x.cuda(), w.to(wd).cuda(), torch.empty(rows, width, device="cuda"), norm_eps)
            assert rel_err(plain, ref) < 2e-6
            for od in (torch.float32, torch.bfloat16):
                tol = 1e-5 if od == torch.float32 else 5e-3
                for kind, bias in ((ops.NEXT_COPY, False), (ops.NEXT_RMS, False), (ops.NEXT_LAYER, False), (ops.NEXT_LAYER, True)):
                    xc = x.cuda()
                    nxt = torch.empty(rows, width, device="cuda", dtype=od)
                    copy = kind == ops.NEXT_COPY
                    ops.stream_join(y.cuda(), xc, w.to(wd).cuda(), xc, norm_eps,
                                    (kind, None if copy else nw.to(wd).cuda(), nb.to(wd).cuda() if bias else None, 1e-4, nxt))
                    assert torch.equal(xc, plain)                                    # in place, whatever comes along
                    if copy:
                        assert torch.equal(nxt, xc.to(od))
                        continue
                    n64, b64 = nw.to(wd).double(), nb.to(wd).double() if bias else 0.0
                    want = pd.layer_norm(ref, n64, b64, 1e-4) if kind == ops.NEXT_LAYER else pd.rms(ref, 1e-4) * n64
                    assert rel_err(nxt, want) < tol, (kind, bias, od)


def test_layer_norm_with_a_bias_and_gathered_rows():
    g = torch.Generator().manual_seed(3)
    for n, width in ((9, 44), (3, 4096), (600, 256)):
        x = torch.randn(n, width, generator=g) * 2 + 3.0
        w, b = torch.randn(width, generator=g), torch.randn(width, generator=g)
        ref = pd.layer_norm(x.double(), w.double(), b.double(), 1e-5)
        out = ops.layernorm(x.cuda(), w.cuda(), 1e-5, torch.empty(n, width, device="cuda"), bias=b.cuda())
        assert rel_err(out, ref) < 5e-6
        rows = torch.tensor([2, 0], dtype=torch.int32, device="cuda")
        assert torch.equal(ops.layernorm(x.cuda(), w.cuda(), 1e-5, torch.empty(2, width, device="cuda"), rows, bias=b.cuda()), out[[2, 0]])


def test_the_token_input_is_gated_by_gelu():
    g = torch.Generator().manual_seed(4)
    for dim, parts, part in ((5, 3, 1), (16, 2, 0), (300, 2, 1)):
        z, table = torch.randn(33, dim, generator=g) * 2, torch.randn(20, dim * parts, generator=g)
        toks = torch.randint(0, 20, (33,), generator=g)
        for td in (torch.float32, torch.bfloat16):
            t = table.to(td)
            ref = pd.gelu_tanh(z.double()) * t.double()[toks][:, part * dim:(part + 1) * dim]
            out = ops.side_gate(z.cuda(), toks.int().cuda(), t.cuda(), part * dim, torch.empty(33, dim, device="cuda"))
            assert rel_err(out, ref) < 2e-6
    bad = ops.side_gate(z.cuda(), torch.full((33,), -1, dtype=torch.int32, device="cuda"), table.cuda(), 0, torch.empty(33, dim, device="cuda"))
    assert bool(torch.isnan(bad).all())                               # an id outside the table stays visible


@pytest.mark.parametrize("M,N,K", [(1, 48, 64), (5, 200, 512), (8, 4096, 256), (20, 96, 1024), (40, 1200, 2048), (64, 512, 4096),
                                   (100, 130, 64), (200, 384, 256), (300, 1024, 512), (700, 2000, 128), (3, 29, 44), (130, 24, 40)])
def test_squared_relu_in_every_product(M, N, K):
    g = torch.Generator().manual_seed(M + N)
    a, w = torch.randn(M, K, generator=g), torch.randn(N, K, generator=g) / math.sqrt(K)
    ref = pd.squared_relu(a.double() @ w.double().T)
    out = ops.linear(a.cuda(), w.cuda(), torch.empty(M, N, device="cuda"), ops.EPI_RELU2)
    assert rel_err(out, ref) < 1e-5
    ab, wb = a.bfloat16(), w.bfloat16()
    ref = pd.squared_relu(ab.double() @ wb.double().T)
    kernels = ["auto", "plain"] + (["tiled", "tc5"] if K % 8 == 0 else []) + (["skinny"] if K % 8 == 0 and M <= 64 else [])
    for kernel in kernels:
        for od in (torch.float32, torch.bfloat16):
            out = ops.linear(ab.cuda(), wb.cuda(), torch.empty(M, N, device="cuda", dtype=od), ops.EPI_RELU2, kernel=kernel)
            assert rel_err(out, ref) < (3e-5 if od == torch.float32 else 8e-3), (kernel, od)


@pytest.mark.parametrize("experts,identity,top,scale", [(5, 3, 3, 1.7), (4, 0, 1, 1.0), (3, 5, 8, 2.5), (40, 20, 6, 1.0), (1, 0, 1, 0.5), (200, 56, 8, 2.0)])
def test_router_softmax_scores(experts, identity, top, scale):
    g = torch.Generator().manual_seed(experts * 7 + top)
    rows, E = 50, experts + identity
    z = torch.randn(rows, E + 1, generator=g) * 2                     # a column more than the router has, as beside a gate
    z[3, :E] = 0.7                                                   # every score the same: the lowest indices win
    z[5, :E] += 90.0                                                 # large logits do not overflow
    corr = torch.randn(E, generator=g) * 0.05
    corr[:] = 0.0 if top == E else corr
    r = {"experts": experts, "identity": identity, "top": top, "scale": scale}
    ids, w = torch.empty(rows, top, dtype=torch.int32, device="cuda"), torch.empty(rows, top, device="cuda")
    ops.moe_route_scored(z.cuda(), corr.cuda(), top, ids, w, scale=scale, renormalize=True, scores="softmax")
    for t in range(rows):
        chosen, weights, gap = pd.route(z[t, :E].double(), corr.double(), r)
        if gap > 1e-6:
            assert sorted(ids[t].tolist()) == sorted(chosen), t
            by = dict(zip(ids[t].tolist(), w[t].cpu().tolist()))
            assert all(by[e] == pytest.approx(v, rel=2e-5) for e, v in zip(chosen, weights)), t
        assert float(w[t].sum()) == pytest.approx(scale, rel=1e-5)
    if float(corr.abs().max()) == 0.0:
        assert ids[3].tolist() == list(range(top))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,experts,identity,top,ff,width", [(1, 4, 2, 3, 24, 40), (9, 5, 3, 3, 24, 64), (70, 3, 1, 2, 9, 44),
                                                               (300, 4, 4, 4, 136, 256), (600, 2, 0, 1, 64, 128), (33, 6, 2, 8, 40, 72)])
def test_experts_identities_and_a_gated_shared_expert(rows, experts, identity, top, ff, width, dtype):
    g = torch.Generator().manual_seed(rows + ff)
    d = DT[dtype]
    h = torch.randn(rows, width, generator=g).to(d)
    up, down = (torch.randn(experts, *s, generator=g).mul(0.1).to(d) for s in ((ff, width), (width, ff)))
    ids = torch.stack([torch.randperm(experts + identity, generator=g)[:top] for _ in range(rows)]).int()
    if identity and rows > 4:
        ids[2] = torch.arange(experts + identity - top, experts + identity).int()       # a row with as many identities as there are
    w = torch.rand(rows, top, generator=g)
    x, shared, gate = torch.randn(rows, width, generator=g), torch.randn(rows, width, generator=g), torch.randn(rows, 7, generator=g)
    s = torch.randn(width, generator=g)
    y = torch.zeros(rows, width, dtype=F)
    h64 = h.double()
    for k in range(top):
        for e in range(experts + identity):
            m = ids[:, k] == e
            if bool(m.any()):
                out = h64[m] if e >= experts else pd.squared_relu(h64[m] @ up[e].double().T) @ down[e].double().T
                y[m] += w[m, k].double().view(-1, 1) * out
    tol = 2e-6 if dtype == "float32" else 1e-2                       # bfloat16: the activations between the products
    dev = [t.cuda() for t in (h, ids, w, up, down)]
    copy = torch.empty(rows, width, device="cuda", dtype=torch.bfloat16)
    xs = x.cuda()
    ops.moe_relu2_join(*dev, xs, shared=shared.cuda(), gate=(gate.cuda(), 4), scale=s.cuda(), copy=copy)
    want = x.double() + s.double() * (y + torch.sigmoid(gate[:, 4:5].double()) * shared.double())
    assert rel_err(xs, want) < tol and torch.equal(copy, xs.bfloat16())
    xs = x.cuda()
    ops.moe_relu2_join(*dev, xs, shared=shared.cuda())
    assert rel_err(xs, x.double() + y + shared.double()) < tol
    xs = x.cuda()
    ops.moe_relu2_join(*dev, xs, scale=s.bfloat16().cuda())
    assert rel_err(xs, x.double() + s.bfloat16().double() * y) < tol


def attend(dtype, seqs, hq, hkv, dim, vdim, chunk, scale, softcap, rel, most, conv_w, kernel="auto", cuts=None):
    """Projection rows of several sequences (float32 [n, q | k | v]) through `conv_heads`, the attention
    kernels and the drop of the padding; a sequence may come in portions (`cuts`)."""
    hd = (max(dim, vdim) + 15) // 16 * 16
    taps, channels = conv_w.shape[1], conv_w.shape[0]
    need = StateNeed((taps - 1, channels), torch.float32) if taps > 1 else None
    cache = Cache([KVNeed(hkv, hd, chunk=chunk)], [need], 8192, DT[dtype], "cuda")
    cache.groups[0].storage.fill_(1e4)                 # stale values of the padding and of keys out of sight would show
    slots = [cache.open() for _ in seqs]
    bias = ops.DistanceBias(bias_by_distance(rel, most, chunk).cuda())
    sink = torch.zeros(hq, device="cuda")
    w = conv_w.cuda()
    outs, at = [[] for _ in seqs], [0] * len(seqs)
    for step in (cuts or [[x.shape[0] for x in seqs]]):
        live = [(i, n) for i, n in enumerate(step) if n]
        for i, n in live:
            cache.reserve(slots[i], cache.length(slots[i]) + n)
        plan = StepPlan(cache, [StepEntry(slots[i], [0] * n, []) for i, n in live], "cuda")
        proj = torch.cat([seqs[i][at[i]:at[i] + n] for i, n in live]).cuda()
        g, storage = plan.groups[0], cache.groups[0].entry_storage(0)
        q = torch.full((proj.shape[0], hq, hd), 1e4, dtype=DT[dtype], device="cuda")
        ops.conv_heads(proj, w, plan, g.page_off, g.page_ids, g.page_size, hq, hkv, dim, vdim,
                       cache.state[0] if taps > 1 else None, storage, q)
        out = torch.empty(proj.shape[0], hq * hd, dtype=DT[dtype], device="cuda")
        ops.attention(q, out, plan, 0, storage, hq, hkv, hd, 0, scale, kernel=kernel, sink=sink, softcap=softcap,
                      chunk=chunk, bias=bias)
        if hd != vdim:
            out = ops.attn_unrotate(out, torch.empty(proj.shape[0], hq * vdim, dtype=DT[dtype], device="cuda"), hq, hd,
                                    vdim, False, None, plan.row_pos)
        out = out.float().cpu()
        row = 0
        for i, n in live:
            outs[i].append(out[row:row + n])
            row += n
            at[i] += n
            cache.advance(slots[i], cache.length(slots[i]) + n)
    return [torch.cat(o) for o in outs]


def attend_ref(x, hq, hkv, dim, vdim, chunk, scale, softcap, rel, most, conv_w):
    """The same on one whole sequence with the plain implementation's functions."""
    T = x.shape[0]
    u = pd.short_conv(x.double(), conv_w.double())
    q, k, v = (t.reshape(T, n, -1) for t, n in zip(u.split([hq * dim, hkv * dim, hkv * vdim], 1), (hq, hkv, hkv)))
    bias, vis = pd.distance_bias(T, rel.double(), most), pd.chunk_mask(T, chunk)
    out = torch.zeros(T, hq, vdim, dtype=F)
    for h in range(hq):
        s = (q[:, h] @ k[:, h // (hq // hkv)].T) * scale
        s = softcap * torch.tanh(s / softcap) if softcap else s
        out[:, h] = pd.softmax_plus_one(s + bias[:, :, h], vis) @ v[:, h // (hq // hkv)]
    return out.reshape(T, hq * vdim)


ATTEND = [
    # hq, hkv, dim, vdim, chunk, softcap, rows of the bias table, its last distance, taps, sequence lengths
    (4, 2, 16, 24, 9, 5.0, 8, 20, 3, (150, 37, 1)),
    (6, 3, 64, 32, 70, 20.0, 32, 55, 4, (150, 37, 1)),
    (2, 1, 64, 64, 0, 0.0, 16, 100, 5, (150, 37, 1)),
    (8, 2, 128, 128, 100, 12.0, 12, 40, 4, (250, 37, 1)),
    (3, 3, 7, 9, 3, 1.5, 2, 3, 2, (150, 37, 1)),
    (4, 1, 96, 80, 64, 9.0, 64, 60, 1, (150, 37, 1)),
    (5, 1, 128, 112, 1, 30.0, 4, 6, 4, (150, 37, 1)),
    (2, 1, 64, 64, 700, 8.0, 20, 300, 4, (1440, 600, 711)),        # chunks of several decode splits
    (1, 1, 128, 128, 1000, 0.0, 32, 2000, 3, (1290, 33, 999)),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", range(len(ATTEND)))
def test_chunked_attention_with_convolutions_and_a_distance_bias(dtype, case):
    """Every attention kernel family: the plain one, the mma.sync ones, and at head sizes 64 and 128
    the tensor-memory prompt kernel and the TMA decode kernel; whole, in portions and one by one."""
    hq, hkv, dim, vdim, chunk, softcap, rows, most, taps, lens = ATTEND[case]
    g = torch.Generator().manual_seed(100 + case)
    width = hq * dim + hkv * (dim + vdim)
    seqs = [torch.randn(n, width, generator=g) * 1.5 for n in lens]
    rel, conv_w = torch.randn(rows, hq, generator=g) * 1.5, torch.randn(width, taps, generator=g) / math.sqrt(taps)
    args = (hq, hkv, dim, vdim, chunk, 1.5 / math.sqrt(dim), softcap, rel, most, conv_w)
    refs = [attend_ref(x, *args) for x in seqs]
    tol = 2e-5 if dtype == "float32" else 3e-2
    kernels = ["auto"] if dtype == "float32" else ["auto", "plain", "mma"] + (["tma"] if max(dim, vdim) in (64, 128) else [])
    a, b, c = lens
    for kernel in kernels:
        for cuts in (None, [[a - 52, b - 9, 0], [2, 7, c], [50, 2, 0]],
                     [[a - 20, b - 9, c]] + [[1, 1 if i < 9 else 0, 0] for i in range(20)]):
            outs = attend(dtype, seqs, *args, kernel=kernel, cuts=cuts)
            for o, r in zip(outs, refs):
                assert rel_err(o, r) < tol, (kernel, cuts and cuts[1])


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5])
def test_convolved_heads_equal_the_convolution_and_the_row_kernel(taps):
    """The fused kernel against `causal_conv` followed by `attn_prep`, to the bit, with the state it leaves."""
    hq, hkv, dim, vdim, hd = 3, 1, 24, 16, 32
    channels = hq * dim + hkv * (dim + vdim)
    g = torch.Generator().manual_seed(taps)
    w = torch.randn(channels, taps, generator=g).bfloat16().cuda()
    need = StateNeed((taps - 1, channels), torch.float32) if taps > 1 else None
    made = []
    rows = [[torch.randn(n, channels, generator=g) for n in step] for step in ((5, 1, 20), (1, 1, 1), (2, 11, 1), (1, 1, 1))]
    for fused in (True, False):
        cache = Cache([KVNeed(hkv, hd)], [need], 512, torch.bfloat16, "cuda")
        slots = [cache.open() for _ in range(3)]
        got = []
        for step in rows:
            for s, x in zip(slots, step):
                cache.reserve(s, cache.length(s) + x.shape[0])
            plan = StepPlan(cache, [StepEntry(s, [0] * x.shape[0], []) for s, x in zip(slots, step)], "cuda")
            proj, p, storage = torch.cat(step).cuda(), plan.groups[0], cache.groups[0].entry_storage(0)
            state = cache.state[0] if taps > 1 else None
            q = torch.empty(proj.shape[0], hq, hd, dtype=torch.bfloat16, device="cuda")
            if fused:
                ops.conv_heads(proj, w, plan, p.page_off, p.page_ids, p.page_size, hq, hkv, dim, vdim, state, storage, q)
            else:
                y = ops.causal_conv(proj, 0, channels, w, None, plan, state, torch.empty_like(proj))
                ops.attn_prep(y, 0, hq * dim, (hq + hkv) * dim, hq, hkv, dim, vdim, hd, 0, False, None, None, None, None, 1e-5,
                              plan.row_seq, plan.row_pos, p.page_off, p.page_ids, p.page_size, storage, q)
            got.append(q.clone())
            for s, x in zip(slots, step):
                cache.advance(s, cache.length(s) + x.shape[0])
        made.append(got + [cache.groups[0].storage.clone()] + ([cache.state[0][slots].clone()] if taps > 1 else []))
    assert all(torch.equal(a, b) for a, b in zip(*made))


# ------------------------------------------------------------------ mechanisms alone: one-layer models
ONE_LAYER = {
    "chunked attention": layer(attention(4, 2, 16, 24, 9, (8, 20), conv=3, scale=0.5)),
    "attention over every key, no cap": layer(attention(2, 1, 32, 32, 0, (6, 30), softcap=0.0)),
    "no convolutions": layer(attention(2, 2, 16, 16, 20, (6, 9), conv=0)),
    "one tap": layer(attention(2, 1, 16, 8, 11, (6, 9), conv=1)),
    "eight taps": layer(attention(2, 1, 16, 16, 30, (6, 9), conv=8)),
    "a head size beyond the tensor-core kernels": layer(attention(1, 1, 272, 16, 25, (6, 9))),
    "dense feed-forward": layer(attention(1, 1, 16, 16, 4, (4, 6)), dense(56)),
    "dense feed-forward, odd size": layer(attention(1, 1, 16, 16, 4, (4, 6)), dense(29)),
    "experts and identities": layer(attention(1, 1, 16, 16, 4, (4, 6)), moe(5, 3, 24, identity=4, scale=1.4, shared=16)),
    "experts, no identities, no shared expert": layer(attention(1, 1, 16, 16, 4, (4, 6)), moe(4, 2, 11)),
    "one expert, one identity": layer(attention(1, 1, 16, 16, 4, (4, 6)), moe(1, 2, 16, identity=1, scale=0.7)),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(ONE_LAYER))
def test_each_mechanism_in_a_model_of_its_own(tmp_path, name, dtype):
    cfg, tensors = write_model(tmp_path / "one", model(90, 48, [ONE_LAYER[name]], side=6 if len(name) % 2 else 0), seed=len(name))
    toks, ref = calm_tokens(cfg, tensors, 75, 9)
    engine = sb.Engine(sb.load_model(tmp_path / "one", dtype=dtype), max_tokens=512)
    for cuts in ([75], [70, 1, 1, 1, 1, 1], [3, 2, 61, 9], [2] * 37 + [1]):
        assert model_err(run_cuts(engine, toks, cuts), ref, dtype) < TOL[dtype], cuts[:4]


def test_the_stream_after_every_layer(folders, engines):
    for name in CONFIGS:
        _, cfg, tensors = folders[name]
        toks = tokens(cfg, 50, 3)
        streams = []
        pd.forward(cfg, tensors, toks, layers_out=streams)
        engine = engines(name, "float32")
        seen = []
        for b in engine.model.blocks:
            inner = b.forward
            b.forward = lambda x, ctx, inner=inner: (lambda y: (seen.append(y.clone()), y)[1])(inner(x, ctx))
        try:
            run_cuts(engine, toks, [50])
        finally:
            for b in engine.model.blocks:
                del b.forward
        assert len(seen) == len(streams)
        for got, ref in zip(seen, streams):
            assert rel_err(got, ref) < 1e-5


# ------------------------------------------------------------------ whole models
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_decoding_and_portions(folders, engines, name, dtype):
    _, cfg, tensors = folders[name]
    toks, ref = calm_tokens(cfg, tensors, 171, 5, key=name)
    engine = engines(name, dtype)
    whole = run_cuts(engine, toks, [171])
    assert model_err(whole, ref, dtype) < TOL[dtype]
    # the first tokens of a sequence one by one, then the rest; most of it at once, then one by one
    # over two page borders (64, 128) and every chunk's edge; portions down to two tokens
    for cuts in ([1, 1, 1, 168], [40] + [1] * 131, [2, 3, 62, 2, 59, 7, 17, 19], [64, 64, 43], [170, 1], [69, 2, 100]):
        got = run_cuts(engine, toks, cuts)
        assert model_err(got, ref, dtype) < TOL[dtype], cuts
        if dtype == "float32":
            assert rel_err(got, whole) < 1e-5, cuts       # rounding: few rows run other kernels
    engine.cache.check()
    assert engine.free_pages() == engine.cache.n_pages


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_unequal_batch_equals_each_alone_and_slots_are_reused(folders, engines, name, dtype):
    from gpu_util import batch_unequal
    _, cfg, tensors = folders[name]
    reqs, refs = zip(*[calm_tokens(cfg, tensors, n, 10 + n, key=name) for n in (1, 70, 131, 23)])
    engine = engines(name, dtype, max_tokens=512)
    # twice in the same engine: the second pass reuses the slots and pages of the first
    for _ in range(2):
        outs = batch_unequal(engine, reqs, [1, 40, 100, 23])
        for o, r in zip(outs, refs):
            assert model_err(o, r, dtype) < TOL[dtype]
        engine.cache.check()
    alone = [run_cuts(engine, r, [k] + [1] * (len(r) - k)) for r, k in zip(reqs, [1, 40, 100, 23])]
    if dtype == "float32":
        for o, a in zip(outs, alone):
            assert rel_err(o, a) < 1e-5
    # a sequence that ends early gives its slot to a new one while the others go on
    a, b = engine.open(), engine.open()
    engine.step([(a, reqs[1][:30], []), (b, reqs[2][:50], [])])
    engine.close(a)
    c = engine.open()
    assert c == a
    lg = engine.step([(b, reqs[2][50:60], list(range(10))), (c, reqs[3], list(range(23)))]).float().cpu()
    assert rel_err(lg[:10], refs[2][50:60]) < TOL[dtype] and rel_err(lg[10:], refs[3]) < TOL[dtype]
    engine.close(b), engine.close(c)


def sharp_model():
    """Large score scales, so that a few keys carry a row's sum: a chunk one position off, a sink left out, a
    bias row off, a lost tap or a far key lost moves the logits by a large multiple of the tolerance."""
    return model(80, 48, [
        layer(attention(2, 1, 16, 16, 13, (8, 12), softcap=30.0, scale=1.2)),
        layer(attention(2, 2, 16, 16, 0, (16, 200), softcap=40.0, scale=0.9), dense(32)),
        layer(attention(2, 2, 64, 64, 100, (10, 80), softcap=25.0, scale=0.4)),
    ], side=4)


def sharpen(t):
    for i in range(3):
        t[f"l{i}.mix.o"] *= 3.0
        t[f"l{i}.mix.rel"] *= 1.5
    t["l1.mix.rel"][-1] += 5.0                          # far keys carry weight


@pytest.mark.parametrize("dtype", DTYPES)
def test_chunk_edges_bias_sink_taps_and_far_keys_show(tmp_path, dtype):
    cfg, tensors = write_model(tmp_path / "w", sharp_model(), seed=9, edit=sharpen)
    toks = tokens(cfg, 420, 21)
    ref = pd.forward(cfg, tensors, toks)
    shows = 100 * TOL["float32"]

    def other(edit_cfg=None, edit_tensors=None, seq=toks):
        c, t = json.loads(json.dumps(cfg)), dict(tensors)
        if edit_cfg:
            edit_cfg(c)
        if edit_tensors:
            edit_tensors(t)
        return pd.forward(c, t, seq)
    for which in (0, 2):
        for delta in (1, -1):
            got = other(lambda c: c["layers"][which]["mixer"]["mask"].update(size=cfg["layers"][which]["mixer"]["mask"]["size"] + delta))
            assert rel_err(got[100:], ref[100:]) > shows, (which, delta)
    for which, most in ((0, 10), (1, 150), (2, 60)):
        assert rel_err(other(lambda c: c["layers"][which]["mixer"].update(bias_max=most)), ref) > shows, which
    for which in range(3):
        for n in ("q", "k", "v"):
            def drop(t):                                # the oldest tap lost
                name = f"l{which}.mix.{n}.conv"
                t[name] = t[name].clone()
                t[name][:, 0] = 0.0
            assert rel_err(other(edit_tensors=drop), ref) > shows, (which, n)
    far = list(toks)
    far[3] = (toks[3] + 1) % cfg["vocab"]
    assert rel_err(other(seq=far)[400:], ref[400:]) > shows
    engine = sb.Engine(sb.load_model(tmp_path / "w", dtype=dtype), max_tokens=1024)
    for cuts in ([420], [380] + [1] * 40, [12, 2, 50, 356], [13] + [1] * 120 + [287], [5, 200, 215], [99, 2, 99, 2, 218]):
        assert rel_err(run_cuts(engine, toks, cuts), ref) < TOL[dtype], cuts[:4]


def test_the_sink_shows_and_a_lone_key_keeps_its_share(tmp_path):
    """The first position of a chunk sees itself alone: with the one in the denominator its weight is
    sigmoid(score), not 1."""
    cfg, tensors = write_model(tmp_path / "s", model(50, 32, [layer(attention(2, 1, 16, 16, 1, (4, 6), scale=0.5))], side=0), seed=4)
    toks = tokens(cfg, 9, 3)
    ref = pd.forward(cfg, tensors, toks)
    plain = pd.softmax_plus_one
    try:
        pd.softmax_plus_one = lambda s, vis: torch.softmax(s.masked_fill(~vis, -math.inf), -1)
        assert rel_err(pd.forward(cfg, tensors, toks), ref) > 0.01
    finally:
        pd.softmax_plus_one = plain
    engine = sb.Engine(sb.load_model(tmp_path / "s", dtype="float32"), max_tokens=256)
    assert rel_err(run_cuts(engine, toks, [4, 1, 1, 3]), ref) < TOL["float32"]


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_gives_pages_back(folders, engines, dtype):
    """Six hundred tokens one by one: chunks end within and at the end of pages, and the pages of past
    chunks are given back."""
    _, cfg, tensors = folders["B"]
    toks, ref = calm_tokens(cfg, tensors, 600, 77, key="B")
    engine = engines("B", dtype, max_tokens=704)
    s = engine.open()
    engine.step([(s, toks[:5], [])])
    rows = []
    for i in range(5, 600):
        lg = engine.step([(s, [toks[i]], [0] if i % 7 == 0 or i > 590 else [])])
        if lg is not None:
            rows.append((i, lg.float().cpu()[0]))
    assert all(sum(p >= 0 for p in engine.cache.page_list(s, g)) <= 2 for g in range(len(engine.cache.groups)))
    engine.close(s)
    got = torch.stack([r for _, r in rows])
    assert rel_err(got, ref[[i for i, _ in rows]]) < TOL[dtype]
    engine.cache.check()
    assert engine.free_pages() == engine.cache.n_pages


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_greedy_generation_through_the_entry_point(folders, name, dtype):
    """`llm.generate_batch`: the scheduler's batches, the captured decode step with the convolutions' state
    in it, and slots given to the next batch."""
    d, cfg, tensors = folders[name]
    m = llm.model_load(d, dtype=dtype)
    assert m.arch == "Debisun" and m.vocab_size == cfg["vocab"]
    prompts = [tokens(cfg, n, 30 + n) for n in (3, 66, 20, 1)]
    n_new = 12
    outs = llm.generate_batch(m, prompts, max_tokens=n_new)
    for p, o in zip(prompts, outs):
        seq = list(p)
        for i, t in enumerate(o):
            gaps = []
            logits = pd.forward(cfg, tensors, seq, gaps=gaps)[-1]
            best = int(torch.argmax(logits))
            if t != best:
                top2 = torch.topk(logits, 2).values
                margin = float(top2[0] - top2[1]) / float(logits.abs().max())
                close_call = min((min(g) for g in gaps), default=1.0) < 0.02
                assert dtype == "bfloat16" and (margin < 2 * TOL[dtype] or close_call), (i, o, margin)
                break
            seq.append(t)
    alone = [llm.generate_batch(m, [p], max_tokens=n_new)[0] for p in prompts]
    small = llm.generate_batch(m, prompts, max_tokens=n_new, max_cache_tokens=192)     # more than one batch
    if dtype == "float32":
        assert alone == outs and small == outs
    s = llm.session_new(m, 128)
    assert llm.generate_tokens(s, prompts[2], n_new) == alone[2]
    s.free()


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay_program(folders, tmp_path, dtype):
    d, cfg, tensors = folders["B"]
    (a, ra), (b, rb) = calm_tokens(cfg, tensors, 75, 1, key="B"), calm_tokens(cfg, tensors, 30, 2, key="B")
    ra, rb = ra.numpy(), rb.numpy()
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:70], "want": [0, 69]},
                                     {"id": "b", "tokens": b[:29], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[70:71], "want": [0]},
                                     {"id": "b", "tokens": b[29:], "want": [0]}], "end": ["b"]}]
    steps += [{"step": i - 69, "entries": [{"id": "a", "tokens": [a[i]], "want": [0] if i % 2 else []}],
               "end": ["a"] if i == 74 else []} for i in range(71, 75)]
    got = replay(d, dtype, steps, tmp_path / "out", 256)
    V = cfg["vocab"]
    want = {0: ra[[0, 69]], 1: np.stack([ra[70], rb[29]]), 2: ra[71:72], 4: ra[73:74]}
    assert set(got) == set(want)
    for k, ref in want.items():
        assert np.abs(got[k].reshape(-1, V) - ref).max() / np.abs(ra).max() < TOL[dtype], k


def test_command_line_generates(folders, tmp_path):
    """`python -m sonicboom_b200 generate` on a Debisun folder: greedy tokens as the plain
    implementation's."""
    import subprocess
    import sys
    from conftest import ROOT
    d, cfg, tensors = folders["A"]
    prompts = [tokens(cfg, n, 50 + n) for n in (7, 33)]
    f = tmp_path / "prompts.txt"
    f.write_text("".join(" ".join(map(str, p)) + "\n" for p in prompts))
    base = [sys.executable, "-m", "sonicboom_b200", "generate", "-m", str(d), "--tokens", str(f), "-n", "6",
            "--dtype", "float32"]
    r = subprocess.run(base, capture_output=True, text=True, cwd=ROOT, timeout=900)
    assert r.returncode == 0, r.stderr[-2000:]
    got = [[int(t) for t in line.split()] for line in r.stdout.strip().splitlines()]
    assert got == [pd.greedy_generate(cfg, tensors, p, 6) for p in prompts]
