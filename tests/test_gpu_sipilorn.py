"""Sipilorn on the device against the plain implementation: every mechanism alone (kernels, then one-layer models),
the stream after every layer, whole prompts, token-by-token decoding, portions, unequal batches, reused slots and
pages, window edges, far keys and far writes, long decoding, greedy generation through the entry point, the command
line and the trace replay program."""
import json

import numpy as np
import pytest
import torch

import plain_sipilorn as ps
import sonicboom_b200 as sb
from sonicboom_b200 import llm, ops
from sonicboom_b200.cache.kv import Cache, StateNeed
from sonicboom_b200.engine.step import StepEntry, StepPlan
from test_gpu_generate import replay
from sipilorn_util import CONFIGS, attention, delta, dense, layer, model, moe, parallel, tokens, write_model

pytestmark = pytest.mark.gpu
# The largest root mean square of a row's difference, over the root mean square of the whole
# reference (a request's logits).  The plain implementation is float64; bfloat16 rounds to 2^-9.
TOL = {"float32": 3e-5, "bfloat16": 8e-2}
DTYPES = ["float32", "bfloat16"]
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
        d = tmp_path_factory.mktemp(f"sipilorn{name}")
        out[name] = (d,) + write_model(d, cfg, seed=80 + ord(name))
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


_REFS = {}


def reference(folders, name, n, seed):
    """(tokens, the plain implementation's logits), worked out once."""
    key = (name, n, seed)
    if key not in _REFS:
        _, cfg, tensors = folders[name]
        toks = tokens(cfg, n, seed)
        _REFS[key] = (toks, ps.forward(cfg, tensors, toks))
    return _REFS[key]


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
def delta_case(H, G, d, dv, taps, T, seed, keys="random", decays="mixed"):
    """Random projection rows and weights of a gated delta mixer, and what its oracle makes of them."""
    g = torch.Generator().manual_seed(seed)
    C = 2 * G * d + H * dv
    q_off, g_off, b_off, a_off = 4, 4 + C, 4 + C + H * dv, 4 + C + H * dv + H
    proj = torch.randn(T, a_off + H + 3, generator=g)
    if keys == "repeated":               # the same key again and again, written with beta near one
        proj[:, q_off + G * d:q_off + 2 * G * d] = torch.randn(G * d, generator=g) + 0.05 * torch.randn(T, G * d, generator=g)
        proj[:, b_off:b_off + H] += 4.0
    conv = torch.randn(C, taps, generator=g) * 0.4
    conv[:, -1] += 1.0
    a_log = torch.randn(H, generator=g) * 2.0 - (5.0 if decays == "slow" else 1.0)
    if decays == "mixed":
        a_log[0], a_log[-1] = -8.0, 4.0   # one head that forgets nothing, one that forgets at once
    dt, norm = torch.randn(H, generator=g), 1.0 + 0.3 * torch.randn(dv, generator=g)
    x = proj.double()
    act = torch.nn.functional.silu(ps.short_conv(x[:, q_off:q_off + C], conv.double()))
    q = ps.unit(act[:, :G * d].view(T, G, d)) * d ** -0.5
    k = ps.unit(act[:, G * d:2 * G * d].view(T, G, d))
    decay = torch.exp(-torch.exp(a_log.double()) * torch.nn.functional.softplus(x[:, a_off:a_off + H] + dt.double(), threshold=200.0))
    raw = ps.gated_delta_rule(q, k, act[:, 2 * G * d:].view(T, H, dv), decay, torch.sigmoid(x[:, b_off:b_off + H]))
    o = ps.rms(raw, 1e-4) * norm.double() * torch.nn.functional.silu(x[:, g_off:g_off + H * dv]).view(T, H, dv)
    return dict(proj=proj, q_off=q_off, g_off=g_off, b_off=b_off, a_off=a_off, conv=conv.cuda(), a_log=a_log.cuda(), dt=dt.cuda(),
                norm=norm.cuda(), sizes=(H, G, d, dv), taps=taps), o.reshape(T, H * dv)


def delta_cache(H, G, d, dv, taps, n_slots):
    need = {"memory": StateNeed((H, dv, d), torch.float32)}
    if taps > 1:
        need["ring"] = StateNeed((taps, 2 * G * d + H * dv), torch.float32)
    cache = Cache([None], [need], 64 * n_slots, torch.float32, "cuda", n_slots=n_slots)
    for t in cache.state.values():
        t.fill_(float("nan"))            # a slot's rows are zeroed when it is taken; ring rows of no position are never read
    return cache


def run_delta(case, cache, slot_rows, kernel="auto", scale=1.0, dtype=torch.float32, pad=5):
    """One step of the mixer: `slot_rows` = [(slot, rows of the projection)], through the cache's state."""
    plan = StepPlan(cache, [StepEntry(s, [0] * r.shape[0], []) for s, r in slot_rows], "cuda")
    rows = torch.cat([r for _, r in slot_rows]).cuda()
    H, G, d, dv = case["sizes"]
    out = torch.full((rows.shape[0], H * dv + 2 * pad), 7.0, device="cuda", dtype=dtype)
    ops.gated_delta(rows, case["q_off"], case["a_off"], case["b_off"], case["g_off"], plan, H, G, d, dv, case["conv"], case["a_log"],
                    case["dt"], d ** -0.5, 1e-6, case["norm"], 1e-4, cache.state.get((0, "ring")), cache.state[(0, "memory")],
                    out, pad, scale, kernel=kernel)
    assert (out[:, :pad] == 7.0).all() and (out[:, pad + H * dv:] == 7.0).all()
    got, at = [], 0
    for s, r in slot_rows:
        got.append(out[at:at + r.shape[0], pad:pad + H * dv].cpu())
        at += r.shape[0]
        cache.advance(s, cache.length(s) + r.shape[0])
    return got


@pytest.mark.parametrize("H,G,d,dv,taps", [
    (1, 1, 8, 8, 4), (6, 2, 16, 24, 3), (2, 2, 17, 33, 2), (3, 1, 32, 16, 1), (4, 4, 64, 64, 4), (2, 1, 128, 128, 4), (1, 1, 100, 70, 9),
    (2, 1, 200, 36, 5), (1, 1, 300, 20, 4), (3, 3, 5, 130, 6)])
def test_the_gated_delta_rule_in_every_cut(H, G, d, dv, taps):
    T = 150
    for seed, keys, decays in ((1, "random", "mixed"), (2, "repeated", "slow"), (3, "random", "slow")):
        case, ref = delta_case(H, G, d, dv, taps, T, seed, keys, decays)
        cuts_list = ([T], [1] * T, [1, 2, 15, 16, 17, 33, 1, 1, 48, 16], [2] * 75, [130] + [1] * 20) if seed == 1 else ([T], [100] + [1] * 50)
        for cpt in (0, 2, 4):
            ops.force_gated_delta_columns(cpt)
            try:
                for cuts in cuts_list if cpt == 0 else ([T],):
                    for kernel in ("auto", "chunks") if 1 in cuts else ("auto",):
                        cache = delta_cache(H, G, d, dv, taps, 2)
                        s, outs, at = cache.open(), [], 0
                        for n in cuts:
                            outs += run_delta(case, cache, [(s, case["proj"][at:at + n])], kernel)
                            at += n
                        assert rel_err(torch.cat(outs), ref) < 2e-5, (keys, decays, cpt, cuts[:3], kernel)
            finally:
                ops.force_gated_delta_columns(0)
    got = run_delta(case, *(lambda c: (c, [(c.open(), case["proj"])]))(delta_cache(H, G, d, dv, taps, 1)), scale=-0.75, dtype=torch.bfloat16)
    assert rel_err(got[0], -0.75 * ref) < 1e-2


def test_the_gated_delta_rule_over_unequal_sequences_and_used_slots():
    H, G, d, dv, taps = 4, 2, 24, 20, 4
    cases = [delta_case(H, G, d, dv, taps, n, 10 + n) for n in (1, 50, 16, 77, 33)]
    base = cases[0][0]
    for c, _ in cases:                                   # one mixer's weights for all
        for name in ("conv", "a_log", "dt", "norm"):
            c[name] = base[name]
    def ref_of(c):
        H, G, d, dv = c["sizes"]
        T, C, x = c["proj"].shape[0], 2 * G * d + H * dv, c["proj"].double()
        act = torch.nn.functional.silu(ps.short_conv(x[:, c["q_off"]:c["q_off"] + C], base["conv"].double().cpu()))
        q, k = ps.unit(act[:, :G * d].view(T, G, d)) * d ** -0.5, ps.unit(act[:, G * d:2 * G * d].view(T, G, d))
        soft = torch.nn.functional.softplus(x[:, c["a_off"]:c["a_off"] + H] + base["dt"].double().cpu(), threshold=200.0)
        raw = ps.gated_delta_rule(q, k, act[:, 2 * G * d:].view(T, H, dv), torch.exp(-torch.exp(base["a_log"].double().cpu()) * soft),
                                  torch.sigmoid(x[:, c["b_off"]:c["b_off"] + H]))
        o = ps.rms(raw, 1e-4) * base["norm"].double().cpu() * torch.nn.functional.silu(x[:, c["g_off"]:c["g_off"] + H * dv]).view(T, H, dv)
        return o.reshape(T, H * dv)
    refs = [ref_of(c) for c, _ in cases]
    cache = delta_cache(H, G, d, dv, taps, 5)
    for _ in range(2):                                   # the second time in the slots of the first
        slots = [cache.open() for _ in cases]
        outs, fed = [[] for _ in cases], [0] * len(cases)
        for portion in ((1, 20, 16, 40, 1), (0, 1, 0, 1, 1), (0, 1, 0, 1, 1), (0, 28, 0, 1, 2), (0, 0, 0, 34, 28)):
            step = [(i, n) for i, n in enumerate(portion) if n]
            got = run_delta(base, cache, [(slots[i], cases[i][0]["proj"][fed[i]:fed[i] + n]) for i, n in step])
            for (i, n), o in zip(step, got):
                outs[i].append(o)
                fed[i] += n
        assert fed == [c["proj"].shape[0] for c, _ in cases]
        for o, r in zip(outs, refs):
            assert rel_err(torch.cat(o), r) < 2e-5
        for s in reversed(slots):
            cache.close(s)
    cache.check()


@pytest.mark.parametrize("rows,width", [(1, 8), (7, 44), (5, 63), (40, 1000), (3, 4096), (600, 2048), (9, 5000), (2, 9000)])
def test_two_norms_of_one_row(rows, width):
    g = torch.Generator().manual_seed(rows + width)
    x, w1, w2, v = (torch.randn(n, generator=g) + 0.2 for n in ((rows, width), (width,), (width,), (width,)))
    for wd in (torch.float32, torch.bfloat16):
        a, b, vec = w1.to(wd).cuda(), w2.to(wd).cuda(), v.to(wd).cuda()
        for od in (torch.float32, torch.bfloat16):
            o1, o2 = (torch.empty(rows, width, device="cuda", dtype=od) for _ in range(2))
            ops.rmsnorm_pair(x.cuda(), a, b, 1e-3, o1, o2)
            for o, w in ((o1, a), (o2, b)):              # the two norms as kernels of their own, to the bit
                assert torch.equal(o, ops.rmsnorm(x.cuda(), w, 1e-3, torch.empty_like(o)))
            tol = 1e-5 if od == torch.float32 else 5e-3
            assert rel_err(o2, ps.rms(x.double(), 1e-3) * b.double().cpu()) < tol
            # riding on a vector that joins the stream
            out = ops.stream_add(x.cuda(), None, vec, torch.empty(rows, width, device="cuda"), (a, 1e-3, o1, b, o2))
            joined = x.double() + vec.double().cpu()
            assert rel_err(out, joined) < 1e-6
            assert rel_err(o1, ps.rms(joined, 1e-3) * a.double().cpu()) < tol and rel_err(o2, ps.rms(joined, 1e-3) * b.double().cpu()) < tol


@pytest.mark.parametrize("M,N,K", [(1, 64, 40), (8, 2048, 4096), (20, 3584, 2048), (64, 2048, 8192), (130, 512, 256), (3, 44, 132)])
def test_two_norms_ride_on_a_product(M, N, K):
    g = torch.Generator().manual_seed(M + N)
    a, w = torch.randn(M, K, generator=g).bfloat16().cuda(), (torch.randn(N, K, generator=g) * K ** -0.5).bfloat16().cuda()
    x, w1, w2 = torch.randn(M, N, generator=g).cuda(), torch.randn(N, generator=g).bfloat16().cuda(), torch.randn(N, generator=g).bfloat16().cuda()
    ref = x.double() + a.double() @ w.double().T
    n1, n2 = (torch.empty(M, N, device="cuda", dtype=torch.bfloat16) for _ in range(2))
    out = ops.linear(a, w, torch.empty(M, N, device="cuda"), ops.EPI_RESIDUAL, residual=x, norm=(w1, 1e-4, n1, w2, n2))
    ref = ref.cpu()
    assert rel_err(out, ref) < 1e-5
    for n, wt in ((n1, w1), (n2, w2)):
        assert rel_err(n, ps.rms(ref, 1e-4) * wt.double().cpu()) < 5e-3
    ops.check_status()


@pytest.mark.parametrize("vocab,width", [(50, 8), (97, 44), (31, 63), (40, 1024), (11, 5000)])
def test_embedding_rows_are_normed(vocab, width):
    g = torch.Generator().manual_seed(width)
    table, w = torch.randn(vocab, width, generator=g), torch.randn(width, generator=g)
    toks = torch.randint(0, vocab, (37,), generator=g).int()
    for td in (torch.float32, torch.bfloat16):
        for scale in (1.0, 2.5):
            out = ops.embed_norm(toks.cuda(), table.to(td).cuda(), w.to(td).cuda(), 1e-2, torch.empty(37, width, device="cuda"), scale)
            assert rel_err(out, ps.rms(table.to(td).double()[toks.long()] * scale, 1e-2) * w.to(td).double()) < 2e-6
    toks[3] = vocab
    out = ops.embed_norm(toks.cuda(), table.cuda(), w.cuda(), 1e-2, torch.empty(37, width, device="cuda"))
    assert out[3].isnan().all() and not out[:3].isnan().any() and not out[4:].isnan().any()


@pytest.mark.parametrize("rows,H,hd,vdim", [(1, 1, 16, 16), (5, 3, 32, 20), (40, 4, 64, 64), (7, 2, 48, 33), (300, 8, 128, 80)])
def test_every_value_of_a_head_has_its_gate(rows, H, hd, vdim):
    g = torch.Generator().manual_seed(rows + hd)
    x, proj = torch.randn(rows, H * hd, generator=g), torch.randn(rows, H * vdim + 12, generator=g) * 3
    for dt, tol in ((torch.float32, 2e-6), (torch.bfloat16, 8e-3)):
        xd = x.to(dt)
        v = xd.double().view(rows, H, hd)[..., :vdim].reshape(rows, H * vdim)
        for off, out_off, wide in ((4, 0, 0), (3, 8, 12), (8, 5, 7)):
            for scale in (1.0, -0.6):
                out = torch.zeros(rows, H * vdim + wide, device="cuda", dtype=dt)
                ops.attn_gate(xd.cuda(), out, H, hd, vdim, (proj.cuda(), off), scale, out_off)
                ref = v * torch.sigmoid(proj[:, off:off + H * vdim].double()) * scale
                assert rel_err(out[:, out_off:out_off + H * vdim], ref) < tol
                assert not out[:, :out_off].any() and not out[:, out_off + H * vdim:].any()
        out = torch.zeros(rows, H * vdim, device="cuda", dtype=dt)
        assert rel_err(ops.attn_gate(xd.cuda(), out, H, hd, vdim), v) < 1e-6


@pytest.mark.parametrize("experts,top,ff,width,rows", [(5, 2, 24, 48, 9), (3, 1, 9, 44, 40), (1, 1, 16, 16, 3), (4, 4, 64, 128, 300), (12, 3, 40, 64, 1000)])
def test_experts_by_token(experts, top, ff, width, rows):
    g = torch.Generator().manual_seed(experts + rows)
    vocab = 30
    table = torch.stack([torch.randperm(experts, generator=g)[:top] for _ in range(vocab)]).int()
    toks = torch.randint(0, vocab, (rows,), generator=g).int()
    for dt, tol in ((torch.float32, 1e-5), (torch.bfloat16, 2e-2)):
        h, up = torch.randn(rows, width, generator=g).to(dt), (torch.randn(experts, ff, width, generator=g) * width ** -0.5).to(dt)
        down, x = (torch.randn(experts, width, ff, generator=g) * ff ** -0.5).to(dt), torch.randn(rows, width, generator=g)
        W = {"table": table, **{f"e{j}.up": up[j].double() for j in range(experts)}, **{f"e{j}.down": down[j].double() for j in range(experts)}}
        ref = ps.experts_by_token(h.double(), W, "", toks.long())
        ids, order, meta = ops.moe_group_by_token(toks.cuda(), table.cuda(), experts, dt, ff, width)
        assert torch.equal(ids.cpu(), table[toks.long()])
        got = x.cuda()
        ops.moe_relu2_join(h.cuda(), ids, 1.0 / top, up.cuda(), down.cuda(), got, grouped=(order, meta))
        assert rel_err(got.cpu() - x, ref) < tol
        again = ops.moe_relu2_join(h.cuda(), ids, torch.full((rows, top), 1.0 / top, device="cuda"), up.cuda(), down.cuda(), x.cuda())
        assert torch.equal(got, again)                  # as with a router's ids and weights


# ------------------------------------------------------------------ mechanisms alone: one-layer models
ONE_LAYER = {
    "delta": layer(delta(4, 2, 16, 24)),
    "delta, one tap": layer(delta(2, 1, 32, 8, conv=1)),
    "delta, twelve taps": layer(delta(2, 2, 16, 16, conv=12)),
    "delta, odd sizes": layer(delta(3, 1, 7, 5, conv=3)),
    "parallel": layer(parallel(attention(4, 2, 16, 24, 9, dims=8), delta(2, 1, 16, 16))),
    "parallel, every earlier key": layer(parallel(attention(2, 1, 32, 32, 0), delta(2, 2, 8, 12, conv=2), 0.5, 2.0)),
    "parallel, a window of one": layer(parallel(attention(2, 2, 16, 8, 1), delta(1, 1, 16, 16), -1.0, 0.3)),
    "parallel, odd sizes": layer(parallel(attention(3, 1, 10, 7, 20, dims=6), delta(3, 3, 9, 11), 1.1, 0.7)),
    "parallel, a head size beyond the tensor-core kernels": layer(parallel(attention(1, 1, 272, 16, 25), delta(1, 1, 8, 8))),
    "dense feed-forward": layer(delta(1, 1, 16, 16), dense(56)),
    "dense feed-forward, odd size": layer(delta(1, 1, 16, 16), dense(29)),
    "experts": layer(delta(1, 1, 16, 16), moe(5, 3, 24)),
    "one expert": layer(delta(1, 1, 16, 16), moe(1, 1, 11)),
    "parallel and experts": layer(parallel(attention(2, 1, 64, 64, 33), delta(2, 1, 64, 64)), moe(4, 2, 16)),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(ONE_LAYER))
def test_each_mechanism_in_a_model_of_its_own(tmp_path, name, dtype):
    loop = (0, 1, 2) if len(name) % 2 else None
    cfg, tensors = write_model(tmp_path / "one", model(90, 48, [ONE_LAYER[name]], loop=loop), seed=len(name))
    toks = tokens(cfg, 75, 9)
    ref = ps.forward(cfg, tensors, toks)
    engine = sb.Engine(sb.load_model(tmp_path / "one", dtype=dtype), max_tokens=512)
    for cuts in ([75], [70, 1, 1, 1, 1, 1], [3, 2, 61, 9], [2] * 37 + [1]):
        assert model_err(run_cuts(engine, toks, cuts), ref, dtype) < TOL[dtype], cuts[:4]


def test_the_stream_after_every_layer(folders, engines):
    for name in CONFIGS:
        _, cfg, tensors = folders[name]
        toks, streams = tokens(cfg, 50, 3), []
        ps.forward(cfg, tensors, toks, streams=streams)
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
        assert len(seen) == len(streams) == len(ps.run_order(cfg))
        for got, ref in zip(seen, streams):
            assert rel_err(got, ref) < 1e-5


@pytest.mark.parametrize("dtype", DTYPES)
def test_sides_that_do_not_share_their_products_give_the_same_sum(tmp_path, dtype):
    """The weighted sum of two mixers that stay closed: each runs by itself and joins by a row kernel."""
    cfg, tensors = write_model(tmp_path / "m", model(60, 32, [layer(parallel(attention(2, 1, 16, 24, 9), delta(2, 1, 16, 8), 1.4, -0.6), dense(24))]), seed=2)
    toks = tokens(cfg, 40, 1)
    ref = ps.forward(cfg, tensors, toks)
    from sonicboom_b200.parts.window_attention import WindowAttention
    opens = WindowAttention.input_matrix
    shared = sb.Engine(sb.load_model(tmp_path / "m", dtype=dtype), max_tokens=256)
    try:
        WindowAttention.input_matrix = lambda self: None
        closed = sb.Engine(sb.load_model(tmp_path / "m", dtype=dtype), max_tokens=256)
    finally:
        WindowAttention.input_matrix = opens
    assert shared.model.blocks[0].mixer.w_in is not None and closed.model.blocks[0].mixer.w_in is None
    for e in (shared, closed):
        for cuts in ([40], [30] + [1] * 10):
            assert rel_err(run_cuts(e, toks, cuts), ref) < TOL[dtype]


# ------------------------------------------------------------------ whole models
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_decoding_and_portions(folders, engines, name, dtype):
    toks, ref = reference(folders, name, 171, 5)
    engine = engines(name, dtype)
    whole = run_cuts(engine, toks, [171])
    assert model_err(whole, ref, dtype) < TOL[dtype]
    # the first tokens of a sequence one by one, then the rest; most of it at once, then one by one over two page
    # borders (64, 128) and every window's edge; portions down to two tokens; chunks of the scan cut everywhere
    for cuts in ([1, 1, 1, 168], [40] + [1] * 131, [2, 3, 62, 2, 59, 7, 17, 19], [64, 64, 43], [170, 1], [69, 2, 100], [16, 15, 17, 123]):
        got = run_cuts(engine, toks, cuts)
        assert model_err(got, ref, dtype) < TOL[dtype], cuts
        if dtype == "float32":
            assert rel_err(got, whole) < 2e-5, cuts       # rounding: few rows run other kernels
    engine.cache.check()
    assert engine.free_pages() == engine.cache.n_pages


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_unequal_batch_equals_each_alone_and_slots_are_reused(folders, engines, name, dtype):
    from gpu_util import batch_unequal
    reqs, refs = zip(*[reference(folders, name, n, 10 + n) for n in (1, 70, 131, 23)])
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
            assert rel_err(o, a) < 2e-5
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
    """Large score scales and slow decays, so that a few keys carry a row: a window one key off, a lost tap, a lost
    write of long ago or a pass without its vector moves the logits by a large multiple of the tolerance."""
    return model(80, 48, [
        layer(parallel(attention(2, 1, 16, 16, 13, scale=1.2), delta(2, 1, 16, 16, conv=3), 1.5, 0.8)),
        layer(delta(4, 2, 32, 16), moe(4, 2, 16)),
        layer(parallel(attention(2, 2, 64, 64, 100, dims=32, scale=0.4), delta(2, 2, 8, 8, conv=2), 1.2, 1.2), dense(32)),
    ], loop=(0, 2, 2), cap=0.0)


def sharpen(t):
    for n in t:
        if n.endswith(".o"):
            t[n] *= 2.0
        if n.endswith("A_log"):
            t[n][:] = -7.0                             # every head remembers for long


@pytest.mark.parametrize("dtype", DTYPES)
def test_window_edges_taps_far_writes_and_passes_show(tmp_path, dtype):
    cfg, tensors = write_model(tmp_path / "w", sharp_model(), seed=9, edit=sharpen)
    toks = tokens(cfg, 420, 21)
    ref = ps.forward(cfg, tensors, toks)
    shows = 100 * TOL["float32"]

    def other(edit_cfg=None, edit_tensors=None, seq=toks):
        c, t = json.loads(json.dumps(cfg)), {n: v.clone() for n, v in tensors.items()}
        if edit_cfg:
            edit_cfg(c)
        if edit_tensors:
            edit_tensors(t)
        return ps.forward(c, t, seq)
    for which in (0, 2):
        for by in (1, -1):
            size = cfg["layers"][which]["mixer"]["left"]["mask"]["size"] + by
            got = other(lambda c: c["layers"][which]["mixer"]["left"]["mask"].update(size=size))
            assert rel_err(got[100:], ref[100:]) > shows, (which, by)
    for name in [n for n in tensors if n.endswith(".conv")]:
        assert rel_err(other(edit_tensors=lambda t: t[name][:, 0].zero_()), ref) > shows, name        # the oldest tap lost
    for name in ("loop.step", "embed.norm", "l1.norm2"):
        assert rel_err(other(edit_tensors=lambda t: t[name][-1].mul_(0.5)), ref) > shows, name
    assert rel_err(other(edit_tensors=lambda t: t["l1.mlp.table"].copy_((t["l1.mlp.table"] + 1) % 4)), ref) > shows
    far = list(toks)
    far[3] = (toks[3] + 1) % cfg["vocab"]              # outside every window: only the state carries it
    assert rel_err(other(seq=far)[400:], ref[400:]) > shows
    engine = sb.Engine(sb.load_model(tmp_path / "w", dtype=dtype), max_tokens=1024)
    tol = TOL[dtype] if dtype == "float32" else 0.15   # scores of a large scale: bfloat16 keys move the weights
    for cuts in ([420], [380] + [1] * 40, [12, 2, 50, 356], [13] + [1] * 120 + [287], [5, 200, 215], [99, 2, 99, 2, 218]):
        assert rel_err(run_cuts(engine, toks, cuts), ref) < tol, cuts[:4]


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_gives_pages_back(folders, engines, dtype):
    """Six hundred tokens one by one: the window leaves pages behind, the state goes on."""
    toks, ref = reference(folders, "B", 600, 77)
    engine = engines("B", dtype, max_tokens=704)
    s = engine.open()
    engine.step([(s, toks[:5], [])])
    rows = []
    for i in range(5, 600):
        lg = engine.step([(s, [toks[i]], [0] if i % 7 == 0 or i > 590 else [])])
        if lg is not None:
            rows.append((i, lg.float().cpu()[0]))
    assert all(sum(p >= 0 for p in engine.cache.page_list(s, g)) <= 3 for g in range(len(engine.cache.groups)))
    engine.close(s)
    assert rel_err(torch.stack([r for _, r in rows]), ref[[i for i, _ in rows]]) < TOL[dtype]
    engine.cache.check()
    assert engine.free_pages() == engine.cache.n_pages


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_greedy_generation_through_the_entry_point(folders, name, dtype):
    """`llm.generate_batch`: the scheduler's batches, the captured decode step with the recurrences' state and
    rings in it, and slots given to the next batch."""
    d, cfg, tensors = folders[name]
    m = llm.model_load(d, dtype=dtype)
    assert m.arch == "Sipilorn" and m.vocab_size == cfg["vocab"]
    prompts = [tokens(cfg, n, 30 + n) for n in (3, 66, 20, 1)]
    n_new = 12
    outs = llm.generate_batch(m, prompts, max_tokens=n_new)
    for p, o in zip(prompts, outs):
        seq = list(p)
        for i, t in enumerate(o):
            logits = ps.forward(cfg, tensors, seq)[-1]
            best = int(torch.argmax(logits))
            if t != best:
                top2 = torch.topk(logits, 2).values
                margin = float(top2[0] - top2[1]) / float(logits.abs().max())
                assert dtype == "bfloat16" and margin < 2 * TOL[dtype], (i, o, margin)
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
    (a, ra), (b, rb) = reference(folders, "B", 75, 1), reference(folders, "B", 30, 2)
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
    """`python -m sonicboom_b200 generate` on a Sipilorn folder: greedy tokens as the plain implementation's."""
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
    want = []
    for p in prompts:
        seq = list(p)
        for _ in range(6):
            seq.append(int(torch.argmax(ps.forward(cfg, tensors, seq)[-1])))
        want.append(seq[len(p):])
    assert got == want


def test_a_random_model_on_the_device_equals_its_folder(tmp_path):
    """Weights made on the device and the folder written from the same seed, expert tables included."""
    from sonicboom_b200 import write_random_model
    cfg = CONFIGS["A"]
    write_random_model(tmp_path / "m", cfg, seed=11, std=0.05)
    a, b = sb.load_model(tmp_path / "m", dtype="bfloat16"), sb.random_model(cfg, seed=11, dtype="bfloat16", std=0.05)
    assert torch.equal(a.blocks[0].feed_forward.table, b.blocks[0].feed_forward.table) and bool(a.blocks[0].feed_forward.table.any())
    toks = tokens(cfg, 30, 4)
    x, y = (run_cuts(sb.Engine(m, max_tokens=256), toks, [20] + [1] * 10) for m in (a, b))
    assert torch.equal(x, y)
