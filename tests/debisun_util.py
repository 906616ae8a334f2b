"""Small Debisun configurations for the tests, and model folders made from them.

The configurations differ from each other in every size and option: layer order, value heads
narrower and wider than the keys, one to three key/value heads, chunks of one position, of a few, over a
page border and none, one to six convolution taps and no convolutions, bias tables of few and many rows
that end within and beyond a chunk, with and without a score cap, layers without a feed-forward, dense
feed-forwards whose size is and is not a multiple of 8, experts with no, one and several identity outputs,
one to four choices, with and without a shared expert, a width that is no multiple of 8, head sizes the
tensor-memory kernels take (64) and others, models with and without token inputs."""
import json
from pathlib import Path

import torch


def attention(heads, kv_heads, dim, vdim, chunk, bias, conv=4, softcap=6.0, scale=None):
    """`bias` = (rows of the table, distance its last row starts at); chunk 0, conv 0, softcap 0: none."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "bias_rows": bias[0], "bias_max": bias[1],
         "scale": scale if scale is not None else dim ** -0.5}
    if chunk:
        m["mask"] = {"size": chunk}
    if conv:
        m["conv"] = conv
    if softcap:
        m["softcap"] = softcap
    return m


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, identity=0, scale=None, shared=0):
    router = {"experts": experts, "top": top}
    if identity:
        router["identity"] = identity
    if scale is not None:
        router["scale"] = scale
    m = {"kind": "moe", "router": router, "expert": {"ff": ff}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def layer(mixer, mlp=None):
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def model(vocab, width, layers, side=12, eps=1e-5):
    d = {"architecture": "Debisun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if side:
        d["token_side"] = {"dim": side}
    return d


CONFIGS = {
    # values wider than keys, chunks of 9; chunks of one position and no feed-forward; no chunks, two taps;
    # six taps (more than the fused kernel takes) and a bias table that ends within the chunk
    "A": model(211, 64, [
        layer(attention(4, 2, 16, 24, 9, (8, 20), conv=3, softcap=5.0, scale=0.3),
              moe(5, 3, 24, identity=3, scale=1.7, shared=40)),
        layer(attention(2, 2, 32, 16, 1, (4, 6), conv=1)),
        layer(attention(3, 1, 16, 16, 0, (12, 40), conv=2, softcap=0.0), dense(40)),
        layer(attention(4, 4, 16, 16, 50, (6, 11), conv=6, softcap=2.0), moe(6, 1, 20, shared=16)),
    ], side=12),
    # head size 64 (the tensor-memory kernels) with three key/value heads, a chunk over a page border; a
    # width that is no multiple of 8; chunks of a page; one identity; no convolution and no cap
    "B": model(150, 44, [
        layer(attention(6, 3, 64, 32, 70, (32, 55), conv=4, softcap=20.0, scale=0.1), dense(30)),
        layer(attention(2, 1, 64, 64, 64, (16, 100), conv=5, softcap=9.0, scale=0.15), moe(3, 2, 9, identity=1, scale=0.8)),
        layer(attention(3, 3, 8, 8, 33, (2, 3), conv=0, softcap=0.0, scale=0.5), moe(4, 4, 16, identity=4, scale=2.2, shared=18)),
    ], side=5, eps=1e-6),
    # no token inputs
    "C": model(97, 40, [
        layer(attention(2, 1, 16, 16, 20, (10, 19), conv=4), moe(4, 2, 16, identity=2, scale=1.3, shared=8)),
        layer(attention(2, 2, 16, 8, 7, (4, 30), conv=3), dense(24)),
    ], side=0),
}
INIT = dict(std=0.1, bias_std=0.3, norm_std=0.2)


def write_model(path, cfg, seed, edit=None):
    """A model folder with seeded random weights; `edit(tensors)` may change them (float32 in,
    stored as bfloat16).  Returns (config as written, float32 tensors as stored)."""
    import plain_model as pm
    from sonicboom_b200 import write_random_model
    from sonicboom_b200.weights.safetensors_io import write_safetensors
    path = Path(path)
    write_random_model(path, cfg, seed=seed, **INIT)
    _, tensors = pm.read_model_dir(path)
    for name in tensors:
        if name.endswith(".router"):
            tensors[name] = tensors[name] * 3.0           # routers that prefer some experts clearly
        if name.endswith(".correction"):
            tensors[name] = tensors[name] * 0.2           # softmax scores are small: corrections beside them
        if name.endswith(".conv"):
            tensors[name] = tensors[name] * 3.0
            tensors[name][:, -1] += 1.0                   # taps that keep most of the newest value
        if name.endswith(".rel"):
            tensors[name] = tensors[name] * 3.0
    if edit is not None:
        edit(tensors)
    stored = {n: t.to(torch.bfloat16) for n, t in tensors.items()}
    write_safetensors(path / "model.safetensors",
                      [(n, t.dtype, tuple(t.shape), (lambda t=t: t)) for n, t in stored.items()])
    (path / "config.json").write_text(json.dumps(cfg))
    return cfg, {n: t.float() for n, t in stored.items()}


def tokens(cfg, n, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


ROUTER_MARGIN = 0.01
_CALM = {}


def calm_tokens(cfg, tensors, n, seed, key=None, margin=ROUTER_MARGIN):
    """`n` seeded random tokens at none of which a router's choice is a close call (the last chosen
    output's choice score is at least `margin` above the best one left out), so that rounding cannot send
    a token to other experts than the plain implementation does.  A position's routing depends on the
    tokens up to it only: the first close call's token is drawn again until none is left.  Returns
    (tokens, the plain implementation's logits)."""
    import plain_debisun as pd
    k = (key, n, seed, margin)
    if key is not None and k in _CALM:
        return _CALM[k]
    g = torch.Generator().manual_seed(seed)
    toks = torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()
    for _ in range(20 * n):
        gaps = []
        ref = pd.forward(cfg, tensors, toks, gaps=gaps)
        close = [t for t in range(n) if any(layer_gaps[t] < margin for layer_gaps in gaps)]
        if not close:
            break
        toks[close[0]] = int(torch.randint(0, cfg["vocab"], (1,), generator=g))
    else:
        raise AssertionError("no tokens without a close router call were found")
    if key is not None:
        _CALM[k] = (toks, ref)
    return toks, ref
