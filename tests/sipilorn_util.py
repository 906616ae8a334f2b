"""Small Sipilorn configurations for the tests, and model folders made from them.

The configurations differ from each other in every size and option: layer order, loops over several layers, over
one, and none, one to three heads per key head, key sizes that are and are not multiples of 4, value sizes smaller
and larger than the key size, one to nine taps, windows of one key, of a few, over a page border and none,
rotated prefixes and none, head sizes the tensor-memory attention kernels take (64) and others, scales of the two
sides that are negative and above one, layers without a feed-forward, dense feed-forwards whose size is and is not
a multiple of 8, one to three experts a token, a width that is no multiple of 8, with and without a logit cap."""
import json
from pathlib import Path

import torch


def delta(heads, kv_heads, dim, vdim, conv=4):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def attention(heads, kv_heads, dim, vdim, window, dims=None, base=10000.0, scale=None):
    a = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else dim ** -0.5,
         "rot": {"base": base, "dims": dim if dims is None else dims}}
    if window:
        a["mask"] = {"size": window}
    return a


def parallel(left, right, left_scale=0.8, right_scale=1.3):
    return {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def layer(mixer, mlp=None):
    return {"type": "parallel" if "left" in mixer else "delta", "mixer": mixer, "mlp": mlp}


def model(vocab, width, layers, loop=None, cap=20.0, eps=1e-5):
    d = {"architecture": "Sipilorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop is not None:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    if cap:
        d["logit_softcap"] = cap
    return d


CONFIGS = {
    # a loop over the middle two layers, run three times; three heads a key head; values wider than keys
    "A": model(211, 64, [
        layer(delta(6, 2, 16, 24), moe(5, 2, 24)),
        layer(parallel(attention(4, 2, 16, 24, 9, dims=8, scale=0.3), delta(2, 1, 24, 16, conv=2), 1.4, -0.6), dense(40)),
        layer(delta(3, 3, 12, 8, conv=6)),
        layer(delta(4, 2, 32, 48, conv=4), moe(3, 1, 16)),
    ], loop=(1, 3, 3)),
    # head size 64 (the tensor-memory kernels), a window over a page border; sizes that are no multiples of 4 or 8;
    # nine taps, one tap; a loop over one layer run once; no cap
    "B": model(150, 44, [
        layer(parallel(attention(6, 3, 64, 32, 70, base=3e5), delta(4, 4, 17, 33, conv=9), -0.7, 0.9), moe(4, 3, 9)),
        layer(delta(2, 1, 40, 64, conv=1), dense(30)),
        layer(parallel(attention(2, 1, 24, 40, 1, dims=0), delta(3, 1, 8, 6, conv=3), 1.0, 1.0)),
    ], loop=(0, 1, 1), cap=0.0, eps=1e-6),
    # no loop; every earlier key in sight
    "C": model(97, 40, [
        layer(parallel(attention(2, 2, 16, 16, 0, dims=4), delta(2, 2, 16, 16)), dense(24)),
        layer(delta(1, 1, 64, 128, conv=3), moe(2, 2, 16)),
    ], cap=7.0),
}
INIT = dict(std=0.1, bias_std=0.3, norm_std=0.2)


def write_model(path, cfg, seed, edit=None):
    """A model folder with seeded random weights; `edit(tensors)` may change them (float32 in,
    stored as bfloat16, tables as int32).  Returns (config as written, tensors as stored)."""
    import plain_model as pm
    from sonicboom_b200 import write_random_model
    from sonicboom_b200.weights.safetensors_io import write_safetensors
    path = Path(path)
    write_random_model(path, cfg, seed=seed, **INIT)
    _, tensors = pm.read_model_dir(path)
    for name in tensors:
        if name.endswith(".conv"):
            tensors[name] = tensors[name] * 3.0
            tensors[name][:, -1] += 1.0                   # taps that keep most of the newest value
        if name.endswith(".A_log"):
            tensors[name] = tensors[name] * 3.0 - 3.0     # decays from near one to short
            tensors[name][0] = -6.0                       # a head that remembers hundreds of tokens
        if name.endswith(".b") or name.endswith(".a"):
            tensors[name] = tensors[name] * 4.0
        if name == "loop.step":
            tensors[name] = tensors[name] * 2.0
    if edit is not None:
        edit(tensors)
    stored = {n: t.to(torch.int32 if n.endswith(".table") else torch.bfloat16) for n, t in tensors.items()}
    write_safetensors(path / "model.safetensors",
                      [(n, t.dtype, tuple(t.shape), (lambda t=t: t)) for n, t in stored.items()])
    (path / "config.json").write_text(json.dumps(cfg))
    return cfg, {n: t if n.endswith(".table") else t.float() for n, t in stored.items()}


def tokens(cfg, n, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()
