"""Small Rupotar models for the tests: configurations as config.json would hold them, and weights under which single keys, slow
decays and the experts' clamps show (with plain random weights a lost key or state would drown)."""
from __future__ import annotations

import torch

from tests.nibelorn_cases import LIMIT, row_errors, write_model  # noqa: F401


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def attention(heads, kv_heads, dim, vdim, size=None, keep=None, gain=1.0, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": gain * dim ** -0.5}
    if size is not None:
        m["mask"] = {"size": size, "keep_first": keep}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def delta(heads, kv_heads, dim, vdim, conv, mlp=None):
    return {"type": "channel_delta", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def wkv(heads, dim, mlp=None):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "mlp": mlp}


def config(width, vocab, layers, loop=None, eps=1e-5, scale=2.5):
    c = {"architecture": "Rupotar", "width": width, "vocab": vocab, "embedding": {"scale": scale}, "norm": {"eps": eps}, "layers": layers}
    if loop is not None:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def case(name, smooth=False):
    """`_case`, with `smooth` every expert of a token chosen: the model is then a smooth function of its weights, and bf16
    rounding cannot change which experts a token takes (and with it everything behind, through the recurrences)."""
    c = _case(name)
    for layer in c["layers"] if smooth else ():
        if layer["mlp"] is not None and layer["mlp"]["kind"] == "moe":
            layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
    return c


def _case(name):
    """name -> config.json as a dict.  mixed: every mixer and feed-forward, a loop in the middle, a layer without feed-forward;
    wide: sizes the tensor-core kernels take, a loop of one layer at the start; odd: rows that do not start on 16 bytes, no loop;
    thin: one head, one expert, one pass over all layers; order: recurrences first, an attention without a window last in the
    loop."""
    if name == "mixed":
        return config(104, 211, [attention(6, 2, 16, 24, 13, 5, mlp=dense(72)), delta(6, 3, 24, 16, 4, moe(6, 3, 40, 0.8)), wkv(3, 24),
                                 attention(4, 4, 8, 16, mlp=moe(5, 2, 24, 2.0))], loop=(1, 3, 2), eps=1e-4)
    if name == "wide":
        return config(256, 320, [attention(8, 2, 64, 96, 70, 3, mlp=moe(9, 2, 128, 0.7)), wkv(5, 64, dense(200)),
                                 delta(4, 4, 32, 64, 2, moe(4, 4, 64, 1.5)), attention(4, 1, 128, 128, 129, 130, mlp=dense(96))], loop=(0, 1, 3))
    if name == "odd":
        return config(50, 101, [attention(3, 1, 5, 9, 7, 2, mlp=moe(3, 3, 11, 0.5)), wkv(3, 7, dense(13)), delta(2, 1, 10, 6, 1, dense(9)),
                                delta(3, 3, 3, 5, 5, moe(7, 1, 5, 3.0))])
    if name == "thin":
        return config(32, 64, [wkv(1, 8, moe(1, 1, 8, 1.0)), delta(1, 1, 8, 8, 3), attention(1, 1, 8, 8, 1, 0, mlp=dense(8))], loop=(0, 3, 1))
    if name == "order":
        return config(72, 130, [delta(4, 2, 40, 48, 3, dense(40)), wkv(2, 40), attention(4, 2, 24, 16, mlp=moe(8, 2, 16, 1.0)),
                                wkv(4, 16, moe(2, 1, 32, 0.6))], loop=(0, 3, 2), scale=0.7)
    raise KeyError(name)


NAMES = ("mixed", "wide", "odd", "thin", "order")


def weights(pkg, cfg_json, seed=0, gain=1.5, rank=6):
    """Random checkpoint tensors, query norms scaled up, the decays of a wide range."""
    w = pkg.rupotar.init_weights(pkg.rupotar.config_from_json(cfg_json), seed, rank=rank)
    g = torch.Generator().manual_seed(seed + 1)
    for name in w:
        if name.endswith("q.norm"):
            w[name] = (w[name].float() * gain).to(torch.bfloat16)
        elif name.endswith((".A_log", ".w0")):
            w[name] = (4.0 * torch.rand(w[name].shape, generator=g) - 5.0).to(torch.bfloat16)
        elif name.endswith((".gate", ".up")):
            w[name] = (w[name].float() * 1.5).to(torch.bfloat16)
    return w
