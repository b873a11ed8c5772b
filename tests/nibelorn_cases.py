"""Small Nibelorn models for the tests: configurations as config.json would hold them, and weights under which attention
is far from uniform (with plain random weights a lost key would drown among the others)."""
from __future__ import annotations

import json

import torch


def latent(heads, dim, rot_dim, vdim, kv_rank, base=500.0, gain=1.0):
    return {"type": "latent_attention", "mlp": {"kind": "dense", "ff": 3 * vdim + 8},
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                      "scale": gain * (dim + rot_dim) ** -0.5, "rot": {"base": base, "dims": rot_dim}}}


def differential(heads, kv_heads, dim, vdim, diff=0.3, cap=15.0, coef=0.4, every=20, gain=1.0):
    return {"type": "attention", "mlp": {"kind": "dense", "ff": 2 * vdim + 24},
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": gain * dim ** -0.5, "diff": diff,
                      "softcap": cap, "q_temp": {"coef": coef, "every": every}}}


def borrowed(layers, j):
    return dict(layers[j], weights_of=j)


def config(width, vocab, layers, eps=1e-5):
    return {"architecture": "Nibelorn", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers}


def case(name):
    """name -> config.json as a dict.  mixed: both mixers, borrowed weights out of order, a layer without feed-forward; wide:
    sizes the tensor-core prefill kernels take; odd: rows that do not start on 16 bytes; thin: heads of one, ratios of one."""
    if name == "mixed":
        layers = [differential(6, 2, 16, 24), latent(3, 24, 8, 40, 56)]
        layers += [dict(differential(4, 4, 8, 16, diff=0.7, cap=4.0, coef=1.1, every=3), mlp=None)]
        layers += [borrowed(layers, 1), borrowed(layers, 0), borrowed(layers, 2)]
        return config(104, 211, layers, eps=1e-4)
    if name == "wide":
        layers = [latent(4, 64, 32, 72, 96, base=1e4), differential(8, 2, 40, 96, every=64)]
        layers += [borrowed(layers, 0), latent(2, 128, 64, 128, 160)]
        return config(192, 320, layers)
    if name == "odd":
        layers = [latent(3, 10, 6, 7, 33), differential(3, 1, 5, 9), dict(latent(1, 3, 2, 5, 11), mlp=None)]
        return config(50, 101, layers + [borrowed(layers, 0)])
    if name == "thin":
        layers = [differential(1, 1, 8, 8, every=1), latent(1, 8, 8, 8, 8)]
        return config(32, 64, layers + [borrowed(layers, 1)])
    raise KeyError(name)


NAMES = ("mixed", "wide", "odd", "thin")


def weights(pkg, cfg_json, seed=0, gain=2.0):
    """Random checkpoint tensors; query projections scaled up so that single keys carry visible weight."""
    cfg = pkg.nibelorn.config_from_json(cfg_json)
    w = pkg.nibelorn.init_weights(cfg, seed)
    g = torch.Generator().manual_seed(seed + 1)
    for name in w:
        if name.endswith("mix.q"):
            w[name] = (w[name].float() * gain).to(torch.bfloat16)
        elif name.endswith(".alpha"):
            w[name] = (0.3 + 0.5 * torch.rand((), generator=g)).to(torch.bfloat16)
    return w


def write_model(folder, cfg_json, tensors):
    """config.json and model.safetensors, written by hand from the format's description."""
    codes = {torch.bfloat16: "BF16", torch.float32: "F32", torch.int32: "I32"}
    header, blobs, at = {"__metadata__": {"format": "pt"}}, [], 0
    for name, t in tensors.items():
        raw = t.contiguous().reshape(-1).view(torch.uint8).numpy().tobytes()
        header[name] = {"dtype": codes[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    text = json.dumps(header).encode()
    (folder / "model.safetensors").write_bytes(len(text).to_bytes(8, "little") + text + b"".join(blobs))
    (folder / "config.json").write_text(json.dumps(cfg_json))


def row_errors(got, want):
    """Root mean square over the vocabulary of the difference (mean taken off), relative to the spread of the logits."""
    d = got.double().cpu() - want.double()
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.double().std()


LIMIT = {torch.float32: 2e-5, torch.bfloat16: 6e-2}
