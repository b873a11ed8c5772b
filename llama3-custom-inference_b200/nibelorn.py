"""Nibelorn: a decoder whose layers mix latent attention and differential attention over a 32-bit residual stream.

Per layer: x += mixer(norm1(x)), then, unless the layer has no feed-forward, x += down(gelu(up(norm2(x)))); the norms
are dynamic tanh (tanh(alpha x) w + b).  A layer may borrow another layer's weights (`weights_of`); its cache is its
own.  Sizes and constants come from config.json or a tensor's shape.

Generation, requests, the cache and the CUDA graph of a decode step are `decode_loop.DecodeLoop`'s; this file holds the
configuration, the weight layout and one forward pass over the mixer kernels (mixers.py).  Matrix products are torch's
(cuBLAS), fused where inputs are shared: query and latent down-projection, or query, key, value and gate, are one.

Latent attention runs in two forms.  Decode and short portions keep the keys and values in the latent: the query is
multiplied into it (q_n W_uk), scores and the weighted sum run over the cached rows alone, and W_uv is applied to the
result.  Long portions expand the cached latents into per-head keys and values first (one product) and run ordinary
attention on the tensor cores.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn.functional as F

from . import mixers, rope_table
from .decode_loop import DecodeLoop, full_precision_products, nvtx_range

EXPAND_FROM = 128   # portions of at least this many tokens expand the latents (a query block of the tcgen05 kernel)


@dataclass(frozen=True)
class LatentAttention:
    heads: int
    dim: int        # unrotated query / key size per head
    rot_dim: int    # rotated size, its key part shared by the heads
    vdim: int
    kv_rank: int
    scale: float
    rot_base: float

    @property
    def planes(self) -> dict:
        return {"latent": (_round8(self.kv_rank + self.rot_dim),)}


@dataclass(frozen=True)
class DifferentialAttention:
    heads: int
    kv_heads: int
    dim: int        # per map
    vdim: int
    scale: float
    diff: float
    softcap: float = 0.0
    temp_coef: float = 0.0
    temp_every: float = 0.0

    @property
    def planes(self) -> dict:
        return {"k": (self.kv_heads, 2 * self.dim), "v": (self.kv_heads, self.vdim)}


@dataclass(frozen=True)
class Layer:
    mixer: object
    ff: Optional[int]      # feed-forward size, None: no feed-forward
    weights: int           # index of the layer that owns the tensors


@dataclass(frozen=True)
class NibelornConfig:
    vocab_size: int
    width: int
    eps: float
    layers: tuple


def _round8(n: int) -> int:
    return (n + 7) // 8 * 8


def _mixer_from_json(kind: str, m: dict):
    if kind == "latent_attention":
        rot = m["rot"]
        if rot["dims"] != m["rot_dim"]:
            raise ValueError("latent attention rotates the whole rotated part: rot.dims must equal rot_dim")
        return LatentAttention(heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"], kv_rank=m["kv_rank"],
                               scale=float(m["scale"]), rot_base=float(rot["base"]))
    if kind == "attention":
        temp = m.get("q_temp") or {"coef": 0.0, "every": 0.0}
        return DifferentialAttention(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"],
                                     scale=float(m["scale"]), diff=float(m["diff"]), softcap=float(m.get("softcap") or 0.0),
                                     temp_coef=float(temp["coef"]), temp_every=float(temp["every"]))
    raise ValueError(f"unknown mixer type {kind!r}")


def config_from_json(config: dict) -> NibelornConfig:
    entries = config["layers"]

    def owner(i):
        seen = set()
        while entries[i].get("weights_of") is not None:
            if i in seen:
                raise ValueError(f"layer {i}: weights_of goes in a circle")
            seen.add(i)
            i = entries[i]["weights_of"]
        return i

    layers = []
    for i, e in enumerate(entries):
        mlp = e.get("mlp")
        if mlp is not None and mlp["kind"] != "dense":
            raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
        layers.append(Layer(_mixer_from_json(e["type"], e["mixer"]), mlp["ff"] if mlp is not None else None, owner(i)))
    return NibelornConfig(vocab_size=config["vocab"], width=config["width"], eps=float(config["norm"]["eps"]), layers=tuple(layers))


def tensor_shapes(cfg: NibelornConfig) -> dict:
    """Name and shape of every tensor of a checkpoint of this configuration."""
    E = cfg.width
    out = {"embed": (cfg.vocab_size, E), "head": (cfg.vocab_size, E)}

    def norm(name):
        out.update({name: (E,), name + ".b": (E,), name + ".alpha": ()})

    norm("final.norm")
    for i, layer in enumerate(cfg.layers):
        if layer.weights != i:
            continue
        m, p = layer.mixer, f"l{i}."
        norm(p + "norm1")
        if isinstance(m, LatentAttention):
            sizes = {"q": (m.heads * (m.dim + m.rot_dim), E), "dkv": (m.kv_rank + m.rot_dim, E), "dkv.norm": (m.kv_rank,),
                     "uk": (m.heads * m.dim, m.kv_rank), "uv": (m.heads * m.vdim, m.kv_rank)}
        else:
            sizes = {"q": (m.heads * 2 * m.dim, E), "k": (m.kv_heads * 2 * m.dim, E), "v": (m.kv_heads * m.vdim, E),
                     "g": (m.heads, E), "lq1": (m.dim,), "lk1": (m.dim,), "lq2": (m.dim,), "lk2": (m.dim,)}
        sizes["o"] = (E, m.heads * m.vdim)
        out.update({p + "mix." + n: s for n, s in sizes.items()})
        if layer.ff is not None:
            norm(p + "norm2")
            out.update({p + "mlp.up": (layer.ff, E), p + "mlp.down": (E, layer.ff)})
    return out


def init_weights(cfg: NibelornConfig, seed: int = 42, device="cpu") -> dict:
    """Random bf16 checkpoint tensors: matrices ~ N(0, 1/in), norm weights near 1, alpha 0.5."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        if name.endswith(".alpha"):
            t = torch.full((), 0.5, device=device)
        elif name == "embed":
            t = torch.randn(shape, generator=g, device=device)
        elif len(shape) == 2:
            t = torch.randn(shape, generator=g, device=device) * shape[1] ** -0.5
        elif name.endswith("norm") or name.endswith("norm1") or name.endswith("norm2"):
            t = 1.0 + 0.1 * torch.randn(shape, generator=g, device=device)
        else:
            t = 0.1 * torch.randn(shape, generator=g, device=device)
        out[name] = t.to(torch.bfloat16)
    return out


class _Norm:
    """Weight and bias in fp32 on the device, alpha as a host number."""

    def __init__(self, tensors: dict, name: str, device):
        self.weight = tensors[name].to(device, torch.float32).contiguous()
        self.bias = tensors[name + ".b"].to(device, torch.float32).contiguous()
        self.alpha = float(tensors[name + ".alpha"].float())

    @property
    def args(self):
        return self.weight, self.bias, self.alpha


class _LayerWeights:
    """A layer's tensors in the form the forward pass takes them: projections of the same input stacked."""

    def __init__(self, tensors: dict, p: str, layer: Layer, device, dtype):
        def get(name):
            return tensors[p + name].to(device, dtype)

        m = layer.mixer
        self.norm1 = _Norm(tensors, p + "norm1", device)
        if isinstance(m, LatentAttention):
            self.proj = torch.cat([get("mix.q"), get("mix.dkv")])
            self.latent_norm = tensors[p + "mix.dkv.norm"].to(device, torch.float32).contiguous()
            self.up = torch.cat([get("mix.uk"), get("mix.uv")])                       # latent -> keys | values of all heads
            split = m.heads * m.dim
            self.uk = self.up[:split].view(m.heads, m.dim, m.kv_rank)
            self.uv = self.up[split:].view(m.heads, m.vdim, m.kv_rank)
        else:
            rows = [get("mix.q"), get("mix.k"), get("mix.v"), get("mix.g")]
            pad = -sum(r.shape[0] for r in rows) % 8                                  # rows of the product start on 16 bytes
            self.proj = torch.cat(rows + [rows[0].new_zeros(pad, rows[0].shape[1])])

            def dot(a, b):
                return float((tensors[p + "mix." + a].double() * tensors[p + "mix." + b].double()).sum().exp())

            self.lambda_ = dot("lq1", "lk1") - dot("lq2", "lk2") + m.diff
        self.o = get("mix.o")
        if layer.ff is not None:
            self.norm2 = _Norm(tensors, p + "norm2", device)
            self.ff_up, self.ff_down = get("mlp.up"), get("mlp.down")


class NibelornDecoder(DecodeLoop):
    """The decoder on one GPU with a static cache; dtype bfloat16 (the serving precision) or float32."""

    def __init__(self, ext, cfg: NibelornConfig, device, max_batch: int, max_len: int, seed: int = 42,
                 weights: Optional[dict] = None, dtype=torch.bfloat16):
        super().__init__(ext, device, [layer.mixer.planes for layer in cfg.layers], max_batch, max_len, dtype)
        self.cfg = cfg
        if weights is None:
            weights = init_weights(cfg, seed)
        for name, shape in tensor_shapes(cfg).items():
            if tuple(weights[name].shape) != shape:
                raise ValueError(f"tensor {name} has shape {tuple(weights[name].shape)}, the configuration says {shape}")
        dev = self.device
        self.embed, self.head = weights["embed"].to(dev, dtype), weights["head"].to(dev, dtype)
        self.final_norm = _Norm(weights, "final.norm", dev)
        own = {i: _LayerWeights(weights, f"l{i}.", layer, dev, dtype) for i, layer in enumerate(cfg.layers) if layer.weights == i}
        self.w = [own[layer.weights] for layer in cfg.layers]
        self._tables = {}
        for layer in cfg.layers:
            m = layer.mixer
            if isinstance(m, LatentAttention) and (m.rot_dim, m.rot_base) not in self._tables:
                self._tables[m.rot_dim, m.rot_base] = rope_table.rotation_table(m.rot_dim, max_len, m.rot_base).to(dev)

    # ---- mixers: h [B, T, width] -> heads' outputs [B, T, heads * vdim] --------------------------------------
    def _latent(self, l: int, h, positions, slots: slice, start_pos: int):
        m, w = self.cfg.layers[l].mixer, self.w[l]
        B, T, _ = h.shape
        H, D, R, C, V = m.heads, m.dim, m.rot_dim, m.kv_rank, m.vdim
        cache = self.cache.layers[l]["latent"][slots]
        qd = F.linear(h, w.proj)
        mixers.latent_cache(qd, self._tables[R, m.rot_base], w.latent_norm, self.cfg.eps, cache, positions, H, D, R, C)
        q = qd[..., :H * (D + R)].view(B, T, H, D + R)
        out = torch.empty(B, T, H, V, dtype=h.dtype, device=h.device)
        if self._expands(m, T):
            S = start_pos + T
            kv = F.linear(cache[:, :S, :C], w.up)
            k_rot = cache[:, :S, None, C:C + R].expand(B, S, H, R)
            mixers.attention(q[..., :D], kv[..., :H * D].view(B, S, H, D), kv[..., H * D:].view(B, S, H, V), out, positions,
                             qb=q[..., D:], kb=k_rot, scale=m.scale, start_pos=start_pos, variant=mixers.TC)
        else:
            q_lat = torch.bmm(q[..., :D].reshape(B * T, H, D).transpose(0, 1), w.uk)               # [H, B * T, C]
            o_lat = torch.empty_like(q_lat)
            mixers.attention(q_lat.view(H, B, T, C).permute(1, 2, 0, 3), cache[:, :, None, :C], cache[:, :, None, :C],
                             o_lat.view(H, B, T, C).permute(1, 2, 0, 3), positions, qb=q[..., D:],
                             kb=cache[:, :, None, C:C + R], scale=m.scale, start_pos=start_pos)
            torch.bmm(o_lat, w.uv.transpose(1, 2), out=out.view(B * T, H, V).transpose(0, 1))
        return out.view(B, T, H * V)

    def _expands(self, m: LatentAttention, T: int) -> bool:
        return (self.dtype == torch.bfloat16 and T >= EXPAND_FROM and mixers.tc_sizes_ok(m.dim, m.rot_dim, m.vdim) and
                m.kv_rank % 8 == 0)

    def _differential(self, l: int, h, positions, slots: slice, start_pos: int):
        m, w = self.cfg.layers[l].mixer, self.w[l]
        B, T, _ = h.shape
        H, G, D, V = m.heads, m.kv_heads, m.dim, m.vdim
        planes = self.cache.layers[l]
        k, v = planes["k"][slots], planes["v"][slots]
        p = F.linear(h, w.proj)
        at_k, at_v, at_g = 2 * H * D, 2 * (H + G) * D, 2 * (H + G) * D + G * V
        mixers.kv_cache_write(p, at_k, at_v, k, v, positions)
        out = torch.empty(B, T, H, V, dtype=h.dtype, device=h.device)
        mixers.attention(p[..., :at_k].view(B, T, H, 2 * D), k, v, out, positions, maps=2, scale=m.scale, softcap=m.softcap,
                         temp_coef=m.temp_coef, temp_every=m.temp_every, gate=p[..., at_g:at_g + H], lambda_=w.lambda_,
                         post=1.0 - m.diff, eps=self.cfg.eps, start_pos=start_pos)
        return out.view(B, T, H * V)

    # ---- one forward pass over T new tokens per sequence ------------------------------------------------------
    def forward(self, tokens: torch.Tensor, positions: torch.Tensor, seq_lens: torch.Tensor, start_pos: int = 0,
                slots: Optional[slice] = None, want=None, keep: Optional[list] = None):
        """See DecodeLoop.forward; `keep` (a list) receives a copy of the residual stream after every layer."""
        layers = self.cfg.layers
        B, T = tokens.shape
        slots = slice(0, B) if slots is None else slots
        start_pos = start_pos if T > 1 else -1       # one token: positions live on the device alone (CUDA graph)
        with full_precision_products():
            x, h = mixers.embed_dyn_tanh(tokens, self.embed, *self.w[0].norm1.args)
            for l, layer in enumerate(layers):
                w = self.w[l]
                following = self.w[l + 1].norm1 if l + 1 < len(layers) else self.final_norm
                with nvtx_range("layer"):
                    mix = self._latent if isinstance(layer.mixer, LatentAttention) else self._differential
                    y = F.linear(mix(l, h, positions, slots, start_pos), w.o)
                    if layer.ff is not None:
                        h = mixers.add_dyn_tanh(y, x, *w.norm2.args)
                        y = F.linear(mixers.gelu_(F.linear(h, w.ff_up)), w.ff_down)
                    h = mixers.add_dyn_tanh(y, x, *following.args)
                    if keep is not None:
                        keep.append(x.clone())
            return self.logits(h, self.head, want)
