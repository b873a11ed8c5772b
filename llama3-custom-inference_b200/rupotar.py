"""Rupotar: a decoder whose layers mix windowed attention and two linear recurrences, with looped layers and experts.

Per layer run: x += norm1b(mixer(norm1(x))), then, unless the layer has no feed-forward, x += norm2b(ff(norm2(x))), over a
32-bit residual stream with layer norms.  A run of layers may be looped: its passes share the weights, each pass has its own
cache and state, and begins with x = W_in [x; embedding output] + step_t.  Mixers:
  attention      grouped queries, RMS norm over the whole query and key rows, a distance bias per head instead of positions, a
                 sliding window with kept first tokens, one added to the softmax's denominator
  channel_delta  gated delta rule with a decay per head and key channel, short convolutions on q, k, v
  wkv            time mixing with the token before and a data-dependent decay per channel, a bonus for the current token
Feed-forward: gated silu, or experts with a clamped activation.  Sizes and constants come from config.json or a tensor's shape.

Generation, requests, the cache and the CUDA graph of a decode step are `decode_loop.DecodeLoop`'s; this file holds the
configuration, the weight layout and one forward pass over the kernels (mixers.py).  Matrix products of one input are fused;
those of the experts are kernels of their own, the others torch's (cuBLAS).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn.functional as F

from . import mixers
from .decode_loop import DecodeLoop, full_precision_products, nvtx_range
from .kv_cache import State

POSITION_BASE = 10000.0     # sinusoidal positions
SLOPE_RANGE = 8.0           # head h of H takes 2^(-8 (h + 1) / H) off a score per position of distance
UNIT_EPS = 1e-6             # of the delta rule's unit vectors
EXPERT_ALPHA = 1.702        # g * sigmoid(alpha g)
MIXES = ("r", "k", "v", "g", "w")


@dataclass(frozen=True)
class Attention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int = 0         # 0: every earlier position
    keep_first: int = 0

    def planes(self, width: int) -> dict:
        return {"k": (self.kv_heads, self.dim), "v": (self.kv_heads, self.vdim)}

    def shapes(self, width: int) -> dict:
        q, k, v = self.heads * self.dim, self.kv_heads * self.dim, self.kv_heads * self.vdim
        return {"q": (q, width), "k": (k, width), "v": (v, width), "q.norm": (q,), "k.norm": (k,), "o": (width, self.heads * self.vdim)}


@dataclass(frozen=True)
class ChannelDelta:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int

    @property
    def channels(self) -> int:
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim

    def planes(self, width: int) -> dict:
        return {"state": State((self.heads, self.dim, self.vdim), torch.float32), "tail": State((self.taps - 1, self.channels))}

    def shapes(self, width: int) -> dict:
        qk, v, H = self.kv_heads * self.dim, self.heads * self.vdim, self.heads
        return {"q": (qk, width), "q.conv": (qk, self.taps), "k": (qk, width), "k.conv": (qk, self.taps), "v": (v, width),
                "v.conv": (v, self.taps), "b": (H, width), "A_log": (H,), "norm": (self.vdim,), "a1": (None, width),
                "a2": (H * self.dim, None), "dt_bias": (H * self.dim,), "g1": (None, width), "g2": (v, None), "o": (width, v)}


@dataclass(frozen=True)
class TimeMix:
    heads: int
    dim: int

    def planes(self, width: int) -> dict:
        return {"state": State((self.heads, self.dim, self.dim), torch.float32), "last": State((width,))}

    def shapes(self, width: int) -> dict:
        n = self.heads * self.dim
        out = {"mu." + s: (width,) for s in MIXES}
        out.update({s: (n, width) for s in "rkvg"})
        out.update({"w1": (None, width), "w2": (n, None), "w0": (n,), "u": (self.heads, self.dim), "norm": (n,), "o": (width, n)})
        return out


@dataclass(frozen=True)
class Dense:
    ff: int

    def shapes(self, width: int) -> dict:
        return {"gate": (self.ff, width), "up": (self.ff, width), "down": (width, self.ff)}


@dataclass(frozen=True)
class Experts:
    ff: int
    limit: float
    experts: int
    top: int

    def shapes(self, width: int) -> dict:
        out = {f"e{e}.{n}": s for e in range(self.experts) for n, s in Dense(self.ff).shapes(width).items()}
        return {**out, "router": (self.experts, width), "router.b": (self.experts,)}


@dataclass(frozen=True)
class Layer:
    mixer: object
    ff: object             # Dense, Experts or None


@dataclass(frozen=True)
class Loop:
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class Run:
    """One run of a layer: `step` is the number of the pass that it opens, None if it opens none."""
    layer: int
    step: Optional[int] = None


@dataclass(frozen=True)
class RupotarConfig:
    vocab_size: int
    width: int
    eps: float
    embed_scale: float
    layers: tuple
    loop: Optional[Loop] = None

    @property
    def runs(self) -> tuple:
        """Layer runs in the order of execution; each has its own cache."""
        n, loop = len(self.layers), self.loop
        if loop is None:
            return tuple(Run(i) for i in range(n))
        passes = [Run(i, t if i == loop.start else None) for t in range(loop.times) for i in range(loop.start, loop.stop)]
        return tuple([Run(i) for i in range(loop.start)] + passes + [Run(i) for i in range(loop.stop, n)])


def _mixer_from_json(kind: str, m: dict):
    if kind == "attention":
        mask = m.get("mask") or {}
        return Attention(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=float(m["scale"]),
                         window=mask.get("size") or 0, keep_first=mask.get("keep_first") or 0)
    if kind == "channel_delta":
        return ChannelDelta(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], taps=m["conv"])
    if kind == "wkv":
        return TimeMix(heads=m["heads"], dim=m["dim"])
    raise ValueError(f"unknown mixer type {kind!r}")


def _ff_from_json(mlp):
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return Dense(mlp["ff"])
    if mlp["kind"] == "moe":
        return Experts(ff=mlp["expert"]["ff"], limit=float(mlp["expert"]["limit"]), experts=mlp["router"]["experts"], top=mlp["router"]["top"])
    raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")


def config_from_json(config: dict) -> RupotarConfig:
    layers = tuple(Layer(_mixer_from_json(e["type"], e["mixer"]), _ff_from_json(e.get("mlp"))) for e in config["layers"])
    loop = config.get("loop")
    if loop is not None:
        loop = Loop(loop["start"], loop["stop"], loop["times"])
        if not 0 <= loop.start < loop.stop <= len(layers) or loop.times < 1:
            raise ValueError(f"loop {loop} does not fit {len(layers)} layers")
    return RupotarConfig(vocab_size=config["vocab"], width=config["width"], eps=float(config["norm"]["eps"]),
                         embed_scale=float(config["embedding"]["scale"]), layers=layers, loop=loop)


def tensor_shapes(cfg: RupotarConfig) -> dict:
    """Name and shape of every tensor of a checkpoint of this configuration; None: a low rank, the tensor's own choice."""
    E = cfg.width
    out = {"embed": (cfg.vocab_size, E), "head": (cfg.vocab_size, E)}

    def norm(name):
        out.update({name: (E,), name + ".b": (E,)})

    norm("final.norm")
    if cfg.loop is not None:
        out.update({"loop.in": (E, 2 * E), "loop.step": (cfg.loop.times, E)})
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        for name in ("norm1", "norm1b") + (("norm2", "norm2b") if layer.ff is not None else ()):
            norm(p + name)
        out.update({p + "mix." + n: s for n, s in layer.mixer.shapes(E).items()})
        if layer.ff is not None:
            out.update({p + "mlp." + n: s for n, s in layer.ff.shapes(E).items()})
    return out


def init_weights(cfg: RupotarConfig, seed: int = 42, device="cpu", rank: int = 16) -> dict:
    """Random bf16 checkpoint tensors: matrices ~ N(0, 1/in), norm weights near 1, slow decays."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        shape = tuple(rank if n is None else n for n in shape)
        z = torch.randn(shape, generator=g, device=device)
        last = name.split(".")[-1]
        if name == "embed":
            t = z
        elif last.startswith("norm"):
            t = 1.0 + 0.1 * z
        elif ".mu." in name:
            t = torch.sigmoid(z)
        elif last in ("A_log", "w0"):
            t = z - 2.0
        elif last == "conv":
            t = z * shape[1] ** -0.5
        elif last == "u":
            t = 0.5 * z
        elif len(shape) == 2 and name != "loop.step":
            t = z * shape[1] ** -0.5
        else:
            t = 0.1 * z
        out[name] = t.to(torch.bfloat16)
    return out


class _LayerWeights:
    """A layer's tensors in the form the forward pass takes them: projections of the same input stacked, every block of
    columns of a product on 16 bytes; norms and the constants of the recurrences in fp32."""

    def __init__(self, tensors: dict, p: str, layer: Layer, device, dtype):
        def get(name):
            return tensors[p + name].to(device, dtype)

        def f32(name):
            return tensors[p + name].to(device, torch.float32).contiguous()

        def stack(*names):
            """One matrix of the blocks' rows, and the first row of each."""
            at, rows, starts = 0, [], []
            for n in names:
                w = get("mix." + n)
                pad = -w.shape[0] % 8
                starts.append(at)
                rows += [w, w.new_zeros(pad, w.shape[1])]
                at += w.shape[0] + pad
            return torch.cat(rows), starts

        m = layer.mixer
        self.norm1, self.norm1b = ((f32(n), f32(n + ".b")) for n in ("norm1", "norm1b"))
        if isinstance(m, Attention):
            rows = [get("mix." + n) for n in "qkv"]
            self.proj = torch.cat(rows)
            self.q_norm, self.k_norm = f32("mix.q.norm"), f32("mix.k.norm")
        elif isinstance(m, ChannelDelta):
            # columns: q | k | v (as the convolution takes them), then b, then the low-rank inputs of decay and gate
            qkv = torch.cat([get("mix." + n) for n in "qkv"])
            tail, starts = stack("b", "a1", "g1")
            pad = -qkv.shape[0] % 8
            self.proj = torch.cat([qkv, qkv.new_zeros(pad, qkv.shape[1]), tail])
            self.at_b, self.at_low = qkv.shape[0] + pad, qkv.shape[0] + pad + starts[1]
            ranks = [tensors[p + "mix." + n].shape[0] for n in ("a1", "g1")]
            low = self.proj.shape[0] - self.at_low
            a2, g2 = get("mix.a2"), get("mix.g2")
            pad = -a2.shape[0] % 8                                            # the gate's columns start on 16 bytes
            self.at_gate = a2.shape[0] + pad
            self.up = a2.new_zeros(self.at_gate + g2.shape[0], low)           # decay and gate from their ranks in one product
            self.up[:a2.shape[0], :ranks[0]] = a2
            at = starts[2] - starts[1]
            self.up[self.at_gate:, at:at + ranks[1]] = g2
            self.conv = torch.cat([f32(f"mix.{n}.conv") for n in "qkv"]).t().contiguous()
            self.a_log, self.dt_bias, self.norm = f32("mix.A_log"), f32("mix.dt_bias"), f32("mix.norm")
        else:
            self.mu = torch.stack([f32("mix.mu." + s) for s in MIXES])
            self.rkvg = torch.stack([get("mix." + s) for s in "rkvg"]).transpose(1, 2)   # [4, width, heads * dim]
            self.w1, self.w2, self.w0 = get("mix.w1"), get("mix.w2"), f32("mix.w0")
            self.u, self.norm = f32("mix.u"), f32("mix.norm").view(m.heads, m.dim)
        self.o = get("mix.o")
        ff = layer.ff
        if ff is not None:
            self.norm2, self.norm2b = ((f32(n), f32(n + ".b")) for n in ("norm2", "norm2b"))
        if isinstance(ff, Dense):
            self.gate_up, self.down = torch.cat([get("mlp.gate"), get("mlp.up")]), get("mlp.down")
        elif isinstance(ff, Experts):
            self.gate_up = torch.stack([torch.stack([get(f"mlp.e{e}.gate"), get(f"mlp.e{e}.up")]) for e in range(ff.experts)])
            self.down = torch.stack([get(f"mlp.e{e}.down") for e in range(ff.experts)])
            self.router, self.router_b = get("mlp.router").contiguous(), f32("mlp.router.b")


class RupotarDecoder(DecodeLoop):
    """The decoder on one GPU with a static cache; dtype bfloat16 (the serving precision) or float32."""

    def __init__(self, ext, cfg: RupotarConfig, device, max_batch: int, max_len: int, seed: int = 42,
                 weights: Optional[dict] = None, dtype=torch.bfloat16):
        self.runs = cfg.runs
        super().__init__(ext, device, [cfg.layers[r.layer].mixer.planes(cfg.width) for r in self.runs], max_batch, max_len, dtype)
        self.cfg = cfg
        if weights is None:
            weights = init_weights(cfg, seed)
        for name, shape in tensor_shapes(cfg).items():
            got = tuple(weights[name].shape)
            if len(got) != len(shape) or any(n is not None and n != g for n, g in zip(shape, got)):
                raise ValueError(f"tensor {name} has shape {got}, the configuration says {shape}")
        dev = self.device
        self.embed, self.head = weights["embed"].to(dev, dtype), weights["head"].to(dev, dtype)
        self.final_norm = tuple(weights["final.norm" + s].to(dev, torch.float32).contiguous() for s in ("", ".b"))
        self.w = [_LayerWeights(weights, f"l{i}.", layer, dev, dtype) for i, layer in enumerate(cfg.layers)]
        if cfg.loop is not None:
            self.loop_in = weights["loop.in"].to(dev, dtype)
            self.loop_step = weights["loop.step"].to(dev, torch.float32).contiguous()
        pairs = torch.arange((cfg.width + 1) // 2, dtype=torch.float64)
        self.freqs = (POSITION_BASE ** (-2.0 * pairs / cfg.width)).to(dev)

    # ---- mixers: h [B, T, width] -> heads' outputs [B, T, heads * vdim] --------------------------------------
    def _attention(self, m: Attention, w: _LayerWeights, planes: dict, h, positions, start_pos: int):
        B, T, _ = h.shape
        qw, kw = m.heads * m.dim, m.kv_heads * m.dim
        qkv = F.linear(h, w.proj)
        k, v = planes["k"], planes["v"]
        mixers.qk_norm_cache(qkv, qw, kw, w.q_norm, w.k_norm, self.cfg.eps, k, v, positions)
        out = torch.empty(B, T, m.heads, m.vdim, dtype=h.dtype, device=h.device)
        mixers.attention(qkv[..., :qw].view(B, T, m.heads, m.dim), k, v, out, positions, scale=m.scale, start_pos=start_pos,
                         window=m.window, keep_first=m.keep_first, bias_range=SLOPE_RANGE, sink=True)
        return out.view(B, T, m.heads * m.vdim)

    def _channel_delta(self, m: ChannelDelta, w: _LayerWeights, planes: dict, h, positions, start_pos: int):
        B, T, E = h.shape
        H, G, D, V = m.heads, m.kv_heads, m.dim, m.vdim
        p = F.linear(h, w.proj)
        low = p.view(B * T, -1)[:, w.at_low:]
        up = torch.mm(low, w.up.t()).view(B, T, -1)
        qk, v, beta, decay = mixers.delta_inputs(p, p[..., w.at_b:w.at_b + H], up[..., :H * D], w.conv, w.a_log, w.dt_bias, planes["tail"],
                                                 positions, H, G, D, V, UNIT_EPS)
        gate = up[..., w.at_gate:w.at_gate + H * V].view(B, T, H, V)
        return mixers.recurrent_scan(qk[:, :, 0], qk[:, :, 1], v, decay, planes["state"], positions, w.norm, gate, act=mixers.SIGMOID,
                                     eps=self.cfg.eps, beta=beta, conv_in=p, tail=planes["tail"], taps=m.taps)

    def _wkv(self, m: TimeMix, w: _LayerWeights, planes: dict, h, positions, start_pos: int):
        B, T, E = h.shape
        mixes = mixers.token_shift(h, w.mu, planes["last"], positions).view(len(MIXES), B * T, E)
        r, k, v, g = torch.bmm(mixes[:4], w.rkvg).view(4, B, T, m.heads, m.dim)
        decay = F.linear(mixers.tanh_(F.linear(mixes[4], w.w1)), w.w2).view(B, T, m.heads, m.dim)
        return mixers.recurrent_scan(r, k, v, decay, planes["state"], positions, w.norm, g, act=mixers.SILU, eps=self.cfg.eps, bonus=w.u,
                                     g_bias=w.w0)

    # ---- feed-forward: what `residual_norm` adds ---------------------------------------------------------------
    def _feed_forward(self, ff, w: _LayerWeights, h):
        if isinstance(ff, Dense):
            return {"y": F.linear(mixers.gated_act(F.linear(h, w.gate_up)), w.down)}
        rows = h.view(-1, h.shape[-1])
        experts, ranks, weights, counts = mixers.moe_route(self._product32(rows, w.router), w.router_b, ff.top)
        x, part_rows = mixers.moe_gather(rows, experts, ranks, counts)
        a = mixers.moe_gemm(x, w.gate_up, counts, limit=ff.limit, alpha=EXPERT_ALPHA)
        return {"y": mixers.moe_gemm(a, w.down, counts), "part_rows": part_rows, "part_weights": weights}

    def _product32(self, x, w):
        """x w^T in fp32: products of two bf16 numbers are exact, the sum is not rounded to bf16."""
        return torch.mm(x, w.t()) if x.dtype == torch.float32 else torch.mm(x, w.t(), out_dtype=torch.float32)

    # ---- one forward pass over T new tokens per sequence ------------------------------------------------------
    def forward(self, tokens: torch.Tensor, positions: torch.Tensor, seq_lens: torch.Tensor, start_pos: int = 0,
                slots: Optional[slice] = None, want=None, keep: Optional[list] = None):
        """See DecodeLoop.forward; `keep` (a list) receives a copy of the residual stream after every layer run."""
        cfg, runs, eps = self.cfg, self.runs, self.cfg.eps
        B, T = tokens.shape
        E = cfg.width
        slots = slice(0, B) if slots is None else slots
        start_pos = start_pos if T > 1 else -1       # one token: positions live on the device alone (CUDA graph)
        # [x; embedding output], the input of a pass
        cat = torch.empty(B, T, 2 * E, dtype=self.dtype, device=self.device) if cfg.loop is not None else None

        def before(r):
            """Where the residual stream goes ahead of run r: the run's first norm, or the input of the pass it opens."""
            if r == len(runs):
                return {"pre": self.final_norm}
            return {"out": cat[..., :E]} if runs[r].step is not None else {"pre": self.w[runs[r].layer].norm1}

        with full_precision_products():
            first = before(0)
            x, h = mixers.embed_residual(tokens, self.embed, cfg.embed_scale, self.freqs, positions, x0=None if cat is None else cat[..., E:],
                                         norm=first.get("pre"), out=first.get("out"), eps=eps)
            for r, run in enumerate(runs):
                layer, w = cfg.layers[run.layer], self.w[run.layer]
                m, ff = layer.mixer, layer.ff
                planes = {name: p[slots] for name, p in self.cache.layers[r].items()}
                mix = self._attention if isinstance(m, Attention) else self._channel_delta if isinstance(m, ChannelDelta) else self._wkv
                with nvtx_range("layer"):
                    if run.step is not None:
                        h = mixers.residual_norm(self._product32(cat.view(B * T, 2 * E), self.loop_in), x, dtype=self.dtype, reset=True, step=self.loop_step[run.step],
                                                 pre=w.norm1, eps=eps)
                    added, post = {"y": F.linear(mix(m, w, planes, h, positions, start_pos), w.o)}, w.norm1b
                    if ff is not None:
                        h = mixers.residual_norm(**added, x=x, dtype=self.dtype, post=post, pre=w.norm2, eps=eps)
                        added, post = self._feed_forward(ff, w, h), w.norm2b
                    h = mixers.residual_norm(**added, x=x, dtype=self.dtype, post=post, eps=eps, **before(r + 1))
                    if keep is not None:
                        keep.append(x.clone())
            return self.logits(h, self.head, want)
