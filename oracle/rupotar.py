"""Plain float64 restatement of the Rupotar decoder, one function per mechanism, one sequence at a time.

Slow on purpose: whole sequences only (no cache, no chunks), heads and tokens in loops, dense masks.  It shares no code
with the product path; the tests compare the kernels, the layers and whole decodes with it.

Notation: x[t, :] is the residual stream of position t, h the normalised input of a mixer or feed-forward.  A weight
matrix is stored [out, in].
"""
from __future__ import annotations

import torch

F64 = torch.float64


# ---- norms and activations ------------------------------------------------------------------------------------
def rms(x, eps):
    """x divided by sqrt(mean(x^2) + eps) along the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def layer_norm(x, weight, bias, eps):
    centred = x - x.mean(dim=-1, keepdim=True)
    return centred / torch.sqrt((centred * centred).mean(dim=-1, keepdim=True) + eps) * weight + bias


def unit(x, eps=1e-6):
    """x divided by sqrt(sum(x^2) + eps) along the last axis."""
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + eps)


def silu(z):
    return z / (1.0 + torch.exp(-z))


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


# ---- embedding --------------------------------------------------------------------------------------------------
def sinusoid(positions, width):
    """[T, width]: sin and cos of p * 10000^(-2i/width) at entries 2i and 2i + 1."""
    out = torch.zeros(len(positions), width, dtype=F64)
    for c in range(width):
        angle = positions.to(F64) * 10000.0 ** (-2.0 * (c // 2) / width)
        out[:, c] = torch.cos(angle) if c % 2 else torch.sin(angle)
    return out


# ---- attention: distance bias, window with kept first tokens, sink -------------------------------------------------
def slope(h, heads):
    return 2.0 ** (-8.0 * (h + 1) / heads)


def sink_softmax(scores, visible):
    """exp(s) / (1 + sum exp(s)) over the visible keys, formed with the larger of 0 and the row's maximum taken off."""
    s = scores.masked_fill(~visible, float("-inf"))
    top = torch.clamp(s.max(dim=-1, keepdim=True).values, min=0.0)
    e = torch.exp(s - top)
    return e / (torch.exp(-top) + e.sum(dim=-1, keepdim=True))


def attention(q, k, v, scale, size, keep):
    """q [T, H, D], k [S, G, D], v [S, G, V], the queries are the last T of the S positions.  Position i sees j <= i with
    i - j < size (None: all) or j < keep.  Returns [T, H, V]."""
    T, H, _ = q.shape
    S, G, _ = k.shape
    i, j = torch.arange(S - T, S)[:, None], torch.arange(S)[None, :]
    visible = j <= i
    if size is not None:
        visible = visible & ((i - j < size) | (j < keep))
    out = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for h in range(H):
        g = h // (H // G)
        scores = q[:, h] @ k[:, g].T * scale - slope(h, H) * (i - j).to(F64)
        out[:, h] = sink_softmax(scores, visible) @ v[:, g]
    return out


def attention_mixer(m, w, h, eps):
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    mask = m.get("mask") or {}
    q = rms(h @ w["q"].T, eps) * w["q.norm"]
    k = rms(h @ w["k"].T, eps) * w["k.norm"]
    v = h @ w["v"].T
    T = h.shape[0]
    o = attention(q.view(T, H, D), k.view(T, G, D), v.view(T, G, V), m["scale"], mask.get("size"), mask.get("keep_first") or 0)
    return o.reshape(T, H * V) @ w["o"].T


# ---- gated delta rule with a decay per key channel -----------------------------------------------------------------
def short_conv(x, taps):
    """y[t, c] = sum_i taps[c, i] x[t - (n - 1) + i, c], zeros before the start."""
    T, C = x.shape
    n = taps.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for i in range(n):
            at = t - (n - 1) + i
            if at >= 0:
                y[t] += taps[:, i] * x[at]
    return y


def delta_scan(q, k, v, g, beta, state=None):
    """q, k, g [T, H, D] (one per state head), v [T, H, V], beta [T, H].  Returns o [T, H, V] and the state [H, D, V]."""
    T, H, D = q.shape
    V = v.shape[-1]
    S = torch.zeros(H, D, V, dtype=F64) if state is None else state.clone()
    o = torch.zeros(T, H, V, dtype=F64)
    for t in range(T):
        for h in range(H):
            S[h] = g[t, h][:, None] * S[h]
            u = beta[t, h] * (v[t, h] - S[h].T @ k[t, h])
            S[h] = S[h] + torch.outer(k[t, h], u)
            o[t, h] = S[h].T @ q[t, h]
    return o, S


def delta_inputs(m, w, h):
    """The scan's inputs (see `delta_scan`) of a whole sequence."""
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q, k, v = (silu(short_conv(h @ w[n].T, w[n + ".conv"])) for n in ("q", "k", "v"))
    q = unit(q.view(T, G, D)) * D ** -0.5
    k = unit(k.view(T, G, D))
    beta = 1.0 / (1.0 + torch.exp(-(h @ w["b"].T)))
    a = softplus(h @ w["a1"].T @ w["a2"].T + w["dt_bias"]).view(T, H, D)
    g = torch.exp(-torch.exp(w["A_log"])[None, :, None] * a)
    of = [i // (H // G) for i in range(H)]
    return q[:, of], k[:, of], v.view(T, H, V), g, beta


def delta_mixer(m, w, h, eps):
    o, _ = delta_scan(*delta_inputs(m, w, h))
    gate = h @ w["g1"].T @ w["g2"].T
    o = rms(o, eps) * w["norm"]
    return (o.reshape(gate.shape) / (1.0 + torch.exp(-gate))) @ w["o"].T


# ---- time mixing with a bonus for the current token ---------------------------------------------------------------
def token_shift(h, mu):
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mu


def wkv_scan(r, k, v, w, u, state=None):
    """r, k, v, w [T, H, D], u [H, D].  Returns o [T, H, D] and the state [H, D, D] (key channel, value channel)."""
    T, H, D = r.shape
    S = torch.zeros(H, D, D, dtype=F64) if state is None else state.clone()
    o = torch.zeros(T, H, D, dtype=F64)
    for t in range(T):
        for h in range(H):
            kv = torch.outer(k[t, h], v[t, h])
            o[t, h] = (S[h] + u[h][:, None] * kv).T @ r[t, h]
            S[h] = w[t, h][:, None] * S[h] + kv
    return o, S


def wkv_inputs(m, w, h):
    T, H, D = h.shape[0], m["heads"], m["dim"]
    r, k, v = ((token_shift(h, w["mu." + n]) @ w[n].T).view(T, H, D) for n in ("r", "k", "v"))
    low = torch.tanh(token_shift(h, w["mu.w"]) @ w["w1"].T)
    decay = torch.exp(-torch.exp(low @ w["w2"].T + w["w0"])).view(T, H, D)
    return r, k, v, decay, w["u"].view(H, D)


def wkv_mixer(m, w, h, eps):
    o, _ = wkv_scan(*wkv_inputs(m, w, h))
    gate = silu(token_shift(h, w["mu.g"]) @ w["g"].T)
    return (rms(o, eps).reshape(gate.shape) * w["norm"] * gate) @ w["o"].T


# ---- feed-forward ----------------------------------------------------------------------------------------------------
def dense_ff(w, h):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def clamped_expert(gate, up, down, h, limit):
    g = torch.clamp(h @ gate.T, max=limit)
    u = torch.clamp(h @ up.T, min=-limit, max=limit)
    return (g / (1.0 + torch.exp(-1.702 * g)) * (u + 1.0)) @ down.T


def route(z, top):
    """Indices and weights [T, top] of the largest logits: softmax over the chosen ones."""
    values, chosen = torch.topk(z, top, dim=-1)
    e = torch.exp(values - values.max(dim=-1, keepdim=True).values)
    return chosen, e / e.sum(dim=-1, keepdim=True)


def moe_ff(mlp, w, h):
    chosen, weight = route(h @ w["router"].T + w["router.b"], mlp["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, p in zip(chosen[t].tolist(), weight[t]):
            out[t] += p * clamped_expert(w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"], h[t], mlp["expert"]["limit"])
    return out


# ---- the decoder -------------------------------------------------------------------------------------------------------
MIXERS = {"attention": attention_mixer, "channel_delta": delta_mixer, "wkv": wkv_mixer}


def layer_runs(config):
    """(layer, pass of the loop or None, whether the run opens a pass) in order of execution."""
    loop = config.get("loop") or {"start": 0, "stop": 0, "times": 0}
    a, b = loop["start"], loop["stop"]
    runs = [(i, None, False) for i in range(a)]
    for t in range(loop["times"]):
        runs += [(i, t, i == a) for i in range(a, b)]
    return runs + [(i, None, False) for i in range(b, len(config["layers"]))]


def forward(config, weights, tokens, keep=None):
    """Logits [T, vocab] of a whole sequence; `keep` (a list) receives the residual stream after every layer run."""
    w = {n: t.to(F64) for n, t in weights.items()}
    eps = config["norm"]["eps"]

    def part(prefix):
        return {n[len(prefix):]: t for n, t in w.items() if n.startswith(prefix)}

    def norm(x, name):
        return layer_norm(x, w[name], w[name + ".b"], eps)

    tokens = torch.as_tensor(tokens)
    x0 = w["embed"][tokens] * config["embedding"]["scale"] + sinusoid(torch.arange(len(tokens)), config["width"])
    x = x0
    for i, t, opens in layer_runs(config):
        if opens:
            x = torch.cat([x, x0], dim=-1) @ w["loop.in"].T + w["loop.step"][t]
        entry, p = config["layers"][i], f"l{i}."
        x = x + norm(MIXERS[entry["type"]](entry["mixer"], part(p + "mix."), norm(x, p + "norm1"), eps), p + "norm1b")
        mlp = entry.get("mlp")
        if mlp is not None:
            h, mw = norm(x, p + "norm2"), part(p + "mlp.")
            x = x + norm(dense_ff(mw, h) if mlp["kind"] == "dense" else moe_ff(mlp, mw, h), p + "norm2b")
        if keep is not None:
            keep.append(x.clone())
    return norm(x, "final.norm") @ w["head"].T
