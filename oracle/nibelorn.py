"""Plain float64 restatement of the Nibelorn decoder, one function per mechanism, one sequence at a time.

Slow on purpose: whole sequences only (no cache), heads in loops, dense masks.  It shares no code with the
product path; the tests compare the kernels, the layers and whole decodes with it.

Notation: x[t, :] is the residual stream of position t, h the normalised input of a mixer or feed-forward.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def dyn_tanh(x, weight, bias, alpha):
    """y = tanh(alpha x) * weight + bias, elementwise; no statistics of x."""
    return torch.tanh(alpha.to(F64) * x) * weight.to(F64) + bias.to(F64)


def rms(x, eps):
    """x divided by sqrt(mean(x^2) + eps) along the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def gelu(z):
    """The exact gelu: z times the normal distribution function of z."""
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def rotate_half(x, positions, base):
    """Rotation of x[t, ..., n] by position: element i pairs with element i + n/2, frequency base^(-2i/n)."""
    n = x.shape[-1]
    out = torch.empty_like(x)
    for i in range(n // 2):
        angle = positions.to(F64) * base ** (-2.0 * i / n)
        c, s = torch.cos(angle), torch.sin(angle)
        while c.dim() < x.dim() - 1:
            c, s = c.unsqueeze(-1), s.unsqueeze(-1)
        u, v = x[..., i], x[..., i + n // 2]
        out[..., i] = u * c - v * s
        out[..., i + n // 2] = v * c + u * s
    return out


def query_temperature(positions, coef, every):
    """1 + coef * ln(floor((p + 1) / every) + 1)."""
    return 1.0 + coef * torch.log(torch.floor((positions.to(F64) + 1.0) / every) + 1.0)


def softcap(scores, cap):
    return cap * torch.tanh(scores / cap)


def causal_softmax(scores):
    """Softmax over the keys j <= i of scores[i, j]."""
    T, S = scores.shape
    hidden = torch.arange(S)[None, :] > torch.arange(T)[:, None]
    s = scores.masked_fill(hidden, -math.inf)
    e = torch.exp(s - s.amax(dim=-1, keepdim=True))
    return e / e.sum(dim=-1, keepdim=True)


def latent_attention(h, w, m, eps):
    """Keys and values of all heads are linear in one latent row per token; a rotated key part is shared by the heads.

    w: q, dkv, dkv.norm, uk, uv, o;  m: heads, dim, rot_dim, vdim, kv_rank, scale, rot.base."""
    T = h.shape[0]
    H, D, R, V, C = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    q = (h @ w["q"].to(F64).T).view(T, H, D + R)
    down = h @ w["dkv"].to(F64).T
    c = rms(down[:, :C], eps) * w["dkv.norm"].to(F64)
    k_rot = rotate_half(down[:, C:], pos, m["rot"]["base"])
    k = (c @ w["uk"].to(F64).T).view(T, H, D)
    v = (c @ w["uv"].to(F64).T).view(T, H, V)
    out = torch.empty(T, H, V, dtype=F64)
    for n in range(H):
        q_rot = rotate_half(q[:, n, D:], pos, m["rot"]["base"])
        s = (q[:, n, :D] @ k[:, n].T + q_rot @ k_rot.T) * m["scale"]
        out[:, n] = causal_softmax(s) @ v[:, n]
    return out.reshape(T, H * V) @ w["o"].to(F64).T


def cached_attention(q, k, v, start, scale, cap=0.0, temp=None):
    """Softmax attention of q[t, H, D] at positions start + t over k[j, G, D], v[j, G, V]: keys j <= start + t."""
    T, H, _ = q.shape
    S, G, _ = k.shape
    pos = torch.arange(start, start + T)
    factor = query_temperature(pos, *temp) if temp else torch.ones(T, dtype=F64)
    hidden = torch.arange(S)[None, :] > pos[:, None]
    out = torch.empty(T, H, v.shape[-1], dtype=F64)
    for n in range(H):
        g = n // (H // G)
        s = (q[:, n].to(F64) * factor[:, None]) @ k[:, g].to(F64).T * scale
        if cap:
            s = softcap(s, cap)
        out[:, n] = torch.softmax(s.masked_fill(hidden, -math.inf), dim=-1) @ v[:, g].to(F64)
    return out


def differential_combine(a1, a2, lam, diff, eps, gate=None):
    """a1, a2 [t, H, V]: the maps' outputs; gate [t, H] before the sigmoid."""
    o = rms(a1 - lam * a2, eps) * (1.0 - diff)
    return o if gate is None else o * torch.sigmoid(gate.to(F64))[..., None]


def differential_lambda(w, diff):
    def dot(a, b):
        return (w[a].to(F64) * w[b].to(F64)).sum()

    return torch.exp(dot("lq1", "lk1")) - torch.exp(dot("lq2", "lk2")) + diff


def differential_attention(h, w, m, eps):
    """Two attention maps per head over the same values; the second is subtracted, lambda times, from the first.

    w: q, k, v, g, o, lq1, lk1, lq2, lk2;  m: heads, kv_heads, dim, vdim, scale, diff, softcap, q_temp."""
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].to(F64).T).view(T, H, 2, D)
    k = (h @ w["k"].to(F64).T).view(T, G, 2, D)
    v = (h @ w["v"].to(F64).T).view(T, G, V)
    temp = query_temperature(torch.arange(T), m["q_temp"]["coef"], m["q_temp"]["every"])
    lam = differential_lambda(w, m["diff"])
    gate = torch.sigmoid(h @ w["g"].to(F64).T)
    out = torch.empty(T, H, V, dtype=F64)
    for n in range(H):
        g = n // (H // G)
        maps = []
        for i in range(2):
            s = (q[:, n, i] * temp[:, None]) @ k[:, g, i].T * m["scale"]
            maps.append(causal_softmax(softcap(s, m["softcap"])) @ v[:, g])
        out[:, n] = rms(maps[0] - lam * maps[1], eps) * (1.0 - m["diff"]) * gate[:, n:n + 1]
    return out.reshape(T, H * V) @ w["o"].to(F64).T


MIXERS = {"latent_attention": latent_attention, "attention": differential_attention}


def feed_forward(h, w):
    return gelu(h @ w["up"].to(F64).T) @ w["down"].to(F64).T


def under(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(config, weights, tokens, keep=None):
    """Logits [T, vocab] of one sequence; `keep` (a list) receives the residual stream after every layer."""
    eps = config["norm"]["eps"]
    x = weights["embed"].to(F64)[torch.as_tensor(tokens)]

    def norm(x, name):
        return dyn_tanh(x, weights[name], weights[name + ".b"], weights[name + ".alpha"])

    for i, layer in enumerate(config["layers"]):
        p = f"l{layer.get('weights_of', i)}."
        x = x + MIXERS[layer["type"]](norm(x, p + "norm1"), under(weights, p + "mix."), layer["mixer"], eps)
        if layer["mlp"] is not None:
            x = x + feed_forward(norm(x, p + "norm2"), under(weights, p + "mlp."))
        if keep is not None:
            keep.append(x.clone())
    return norm(x, "final.norm") @ weights["head"].to(F64).T


def greedy(config, weights, prompt, n):
    """n tokens after `prompt`, each the argmax of the whole sequence's last logits."""
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(forward(config, weights, seq)[-1].argmax()))
    return seq[len(prompt):]
