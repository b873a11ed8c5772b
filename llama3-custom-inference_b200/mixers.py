"""ctypes binding of include/l3ci_mixers.h (lib/libl3ci_mixers.so) over torch device tensors: the layer parts of the
decoders other than Llama-3.  As in capi.py, torch owns the memory and names the stream; nothing here computes."""
from __future__ import annotations

import ctypes as C
from pathlib import Path

import torch

from .capi import OK, L3ciError, _on, _stream

LIB_PATH = Path(__file__).resolve().parent / "lib" / "libl3ci_mixers.so"

EXPORTS = ("l3ci_mixers_last_error", "l3ci_mixers_set_programmatic_launch", "l3ci_add_dyn_tanh", "l3ci_gelu",
           "l3ci_latent_cache", "l3ci_kv_cache_write", "l3ci_mixer_attention", "l3ci_mixer_attention_scratch_bytes",
           "l3ci_mixer_attention_variant", "l3ci_residual_norm", "l3ci_tanh", "l3ci_gated_act", "l3ci_qk_norm_cache",
           "l3ci_token_shift", "l3ci_delta_inputs", "l3ci_recurrent_scan", "l3ci_moe_route", "l3ci_moe_gather",
           "l3ci_moe_gemm", "l3ci_moe_gemm_variant")

DTYPE_CODES = {torch.bfloat16: 0, torch.float32: 1}
ROWS, MMA, TC = 1, 2, 3   # variants of l3ci_mixer_attention (0: choose)


class AttnArgs(C.Structure):
    """struct l3ci_mixer_attn_args"""
    _fields_ = [
        ("qa", C.c_void_p), ("qb", C.c_void_p), ("ka", C.c_void_p), ("kb", C.c_void_p), ("v", C.c_void_p),
        ("gate", C.c_void_p), ("out", C.c_void_p), ("positions", C.c_void_p), ("scratch", C.c_void_p),
        ("scratch_bytes", C.c_size_t), ("status", C.c_void_p),
        *[(n, C.c_int64) for n in ("qa_sb", "qa_st", "qa_sh", "qb_sb", "qb_st", "qb_sh", "ka_sb", "ka_st", "ka_sh",
                                   "kb_sb", "kb_st", "kb_sh", "v_sb", "v_st", "v_sh", "o_sb", "o_st", "o_sh", "g_sb", "g_st")],
        *[(n, C.c_int32) for n in ("dtype", "B", "T", "H", "G", "maps", "Da", "Db", "Dv", "n_keys", "start_pos", "variant",
                                   "window", "keep_first", "sink")],
        *[(n, C.c_float) for n in ("scale", "softcap", "temp_coef", "temp_every", "lambda_", "post", "eps", "bias_range")],
        ("stream", C.c_void_p),
    ]


def _fields(pointers: str, longs: str, ints: str, floats: str):
    kinds = ((pointers, C.c_void_p), (longs, C.c_int64), (ints, C.c_int32), (floats, C.c_float))
    return [(n, kind) for names, kind in kinds for n in names.split()] + [("stream", C.c_void_p)]


class ResidualNormArgs(C.Structure):
    """struct l3ci_residual_norm_args"""
    _fields_ = _fields("x y part_weights part_rows post_w post_b step pre_w pre_b out tokens table freqs positions x0",
                       "out_stride x0_stride vocab rows width", "parts reset T dtype y_dtype", "eps embed_scale")


class DeltaInputsArgs(C.Structure):
    """struct l3ci_delta_inputs_args"""
    _fields_ = _fields("p b a conv a_log dt_bias tail positions qk_out beta_out decay_out v_out", "p_st b_st a_st tail_sb",
                       "B T H G D V taps dtype", "unit_eps")


class RecurrentScanArgs(C.Structure):
    """struct l3ci_recurrent_scan_args"""
    _fields_ = _fields("q k v g beta bonus g_bias norm gate state out conv_in tail positions status",
                       "qk_st qk_sh v_st v_sh g_st g_sh gate_st gate_sh out_st out_sh norm_sh state_sb conv_st tail_sb",
                       "kind B T H G D V act taps dtype", "eps")


class MoeGemmArgs(C.Structure):
    """struct l3ci_moe_gemm_args"""
    _fields_ = _fields("x w out counts status", "rows", "K N n_experts gated dtype variant", "limit alpha")


SIGMOID, SILU = 0, 1   # gates of a recurrent head's output


def tc_sizes_ok(Da: int, Db: int, Dv: int) -> bool:
    """Sizes the tcgen05 kernel of `attention` takes for one map (variant TC): parts that fit its shared-memory tiles, rows of
    whole 16-byte vectors."""
    return 0 < Da <= 128 and Db <= 64 and Dv <= 128 and Da % 8 == 0 and Db % 8 == 0 and Dv % 8 == 0


_lib = None


def load() -> C.CDLL:
    """Loads lib/libl3ci_mixers.so once and declares the prototypes.  Raises OSError if it is not built."""
    global _lib
    if _lib is not None:
        return _lib
    if not LIB_PATH.exists():
        raise OSError(f"{LIB_PATH} is missing: run build.py in this directory; there is no fallback")
    lib = C.CDLL(str(LIB_PATH))
    i64, i32, vp, f32 = C.c_int64, C.c_int32, C.c_void_p, C.c_float
    lib.l3ci_mixers_last_error.restype = C.c_char_p
    lib.l3ci_mixers_set_programmatic_launch.argtypes = [C.c_int]
    lib.l3ci_add_dyn_tanh.argtypes = [vp, vp, vp, i64, vp, vp, vp, f32, vp, i64, i64, i32, vp]
    lib.l3ci_gelu.argtypes = [vp, vp, i64, i32, vp]
    lib.l3ci_latent_cache.argtypes = [vp, i64, vp, i64, vp, f32, vp, i64, i64, i64, vp] + [i32] * 7 + [vp]
    lib.l3ci_kv_cache_write.argtypes = [vp] + [i64] * 5 + [vp, i64, i64, vp, i64, i64, i64, vp, i32, i32, i32, vp]
    lib.l3ci_mixer_attention.argtypes = [C.POINTER(AttnArgs)]
    lib.l3ci_mixer_attention_variant.argtypes = [C.POINTER(AttnArgs)]
    lib.l3ci_mixer_attention_scratch_bytes.argtypes = [C.POINTER(AttnArgs)]
    lib.l3ci_mixer_attention_scratch_bytes.restype = C.c_size_t
    lib.l3ci_residual_norm.argtypes = [C.POINTER(ResidualNormArgs)]
    lib.l3ci_tanh.argtypes = [vp, vp, i64, i32, vp]
    lib.l3ci_gated_act.argtypes = [vp, vp, i64, i64, f32, f32, i32, vp]
    lib.l3ci_qk_norm_cache.argtypes = [vp, i64, i64, i64, i64, vp, vp, f32, vp, i64, i64, vp, i64, i64, i64, vp, i32, i32, i32, vp]
    lib.l3ci_token_shift.argtypes = [vp, vp, vp, i64, vp, vp, i32, i32, i32, i64, i32, vp]
    lib.l3ci_delta_inputs.argtypes = [C.POINTER(DeltaInputsArgs)]
    lib.l3ci_recurrent_scan.argtypes = [C.POINTER(RecurrentScanArgs)]
    lib.l3ci_moe_route.argtypes = [vp, vp, vp, vp, vp, vp, i64, i32, i32, vp]
    lib.l3ci_moe_gather.argtypes = [vp, vp, vp, vp, vp, vp, i64, i64, i32, i32, i32, vp]
    lib.l3ci_moe_gemm.argtypes = [C.POINTER(MoeGemmArgs)]
    lib.l3ci_moe_gemm_variant.argtypes = [C.POINTER(MoeGemmArgs)]
    _lib = lib
    return lib


def _check(status: int, what: str) -> None:
    if status != OK:
        raise L3ciError(status, what, load().l3ci_mixers_last_error().decode())


def _cuda(*tensors):
    for t in tensors:
        if not t.is_cuda:
            raise ValueError("the mixer kernels take CUDA tensors: there is no CPU path")


def embed_dyn_tanh(tokens, table, weight, bias, alpha: float):
    """x = table[tokens] in fp32 and tanh(alpha x) * weight + bias in the table's type; tokens int64, contiguous."""
    _cuda(tokens, table)
    E = table.shape[1]
    x = torch.empty(*tokens.shape, E, dtype=torch.float32, device=tokens.device)
    out = torch.empty(x.shape, dtype=table.dtype, device=tokens.device)
    with _on(x):
        _check(load().l3ci_add_dyn_tanh(None, tokens.data_ptr(), table.data_ptr(), table.shape[0], x.data_ptr(),
                                        weight.data_ptr(), bias.data_ptr(), alpha, out.data_ptr(), tokens.numel(), E,
                                        DTYPE_CODES[table.dtype], _stream(x)), "l3ci_add_dyn_tanh")
    return x, out


def add_dyn_tanh(y, x, weight, bias, alpha: float):
    """x += y in place (x: the fp32 residual stream); returns tanh(alpha x) * weight + bias in y's type."""
    _cuda(x, y)
    assert y.is_contiguous() and x.is_contiguous() and x.dtype == torch.float32 and y.numel() == x.numel()
    out = torch.empty_like(y)
    E = x.shape[-1]
    with _on(x):
        _check(load().l3ci_add_dyn_tanh(y.data_ptr(), None, None, 0, x.data_ptr(), weight.data_ptr(), bias.data_ptr(), alpha,
                                        out.data_ptr(), x.numel() // E, E, DTYPE_CODES[y.dtype], _stream(x)),
               "l3ci_add_dyn_tanh")
    return out


def gelu_(z):
    """Exact gelu in place."""
    _cuda(z)
    assert z.is_contiguous()
    with _on(z):
        _check(load().l3ci_gelu(z.data_ptr(), z.data_ptr(), z.numel(), DTYPE_CODES[z.dtype], _stream(z)), "l3ci_gelu")
    return z


def tanh_(z):
    """tanh in place."""
    _cuda(z)
    assert z.is_contiguous()
    with _on(z):
        _check(load().l3ci_tanh(z.data_ptr(), z.data_ptr(), z.numel(), DTYPE_CODES[z.dtype], _stream(z)), "l3ci_tanh")
    return z


def gated_act(gu, limit: float = 0.0, alpha: float = 1.702):
    """gu [..., 2 ff] = gate | up: silu(gate) * up, or the clamped form (limit > 0)."""
    _cuda(gu)
    assert gu.is_contiguous()
    ff = gu.shape[-1] // 2
    out = torch.empty(*gu.shape[:-1], ff, dtype=gu.dtype, device=gu.device)
    with _on(gu):
        _check(load().l3ci_gated_act(gu.data_ptr(), out.data_ptr(), out.numel() // ff, ff, limit, alpha, DTYPE_CODES[gu.dtype],
                                     _stream(gu)), "l3ci_gated_act")
    return out


def _row_stride(t) -> int:
    """Elements between consecutive rows of t [B, T, ...], (b, t) pairs counted as one axis."""
    B, T = t.shape[:2]
    assert t.stride(-1) == 1 and (B == 1 or T == 1 or t.stride(0) == T * t.stride(1))
    return t.stride(1) if T > 1 else t.stride(0) if B > 1 else t[0, 0].numel()


def _residual(a: ResidualNormArgs, x, out):
    a.x, a.rows, a.width = x.data_ptr(), x.numel() // x.shape[-1], x.shape[-1]
    if out is not None:
        a.out, a.out_stride = out.data_ptr(), _row_stride(out if out.dim() > 2 else out[None])
    a.stream = _stream(x)
    with _on(x):
        _check(load().l3ci_residual_norm(C.byref(a)), "l3ci_residual_norm")


def embed_residual(tokens, table, scale: float, freqs, positions, x0=None, norm=None, eps: float = 0.0, out=None):
    """The residual stream [B, T, width] (fp32) of tokens [B, T]: table[tokens] * scale, plus the sinusoidal vector of the
    position (freqs: float64 [width / 2] rounded up, or None).  x0 [B, T, width] (any row stride) receives a copy in the table's
    type.  Returns x and layer_norm(x) with `norm` (weight, bias), else x in the table's type if `out` is given for it, else
    None."""
    _cuda(tokens, table, positions)
    B, T = tokens.shape
    E = table.shape[1]
    assert tokens.is_contiguous() and table.is_contiguous()
    x = torch.empty(B, T, E, dtype=torch.float32, device=tokens.device)
    if norm is not None and out is None:
        out = torch.empty(B, T, E, dtype=table.dtype, device=tokens.device)
    a = ResidualNormArgs(tokens=tokens.data_ptr(), table=table.data_ptr(), vocab=table.shape[0], positions=positions.data_ptr(), T=T,
                         embed_scale=scale, dtype=DTYPE_CODES[table.dtype], eps=eps)
    if freqs is not None:
        assert freqs.dtype == torch.float64 and freqs.numel() == (E + 1) // 2
        a.freqs = freqs.data_ptr()
    if x0 is not None:
        assert x0.dtype == table.dtype
        a.x0, a.x0_stride = x0.data_ptr(), _row_stride(x0)
    if norm is not None:
        a.pre_w, a.pre_b = norm[0].data_ptr(), norm[1].data_ptr()
    _residual(a, x, out)
    return x, out


def residual_norm(y, x, *, dtype, post=None, pre=None, step=None, reset: bool = False, eps: float = 0.0, part_rows=None,
                  part_weights=None, out=None):
    """x [B, T, width] (fp32, in place) <- (0 if reset else x) + (layer_norm(y) if post else y) + step; returns layer_norm(x)
    if pre, x itself in `dtype` if `out` is given, else None.  post, pre: (weight, bias).  With part_rows, part_weights
    [rows, parts] y holds rows in any order and a row's y is the weighted sum of its parts."""
    _cuda(x)
    a = ResidualNormArgs(dtype=DTYPE_CODES[dtype], reset=int(reset), eps=eps, parts=1, y_dtype=DTYPE_CODES[dtype])
    assert x.is_contiguous() and x.dtype == torch.float32
    if y is not None:
        assert y.is_contiguous()
        a.y, a.y_dtype = y.data_ptr(), DTYPE_CODES[y.dtype]
        if part_rows is not None:
            assert part_rows.is_contiguous() and part_weights.is_contiguous() and part_rows.dtype == torch.int32
            a.part_rows, a.part_weights, a.parts = part_rows.data_ptr(), part_weights.data_ptr(), part_rows.shape[-1]
    if post is not None:
        a.post_w, a.post_b = post[0].data_ptr(), post[1].data_ptr()
    if step is not None:
        a.step = step.data_ptr()
    if pre is not None:
        a.pre_w, a.pre_b = pre[0].data_ptr(), pre[1].data_ptr()
        out = torch.empty(x.shape, dtype=dtype, device=x.device) if out is None else out
    _residual(a, x, out)
    return out


def qk_norm_cache(qkv, q_width: int, k_width: int, q_norm, k_norm, eps: float, cache_k, cache_v, positions):
    """Rows [q | k | v] of qkv [B, T, W]: whole-row RMS norm of q (in place) and k, k and v into cache_k, cache_v."""
    _cuda(qkv, cache_k, cache_v, positions)
    B, T, W = qkv.shape
    vw = cache_v.shape[2] * cache_v.shape[3]
    assert qkv.is_contiguous() and cache_k.dtype == cache_v.dtype == qkv.dtype and cache_k.shape[0] == B
    assert cache_k[0, 0].is_contiguous() and cache_v[0, 0].is_contiguous()
    with _on(qkv):
        _check(load().l3ci_qk_norm_cache(qkv.data_ptr(), W, q_width, k_width, vw, q_norm.data_ptr(), k_norm.data_ptr(), eps,
                                         cache_k.data_ptr(), cache_k.stride(0), cache_k.stride(1), cache_v.data_ptr(),
                                         cache_v.stride(0), cache_v.stride(1), cache_k.shape[1], positions.data_ptr(), B, T,
                                         DTYPE_CODES[qkv.dtype], _stream(qkv)), "l3ci_qk_norm_cache")


def token_shift(h, mu, last, positions):
    """Mixes [n, B, T, width] of h [B, T, width] with the token before, factors mu [n, width]; last [B, width] is carried."""
    _cuda(h, mu, last, positions)
    B, T, E = h.shape
    assert h.is_contiguous() and mu.is_contiguous() and last.stride(1) == 1 and last.dtype == h.dtype
    out = torch.empty(mu.shape[0], B, T, E, dtype=h.dtype, device=h.device)
    with _on(h):
        _check(load().l3ci_token_shift(h.data_ptr(), mu.data_ptr(), last.data_ptr(), last.stride(0), positions.data_ptr(), out.data_ptr(),
                                       mu.shape[0], B, T, E, DTYPE_CODES[h.dtype], _stream(h)), "l3ci_token_shift")
    return out


def delta_inputs(p, b, a_proj, conv, a_log, dt_bias, tail, positions, H: int, G: int, D: int, V: int, unit_eps: float = 1e-6):
    """p [B, T, W] with columns q | k | v first, b [B, T, H] and a_proj [B, T, H * D] (any row stride), conv [taps, channels],
    tail [B, taps - 1, channels].  Returns qk [B, T, 2, G, D], v [B, T, H, V], beta [B, T, H], decay [B, T, H, D]."""
    _cuda(p, b, a_proj, tail, positions)
    B, T, _ = p.shape
    dev, f32 = p.device, torch.float32
    assert b.dtype == a_proj.dtype == p.dtype
    assert conv.is_contiguous() and tail[0].is_contiguous() and tail.dtype == p.dtype
    qk, beta = torch.empty(B, T, 2, G, D, dtype=f32, device=dev), torch.empty(B, T, H, dtype=f32, device=dev)
    decay, v = torch.empty(B, T, H, D, dtype=f32, device=dev), torch.empty(B, T, H, V, dtype=p.dtype, device=dev)
    a = DeltaInputsArgs(p=p.data_ptr(), b=b.data_ptr(), a=a_proj.data_ptr(), conv=conv.data_ptr(), a_log=a_log.data_ptr(),
                        dt_bias=dt_bias.data_ptr(), tail=tail.data_ptr(), positions=positions.data_ptr(), qk_out=qk.data_ptr(),
                        beta_out=beta.data_ptr(), decay_out=decay.data_ptr(), v_out=v.data_ptr(), p_st=_row_stride(p), b_st=_row_stride(b),
                        a_st=_row_stride(a_proj), tail_sb=tail.stride(0), B=B, T=T, H=H, G=G, D=D, V=V, taps=conv.shape[0],
                        dtype=DTYPE_CODES[p.dtype], unit_eps=unit_eps, stream=_stream(p))
    with _on(p):
        _check(load().l3ci_delta_inputs(C.byref(a)), "l3ci_delta_inputs")
    return qk, v, beta, decay


def recurrent_scan(q, k, v, g, state, positions, norm, gate, *, act: int, eps: float, beta=None, bonus=None, g_bias=None,
                   conv_in=None, tail=None, taps: int = 1, status=None):
    """q, k [B, T, G, D], v, gate [B, T, H, V], g [B, T, H, D], state [B, H, D, V] (fp32, carried), norm [V] or [H, V].  beta (delta rule) or bonus
    and g_bias (time mixing) choose the recurrence.  Returns the normed and gated output [B, T, H * V].  conv_in [B, T, W],
    tail: the convolution's inputs and its carried ones, moved on."""
    _cuda(q, k, v, g, state, positions, gate)
    B, T, H, V = v.shape
    G, D = q.shape[2:]
    out = torch.empty(B, T, H, V, dtype=v.dtype, device=v.device)
    assert _row_stride(k) == _row_stride(q) and k.stride(2) == q.stride(2) and gate.dtype == v.dtype and state.dtype == torch.float32 and state[0].is_contiguous()
    assert q.dtype == k.dtype == g.dtype == (torch.float32 if beta is not None else v.dtype) and norm.is_contiguous()
    a = RecurrentScanArgs(q=q.data_ptr(), k=k.data_ptr(), v=v.data_ptr(), g=g.data_ptr(), norm=norm.data_ptr(), gate=gate.data_ptr(),
                          state=state.data_ptr(), out=out.data_ptr(), positions=positions.data_ptr(), qk_st=_row_stride(q), qk_sh=q.stride(2),
                          v_st=_row_stride(v), v_sh=v.stride(2), g_st=_row_stride(g), g_sh=g.stride(2), gate_st=_row_stride(gate),
                          gate_sh=gate.stride(2), out_st=H * V, out_sh=V, norm_sh=V if norm.dim() == 2 else 0,
                          state_sb=state.stride(0), kind=0 if beta is not None else 1, B=B, T=T, H=H, G=G, D=D, V=V, act=act,
                          taps=taps, dtype=DTYPE_CODES[v.dtype], eps=eps, stream=_stream(v))
    for name, t in (("beta", beta), ("bonus", bonus), ("g_bias", g_bias)):
        if t is not None:
            assert t.is_contiguous() and t.dtype == torch.float32
            setattr(a, name, t.data_ptr())
    if status is not None:
        a.status = status.data_ptr()
    if tail is not None:
        assert tail[0].is_contiguous() and conv_in.dtype == tail.dtype == v.dtype
        a.conv_in, a.conv_st, a.tail, a.tail_sb = conv_in.data_ptr(), _row_stride(conv_in), tail.data_ptr(), tail.stride(0)
    with _on(v):
        _check(load().l3ci_recurrent_scan(C.byref(a)), "l3ci_recurrent_scan")
    return out.view(B, T, H * V)


def moe_route(logits, bias, top: int):
    """logits fp32 [rows, experts] -> experts, ranks (int32 [rows, top]), weights [rows, top], counts [experts]."""
    _cuda(logits, bias)
    rows, E = logits.shape
    assert logits.is_contiguous() and logits.dtype == bias.dtype == torch.float32
    i32 = dict(dtype=torch.int32, device=logits.device)
    experts, ranks, counts = torch.empty(rows, top, **i32), torch.empty(rows, top, **i32), torch.empty(E, **i32)
    weights = torch.empty(rows, top, dtype=torch.float32, device=logits.device)
    with _on(logits):
        _check(load().l3ci_moe_route(logits.data_ptr(), bias.data_ptr(), experts.data_ptr(), ranks.data_ptr(), weights.data_ptr(),
                                     counts.data_ptr(), rows, E, top, _stream(logits)), "l3ci_moe_route")
    return experts, ranks, weights, counts


def moe_gather(h, experts, ranks, counts):
    """h's rows in the order of the experts [rows * top, width], and the place of every (row, choice) pair."""
    _cuda(h, experts, ranks, counts)
    rows, top = experts.shape
    out = torch.empty(rows * top, h.shape[1], dtype=h.dtype, device=h.device)
    part_rows = torch.empty(rows, top, dtype=torch.int32, device=h.device)
    with _on(h):
        _check(load().l3ci_moe_gather(h.data_ptr(), experts.data_ptr(), ranks.data_ptr(), counts.data_ptr(), out.data_ptr(),
                                      part_rows.data_ptr(), rows, h.shape[1], counts.numel(), top, DTYPE_CODES[h.dtype], _stream(h)),
               "l3ci_moe_gather")
    return out, part_rows


def moe_gemm(x, w, counts, *, limit: float = 0.0, alpha: float = 1.702, variant: int = 0, status=None):
    """Sorted rows x [rows, K] times their expert's matrix: w [experts, N, K], or, gated, w [experts, 2, N, K] (gate, up)."""
    _cuda(x, w, counts)
    assert x.is_contiguous() and w.is_contiguous() and w.dtype == x.dtype and w.shape[-1] == x.shape[1]
    gated, N = int(w.dim() == 4), w.shape[-2]
    out = torch.empty(x.shape[0], N, dtype=x.dtype, device=x.device)
    a = MoeGemmArgs(x=x.data_ptr(), w=w.data_ptr(), out=out.data_ptr(), counts=counts.data_ptr(), rows=x.shape[0], K=x.shape[1], N=N,
                    n_experts=w.shape[0], gated=gated, dtype=DTYPE_CODES[x.dtype], variant=variant, limit=limit, alpha=alpha,
                    stream=_stream(x))
    if status is not None:
        a.status = status.data_ptr()
    with _on(x):
        _check(load().l3ci_moe_gemm(C.byref(a)), "l3ci_moe_gemm")
    return out


def latent_cache(qd, table, norm_weight, eps: float, cache, positions, heads: int, dim: int, rot_dim: int, rank: int):
    """qd [B, T, W]: rotates the query heads in place and writes the latent rows of `cache` [B, L, width]."""
    _cuda(qd, cache, positions)
    B, T, W = qd.shape
    assert qd.is_contiguous() and cache.stride(2) == 1 and cache.dtype == qd.dtype and cache.shape[0] == B
    with _on(qd):
        _check(load().l3ci_latent_cache(qd.data_ptr(), W, table.data_ptr(), table.shape[0], norm_weight.data_ptr(), eps,
                                        cache.data_ptr(), cache.stride(0), cache.stride(1), cache.shape[1],
                                        positions.data_ptr(), B, T, heads, dim, rot_dim, rank, DTYPE_CODES[qd.dtype],
                                        _stream(qd)), "l3ci_latent_cache")


def kv_cache_write(src, k_col: int, v_col: int, cache_k, cache_v, positions):
    """Columns of src [B, T, W] into cache_k, cache_v [B, L, heads, size] at the sequences' positions."""
    _cuda(src, cache_k, cache_v, positions)
    B, T, W = src.shape
    kw, vw = cache_k.shape[2] * cache_k.shape[3], cache_v.shape[2] * cache_v.shape[3]
    assert src.is_contiguous() and cache_k.dtype == cache_v.dtype == src.dtype and cache_k.shape[0] == B
    assert cache_k[0, 0].is_contiguous() and cache_v[0, 0].is_contiguous()
    with _on(src):
        _check(load().l3ci_kv_cache_write(src.data_ptr(), W, k_col, kw, v_col, vw, cache_k.data_ptr(), cache_k.stride(0),
                                          cache_k.stride(1), cache_v.data_ptr(), cache_v.stride(0), cache_v.stride(1),
                                          cache_k.shape[1], positions.data_ptr(), B, T, DTYPE_CODES[src.dtype],
                                          _stream(src)), "l3ci_kv_cache_write")


def attention(qa, ka, v, out, positions, *, qb=None, kb=None, maps: int = 1, scale: float, softcap: float = 0.0,
              temp_coef: float = 0.0, temp_every: float = 0.0, gate=None, lambda_: float = 0.0, post: float = 1.0,
              eps: float = 0.0, start_pos: int = -1, variant: int = 0, status=None, window: int = 0, keep_first: int = 0,
              bias_range: float = 0.0, sink: bool = False):
    """`l3ci_mixer_attention`.  qa [B, T, H, maps * Da], qb [B, T, H, Db], ka [B, S, G, maps * Da], kb [B, S, G, Db] (a
    part shared by the heads: a stride-0 head axis), v [B, S, G, Dv], out [B, T, H, Dv], gate [B, T, H]: any strides with
    a contiguous last axis (gate: contiguous heads)."""
    _cuda(qa, ka, v, out, positions)
    a = AttnArgs()
    a.B, a.T, a.H = qa.shape[:3]
    a.n_keys, a.G = ka.shape[1], ka.shape[2]
    a.maps, a.Da, a.Dv = maps, qa.shape[3] // maps, v.shape[3]
    a.Db = qb.shape[3] if qb is not None else 0

    def put(name, t, head_axis=True):
        assert t.dtype == qa.dtype and t.stride(-1) == 1, name
        short = {"out": "o", "gate": "g"}.get(name, name)
        setattr(a, name, t.data_ptr())
        setattr(a, short + "_sb", t.stride(0))
        setattr(a, short + "_st", t.stride(1))
        if head_axis:
            setattr(a, short + "_sh", t.stride(2))

    for name, t in (("qa", qa), ("qb", qb), ("ka", ka), ("kb", kb), ("v", v), ("out", out)):
        if t is not None:
            put(name, t)
    if gate is not None:
        put("gate", gate, head_axis=False)
    a.positions, a.dtype, a.start_pos, a.variant = positions.data_ptr(), DTYPE_CODES[qa.dtype], start_pos, variant
    a.status = status.data_ptr() if status is not None else None
    a.scale, a.softcap, a.temp_coef, a.temp_every = scale, softcap, temp_coef, temp_every
    a.lambda_, a.post, a.eps = lambda_, post, eps
    a.window, a.keep_first, a.bias_range, a.sink = window, keep_first, bias_range, int(sink)
    a.stream = _stream(qa)
    with _on(qa):
        need = load().l3ci_mixer_attention_scratch_bytes(C.byref(a))
        if need:
            scratch = torch.empty(need, dtype=torch.uint8, device=qa.device)
            a.scratch, a.scratch_bytes = scratch.data_ptr(), need
        _check(load().l3ci_mixer_attention(C.byref(a)), "l3ci_mixer_attention")
    return out
