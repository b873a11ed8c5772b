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
           "l3ci_mixer_attention_variant")

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
        *[(n, C.c_int32) for n in ("dtype", "B", "T", "H", "G", "maps", "Da", "Db", "Dv", "n_keys", "start_pos", "variant")],
        *[(n, C.c_float) for n in ("scale", "softcap", "temp_coef", "temp_every", "lambda_", "post", "eps")],
        ("stream", C.c_void_p),
    ]


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
              eps: float = 0.0, start_pos: int = -1, variant: int = 0, status=None):
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
    a.stream = _stream(qa)
    with _on(qa):
        need = load().l3ci_mixer_attention_scratch_bytes(C.byref(a))
        if need:
            scratch = torch.empty(need, dtype=torch.uint8, device=qa.device)
            a.scratch, a.scratch_bytes = scratch.data_ptr(), need
        _check(load().l3ci_mixer_attention(C.byref(a)), "l3ci_mixer_attention")
    return out
