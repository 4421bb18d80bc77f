"""Python mirror of the row-wise operators (include/fa_b200_rows.h): tensors in, tensors out, on the current stream.  T is the
activation type, bfloat16 or float32; there is no CPU path."""
from __future__ import annotations

import ctypes

import torch

from . import _lib

_DTYPE = {torch.float32: 0, torch.bfloat16: 1}


def _p(t):
    return None if t is None else ctypes.c_void_p(t.data_ptr())


def _stream(t):
    return ctypes.c_void_p(torch.cuda.current_stream(t.device).cuda_stream)


def _check(t, name, dtype, contiguous=True):
    if not t.is_cuda:
        raise RuntimeError(f"{name} must be a CUDA tensor")
    if t.dtype != dtype:
        raise RuntimeError(f"{name} must be {dtype}, got {t.dtype}")
    if contiguous and not t.is_contiguous():
        raise RuntimeError(f"{name} must be contiguous")


def _workspace(nbytes, device):
    return torch.empty(nbytes, dtype=torch.uint8, device=device) if nbytes else None


def _type(t, name):
    if t.dtype not in _DTYPE:
        raise RuntimeError(f"{name} must be bfloat16 or float32, got {t.dtype}")
    return t.dtype


def _check_rows(t, name, dtype, rows, cols):
    """A [rows, cols] matrix with contiguous rows at any stride."""
    _check(t, name, dtype, contiguous=False)
    if t.shape != (rows, cols) or t.stride(1) != 1 or (rows > 1 and t.stride(0) < cols):
        raise RuntimeError(f"{name} must be [{rows}, {cols}] with contiguous rows")


def _out_rows(out, name, dtype, rows, cols, device):
    if out is None:
        return torch.empty((rows, cols), dtype=dtype, device=device)
    _check_rows(out, name, dtype, rows, cols)
    return out


def _row_stride(t):
    return max(t.stride(0), t.size(1))      # (the stride of a single row says nothing)


def _check_rc(rc):
    _lib.check(rc, "rows")


def residual_norm(x, w=None, eps=1e-5, *, delta=None, delta_w=None, embed=None, tokens=None, init=False, embed_scale=1.0, more=(), w2=None,
                  out=True, dtype=None):
    """x [rows, cols] fp32, in place: x = embed[tokens] * embed_scale + table[index] for every (table, int32 index) of `more` (`init`),
    or x += embed[tokens], then x += delta or x += rmsnorm(delta) * delta_w.  Returns rmsnorm(x) * w, or x itself when w is
    None, in the activation type, with w2 a pair with rmsnorm(x) * w2; None when `out` is False."""
    _check(x, "x", torch.float32)
    like = next((t for t in (delta, embed, w) if t is not None), None)
    T = dtype or (_type(like, "delta / embed / w") if like is not None else None)
    if T is None:
        raise RuntimeError("residual_norm needs dtype when neither delta, embed nor w is given")
    for name, t in (("delta", delta), ("delta_w", delta_w), ("embed", embed), ("w", w), ("w2", w2)):
        if t is not None:
            _check(t, name, T)
    rows, cols = x.shape
    if delta is not None and delta.shape != x.shape:
        raise RuntimeError("delta must have the shape of x")
    for name, t in (("delta_w", delta_w), ("w", w), ("w2", w2)):
        if t is not None and t.numel() != cols:
            raise RuntimeError(f"{name} must have {cols} elements")
    if embed is not None:
        _check(tokens, "tokens", torch.int64)
        if tokens.numel() != rows or embed.size(1) != cols:
            raise RuntimeError("tokens must have one entry per row and embed the width of x")
    if (more or embed_scale != 1.0) and not init:
        raise RuntimeError("embed_scale and further tables go with init")
    new = lambda: torch.empty((rows, cols), dtype=T, device=x.device)
    res, res2 = new() if out else None, new() if out and w2 is not None else None
    a = _lib.ResidualNorm(x=_p(x), delta=_p(delta), delta_w=_p(delta_w), embed=_p(embed), tokens=_p(tokens) if embed is not None else None,
                          embed_mode=0 if embed is None else (2 if init else 1), vocab=embed.size(0) if embed is not None else 0,
                          embed_scale=embed_scale, eps=eps, w=_p(w) if out else None, w2=_p(w2) if out else None, out=_p(res), out2=_p(res2),
                          rows=rows, cols=cols, dtype=_DTYPE[T])
    for k, (table, index) in enumerate(more):
        _check(table, "table", T)
        _check(index, "index", torch.int32)
        if index.numel() != rows or table.size(1) != cols:
            raise RuntimeError("an index must have one entry per row and its table the width of x")
        a.more[k], a.more_rows[k], a.more_n[k] = table.data_ptr(), index.data_ptr(), table.size(0)
    _check_rc(_lib.library("rows").far_residual_norm(ctypes.byref(a), _stream(x)))
    return res if w2 is None else (res, res2)


def gated_norm(o, g, w, eps, *, group=0, silu_first=False, out=None):
    """rmsnorm(o) * w * sigmoid(g), or rmsnorm(o * silu(g)) * w (`silu_first`); the norm is taken over every `group` columns (0: the
    whole row).  o [rows, cols], g and `out` [rows, cols] with any row stride."""
    T = _type(o, "o")
    _check(o, "o", T)
    _check(w, "w", T)
    rows, cols = o.shape
    _check_rows(g, "g", T, rows, cols)
    if w.numel() != cols:
        raise RuntimeError("w must have one element per column")
    out = _out_rows(out, "out", T, rows, cols, o.device)
    _check_rc(_lib.library("rows").far_gated_norm(_p(o), _p(g), _row_stride(g), _p(w), _p(out), _row_stride(out), rows, cols, group or cols,
                                                  int(silu_first), eps, _DTYPE[T], _stream(o)))
    return out


def gelu(z, *, out=None):
    """gelu_tanh(z); z and `out` [rows, n] with any row stride."""
    T = _type(z, "z")
    rows, n = z.shape
    _check_rows(z, "z", T, rows, n)
    out = _out_rows(out, "out", T, rows, n, z.device)
    _check_rc(_lib.library("rows").far_gelu(_p(z), _row_stride(z), _p(out), _row_stride(out), rows, n, _DTYPE[T], _stream(z)))
    return out


def bigram_rows(tokens, starts, slots, last, buckets, mul_prev, mul_cur, status, *, cu_seqlens=None):
    """int32 row of a bigram table for every token: (previous * mul_prev + token * mul_cur) mod buckets, `buckets` for the first token
    of a sequence; last [n_slots] int32 holds the token before the call and receives the call's last."""
    _check(tokens, "tokens", torch.int64)
    for name, t in (("starts", starts), ("slots", slots), ("last", last), ("status", status)):
        _check(t, name, torch.int32)
    n_seq = slots.numel()
    if cu_seqlens is not None:
        _check(cu_seqlens, "cu_seqlens", torch.int32)
    if starts.numel() != n_seq or (cu_seqlens is not None and cu_seqlens.numel() != n_seq + 1):
        raise RuntimeError("starts, slots and cu_seqlens must describe the same sequences")
    out = torch.empty(tokens.numel(), dtype=torch.int32, device=tokens.device)
    _check_rc(_lib.library("rows").far_bigram_rows(_p(tokens), _p(cu_seqlens), _p(starts), _p(slots), _p(last), last.numel(), n_seq, tokens.numel(),
                                                   buckets, mul_prev, mul_cur, _p(out), _p(status), _stream(tokens)))
    return out


def clamped_glu(gu, limit, alpha, shift):
    """gu [rows, 2n] = gate | linear branch: g sigmoid(alpha g) (u + shift) of the clamped branches."""
    T = _type(gu, "gu")
    _check(gu, "gu", T)
    n = gu.size(1) // 2
    out = torch.empty((gu.size(0), n), dtype=T, device=gu.device)
    _check_rc(_lib.library("rows").far_clamped_glu(_p(gu), _p(out), gu.size(0), n, limit, alpha, shift, _DTYPE[T], _stream(gu)))
    return out


def side_gate(z, side, tokens, off):
    """gelu_tanh(z) * side[tokens, off : off + n]; z [rows, n]."""
    T = _type(z, "z")
    _check(z, "z", T)
    _check(side, "side", T)
    _check(tokens, "tokens", torch.int64)
    if tokens.numel() != z.size(0):
        raise RuntimeError("tokens must have one entry per row")
    out = torch.empty_like(z)
    _check_rc(_lib.library("rows").far_side_gate(_p(z), _p(side), _p(tokens), side.size(0), side.size(1), off, _p(out), z.size(0),
                                                 z.size(1), _DTYPE[T], _stream(z)))
    return out
