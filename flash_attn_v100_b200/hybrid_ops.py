"""Python mirror of the hybrid decoder's operators (include/fa_b200_hybrid.h): tensors in, tensors out, on the current
stream.  T is the activation type, bfloat16 or float32; there is no CPU path."""
from __future__ import annotations

import torch

from . import _lib
from .row_ops import _DTYPE, _check, _p, _stream, _type, _workspace
from .row_ops import clamped_glu, gated_norm, residual_norm, side_gate  # noqa: F401  (the row-wise operators of the same decoder)


def _check_rc(rc):
    _lib.check(rc, "hybrid")


def lightning(qkv, offsets, heads, dk, dv, decay, state, slots, starts, status, *, cu_seqlens=None, max_len=0):
    """Decayed linear attention over packed prompts (cu_seqlens [n_seq + 1], the longest of max_len tokens) or one token per
    sequence.
    qkv [tokens, stride], offsets = columns of q, k, v; state [n_slots, heads, dk, dv] fp32, updated in place;
    slots / starts [n_seq].  Returns [tokens, heads * dv]."""
    T = _type(qkv, "qkv")
    _check(qkv, "qkv", T)
    _check(state, "state", torch.float32)
    _check(decay, "decay", torch.float32)
    for name, t in (("slots", slots), ("starts", starts), ("status", status)):
        _check(t, name, torch.int32)
    if state.shape[1:] != (heads, dk, dv) or decay.numel() != heads:
        raise RuntimeError("state must be [n_slots, heads, dk, dv] and decay [heads]")
    n_seq = slots.numel()
    if cu_seqlens is not None:
        _check(cu_seqlens, "cu_seqlens", torch.int32)
        if cu_seqlens.numel() != n_seq + 1:
            raise RuntimeError("cu_seqlens must have one entry more than slots")
    if starts.numel() != n_seq:
        raise RuntimeError("starts must have one entry per sequence")
    tokens = qkv.size(0)
    out = torch.empty((tokens, heads * dv), dtype=T, device=qkv.device)
    lib, ws = _lib.library("hybrid"), None
    if cu_seqlens is not None:
        ws = _workspace(lib.fah_lightning_workspace(n_seq, heads, dk, dv, max_len, _DTYPE[T]), qkv.device)
    _check_rc(lib.fah_lightning(
        _p(qkv), qkv.size(1), *offsets, heads, dk, dv, _p(decay), _p(state), state.size(0), _p(slots), _p(starts), _p(cu_seqlens), n_seq, max_len,
        tokens, _p(out), _p(ws), ws.numel() if ws is not None else 0, _p(status), _DTYPE[T], _stream(qkv)))
    return out


def _check_paging(pool, block_table, tok_seq, positions, status):
    for name, t in (("block_table", block_table), ("tok_seq", tok_seq), ("positions", positions), ("status", status)):
        _check(t, name, torch.int32, contiguous=name != "block_table")
    if block_table.stride(1) != 1 or block_table.stride(0) != block_table.size(1):
        raise RuntimeError("block_table rows must be contiguous")
    if pool.dim() != 3 or pool.size(1) != 16:
        raise RuntimeError("pool must be [n_blocks, 16, stride]")


def latent_prep(down, off_q, q_rank, off_kv, kv_rank, off_r, rot_dim, wq, wkv, eps, cos, sin, pool, block_table, tok_seq, positions, status,
                *, contiguous_kv=False):
    """Norms of the query and key/value latents, rotation of the shared key part, append of (latent, rotated part) to the
    pages.  Returns (normed query latent [rows, q_rank], latent [rows, kv_rank] or None, rotated part or None)."""
    T = _type(down, "down")
    for name, t in (("down", down), ("wq", wq), ("wkv", wkv), ("pool", pool)):
        _check(t, name, T)
    for name, t in (("cos", cos), ("sin", sin)):
        _check(t, name, torch.float32)
    _check_paging(pool, block_table, tok_seq, positions, status)
    rows = down.size(0)
    if tok_seq.numel() != rows or positions.numel() != rows or cos.shape != (rows, rot_dim // 2) or sin.shape != cos.shape:
        raise RuntimeError("tok_seq, positions, cos and sin must have one row per token")
    new = lambda n: torch.empty((rows, n), dtype=T, device=down.device)
    cq = new(q_rank)
    c, r = (new(kv_rank), new(rot_dim)) if contiguous_kv else (None, None)
    _check_rc(_lib.library("hybrid").fah_latent_prep(
        _p(down), down.size(1), off_q, q_rank, off_kv, kv_rank, off_r, rot_dim, _p(wq), _p(wkv), eps, _p(cos), _p(sin), _p(cq), _p(c), _p(r),
        _p(pool), pool.size(2), pool.size(0), _p(block_table), block_table.size(1), block_table.size(0), _p(tok_seq), _p(positions), rows,
        _p(status), _DTYPE[T], _stream(down)))
    return cq, c, r


def rotate_heads_(q, cos, sin, heads, head_stride, off, rot_dim):
    """Rotates columns [off, off + rot_dim) of every head of q [rows, heads * head_stride] in place."""
    T = _type(q, "q")
    _check(q, "q", T)
    _check(cos, "cos", torch.float32)
    _check(sin, "sin", torch.float32)
    if q.size(1) != heads * head_stride or cos.shape != (q.size(0), rot_dim // 2) or sin.shape != cos.shape:
        raise RuntimeError("q must be [rows, heads * head_stride], cos and sin [rows, rot_dim / 2]")
    _check_rc(_lib.library("hybrid").fah_rotate_heads(_p(q), _p(cos), _p(sin), q.size(0), heads, head_stride, off, rot_dim, _DTYPE[T],
                                                          _stream(q)))
    return q


def latent_attention(q_abs, q, q_off, cos, sin, pool, block_table, tok_seq, positions, gate, kv_rank, rot_dim, scale, status):
    """Attention over cached latent rows: q_abs [rows, heads, kv_rank], q [rows, heads, n] with the part to rotate at column
    q_off; every row sees the keys 0 .. positions[row].  gate [rows, heads] (any row stride) or None.
    Returns the weighted latents [rows, heads, kv_rank]."""
    T = _type(q_abs, "q_abs")
    for name, t in (("q_abs", q_abs), ("q", q), ("pool", pool)):
        _check(t, name, T)
    _check(cos, "cos", torch.float32)
    _check(sin, "sin", torch.float32)
    _check_paging(pool, block_table, tok_seq, positions, status)
    rows, heads, _ = q_abs.shape
    if q.shape[:2] != (rows, heads) or tok_seq.numel() != rows or positions.numel() != rows or cos.shape != (rows, rot_dim // 2):
        raise RuntimeError("q, tok_seq, positions, cos and sin must have one row per query")
    if gate is not None:
        _check(gate, "gate", T, contiguous=False)
        if gate.shape != (rows, heads) or gate.stride(1) != 1:
            raise RuntimeError("gate must be [rows, heads] with contiguous rows")
    out = torch.empty_like(q_abs)
    lib = _lib.library("hybrid")
    ws = _workspace(lib.fah_latent_attention_workspace(heads, kv_rank, rot_dim, rows, _DTYPE[T]), q_abs.device)
    _check_rc(lib.fah_latent_attention(
        _p(q_abs), _p(q), q.size(2), q_off, _p(cos), _p(sin), _p(pool), pool.size(2), pool.size(0), _p(block_table), block_table.size(1),
        block_table.size(0), _p(tok_seq), _p(positions), _p(gate), gate.stride(0) if gate is not None else 0, heads, kv_rank, rot_dim, scale,
        _p(out), rows, _p(ws), ws.numel() if ws is not None else 0, _p(status), _DTYPE[T], _stream(q_abs)))
    return out


def latent_prefill_supported(dim, rot_dim, vdim, scale, dtype):
    """Whether `latent_prefill` is built for these sizes."""
    return dtype in _DTYPE and bool(_lib.library("hybrid").fah_latent_prefill_supported(dim, rot_dim, vdim, scale, _DTYPE[dtype]))


def latent_prefill(q, kv, kr, gate, cu_q, cu_kv, max_q, heads, dim, vdim, scale, status):
    """Causal prompt attention on expanded latents (bfloat16): q [total_q, heads * (dim + rot_dim)] rotated, kv [total_kv,
    heads * (dim + vdim)] = keys | values, kr [total_kv, rot_dim].  A sequence's queries are its last keys.
    Returns [total_q, heads * vdim], head h times sigmoid(gate[:, h])."""
    T = torch.bfloat16
    for name, t in (("q", q), ("kv", kv), ("kr", kr)):
        _check(t, name, T)
    for name, t in (("cu_q", cu_q), ("cu_kv", cu_kv), ("status", status)):
        _check(t, name, torch.int32)
    rot_dim = kr.size(1)
    if q.size(1) != heads * (dim + rot_dim) or kv.shape != (kr.size(0), heads * (dim + vdim)) or cu_q.numel() != cu_kv.numel():
        raise RuntimeError("q, kv and kr do not fit the head sizes")
    if gate is not None:
        _check(gate, "gate", T, contiguous=False)
        if gate.shape != (q.size(0), heads) or gate.stride(1) != 1:
            raise RuntimeError("gate must be [total_q, heads] with contiguous rows")
    out = torch.empty((q.size(0), heads * vdim), dtype=T, device=q.device)
    _check_rc(_lib.library("hybrid").fah_latent_prefill(
        _p(q), _p(kv), _p(kr), _p(gate), gate.stride(0) if gate is not None else 0, _p(cu_q), _p(cu_kv), cu_q.numel() - 1, max_q, q.size(0),
        kv.size(0), heads, dim, rot_dim, vdim, scale, _p(out), _p(status), _stream(q)))
    return out


def latent_gather(pool, block_table, cu_kv, total_kv, kv_rank, rot_dim, status):
    """The cached latent rows of every sequence as contiguous rows: ([total_kv, kv_rank], [total_kv, rot_dim])."""
    T = _type(pool, "pool")
    _check(pool, "pool", T)
    for name, t in (("cu_kv", cu_kv), ("status", status), ("block_table", block_table)):
        _check(t, name, torch.int32)
    if block_table.size(0) != cu_kv.numel() - 1:
        raise RuntimeError("cu_kv must have one entry more than block_table has rows")
    c = torch.empty((total_kv, kv_rank), dtype=T, device=pool.device)
    r = torch.empty((total_kv, rot_dim), dtype=T, device=pool.device)
    _check_rc(_lib.library("hybrid").fah_latent_gather(
        _p(pool), pool.size(2), pool.size(0), _p(block_table), block_table.size(1), block_table.size(0), _p(cu_kv), total_kv, kv_rank, rot_dim,
        _p(c), _p(r), _p(status), _DTYPE[T], _stream(pool)))
    return c, r
