"""Python mirror of the further sequence mixers (include/fa_b200_mixers.h): tensors in, tensors out, on the current stream.  T is
the activation type, bfloat16 or float32; there is no CPU path."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Optional

import torch

from . import _lib
from .row_ops import _DTYPE, _check, _check_rows, _out_rows, _p, _row_stride, _stream, _type, _workspace


def _mixers():
    return _lib.library("mixers")


def _check_rc(rc):
    _lib.check(rc, "mixers")


# ---- gated linear recurrences ----------------------------------------------------------------------------------
@dataclass(frozen=True)
class Sequences:
    """The sequences of a pass: state slots and first positions [n_seq] int32, cu_seqlens [n_seq + 1] int32 (None: one token
    each) with the longest sequence's tokens."""
    slots: torch.Tensor
    starts: torch.Tensor
    cu_seqlens: Optional[torch.Tensor] = None
    max_len: int = 1

    def check(self, status):
        for name, t in (("slots", self.slots), ("starts", self.starts), ("status", status)):
            _check(t, name, torch.int32)
        if self.starts.numel() != self.slots.numel():
            raise RuntimeError("starts must have one entry per sequence")
        if self.cu_seqlens is not None:
            _check(self.cu_seqlens, "cu_seqlens", torch.int32)
            if self.cu_seqlens.numel() != self.slots.numel() + 1:
                raise RuntimeError("cu_seqlens must have one entry more than slots")


def _recurrence_args(x, offsets, heads, groups, dk, dv, q_scale, state, seqs, status, norm, norm_eps, skip):
    T = _type(x, "x")
    _check(x, "x", T)
    _check(state, "state", torch.float32)
    if state.shape[1:] != (heads, dk, dv):
        raise RuntimeError(f"state must be [n_slots, {heads}, {dk}, {dv}]")
    seqs.check(status)
    if skip is not None:
        _check(skip, "skip", torch.float32)
        if skip.numel() != heads:
            raise RuntimeError("skip must have one entry per head")
    if norm is not None:
        _check(norm, "norm", torch.float32)
        if norm.shape != (state.size(0), 2, heads, dk):
            raise RuntimeError("norm must be [n_slots, 2, heads, dk]")
    out = torch.empty((x.size(0), heads * dv), dtype=T, device=x.device)
    off_q, off_k, off_v = offsets
    a = _lib.Recurrence(x=_p(x), stride=x.size(1), total=x.size(0), off_q=off_q, off_k=off_k, off_v=off_v, heads=heads, groups=groups, dk=dk, dv=dv,
                        n_slots=state.size(0), n_seq=seqs.slots.numel(), max_len=seqs.max_len, dtype=_DTYPE[T], q_scale=q_scale, norm_eps=norm_eps,
                        skip=_p(skip), norm=_p(norm), state=_p(state), slots=_p(seqs.slots), starts=_p(seqs.starts), cu_seqlens=_p(seqs.cu_seqlens),
                        out=_p(out), status=_p(status))
    return a, out


def recurrence(x, offsets, heads, groups, dk, dv, la, b, state, seqs, status, *, q_scale=1.0, floor=None, n0=None, norm=None, norm_eps=0.0, skip=None):
    """S = exp(la) S + b k v^T, y = S^T (q_scale q) per head and token, divided by max(|n . q|, floor) + norm_eps with `floor` (n follows S with k
    alone, from n0 [n_seq, heads, dk]; left in norm [n_slots, 2, heads, dk]), plus skip v.  x [tokens, stride] with q, k, v at the columns
    `offsets` (queries and keys of `groups` groups of heads); la, b, floor [heads, tokens] fp32; state [n_slots, heads, dk, dv] fp32, in
    place.  Returns [tokens, heads * dv]."""
    a, out = _recurrence_args(x, offsets, heads, groups, dk, dv, q_scale, state, seqs, status, norm, norm_eps, skip)
    for name, t in (("la", la), ("b", b), ("floor", floor)):
        if t is not None:
            _check(t, name, torch.float32)
            if t.shape != (heads, x.size(0)):
                raise RuntimeError(f"{name} must be [heads, tokens]")
    if floor is not None:
        _check(n0, "n0", torch.float32)
        if n0.shape != (seqs.slots.numel(), heads, dk) or norm is None:
            raise RuntimeError("floor needs n0 [n_seq, heads, dk] and norm")
        a.floor, a.n0 = _p(floor), _p(n0)
    a.la, a.b = _p(la), _p(b)
    ws = _workspace(_mixers().fam_recurrence_workspace(ctypes.byref(a)), x.device)
    if ws is not None:
        a.workspace, a.workspace_bytes = _p(ws), ws.numel()
    _check_rc(_mixers().fam_recurrence(ctypes.byref(a), _stream(x)))
    return out


def max_gates(x, off_i, off_f, bias_i, bias_f, cap, m, norm, seqs, status):
    """Gates with a running maximum: i = cap tanh((x_i + bias_i) / cap), f = logsigmoid(cap tanh((x_f + bias_f) / cap)), m' = max(f + m, i).
    Returns (la = f + m - m', b = e^(i - m'), floor = e^(-m')) [heads, tokens] and the normaliser before the call [n_seq, heads, dk]; m
    [n_slots, 2, heads] in place."""
    T = _type(x, "x")
    _check(x, "x", T)
    _check(bias_i, "bias_i", T)
    _check(bias_f, "bias_f", T)
    _check(m, "m", torch.float32)
    _check(norm, "norm", torch.float32)
    seqs.check(status)
    heads = bias_i.numel()
    if m.shape[1:] != (2, heads) or norm.shape[:3] != m.shape or bias_f.numel() != heads:
        raise RuntimeError("m must be [n_slots, 2, heads], norm [n_slots, 2, heads, dk], the biases [heads]")
    n_seq, dk = seqs.slots.numel(), norm.size(3)
    la, b, floor = torch.empty((3, heads, x.size(0)), dtype=torch.float32, device=x.device)
    n0 = torch.empty((n_seq, heads, dk), dtype=torch.float32, device=x.device)
    _check_rc(_mixers().fam_max_gates(
        _p(x), x.size(1), off_i, off_f, heads, _p(bias_i), _p(bias_f), cap, _p(m), _p(norm), _p(n0), dk, m.size(0), _p(seqs.slots), _p(seqs.starts),
        _p(seqs.cu_seqlens), n_seq, x.size(0), _p(la), _p(b), _p(floor), _p(status), _DTYPE[T], _stream(x)))
    return la, b, floor, n0


def step_gates(x, off, bias, a_log):
    """dt = softplus(x[:, off:] + bias); returns (la = -exp(a_log) dt, b = dt) [heads, tokens] fp32."""
    T = _type(x, "x")
    _check(x, "x", T)
    _check(bias, "bias", torch.float32)
    _check(a_log, "a_log", torch.float32)
    heads = bias.numel()
    if a_log.numel() != heads:
        raise RuntimeError("bias and a_log must have one entry per head")
    la, b = torch.empty((2, heads, x.size(0)), dtype=torch.float32, device=x.device)
    _check_rc(_mixers().fam_step_gates(_p(x), x.size(1), off, heads, _p(bias), _p(a_log), x.size(0), _p(la), _p(b), _DTYPE[T], _stream(x)))
    return la, b


def conv_silu(x, off, w, bias, ring, seqs, tok_seq, positions, status):
    """silu of the causal convolution per channel of x[:, off : off + channels]; w [taps, channels] (last row: the current token), ring
    [n_slots, taps, channels] with the inputs of earlier calls, in place.  Returns [tokens, channels]."""
    T = _type(x, "x")
    for name, t in (("x", x), ("w", w), ("bias", bias), ("ring", ring)):
        _check(t, name, T)
    for name, t in (("tok_seq", tok_seq), ("positions", positions)):
        _check(t, name, torch.int32)
        if t.numel() != x.size(0):
            raise RuntimeError(f"{name} must have one entry per token")
    seqs.check(status)
    taps, channels = w.shape
    if ring.shape[1:] != (taps, channels) or bias.numel() != channels:
        raise RuntimeError("ring must be [n_slots, taps, channels] and bias [channels]")
    out = torch.empty((x.size(0), channels), dtype=T, device=x.device)
    _check_rc(_mixers().fam_conv_silu(
        _p(x), x.size(1), off, channels, taps, _p(w), _p(bias), _p(ring), ring.size(0), _p(seqs.slots), _p(seqs.starts), _p(seqs.cu_seqlens), _p(tok_seq),
        _p(positions), seqs.slots.numel(), x.size(0), _p(out), _p(status), _DTYPE[T], _stream(x)))
    return out


def recurrence_step_supported(dk, dv):
    """Whether the one-kernel decode steps are built for these sizes."""
    return bool(_mixers().fam_recurrence_step_supported(dk, dv))


def max_gate_step(x, offsets, heads, dk, dv, off_i, off_f, bias_i, bias_f, cap, state, norm, m, seqs, status, *, q_scale, norm_eps):
    """`max_gates` and `recurrence` of one token per sequence in one kernel."""
    a, out = _recurrence_args(x, offsets, heads, heads, dk, dv, q_scale, state, seqs, status, norm, norm_eps, None)
    _check(bias_i, "bias_i", x.dtype)
    _check(bias_f, "bias_f", x.dtype)
    _check(m, "m", torch.float32)
    if m.shape != (state.size(0), 2, heads):
        raise RuntimeError("m must be [n_slots, 2, heads]")
    _check_rc(_mixers().fam_max_gate_step(ctypes.byref(a), off_i, off_f, _p(bias_i), _p(bias_f), cap, _p(m), _stream(x)))
    return out


def ssd_step(x, off_x, heads, groups, dk, dv, off_dt, dt_bias, a_log, skip, conv_w, conv_b, ring, state, seqs, status):
    """`conv_silu`, `step_gates` and `recurrence` of one token per sequence in one kernel; x holds v | k | q from column off_x on."""
    off_k = off_x + heads * dv
    a, out = _recurrence_args(x, (off_k + groups * dk, off_k, off_x), heads, groups, dk, dv, 1.0, state, seqs, status, None, 0.0, skip)
    for name, t in (("conv_w", conv_w), ("conv_b", conv_b), ("ring", ring)):
        _check(t, name, x.dtype)
    for name, t in (("dt_bias", dt_bias), ("a_log", a_log)):
        _check(t, name, torch.float32)
    if ring.shape != (state.size(0),) + conv_w.shape or conv_w.size(1) != heads * dv + 2 * groups * dk:
        raise RuntimeError("ring must be [n_slots, taps, channels], conv_w [taps, channels]")
    _check_rc(_mixers().fam_ssd_step(ctypes.byref(a), off_dt, _p(dt_bias), _p(a_log), _p(conv_w), _p(conv_b), _p(ring), conv_w.size(0), _stream(x)))
    return out


# ---- attention on paged keys and values ----------------------------------------------------------------------------
@dataclass(frozen=True)
class Pages:
    """Pools [n_blocks, kv_heads, 16, dim] and [n_blocks, kv_heads, 16, vdim] behind block_table [n_seq, max_blocks]; rows of a
    pass are the tokens at `positions` of the sequences `tok_seq`."""
    k_pool: torch.Tensor
    v_pool: torch.Tensor
    block_table: torch.Tensor
    tok_seq: torch.Tensor
    positions: torch.Tensor
    status: torch.Tensor

    def args(self, heads):
        T = _type(self.k_pool, "k_pool")
        _check(self.k_pool, "k_pool", T)
        _check(self.v_pool, "v_pool", T)
        for name, t in (("block_table", self.block_table), ("tok_seq", self.tok_seq), ("positions", self.positions), ("status", self.status)):
            _check(t, name, torch.int32, contiguous=name != "block_table")
        bt = self.block_table
        if bt.stride(1) != 1 or (bt.size(0) > 1 and bt.stride(0) != bt.size(1)):
            raise RuntimeError("block_table rows must be contiguous")
        n_blocks, kv_heads, page, dim = self.k_pool.shape
        if self.v_pool.shape[:3] != (n_blocks, kv_heads, 16) or page != 16:
            raise RuntimeError("pools must be [n_blocks, kv_heads, 16, dim] and [n_blocks, kv_heads, 16, vdim]")
        if self.positions.numel() != self.tok_seq.numel():
            raise RuntimeError("tok_seq and positions must have one entry per token")
        return _lib.Pages(k_pool=_p(self.k_pool), v_pool=_p(self.v_pool), block_table=_p(bt), tok_seq=_p(self.tok_seq), positions=_p(self.positions),
                          n_blocks=n_blocks, max_blocks=bt.size(1), n_seq=bt.size(0), heads=heads, kv_heads=kv_heads, dim=dim,
                          vdim=self.v_pool.size(3), dtype=_DTYPE[T], rows=self.tok_seq.numel(), status=_p(self.status))


def kv_prep(pages, x, offsets, heads, wq, wk, eps, *, v_first=None, lam=0.0, contiguous_kv=False):
    """RMS norms of queries and keys over all heads at once, values mixed with v_first ((1 - lam) v + lam v_first, [rows, kv_heads * vdim] with
    any row stride), append to the pages.  Returns (queries [rows, heads * dim], keys, values), the last two None without
    `contiguous_kv`."""
    a = pages.args(heads)
    T = _type(x, "x")
    for name, t in (("x", x), ("wq", wq), ("wk", wk), ("pools", pages.k_pool)):
        _check(t, name, T)
    rows = x.size(0)
    if rows != a.rows or wq.numel() != heads * a.dim or wk.numel() != a.kv_heads * a.dim:
        raise RuntimeError("x must have one row per token, the norm weights one element per column")
    if v_first is not None:
        _check_rows(v_first, "v_first", T, rows, a.kv_heads * a.vdim)
    new = lambda n: torch.empty((rows, n), dtype=T, device=x.device)
    q = new(heads * a.dim)
    k, v = (new(a.kv_heads * a.dim), new(a.kv_heads * a.vdim)) if contiguous_kv else (None, None)
    _check_rc(_mixers().fam_kv_prep(ctypes.byref(a), _p(x), x.size(1), *offsets, _p(wq), _p(wk), eps, _p(v_first),
                                    _row_stride(v_first) if v_first is not None else 0, lam, _p(q), _p(k), _p(v), _stream(x)))
    return q, k, v


def _attention_rows(q, gate, out, rows, cols, T):
    if gate is not None:
        _check_rows(gate, "gate", T, rows, cols)
    return _out_rows(out, "out", T, rows, cols, q.device)


def kv_attention(pages, q, heads, chunk, scale, *, slopes=None, gate=None, out=None):
    """Every row attends to the cached keys of its chunk up to its own position; scores scale (q . k) - slopes_h distance; the result times
    sigmoid(gate), [rows, heads * vdim]."""
    a = pages.args(heads)
    T = _type(q, "q")
    _check(q, "q", T)
    _check(pages.k_pool, "k_pool", T)
    if q.shape != (a.rows, heads * a.dim):
        raise RuntimeError("q must be [rows, heads * dim]")
    if slopes is not None:
        _check(slopes, "slopes", torch.float32)
        if slopes.numel() != heads:
            raise RuntimeError("slopes must have one entry per head")
    out = _attention_rows(q, gate, out, a.rows, heads * a.vdim, T)
    ws = _workspace(_mixers().fam_kv_attention_workspace(ctypes.byref(a), chunk), q.device)
    _check_rc(_mixers().fam_kv_attention(ctypes.byref(a), _p(q), _p(slopes), _p(gate), _row_stride(gate) if gate is not None else 0, chunk, scale, _p(out),
                                         _row_stride(out), _p(ws), ws.numel() if ws is not None else 0, _stream(q)))
    return out


def kv_gather(pages, heads, piece_seq, piece_key0, cu_kv, total_kv):
    """The cached keys and values of pieces of sequences as contiguous rows [total_kv, ...]: piece i starts at position piece_key0[i] of
    sequence piece_seq[i]."""
    a = pages.args(heads)
    for name, t in (("piece_seq", piece_seq), ("piece_key0", piece_key0), ("cu_kv", cu_kv)):
        _check(t, name, torch.int32)
    if piece_key0.numel() != piece_seq.numel() or cu_kv.numel() != piece_seq.numel() + 1:
        raise RuntimeError("cu_kv must have one entry more than there are pieces")
    k = torch.empty((total_kv, a.kv_heads * a.dim), dtype=pages.k_pool.dtype, device=cu_kv.device)
    v = torch.empty((total_kv, a.kv_heads * a.vdim), dtype=pages.k_pool.dtype, device=cu_kv.device)
    _check_rc(_mixers().fam_kv_gather(ctypes.byref(a), _p(piece_seq), _p(piece_key0), _p(cu_kv), piece_seq.numel(), total_kv, _p(k), _p(v), _stream(cu_kv)))
    return k, v


def kv_prefill_supported(heads, kv_heads, dim, vdim, scale, dtype):
    """Whether `kv_prefill` is built for these sizes."""
    return dtype in _DTYPE and bool(_mixers().fam_kv_prefill_supported(heads, kv_heads, dim, vdim, scale, _DTYPE[dtype]))


def kv_prefill(q, k, v, cu_q, cu_kv, max_q, heads, kv_heads, scale, slopes, status, *, gate=None, out=None):
    """Prompt attention (bfloat16) on contiguous rows: a piece's queries are its last keys, causal; scores, gate and result as
    `kv_attention`.  q [total_q, heads * dim], k [total_kv, kv_heads * dim], v [total_kv, kv_heads * vdim]."""
    T = torch.bfloat16
    for name, t in (("q", q), ("k", k), ("v", v)):
        _check(t, name, T)
    for name, t in (("cu_q", cu_q), ("cu_kv", cu_kv), ("status", status)):
        _check(t, name, torch.int32)
    _check(slopes, "slopes", torch.float32)
    dim, vdim = k.size(1) // kv_heads, v.size(1) // kv_heads
    if q.size(1) != heads * dim or v.size(0) != k.size(0) or slopes.numel() != heads or cu_q.numel() != cu_kv.numel():
        raise RuntimeError("q, k, v, slopes and the offsets do not fit")
    out = _attention_rows(q, gate, out, q.size(0), heads * vdim, T)
    _check_rc(_mixers().fam_kv_prefill(
        _p(q), _p(k), _p(v), _p(cu_q), _p(cu_kv), cu_q.numel() - 1, max_q, q.size(0), k.size(0), heads, kv_heads, dim, vdim, scale, _p(slopes), _p(gate),
        _row_stride(gate) if gate is not None else 0, _p(out), _row_stride(out), _p(status), _stream(q)))
    return out
