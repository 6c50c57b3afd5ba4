"""Launchers between a layer's input projections and its output (``csrc/mixer_post.cu``, ``rglru.cu``, the step in
``gemv_float.cu``): head rows to query buffer and pages, the short convolution, the gated linear recurrence."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Optional

import torch

from ..core import native as N
from .kernels import _check_device, _dt, _p, _stream

c_vp, c_ll, c_int = C.c_void_p, C.c_longlong, C.c_int
NORM_CODES = {"none": 0, "head": 1, "rows": 2, "unit": 3}


class _HeadRows(C.Structure):
    _fields_ = [("x", c_vp), ("stride", c_ll), ("bias", c_vp), ("gain", c_vp), ("heads", c_int), ("dim", c_int),
                ("gain_heads", c_int)]


class _PostArgs(C.Structure):
    _fields_ = [("q", _HeadRows), ("k", _HeadRows), ("v", _HeadRows), ("freq", c_vp), ("q_out", c_vp), ("kv_cache", c_vp),
                ("block_table", c_vp), ("slot", c_vp), ("pos", c_vp), ("cx", c_vp), ("cx_stride", c_ll), ("cx_bias", c_vp),
                ("cw", c_vp), ("cb", c_vp), ("cstate", c_vp), ("cjournal", c_vp), ("seg_start", c_vp), ("seg_slot", c_vp),
                ("tok_seg", c_vp), ("u", c_vp), ("u_ts", c_ll), ("u_bs", c_ll), ("C", c_int), ("block_cols", c_int),
                ("taps", c_int), ("n_slots", c_int), ("T", c_int), ("in_dtype", c_int), ("out_f32", c_int), ("norm", c_int),
                ("rot_dims", c_int), ("halves", c_int), ("D", c_int), ("page", c_int), ("max_pages", c_int),
                ("heads_per_cta", c_int), ("conv_tokens", c_int), ("eps", C.c_float), ("amp", C.c_float)]


class _RglruArgs(C.Structure):
    _fields_ = [("g", c_vp), ("g_ts", c_ll), ("g_bs", c_ll), ("gw", c_vp), ("gb", c_vp), ("decay", c_vp), ("u", c_vp),
                ("u_ts", c_ll), ("u_bs", c_ll), ("y", c_vp), ("yb", c_vp), ("x", c_vp), ("xb", c_vp), ("row_stride", c_ll),
                ("S", c_vp), ("cstate", c_vp), ("journal", c_vp), ("seg_start", c_vp), ("seg_slot", c_vp), ("out", c_vp),
                ("out_stride", c_ll), ("C", c_int), ("block_cols", c_int), ("taps", c_int), ("n_slots", c_int),
                ("n_seg", c_int), ("T", c_int), ("row_dtype", c_int), ("act_f32", c_int)]


_ABI_OK = False


def _lib():
    global _ABI_OK
    L = N.lib()
    if not _ABI_OK:
        for fn, st in (("he_mixer_post_args_size", _PostArgs), ("he_rglru_args_size", _RglruArgs)):
            if hasattr(L, fn) and getattr(L, fn)() != C.sizeof(st):      # a library built from a subset of the sources lacks some
                raise RuntimeError(f"ABI mismatch for {st.__name__}: C={getattr(L, fn)()} Python={C.sizeof(st)}")
        _ABI_OK = True
    return L


@dataclass
class HeadRows:
    """One projection's rows: ``x`` [T, heads * dim, padded to eight columns] (a column range of a wider buffer is fine)."""
    x: torch.Tensor
    heads: int
    dim: int
    bias: Optional[torch.Tensor] = None     # fp32, padded like x
    gain: Optional[torch.Tensor] = None     # fp32: [dim] or [heads, dim] (norm "head"), or padded like x (norm "rows")


@dataclass
class ConvRows:
    """Inputs of a recurrence on their way through the convolution to ``u`` [T, blocks, block_cols] (any strides)."""
    x: torch.Tensor
    bias: torch.Tensor                      # fp32 [C]
    w: torch.Tensor                         # fp32 [taps, C], oldest first
    conv_bias: torch.Tensor                 # fp32 [C]
    u: torch.Tensor
    state: Optional[torch.Tensor] = None    # fp32 [n_slots, taps - 1, C]; None: one tap
    journal: Optional[torch.Tensor] = None  # fp32 [T, taps - 1, C]


def mixer_post(q: HeadRows, k: Optional[HeadRows], v: Optional[HeadRows], norm: str, rot, freq: torch.Tensor, amp: float,
               q_out: torch.Tensor, kv_cache: Optional[torch.Tensor], page: int, batch, block_table: torch.Tensor, eps: float,
               conv: Optional[ConvRows] = None) -> None:
    """Bias, norm and rotation of query and key rows, page write of keys and values (``k`` without ``v``: the plain keys are the
    values; no ``k``: nothing is cached), and the convolution, in one launch.  ``rot``: ``RotarySpec`` (or None) with its
    frequencies ``freq`` (fp64) and amplitude; ``batch``: ``BatchDesc``."""
    _check_device(q.x)
    a = _PostArgs()
    for dst, r in ((a.q, q), (a.k, k), (a.v, v)):
        if r is None:
            continue
        assert r.x.dtype == q.x.dtype and r.x.stride(1) == 1 and r.x.shape[1] == -(-r.heads * r.dim // 8) * 8
        assert (r.bias is None or r.bias.numel() == r.x.shape[1]) and (norm != "rows" or r is v or r.gain.numel() == r.x.shape[1])
        dst.x, dst.stride, dst.bias, dst.gain, dst.heads, dst.dim = (r.x.data_ptr(), r.x.stride(0), _p(r.bias), _p(r.gain),
                                                                     r.heads, r.dim)
        dst.gain_heads = int(r.gain is not None and r.gain.dim() == 2)
        assert not dst.gain_heads or (norm == "head" and r.gain.shape == (r.heads, r.dim) and r.gain.is_contiguous())
    T, D = q.x.shape[0], q_out.shape[2]
    assert q_out.is_contiguous() and q_out.shape == (T, q.heads, D)
    assert k is None or (kv_cache.dtype == q_out.dtype and kv_cache.shape[1:] == (2, k.heads, page, D))
    a.freq, a.q_out, a.kv_cache = freq.data_ptr(), q_out.data_ptr(), _p(kv_cache)
    a.block_table, a.max_pages = block_table.data_ptr(), block_table.shape[1]
    a.slot, a.pos = batch.slot.data_ptr(), batch.pos.data_ptr()
    a.T, a.in_dtype, a.out_f32, a.norm, a.D, a.page = T, _dt(q.x), int(q_out.dtype == torch.float32), NORM_CODES[norm], D, page
    a.rot_dims, a.halves, a.eps, a.amp = (rot.dims if rot else 0), int(bool(rot and rot.halves)), eps, amp
    if conv is not None:
        taps, ch = conv.w.shape
        assert conv.x.dtype == q.x.dtype and conv.u.dtype == q_out.dtype and conv.u.stride(2) == 1
        assert conv.w.is_contiguous() and conv.bias.numel() == conv.conv_bias.numel() == ch == conv.u.shape[1] * conv.u.shape[2]
        a.cx, a.cx_stride, a.cx_bias = conv.x.data_ptr(), conv.x.stride(0), conv.bias.data_ptr()
        a.cw, a.cb, a.cstate, a.cjournal = conv.w.data_ptr(), conv.conv_bias.data_ptr(), _p(conv.state), _p(conv.journal)
        a.u, a.u_ts, a.u_bs = conv.u.data_ptr(), conv.u.stride(0), conv.u.stride(1)
        a.seg_start, a.seg_slot, a.tok_seg = batch.seg_start.data_ptr(), batch.seg_slot.data_ptr(), batch.tok_seg.data_ptr()
        a.C, a.block_cols, a.taps = ch, conv.u.shape[2], taps
        a.n_slots = conv.state.shape[0] if conv.state is not None else 1 << 30
    N.check(_lib().he_mixer_post(C.byref(a), _stream()), "he_mixer_post")


@dataclass
class Recurrence:
    """Parameters of one RG-LRU."""
    gate_w: torch.Tensor                    # bf16 [blocks, 2 * block_cols, block_cols]: maps of gate r, then of gate i
    gate_b: torch.Tensor                    # fp32 [blocks, 2 * block_cols]
    decay: torch.Tensor                     # fp32 [C]: -8 softplus(lambda)
    y_bias: torch.Tensor                    # fp32 [C]
    x_bias: torch.Tensor                    # fp32 [C]
    taps: int


def _rglru(p: Recurrence, u: torch.Tensor, y: torch.Tensor, x: torch.Tensor, S: torch.Tensor, cstate: Optional[torch.Tensor],
           batch, out: torch.Tensor) -> _RglruArgs:
    _check_device(u)
    a = _RglruArgs()
    blocks, _, bc = p.gate_w.shape
    assert u.dtype == out.dtype and u.stride(2) == 1 and u.shape[1:] == (blocks, bc) and out.stride(1) == 1
    assert y.dtype == x.dtype and y.stride(0) == x.stride(0) and S.is_contiguous() and S.shape[1] == blocks * bc
    assert p.taps == 1 or cstate.shape == (S.shape[0], p.taps - 1, blocks * bc)
    a.gw, a.gb, a.decay, a.yb, a.xb = (t.data_ptr() for t in (p.gate_w, p.gate_b, p.decay, p.y_bias, p.x_bias))
    a.u, a.u_ts, a.u_bs = u.data_ptr(), u.stride(0), u.stride(1)
    a.y, a.x, a.row_stride, a.row_dtype = y.data_ptr(), x.data_ptr(), y.stride(0), _dt(y)
    a.S, a.cstate, a.seg_start, a.seg_slot = S.data_ptr(), _p(cstate), batch.seg_start.data_ptr(), batch.seg_slot.data_ptr()
    a.out, a.out_stride, a.act_f32 = out.data_ptr(), out.stride(0), int(out.dtype == torch.float32)
    a.C, a.block_cols, a.taps, a.n_slots, a.n_seg, a.T = blocks * bc, bc, p.taps, S.shape[0], batch.n_seg, batch.T
    return a


def rglru_step(p: Recurrence, u: torch.Tensor, y: torch.Tensor, x: torch.Tensor, S: torch.Tensor, cstate: Optional[torch.Tensor],
               batch, out: torch.Tensor) -> None:
    """One token per segment (1..16 segments, bf16): gate products, recurrence, output gate and both states in one launch."""
    assert batch.n_seg == batch.T
    a = _rglru(p, u, y, x, S, cstate, batch, out)
    N.check(_lib().he_rglru_step(C.byref(a), _stream()), "he_rglru_step")


def rglru_scan(p: Recurrence, gates: torch.Tensor, u: torch.Tensor, y: torch.Tensor, x: torch.Tensor, S: torch.Tensor,
               cstate: Optional[torch.Tensor], batch, out: torch.Tensor, journal: Optional[torch.Tensor] = None) -> None:
    """Segments of any lengths; ``gates`` fp32 [T, blocks, 2 * block_cols] (any strides) = u times the gate maps.  With
    ``journal`` [T, C] the state after every token goes there and the states stay."""
    a = _rglru(p, u, y, x, S, cstate, batch, out)
    assert gates.dtype == torch.float32 and gates.stride(2) == 1 and gates.shape[1:] == p.gate_w.shape[:2]
    a.g, a.g_ts, a.g_bs, a.journal = gates.data_ptr(), gates.stride(0), gates.stride(1), _p(journal)
    N.check(_lib().he_rglru_scan(C.byref(a), _stream()), "he_rglru_scan")
