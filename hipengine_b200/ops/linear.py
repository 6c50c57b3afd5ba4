"""Launchers of linear attention with a matrix state (``csrc/linear_attn.cu``, ``linear_chunk.cu``: retention and the gated delta
rule) and of the grouped norms with the convolution ahead of a mixer (``csrc/norm_conv.cu``)."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Optional, Tuple

import torch

from ..core import native as N
from .kernels import _check_device, _dt, _p, _stream

c_vp, c_ll, c_int, c_f = C.c_void_p, C.c_longlong, C.c_int, C.c_float
CHUNK = 64                     # tokens per chunk of the prompt form
CHUNK_MAX_DIM = 128            # widest query / key head it is built for


class _NormConvArgs(C.Structure):
    _fields_ = [("x", c_vp), ("ldx", c_ll), ("w1", c_vp), ("w2", c_vp), ("cw", c_vp), ("state", c_vp), ("journal", c_vp),
                ("seg_start", c_vp), ("seg_slot", c_vp), ("a", c_vp), ("b", c_vp), ("T", c_int), ("H", c_int), ("groups", c_int),
                ("gw", c_int), ("taps", c_int), ("n_seg", c_int), ("n_slots", c_int), ("out_bf16", c_int), ("tile", c_int),
                ("eps", c_f)]


_PTRS_1 = ("gm", "pw", "rate", "dt", "cw", "freq", "gain", "S", "ring", "jS", "jring", "seg_start", "seg_slot", "tok_seg", "pos",
           "qf", "kf", "vf", "g1", "beta", "o", "out", "qk", "vb", "mats", "lg")
_INTS = ("T", "n_seg", "n_slots", "H", "G", "dim", "vdim", "vcols", "taps", "C", "ck", "cv", "cz", "ca", "rot_dims", "delta",
         "row_dtype", "out_f32", "chunks")


class _LinearArgs(C.Structure):
    _fields_ = ([("rows", c_vp), ("stride", c_ll), ("ab", c_vp), ("ab_stride", c_ll)] + [(n, c_vp) for n in _PTRS_1]
                + [(n, c_int) for n in _INTS] + [("eps", c_f), ("kscale", c_f), ("qscale", c_f)])


_ABI_OK = False


def _lib():
    global _ABI_OK
    L = N.lib()
    if not _ABI_OK:
        for fn, st in (("he_norm_conv_args_size", _NormConvArgs), ("he_linear_args_size", _LinearArgs)):
            if getattr(L, fn)() != C.sizeof(st):
                raise RuntimeError(f"ABI mismatch for {st.__name__}: C={getattr(L, fn)()} Python={C.sizeof(st)}")
        _ABI_OK = True
    return L


# ----------------------------------------------------------------------------- norms over groups of channels
def _norm_args(x: torch.Tensor, w: torch.Tensor, groups: int, n: int, eps: float, out: torch.Tensor) -> _NormConvArgs:
    _check_device(x)
    assert x.dtype == w.dtype == torch.float32 and x.stride(1) == 1 and out.is_contiguous() and out.shape == x.shape
    assert w.numel() == x.shape[1] and n % groups == 0
    a = _NormConvArgs()
    a.x, a.ldx, a.w1, a.a, a.out_bf16 = x.data_ptr(), x.stride(0), w.data_ptr(), out.data_ptr(), int(out.dtype == torch.bfloat16)
    a.T, a.H, a.groups, a.gw, a.taps, a.eps = x.shape[0], x.shape[1], groups, n // groups, 1, eps
    return a


def grouped_norm(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, groups: int, eps: float, n: int = 0) -> torch.Tensor:
    """out = RMS norm of fp32 rows over ``groups`` equal runs of the first ``n`` columns (0: all), times gains ``w``; further
    columns are written as zeros."""
    a = _norm_args(x, w, groups, n or x.shape[1], eps, out)
    N.check(_lib().he_norm_conv(C.byref(a), _stream()), "he_norm_conv")
    return out


def norm_conv(x: torch.Tensor, w1: torch.Tensor, w2: Optional[torch.Tensor], conv: torch.Tensor, state: Optional[torch.Tensor],
              batch, mixer_rows: torch.Tensor, plain_rows: Optional[torch.Tensor], groups: int, eps: float, n: int,
              journal: Optional[torch.Tensor] = None) -> None:
    """mixer_rows = h + causal convolution of h over time, h = grouped norm of ``x`` times ``w1``; plain_rows = the same norm
    times ``w2``.  ``conv`` fp32 [taps, H] oldest first; ``state`` [n_slots, taps - 1, H] the normalised rows ahead of a
    segment, which it then replaces (with ``journal`` [T, taps - 1, H] it stays and every state is recorded there)."""
    a = _norm_args(x, w1, groups, n, eps, mixer_rows)
    taps, H = conv.shape
    assert conv.is_contiguous() and H == x.shape[1] and (w2 is None) == (plain_rows is None)
    assert taps == 1 or (state.is_contiguous() and state.shape[1:] == (taps - 1, H) and state.dtype == torch.float32)
    assert plain_rows is None or (plain_rows.dtype == mixer_rows.dtype and plain_rows.is_contiguous() and plain_rows.shape == x.shape)
    a.w2, a.b, a.cw, a.taps = _p(w2), _p(plain_rows), conv.data_ptr(), taps
    a.state, a.journal, a.n_slots = _p(state), _p(journal), state.shape[0] if state is not None else 1 << 30
    a.seg_start, a.seg_slot, a.n_seg = batch.seg_start.data_ptr(), batch.seg_slot.data_ptr(), batch.n_seg
    N.check(_lib().he_norm_conv(C.byref(a), _stream()), "he_norm_conv")


# ----------------------------------------------------------------------------- linear attention
@dataclass
class LinearParams:
    """One layer's constants; ``spec``: ``LinearAttentionSpec``.  Columns of the projected rows: queries at 0, keys, values (these
    are the convolution's columns), the output gate."""
    spec: object
    ck: int
    cv: int
    cz: int
    freq: Optional[torch.Tensor] = None       # fp64 [rot dims / 2]
    g1: Optional[torch.Tensor] = None         # retention: fp32 [H] decay - 1
    powers: Optional[torch.Tensor] = None     # retention: fp32 [H, CHUNK + 1]
    rate: Optional[torch.Tensor] = None       # delta: fp32 [H] exp(A_log)
    dt: Optional[torch.Tensor] = None         # delta: fp32 [H]
    conv: Optional[torch.Tensor] = None       # delta: fp32 [taps, conv columns], oldest first
    gain: Optional[torch.Tensor] = None       # fp32 [vdim] or none


def decay_powers(decay) -> torch.Tensor:
    d = torch.tensor(decay, dtype=torch.float64)
    return torch.pow(d[:, None], torch.arange(CHUNK + 1, dtype=torch.float64)[None]).float()


def linear_attention(p: LinearParams, rows: torch.Tensor, ab: Optional[torch.Tensor], ca: int, S: torch.Tensor,
                     ring: Optional[torch.Tensor], batch, out: torch.Tensor, eps: float, scratch,
                     jS: Optional[torch.Tensor] = None, jring: Optional[torch.Tensor] = None) -> None:
    """out [T, H * vcols] = the gated output of a layer's linear attention; ``S`` and ``ring`` (the states of all slots) advance,
    or with journals stay while the state after every token is recorded.  ``ab`` (delta rule): fp32 rows with the step size's
    logits at column 0 and the decay's inputs at column ``ca``."""
    a, steps = plan(p, rows, ab, ca, S, ring, batch, out, eps, scratch, jS, jring)
    for name in steps:
        launch(name, a)


def launch(name: str, a: _LinearArgs) -> None:
    N.check(getattr(_lib(), name)(C.byref(a), _stream()), name)


def plan(p: LinearParams, rows: torch.Tensor, ab: Optional[torch.Tensor], ca: int, S: torch.Tensor, ring: Optional[torch.Tensor],
         batch, out: torch.Tensor, eps: float, scratch, jS: Optional[torch.Tensor] = None,
         jring: Optional[torch.Tensor] = None) -> Tuple[_LinearArgs, Tuple[str, ...]]:
    """(arguments, kernels in order) of ``linear_attention``."""
    s, T = p.spec, rows.shape[0]
    _check_device(rows)
    a = _LinearArgs()
    f32 = out.dtype == torch.float32
    assert rows.stride(1) == 1 and S.is_contiguous() and S.shape[1:] == (s.heads, s.dim, s.vcols)
    assert out.is_contiguous() and out.shape == (T, s.heads * s.vcols)
    a.rows, a.stride, a.row_dtype, a.out_f32 = rows.data_ptr(), rows.stride(0), _dt(rows), int(f32)
    if s.delta:
        assert ab.dtype == torch.float32 and ab.stride(1) == 1 and p.conv.shape == (s.taps, s.conv_cols) and p.conv.is_contiguous()
        assert s.taps == 1 or (ring.is_contiguous() and ring.shape[1:] == (s.taps, s.conv_cols))
        a.ab, a.ab_stride, a.ca = ab.data_ptr(), ab.stride(0), ca
        a.rate, a.dt, a.cw, a.ring, a.jring = p.rate.data_ptr(), p.dt.data_ptr(), p.conv.data_ptr(), _p(ring), _p(jring)
        a.taps, a.C, a.qscale, a.kscale = s.taps, s.conv_cols, s.dim ** -0.5, 1.0
    else:
        a.gm, a.pw, a.freq, a.rot_dims = p.g1.data_ptr(), p.powers.data_ptr(), _p(p.freq), s.rot.dims if s.rot else 0
        a.taps, a.qscale, a.kscale = 1, 1.0, s.dim ** -0.5
    a.gain, a.S, a.jS, a.out, a.eps = _p(p.gain), S.data_ptr(), _p(jS), out.data_ptr(), eps
    a.seg_start, a.seg_slot, a.tok_seg, a.pos = (t.data_ptr() for t in (batch.seg_start, batch.seg_slot, batch.tok_seg, batch.pos))
    a.T, a.n_seg, a.n_slots, a.H, a.G = T, batch.n_seg, S.shape[0], s.heads, s.kv_heads
    a.dim, a.vdim, a.vcols, a.ck, a.cv, a.cz, a.delta = s.dim, s.vdim, s.vcols, p.ck, p.cv, p.cz, int(s.delta)
    if batch.n_seg == T and jS is None:
        return a, ("he_linear_step",)
    get = lambda name, n, dtype=torch.float32: scratch.get("lin_" + name, (n,), dtype).data_ptr()
    a.o = get("o", T * s.heads * s.vcols)
    if use_chunks(s, batch, f32 or jS is not None):
        dk = 64 if s.dim <= 64 else 128
        a.chunks = T // CHUNK + batch.n_seg
        a.qk, a.vb = get("qk", 4 * T * s.kv_heads * dk, torch.bfloat16), get("vb", T * s.heads * s.vcols, torch.bfloat16)
        a.mats = get("mats", 4 * a.chunks * s.heads * CHUNK * CHUNK, torch.bfloat16)
        a.lg, a.beta = get("lg", T * s.heads), get("beta", T * s.heads)
        return a, ("he_linear_chunk_prepare", "he_linear_chunk_scan", "he_linear_out")
    a.qf, a.kf = get("q", T * s.kv_heads * s.dim), get("k", T * s.kv_heads * s.dim)
    a.vf, a.g1, a.beta = get("v", T * s.heads * s.vcols), get("g1", T * s.heads), get("beta", T * s.heads)
    return a, ("he_linear_prepare", "he_linear_scan", "he_linear_out")


def use_chunks(s, batch, serial: bool) -> bool:
    """Prompt portions take the chunked form; fp32, journals, wider heads and batches of short portions the serial one."""
    return not serial and s.dim <= CHUNK_MAX_DIM and batch.T >= 16 * batch.n_seg
