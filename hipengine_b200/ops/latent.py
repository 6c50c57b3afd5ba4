"""Launchers of the latent attention kernels (``csrc/latent_attn.cu``, ``latent_prefill.cu``, ``latent_prefill_tc.cu``).

A cache plane is ``[n_pages, page, W]`` in bf16 (fp32 for the float32 compute dtype): latent columns, then the rotated key
part, zero-padded.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Optional, Sequence, Tuple

import torch

from ..core import native as N
from .kernels import _check_device, _dt, _p, _stream, status_tensor

c_vp, c_ll, c_int = C.c_void_p, C.c_longlong, C.c_int


class _PostArgs(C.Structure):
    _fields_ = [("down", c_vp), ("q", c_vp), ("norm_w", c_vp), ("freq", c_vp), ("cache", c_vp), ("q_out", c_vp),
                ("q_lat", c_vp), ("block_table", c_vp), ("slot", c_vp), ("pos", c_vp), ("down_stride", c_ll),
                ("q_stride", c_ll), ("down_dtype", c_int), ("q_dtype", c_int), ("out_f32", c_int), ("T", c_int),
                ("H", c_int), ("dn", c_int), ("rot_dim", c_int), ("q_cols", c_int), ("rank", c_int), ("rank_cols", c_int),
                ("W", c_int), ("page", c_int), ("max_pages", c_int), ("eps", C.c_float), ("amp", C.c_float)]


class _DecArgs(C.Structure):
    _fields_ = [("q", c_vp), ("cache", c_vp), ("block_table", c_vp), ("slot", c_vp), ("ctx_len", c_vp),
                ("partial", c_vp), ("out", c_vp), ("sink", c_vp), ("R", c_int), ("H", c_int),
                ("W", c_int), ("rank_cols", c_int), ("page", c_int), ("max_pages", c_int), ("window", c_int),
                ("spans", c_int), ("cluster", c_int), ("tile", c_int), ("scale", C.c_float), ("status", c_vp)]


class _GatherArgs(C.Structure):
    _fields_ = [("cache", c_vp), ("block_table", c_vp), ("seg_start", c_vp), ("seg_slot", c_vp), ("pos", c_vp),
                ("out", c_vp), ("n_seg", c_int), ("keys", c_int), ("W", c_int), ("page", c_int), ("max_pages", c_int),
                ("window", c_int)]


class _PrefillArgs(C.Structure):
    _fields_ = [("q", c_vp), ("kx", c_vp), ("v", c_vp), ("lat", c_vp), ("sink", c_vp), ("seg_start", c_vp), ("pos", c_vp),
                ("out", c_vp), ("status", c_vp), ("n_seg", c_int), ("tiles", c_int), ("H", c_int), ("head0", c_int),
                ("n_heads", c_int), ("dn", c_int), ("dv", c_int), ("qd", c_int), ("W", c_int), ("rank_cols", c_int),
                ("window", c_int), ("rows", c_int), ("keys", c_int), ("scale", C.c_float)]


SEG_ALIGN = 8             # gathered rows of a segment are padded to a multiple of this
_ABI_OK = False


def _lib():
    global _ABI_OK
    L = N.lib()
    if not _ABI_OK:
        for fn, st in (("he_latent_post_args_size", _PostArgs), ("he_latent_dec_args_size", _DecArgs),
                       ("he_latent_gather_args_size", _GatherArgs), ("he_latent_prefill_args_size", _PrefillArgs)):
            if getattr(L, fn)() != C.sizeof(st):
                raise RuntimeError(f"ABI mismatch for {st.__name__}: C={getattr(L, fn)()} Python={C.sizeof(st)}")
        _ABI_OK = True
    return L


def latent_post(down: torch.Tensor, q: torch.Tensor, norm_w: torch.Tensor, freq: torch.Tensor, amp: float,
                cache: torch.Tensor, block_table: torch.Tensor, slot: torch.Tensor, pos: torch.Tensor, heads: int, dn: int,
                rot_dim: int, rank: int, rank_cols: int, eps: float, q_out: Optional[torch.Tensor] = None,
                q_lat: Optional[torch.Tensor] = None) -> None:
    """Norm the latent (first ``rank`` columns of ``down``), rotate the shared key part behind it, write both into the
    request's page; rotate the queries ``q`` [T, heads * (dn + rotated)] into ``q_out`` (same layout, the cache's type; may
    be ``q``) and the rotated part alone into columns ``rank_cols..`` of ``q_lat`` [T, heads, W]."""
    _check_device(q)
    T, W, act = q.shape[0], cache.shape[2], cache.dtype
    assert freq.dtype == torch.float64 and freq.numel() == rot_dim // 2 and norm_w.numel() == rank_cols
    assert (q_out is None or (q_out.dtype == act and q_out.is_contiguous())) and \
        (q_lat is None or (q_lat.dtype == act and q_lat.is_contiguous() and q_lat.shape == (T, heads, W)))
    a = _PostArgs()
    a.down, a.down_stride, a.down_dtype = down.data_ptr(), down.stride(0), _dt(down)
    a.q, a.q_stride, a.q_dtype, a.q_cols = q.data_ptr(), q.stride(0), _dt(q), q.shape[1] // heads
    a.norm_w, a.freq, a.amp, a.eps = norm_w.data_ptr(), freq.data_ptr(), amp, eps
    a.cache, a.q_out, a.q_lat, a.out_f32 = cache.data_ptr(), _p(q_out), _p(q_lat), int(act == torch.float32)
    a.block_table, a.slot, a.pos = block_table.data_ptr(), slot.data_ptr(), pos.data_ptr()
    a.T, a.H, a.dn, a.rot_dim, a.rank, a.rank_cols, a.W = T, heads, dn, rot_dim, rank, rank_cols, W
    a.page, a.max_pages = cache.shape[1], block_table.shape[1]
    N.check(_lib().he_latent_post(C.byref(a), _stream()), "he_latent_post")


@dataclass(frozen=True)
class DecodePlan:
    """How a latent-space launch cuts the keys of a row: ``spans`` CTAs, ``cluster`` of them merging on chip, key tiles of
    ``tile``."""
    spans: int
    cluster: int
    tile: int

    @property
    def clusters(self) -> int:
        return self.spans // self.cluster

    def scratch_floats(self, rows: int, heads: int, rank_cols: int) -> int:
        """Cluster sums and their (maximum, sum) pairs; none when one cluster covers a row."""
        return rows * heads * self.clusters * (rank_cols + 2) if self.clusters > 1 else 0


def decode_plan(span: int, rows: int, heads: int, W: int) -> DecodePlan:
    """Plan for ``rows`` rows of up to ``span`` visible keys: about one round of CTAs over the GPU, no more spans than
    tiles, tiles of 32 keys where tiles of 64 would leave SMs idle.  Clusters of four pack the SMs; wider ones do not."""
    chunks, tile_rows = (-(-heads // 32), 32) if heads > 16 else (1, 16)
    per_sm = max(1, min(4, int(227e3 // ((tile_rows + 128) * (2 * W + 16) + tile_rows * 1300))))
    want = max(1, 128 * per_sm // (max(rows, 1) * chunks))
    tile = 64 if -(-span // 64) >= min(want, 64) else 32
    spans = min(want, -(-span // tile))
    if spans > 4:
        return DecodePlan(min(512, spans // 4 * 4), 4, tile)
    return DecodePlan(spans, spans, tile)


def _dec_args(q, cache, block_table, slot, ctx_len, out, rank_cols, scale, window, sink) -> _DecArgs:
    _check_device(q)
    assert q.is_contiguous() and out.is_contiguous() and q.dtype == cache.dtype == out.dtype and cache.is_contiguous()
    R, H, W = q.shape
    assert cache.shape[2] == W and out.numel() == R * H * rank_cols and (sink is None or sink.numel() == H)
    a = _DecArgs()
    a.q, a.cache, a.block_table, a.slot, a.ctx_len = (t.data_ptr() for t in (q, cache, block_table, slot, ctx_len))
    a.out, a.sink, a.R, a.H, a.W, a.rank_cols = out.data_ptr(), _p(sink), R, H, W, rank_cols
    a.page, a.max_pages, a.window, a.scale = cache.shape[1], block_table.shape[1], window, scale
    a.status = status_tensor(q.device).data_ptr()
    return a


def latent_decode(q: torch.Tensor, cache: torch.Tensor, block_table: torch.Tensor, slot: torch.Tensor,
                  ctx_len: torch.Tensor, partial: torch.Tensor, out: torch.Tensor, rank_cols: int, scale: float,
                  plan: DecodePlan, window: int = 0, sink: Optional[torch.Tensor] = None) -> None:
    """Every row of ``q`` [R, H, W] (latent-space queries) against its request's cache rows; ``out`` [R, H, rank_cols] is
    the weighted sum of latents.  ``partial`` holds ``plan.scratch_floats``."""
    a = _dec_args(q, cache, block_table, slot, ctx_len, out, rank_cols, scale, window, sink)
    a.partial, a.spans, a.cluster, a.tile = partial.data_ptr(), plan.spans, plan.cluster, plan.tile
    assert q.dtype == torch.bfloat16 and partial.numel() >= plan.scratch_floats(a.R, a.H, rank_cols)
    N.check(_lib().he_latent_decode(C.byref(a), _stream()), "he_latent_decode")


def latent_exact(q: torch.Tensor, cache: torch.Tensor, block_table: torch.Tensor, slot: torch.Tensor,
                 ctx_len: torch.Tensor, out: torch.Tensor, rank_cols: int, scale: float, window: int = 0,
                 sink: Optional[torch.Tensor] = None) -> None:
    """``latent_decode`` in fp32 throughout (fp32 pages)."""
    a = _dec_args(q, cache, block_table, slot, ctx_len, out, rank_cols, scale, window, sink)
    assert q.dtype == torch.float32
    N.check(_lib().he_latent_exact(C.byref(a), _stream()), "he_latent_exact")


def gathered_rows(segs: Sequence[Tuple[int, int, int]], window: int) -> int:
    """Rows of the gathered keys of (slot, first position, rows) segments: what each can see, padded."""
    seen = (p0 + n - (max(0, p0 - window + 1) if window > 0 else 0) for _, p0, n in segs)
    return sum(-(-n // SEG_ALIGN) * SEG_ALIGN for n in seen)


def latent_gather(cache: torch.Tensor, block_table: torch.Tensor, seg_start: torch.Tensor, seg_slot: torch.Tensor,
                  pos: torch.Tensor, n_seg: int, window: int, out: torch.Tensor) -> None:
    """The cache rows the segments can see, side by side in segment order: ``out`` [``gathered_rows``, W]."""
    a = _GatherArgs()
    a.cache, a.block_table, a.seg_start = cache.data_ptr(), block_table.data_ptr(), seg_start.data_ptr()
    a.seg_slot, a.pos, a.out, a.n_seg, a.keys = seg_slot.data_ptr(), pos.data_ptr(), out.data_ptr(), n_seg, out.shape[0]
    a.W, a.page, a.max_pages, a.window = cache.shape[2], cache.shape[1], block_table.shape[1], window
    assert cache.dtype == out.dtype == torch.bfloat16 and out.is_contiguous() and out.shape[1] == a.W
    N.check(_lib().he_latent_gather(C.byref(a), _stream()), "he_latent_gather")


TC_TILE_ROWS = 256


def prefill_tile_rows(q_cols: int, dv: int) -> int:
    """Query rows per tile of the register form of prefill for this head shape (0: it has none)."""
    return int(_lib().he_latent_prefill_tile_rows(c_int(q_cols), c_int(dv)))


def prefill_tc_ok(dn: int, q_cols: int, dv: int) -> bool:
    """Does the tensor-memory form take this head shape?"""
    return bool(_lib().he_latent_prefill_tc_ok(c_int(dn), c_int(q_cols), c_int(dv)))


def latent_prefill(q: torch.Tensor, kx: torch.Tensor, v: torch.Tensor, lat: torch.Tensor, seg_start: torch.Tensor,
                   pos: torch.Tensor, seg_rows: Sequence[int], out: torch.Tensor, heads: int, head0: int, n_heads: int,
                   dn: int, dv: int, rank_cols: int, scale: float, window: int = 0, sink: Optional[torch.Tensor] = None,
                   transposed: bool = False) -> None:
    """Heads head0 .. head0 + n_heads of the segments' rows: ``q`` [T, heads, q_cols] rotated queries, ``kx``
    [keys, n_heads * dn] and ``v`` [keys, n_heads * dv] expanded from the rows gathered into ``lat``; ``out``
    [T, heads * dv].  ``transposed``: ``v`` is [n_heads * dv, keys] and the tensor-memory form runs."""
    a, keys, qd = _PrefillArgs(), lat.shape[0], q.shape[2]
    assert q.is_contiguous() and kx.is_contiguous() and v.is_contiguous() and out.is_contiguous() and lat.is_contiguous()
    assert kx.shape == (keys, n_heads * dn) and out.shape == (q.shape[0], heads * dv) and q.shape[1] == heads
    assert v.shape == ((n_heads * dv, keys) if transposed else (keys, n_heads * dv))
    a.q, a.kx, a.v, a.lat, a.sink = q.data_ptr(), kx.data_ptr(), v.data_ptr(), lat.data_ptr(), _p(sink)
    a.seg_start, a.pos, a.out, a.n_seg = seg_start.data_ptr(), pos.data_ptr(), out.data_ptr(), len(seg_rows)
    bm = TC_TILE_ROWS if transposed else prefill_tile_rows(qd, dv)
    assert bm > 0
    a.tiles, a.status = sum(-(-n // bm) for n in seg_rows), status_tensor(q.device).data_ptr()
    a.H, a.head0, a.n_heads, a.dn, a.dv, a.qd = heads, head0, n_heads, dn, dv, qd
    a.W, a.rank_cols, a.window, a.scale, a.rows, a.keys = lat.shape[1], rank_cols, window, scale, q.shape[0], keys
    fn = "he_latent_prefill_tc" if transposed else "he_latent_prefill"
    N.check(getattr(_lib(), fn)(C.byref(a), _stream()), fn)
