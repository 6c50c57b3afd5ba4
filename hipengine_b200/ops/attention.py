"""Prefill (flash) attention launcher.  The decode/split-K launcher lives in ``ops.kernels``."""
from __future__ import annotations

import ctypes as C

import torch

from ..core import native as N
from .kernels import _dt


def flash_prefill_available(head_dim: int) -> bool:
    try:
        return head_dim in (64, 128, 256) and hasattr(N.lib(), "he_flash_prefill")
    except Exception:
        return False


FLASH_TILE_ROWS = 64


def flash_prefill_segs(q, gate, kv_cache, block_table, seg_start, seg_slot, pos, seg_rows, out, H, Hkv, D, page, scale,
                       window: int = 0, softcap: float = 0.0, sink=None, head_gate=None, keep_first: int = 0) -> None:
    """``flash_prefill`` for several segments in one launch: ``seg_start`` (device, n + 1 absolute row offsets),
    ``seg_slot`` (device), ``pos`` (device, per row) and ``seg_rows`` (host row counts, sizes the grid).  ``sink`` (fp32 [H]):
    scores of a term in the softmax denominator; ``head_gate`` ([rows, H], fp32 or bf16): logits of a gate per head; with a
    ``window`` the sequence's first ``keep_first`` keys stay visible."""
    tiles = sum(-(-n // FLASH_TILE_ROWS) for n in seg_rows)
    N.check(N.lib().he_flash_prefill_segs(
        C.c_void_p(q.data_ptr()), C.c_void_p(None if gate is None else gate.data_ptr()),
        C.c_void_p(kv_cache.data_ptr()), C.c_void_p(block_table.data_ptr()), C.c_int(block_table.shape[1]),
        C.c_void_p(seg_start.data_ptr()), C.c_void_p(seg_slot.data_ptr()), C.c_void_p(pos.data_ptr()),
        C.c_int(len(seg_rows)), C.c_int(tiles), C.c_void_p(out.data_ptr()), C.c_int(H), C.c_int(Hkv), C.c_int(D),
        C.c_int(page), C.c_float(scale), C.c_int(window), C.c_float(softcap),
        C.c_void_p(None if sink is None else sink.data_ptr()),
        C.c_void_p(None if head_gate is None else head_gate.data_ptr()),
        C.c_longlong(0 if head_gate is None else head_gate.stride(0)), C.c_int(0 if head_gate is None else _dt(head_gate)),
        C.c_int(keep_first),
        C.c_void_p(torch.cuda.current_stream().cuda_stream)), "he_flash_prefill_segs")


def flash_prefill(q, gate, kv_cache, block_table, slot: int, pos0: int, out, H, Hkv, D, page, scale,
                  window: int = 0) -> None:
    """Causal paged GQA attention over one segment's rows (append-then-attend) with the sigmoid gate fused.

    ``q`` / ``gate`` / ``out`` hold the T rows of the segment, which sit at positions pos0 .. pos0+T-1 of the
    request that owns block-table row ``slot``.
    """
    L = N.lib()
    T = q.shape[0]
    bt_row = block_table[slot]
    N.check(L.he_flash_prefill(C.c_void_p(q.data_ptr()), C.c_void_p(None if gate is None else gate.data_ptr()),
                               C.c_void_p(kv_cache.data_ptr()), C.c_void_p(bt_row.data_ptr()),
                               C.c_void_p(out.data_ptr()), C.c_int(T), C.c_int(H), C.c_int(Hkv), C.c_int(D),
                               C.c_int(page), C.c_int(pos0), C.c_float(scale), C.c_int(window),
                               C.c_void_p(torch.cuda.current_stream().cuda_stream)), "he_flash_prefill")
