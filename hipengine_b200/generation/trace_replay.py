"""Replay of recorded token streams through an engine's runner: given ids in, logits out, nothing sampled.

A trace step names the requests it touches, the next tokens of each and the places among them whose logits are wanted.
The whole step is one packed batch of the runner (``GpuRunner.forward_segments``; when every entry continues a request
by one token, the decode-graph step the generation path uses), requests are admitted and released through the same slot
ledger and page pool as generated ones.  A request grows page by page: its final length is not known when it enters.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, replace
from typing import Any, Dict, IO, List, Mapping, Optional, Sequence

import torch

from ..config import EngineConfig
from .gpu_runner import GpuRunner
from .scheduler import RequestState
from .types import GenerationRequest

MAX_LIVE_REQUESTS = 4
POOL_GRANULE_TOKENS = 64


class TraceError(ValueError):
    """The trace asks for something the engine was not sized for, or that is not well formed."""


@dataclass
class _Live:
    rs: RequestState
    tokens: int = 0                # tokens already in the cache


def trace_engine_config(max_tokens: int, dtype: str = "bfloat16", max_live: int = MAX_LIVE_REQUESTS) -> EngineConfig:
    """Engine sized for ``max_tokens`` tokens of live requests in total (plus the pool's null page)."""
    base = EngineConfig.from_env()
    tokens = -(-max(1, max_tokens) // POOL_GRANULE_TOKENS) * POOL_GRANULE_TOKENS
    page = base.kv.page_tokens
    return replace(base, max_sequence_length=tokens, compute_dtype=dtype,
                   scheduler=replace(base.scheduler, max_active_requests=max_live),
                   kv=replace(base.kv, pool_pages=tokens // page + 1, prefix_cache="off", cold_tier_bytes=0),
                   speculative=replace(base.speculative, mode="off"))


class TraceReplay:
    def __init__(self, runner: GpuRunner):
        self.runner = runner
        self.live: Dict[str, _Live] = {}

    def _admit(self, rid: str, tokens: Sequence[int]) -> _Live:
        rs = RequestState(GenerationRequest(prompt_token_ids=list(tokens), max_tokens=0))
        if not self.runner.admit(rs):
            raise TraceError(f"request {rid!r}: no state slot or not enough free pages")
        lv = self.live[rid] = _Live(rs)
        return lv

    @torch.no_grad()
    def step(self, entries: Sequence[Mapping[str, Any]], end: Sequence[str] = ()) -> Optional[torch.Tensor]:
        """Run one step; returns the wanted logits [wanted, vocab] in entry order (None when nothing is wanted)."""
        r = self.runner
        segs, rows, row, decode = [], [], 0, bool(entries)
        for e in entries:
            rid, toks = str(e["id"]), [int(t) for t in e["tokens"]]
            if not toks or min(toks) < 0 or max(toks) >= r.vocab:
                raise TraceError(f"request {rid!r}: token ids must be in [0, {r.vocab}) and there must be some")
            lv = self.live.get(rid)
            if lv is None:
                lv = self._admit(rid, toks)
                decode = False
            decode = decode and len(toks) == 1
            if lv.tokens + len(toks) > r.max_context:
                raise TraceError(f"request {rid!r}: longer than the engine's context {r.max_context}")
            r._ensure_pages(lv.rs, lv.tokens + len(toks))
            segs.append((lv.rs.slot, lv.tokens, toks))
            for w in e.get("want", ()):
                if not 0 <= int(w) < len(toks):
                    raise TraceError(f"request {rid!r}: wanted place {w} of {len(toks)} tokens")
                rows.append(row + int(w))
            row += len(toks)
            lv.tokens += len(toks)
        out = None
        if segs:
            if decode:
                r.graphs.set_rows([s for s, _, _ in segs], [t[0] for _, _, t in segs], [p for _, p, _ in segs])
                r.resident_key = ()
                r.graphs.step(len(segs), max(p + 1 for _, p, _ in segs), greedy=False)
                logits = r.graphs.logits[:len(segs)]
                out = logits[rows] if rows else None
            else:
                _, h = r.forward_segments(segs)
                if rows:
                    out = r.ex.logits(h.index_select(0, torch.tensor(rows, device=r.device)))
            r._sync_checked("trace")
        for rid in end:
            lv = self.live.pop(str(rid), None)
            if lv is None:
                raise TraceError(f"request {rid!r} ends but is not live")
            r.release(lv.rs)
        return out


def replay_stream(replay: TraceReplay, lines: IO[str], out_dir: str, done: IO[str]) -> int:
    """Steps as JSON lines from ``lines``; ``<step>.f32`` files (little-endian fp32 [wanted, vocab]) into ``out_dir``;
    ``done <step>`` on ``done`` after every step."""
    n = 0
    for line in lines:
        if not line.strip():
            continue
        st = json.loads(line)
        got = replay.step(st["entries"], st.get("end", ()))
        if got is not None:
            data = got.to("cpu", torch.float32).contiguous().numpy().astype("<f4", copy=False).tobytes()
            with open(os.path.join(out_dir, f"{st['step']}.f32"), "wb") as f:
                f.write(data)
        done.write(f"done {st['step']}\n")
        done.flush()
        n += 1
    return n


def main(argv: Optional[List[str]] = None) -> int:
    import argparse
    import sys
    ap = argparse.ArgumentParser(prog="trace_run", description="feed recorded token ids through a model, write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors (or a GGUF artifact)")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens live requests hold at any time")
    a = ap.parse_args(argv)
    from ..loading.model_loader import load_model
    from ..models.registry import plugin_for
    weights = load_model(a.model)
    plugin = plugin_for(weights.config.arch)
    if a.dtype not in plugin.compute_dtypes:
        print(f"{plugin.name}: compute dtype {a.dtype} is not built", file=sys.stderr)
        return 3
    from ..core import build
    build.ensure(plugin.native_sources)
    torch.cuda.set_device(0)
    runner = GpuRunner(weights, trace_engine_config(a.max_tokens, a.dtype))
    replay_stream(TraceReplay(runner), sys.stdin, a.out, sys.stdout)
    runner.close()
    return 0
