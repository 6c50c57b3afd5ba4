"""Checkpoint folders: ``config.json`` beside ``model.safetensors``.

A safetensors file is an 8-byte little-endian header length, that many bytes of JSON (name -> dtype, shape,
data_offsets into the rest) and the tensor bytes.  The registry finds the model family by ``architecture`` in config.json
and names the module with its configuration reader and tensor list (``folder_family.py``).
"""
from __future__ import annotations

import json
import struct
from importlib import import_module
from pathlib import Path
from typing import Any, Dict, Optional, Tuple

import torch

from ..quant.ggml import GGMLType
from .weights import ModelWeights, QTensor

CONFIG_FILE, TENSOR_FILE = "config.json", "model.safetensors"
_GGML_OF = {"BF16": GGMLType.BF16, "F32": GGMLType.F32, "F16": GGMLType.F16}
_ITEM_BYTES = {"BF16": 2, "F32": 4, "F16": 2}


def is_checkpoint_dir(path) -> bool:
    p = Path(str(path))
    return p.is_dir() and (p / CONFIG_FILE).is_file() and (p / TENSOR_FILE).is_file()


def read_header(path) -> Tuple[Dict[str, Dict[str, Any]], int]:
    """(entries, offset of the data) of a safetensors file."""
    size = Path(path).stat().st_size
    with open(path, "rb") as f:
        head = f.read(8)
        if len(head) != 8:
            raise ValueError(f"{path}: no safetensors header")
        n = struct.unpack("<Q", head)[0]
        if 8 + n > size:
            raise ValueError(f"{path}: header of {n} bytes in a file of {size}")
        entries = json.loads(f.read(n))
    entries.pop("__metadata__", None)
    for name, e in entries.items():
        a, b = e["data_offsets"]
        count = 1
        for d in e["shape"]:
            count *= int(d)
        if e["dtype"] not in _ITEM_BYTES:
            raise ValueError(f"{path}: {name} is stored as {e['dtype']} (supported: {sorted(_ITEM_BYTES)})")
        if not 0 <= a <= b <= size - 8 - n or b - a != count * _ITEM_BYTES[e["dtype"]]:
            raise ValueError(f"{path}: {name} has offsets {a}..{b} for shape {e['shape']}")
    return entries, 8 + n


def read_tensors(path, device="cpu", pin: bool = False) -> Dict[str, QTensor]:
    """Tensors as stored; on the host they are views of the mapped file."""
    entries, base = read_header(path)
    data = torch.from_file(str(path), size=Path(path).stat().st_size, dtype=torch.uint8, shared=False)
    dev = torch.device(device)
    out: Dict[str, QTensor] = {}
    for name, e in entries.items():
        a, b = e["data_offsets"]
        shape = tuple(int(d) for d in e["shape"])
        cols = shape[-1] if shape else 1
        host = data[base + a:base + b]
        if (base + a) % 4:                       # a mapped view must start where its element type may
            host = host.clone()
        host = host.reshape(-1, max(1, cols * _ITEM_BYTES[e["dtype"]]))
        if pin and dev.type == "cuda":
            host = host.pin_memory()
        raw = host.to(dev, non_blocking=pin) if dev.type != "cpu" else host
        out[name] = QTensor(name, _GGML_OF[e["dtype"]], shape, raw)
    return out


def write_tensors(path, tensors: Dict[str, torch.Tensor]) -> None:
    """Write float tensors (bfloat16 / float32 / float16) as a safetensors file."""
    names = {torch.bfloat16: "BF16", torch.float32: "F32", torch.float16: "F16"}
    entries: Dict[str, Any] = {}
    blobs, at = [], 0
    for name, t in tensors.items():
        raw = t.detach().cpu().contiguous().reshape(-1).view(torch.uint8).numpy().tobytes()
        entries[name] = {"dtype": names[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    head = json.dumps(entries).encode()
    head += b" " * (-len(head) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head)
        for b in blobs:
            f.write(b)


def config_of(path):
    """(``ModelConfig``, decoded config.json) of a checkpoint folder."""
    with open(Path(path) / CONFIG_FILE) as f:
        raw = json.load(f)
    from ..models.registry import folder_plugin
    try:
        plugin = folder_plugin(str(raw.get("architecture", "")))
    except KeyError as e:
        raise ValueError(f"{path}/{CONFIG_FILE}: {e.args[0]}") from None
    return import_module(plugin.folder_reader).config_from_json(raw), raw


def load_checkpoint_dir(path, device="cpu", pin: bool = False, validate: bool = True) -> ModelWeights:
    cfg, raw = config_of(path)
    tensors = read_tensors(Path(path) / TENSOR_FILE, device, pin)
    if validate:
        from .folder_family import check_tensors
        check_tensors(cfg, {n: t.shape for n, t in tensors.items()})
    return ModelWeights(cfg, tensors, {"general.architecture": cfg.arch, "general.name": str(path), "config": raw})


def describe_checkpoint_dir(path) -> Optional[Dict[str, Any]]:
    """Header-only description of a checkpoint folder (None when ``path`` is not one)."""
    if not is_checkpoint_dir(path):
        return None
    f = Path(path) / TENSOR_FILE
    out: Dict[str, Any] = {"source": "safetensors", "path": str(path), "file_bytes": f.stat().st_size}
    try:
        cfg, _ = config_of(path)
        entries, _base = read_header(f)
    except Exception as e:
        return {**out, "error": f"{type(e).__name__}: {e}"}
    hist: Dict[str, int] = {}
    for e in entries.values():
        hist[e["dtype"]] = hist.get(e["dtype"], 0) + e["data_offsets"][1] - e["data_offsets"][0]
    return {**out, "tensors": len(entries), "weight_bytes": sum(hist.values()), "bytes_by_block_type": hist, "config": cfg}
