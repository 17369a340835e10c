"""Reading and writing model folders: ``config.json`` beside ``model.safetensors``.

A safetensors file is an 8-byte little-endian header length, that many bytes of JSON (name -> dtype,
shape, data_offsets relative to the end of the header) and the raw tensors.
"""
from __future__ import annotations

import json
import mmap
import struct
from pathlib import Path

import torch

_DTYPES = {
    "F64": torch.float64, "F32": torch.float32, "F16": torch.float16, "BF16": torch.bfloat16,
    "I64": torch.int64, "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool,
}
_NAMES = {v: k for k, v in _DTYPES.items()}


def read_safetensors(path) -> dict[str, torch.Tensor]:
    """Tensors by name, as views of a private memory map of the file (nothing is copied here)."""
    with open(path, "rb") as f:
        buf = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_COPY)
    if len(buf) < 8:
        raise ValueError(f"{path}: not a safetensors file")
    n = struct.unpack("<Q", buf[:8])[0]
    if n > len(buf) - 8:
        raise ValueError(f"{path}: the header is longer than the file")
    header = json.loads(buf[8:8 + n])
    out = {}
    for name, entry in header.items():
        if name == "__metadata__":
            continue
        lo, hi = entry["data_offsets"]
        dtype = _DTYPES.get(entry["dtype"])
        if dtype is None:
            raise ValueError(f"{path}: {name} has the unsupported type {entry['dtype']}")
        shape = [int(d) for d in entry["shape"]]
        count = 1
        for d in shape:
            count *= d
        size = torch.empty((), dtype=dtype).element_size()
        if hi - lo != count * size or 8 + n + hi > len(buf):
            raise ValueError(f"{path}: {name} does not fit its data range")
        at = 8 + n + lo
        if count == 0:
            out[name] = torch.empty(shape, dtype=dtype)
        elif at % size:
            out[name] = torch.frombuffer(bytearray(buf[at:at + count * size]), dtype=dtype).view(shape)
        else:
            out[name] = torch.frombuffer(buf, dtype=dtype, count=count, offset=at).view(shape)
    return out


def write_safetensors(path, tensors: dict[str, torch.Tensor]) -> None:
    header, blobs, at = {}, [], 0
    for name, t in tensors.items():
        t = t.detach().cpu().contiguous()
        raw = t.view(torch.uint8).numpy().tobytes() if t.numel() else b""
        header[name] = {"dtype": _NAMES[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    head = json.dumps(header).encode()
    head += b" " * (-len(head) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head)
        for b in blobs:
            f.write(b)


def read_model_folder(folder) -> tuple[dict, dict[str, torch.Tensor]]:
    folder = Path(folder)
    config = json.loads((folder / "config.json").read_text())
    return config, read_safetensors(folder / "model.safetensors")


def write_model_folder(folder, config: dict, tensors: dict[str, torch.Tensor]) -> None:
    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(config, indent=1))
    write_safetensors(folder / "model.safetensors", tensors)
