"""Reader and writer of safetensors files: an 8-byte little-endian header length, a JSON header
``name -> {dtype, shape, data_offsets}`` and the tensors' bytes.  Tensors are views of one memory-mapped
buffer until they are copied."""
from __future__ import annotations

import json
from pathlib import Path
from typing import Any

import torch

_DTYPES = {"F64": torch.float64, "F32": torch.float32, "F16": torch.float16, "BF16": torch.bfloat16, "I64": torch.int64,
           "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}
_NAMES = {v: k for k, v in _DTYPES.items()}


def load_safetensors(path: str | Path) -> dict[str, torch.Tensor]:
    path = Path(path)
    size = path.stat().st_size
    with open(path, "rb") as fh:
        n = int.from_bytes(fh.read(8), "little")
        if n <= 0 or 8 + n > size:
            raise ValueError(f"{path}: not a safetensors file (header of {n} bytes, file of {size})")
        header: dict[str, Any] = json.loads(fh.read(n))
    base = 8 + n
    buf = torch.from_file(str(path), shared=False, size=size, dtype=torch.uint8)
    out: dict[str, torch.Tensor] = {}
    for name, meta in header.items():
        if name == "__metadata__":
            continue
        dt = _DTYPES.get(meta["dtype"])
        if dt is None:
            raise ValueError(f"{path}: tensor {name} has unsupported dtype {meta['dtype']}")
        lo, hi = meta["data_offsets"]
        shape = [int(s) for s in meta["shape"]]
        numel = 1
        for s in shape:
            numel *= s
        if lo < 0 or base + hi > size or hi - lo != numel * dt.itemsize:
            raise ValueError(f"{path}: tensor {name} does not fit its data range")
        raw = buf[base + lo: base + hi]
        # the data of a tensor need not be aligned to its element size
        out[name] = (raw if raw.data_ptr() % dt.itemsize == 0 else raw.clone()).view(dt).view(shape)
    return out


def save_safetensors(tensors: dict[str, torch.Tensor], path: str | Path) -> None:
    header, at = {}, 0
    for name, t in tensors.items():
        n = t.numel() * t.element_size()
        header[name] = {"dtype": _NAMES[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + n]}
        at += n
    head = json.dumps(header).encode()
    head += b" " * (-len(head) % 8)
    with open(path, "wb") as fh:
        fh.write(len(head).to_bytes(8, "little"))
        fh.write(head)
        for t in tensors.values():
            fh.write(t.detach().cpu().contiguous().view(-1).view(torch.uint8).numpy().tobytes())
