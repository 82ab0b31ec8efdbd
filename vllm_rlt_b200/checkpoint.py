"""Reading model folders: `config.json` and `model.safetensors`.

A safetensors file is an 8-byte little-endian header length, that many bytes of JSON (tensor name ->
dtype, shape, byte range) and the data.  The file is mapped, not read: a tensor costs memory when it is
moved to the device.
"""

from __future__ import annotations

import json
import mmap
import struct
from pathlib import Path

import torch

DTYPES = {"F64": torch.float64, "F32": torch.float32, "F16": torch.float16, "BF16": torch.bfloat16, "I64": torch.int64,
          "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}


def read_safetensors(path) -> dict[str, torch.Tensor]:
    """name -> CPU tensor over the mapped file (read only: copy before writing)."""
    with open(path, "rb") as f:
        mapped = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_COPY)
    if len(mapped) < 8:
        raise ValueError(f"{path} is not a safetensors file")
    (length,) = struct.unpack("<Q", mapped[:8])
    if length > len(mapped) - 8:
        raise ValueError(f"{path} is truncated: its header does not fit")
    tensors = {}
    for name, entry in json.loads(mapped[8:8 + length]).items():
        if name == "__metadata__":
            continue
        dtype = DTYPES.get(entry["dtype"])
        if dtype is None:
            raise ValueError(f"{name}: unsupported dtype {entry['dtype']}")
        begin, end = entry["data_offsets"]
        count = 1
        for size in entry["shape"]:
            count *= size
        if end - begin != count * dtype.itemsize or 8 + length + end > len(mapped):
            raise ValueError(f"{name}: its byte range does not fit its shape or the file")
        if count == 0:
            tensors[name] = torch.empty(entry["shape"], dtype=dtype)
        elif (8 + length + begin) % dtype.itemsize:
            tensors[name] = torch.frombuffer(bytearray(mapped[8 + length + begin:8 + length + end]), dtype=dtype).reshape(entry["shape"])
        else:
            tensors[name] = torch.frombuffer(mapped, dtype=dtype, count=count, offset=8 + length + begin).reshape(entry["shape"])
    return tensors


def read_config(folder) -> dict:
    with open(Path(folder) / "config.json") as f:
        return json.load(f)


def read_weights(folder) -> dict[str, torch.Tensor]:
    """All tensors of a model folder (`model.safetensors`, or every `*.safetensors` shard in it)."""
    folder = Path(folder)
    single = folder / "model.safetensors"
    files = [single] if single.exists() else sorted(folder.glob("*.safetensors"))
    if not files:
        raise FileNotFoundError(f"no safetensors file in {folder}")
    tensors: dict[str, torch.Tensor] = {}
    for file in files:
        tensors.update(read_safetensors(file))
    return tensors
