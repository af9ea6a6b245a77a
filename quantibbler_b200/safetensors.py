"""Reader of safetensors files: an 8-byte little-endian length, that many bytes of JSON (name ->
dtype, shape, data_offsets), then the data.  The data stays a memory map; a tensor is copied when
it is first used."""

from __future__ import annotations

import json
import os

import numpy as np

_WIDTH = {"BF16": 2, "F16": 2, "F32": 4, "F64": 8, "I32": 4, "I64": 8, "U8": 1, "I8": 1}


class SafetensorsError(ValueError):
    """A malformed file; the text names it."""


def load(path: str) -> dict:
    """{name: torch tensor} of every tensor in the file (bfloat16 stays bfloat16)."""
    import torch
    dtypes = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64,
              "I32": torch.int32, "I64": torch.int64, "U8": torch.uint8, "I8": torch.int8}
    path = os.fspath(path)
    size = os.path.getsize(path)
    if size < 8:
        raise SafetensorsError(f"{path}: {size} bytes; too short for a header")
    data = np.memmap(path, dtype=np.uint8, mode="r")
    header_bytes = int.from_bytes(data[:8].tobytes(), "little")
    if header_bytes > size - 8:
        raise SafetensorsError(f"{path}: header of {header_bytes} bytes in a file of {size}")
    try:
        header = json.loads(data[8:8 + header_bytes].tobytes())
    except ValueError as e:
        raise SafetensorsError(f"{path}: header is not valid JSON: {e}") from None
    body = data[8 + header_bytes:]
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        kind, shape, (begin, end) = info["dtype"], tuple(info["shape"]), info["data_offsets"]
        if kind not in _WIDTH:
            raise SafetensorsError(f"{path}: tensor {name!r} has unsupported dtype {kind}")
        count = int(np.prod(shape, dtype=np.int64)) if shape else 1
        if not 0 <= begin <= end <= body.size or end - begin != count * _WIDTH[kind]:
            raise SafetensorsError(f"{path}: tensor {name!r} of shape {list(shape)} has bytes {begin}..{end}")
        raw = torch.from_numpy(np.array(body[begin:end]))
        out[name] = raw.view(dtypes[kind]).reshape(shape)
    return out
