"""Reads and writes safetensors files: an 8-byte little-endian header length, a JSON header (name ->
dtype, shape, data_offsets) and the tensors' bytes."""

from __future__ import annotations

import json
import struct
from pathlib import Path
from typing import Dict

import torch

_DTYPES = {"F64": torch.float64, "F32": torch.float32, "F16": torch.float16, "BF16": torch.bfloat16,
           "I64": torch.int64, "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8,
           "BOOL": torch.bool}
_NAMES = {dtype: name for name, dtype in _DTYPES.items()}


def load_safetensors(path: str | Path) -> Dict[str, torch.Tensor]:
    """All tensors of a file, on the CPU, in their stored dtypes."""

    data = bytearray(Path(path).read_bytes())
    if len(data) < 8:
        raise ValueError(f"{path} is not a safetensors file")
    size = struct.unpack_from("<Q", data)[0]
    if size > len(data) - 8:
        raise ValueError(f"{path}: the header is longer than the file")
    header = json.loads(bytes(data[8:8 + size]))
    tensors: Dict[str, torch.Tensor] = {}
    for name, entry in header.items():
        if name == "__metadata__":
            continue
        dtype = _DTYPES.get(entry["dtype"])
        if dtype is None:
            raise ValueError(f"{path}: tensor {name} has unsupported dtype {entry['dtype']}")
        begin, end = entry["data_offsets"]
        count = 1
        for extent in entry["shape"]:
            count *= extent
        itemsize = torch.empty(0, dtype=dtype).element_size()
        if not 0 <= begin <= end <= len(data) - 8 - size or end - begin != count * itemsize:
            raise ValueError(f"{path}: tensor {name} does not lie inside the file")
        piece = torch.frombuffer(data, dtype=torch.uint8, count=end - begin, offset=8 + size + begin) \
            if end > begin else torch.empty(0, dtype=torch.uint8)
        tensors[name] = piece.clone().view(dtype).reshape(entry["shape"])
    return tensors


def save_safetensors(tensors: Dict[str, torch.Tensor], path: str | Path) -> None:
    header, offset, blobs = {}, 0, []
    for name, tensor in tensors.items():
        flat = tensor.detach().cpu().contiguous().reshape(-1)
        blob = flat.view(torch.uint8).numpy().tobytes() if flat.numel() else b""
        header[name] = {"dtype": _NAMES[tensor.dtype], "shape": list(tensor.shape),
                        "data_offsets": [offset, offset + len(blob)]}
        offset += len(blob)
        blobs.append(blob)
    text = json.dumps(header).encode()
    text += b" " * (-len(text) % 8)
    with open(path, "wb") as file:
        file.write(struct.pack("<Q", len(text)))
        file.write(text)
        for blob in blobs:
            file.write(blob)
