"""Reading and writing safetensors files.

Layout: a little-endian 64-bit length, that many bytes of JSON {name: {"dtype", "shape", "data_offsets"}}, then the
tensors' bytes; offsets count from the end of the JSON.
"""

from __future__ import annotations

import json
import struct

import numpy as np
import torch

_DTYPES = {
    "F64": torch.float64, "F32": torch.float32, "F16": torch.float16, "BF16": torch.bfloat16,
    "I64": torch.int64, "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool,
}
_NAMES = {v: k for k, v in _DTYPES.items()}


def read_safetensors(path: str) -> dict[str, torch.Tensor]:
    """Tensors on the host, views of the mapped file (copy-on-write)."""
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(n))
    data = torch.from_numpy(np.memmap(path, dtype=np.uint8, mode="c"))[8 + n :]
    out = {}
    for name, entry in header.items():
        if name == "__metadata__":
            continue
        if entry["dtype"] not in _DTYPES:
            raise ValueError(f"{path}: {name} has dtype {entry['dtype']}, which is not read")
        dtype, shape = _DTYPES[entry["dtype"]], entry["shape"]
        begin, end = entry["data_offsets"]
        size = int(np.prod(shape, dtype=np.int64)) * torch.empty(0, dtype=dtype).element_size()
        if not 0 <= begin <= end <= data.numel() or end - begin != size:
            raise ValueError(f"{path}: {name} does not fit its bytes")
        raw = data[begin:end]
        if raw.data_ptr() % torch.empty(0, dtype=dtype).element_size():
            raw = raw.clone()
        out[name] = raw.view(dtype).reshape(shape)
    return out


def write_safetensors(path: str, tensors: dict[str, torch.Tensor]) -> None:
    header, blobs, at = {}, [], 0
    for name, t in tensors.items():
        raw = t.detach().cpu().contiguous().reshape(-1).view(torch.uint8).numpy().tobytes()
        header[name] = {"dtype": _NAMES[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        at += len(raw)
        blobs.append(raw)
    text = json.dumps(header).encode()
    text += b" " * (-len(text) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(text)))
        f.write(text)
        for raw in blobs:
            f.write(raw)
