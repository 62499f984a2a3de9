"""Model folders on disk: config.json and *.safetensors (an 8-byte little-endian length, that many bytes of JSON with name ->
dtype, shape, data_offsets, then the data), read without a library."""

import json
import struct
from pathlib import Path

import numpy as np
import torch
from torch import Tensor

DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64, "I8": torch.int8,
          "U8": torch.uint8, "I16": torch.int16, "I32": torch.int32, "I64": torch.int64, "BOOL": torch.bool}


def read_safetensors(path: "str | Path") -> dict[str, Tensor]:
    """The file's tensors by name, as views of its memory map (copied when they are moved or cast)."""
    path = Path(path)
    size = path.stat().st_size
    with open(path, "rb") as f:
        length = struct.unpack("<Q", f.read(8))[0]
        if length > size - 8:
            raise ValueError(f"{path}: header of {length} bytes in a file of {size}")
        header = json.loads(f.read(length))
    data = torch.from_numpy(np.memmap(path, dtype=np.uint8, mode="c", offset=8 + length, shape=(size - 8 - length,))) \
        if size > 8 + length else torch.empty(0, dtype=torch.uint8)
    tensors = {}
    for name, entry in header.items():
        if name == "__metadata__":
            continue
        begin, end = entry["data_offsets"]
        dtype = DTYPES[entry["dtype"]]
        count = int(np.prod(entry["shape"], dtype=np.int64))
        if not 0 <= begin <= end <= data.numel() or end - begin != count * dtype.itemsize:
            raise ValueError(f"{path}: {name} lies at {begin}..{end}, which is not {entry['shape']} of {entry['dtype']}")
        tensors[name] = data[begin:end].clone().view(dtype).view(entry["shape"])
    return tensors


def read_folder(folder: "str | Path") -> tuple[dict, dict[str, Tensor]]:
    """(config, tensors) of a model folder; the tensors of all its *.safetensors files together."""
    folder = Path(folder)
    tensors: dict[str, Tensor] = {}
    for path in sorted(folder.glob("*.safetensors")):
        tensors.update(read_safetensors(path))
    if not tensors:
        raise FileNotFoundError(f"{folder}: no *.safetensors file")
    return read_config(folder), tensors


def read_config(folder: "str | Path") -> dict:
    return json.loads((Path(folder) / "config.json").read_text())
