"""Reading `.safetensors` files: an 8-byte little-endian header length, a JSON header `name -> dtype, shape, data_offsets`,
then the tensor data. The data is memory-mapped; tensors are views of the map until they are copied somewhere."""
import json
import mmap
import struct
from typing import Dict

import torch

__all__ = ["read_safetensors"]

_DTYPES = {"F64": torch.float64, "F32": torch.float32, "F16": torch.float16, "BF16": torch.bfloat16, "I64": torch.int64,
           "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}


def read_safetensors(path: str) -> Dict[str, torch.Tensor]:
    with open(path, "rb") as f:
        buf = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_COPY)
    if len(buf) < 8:
        raise ValueError(f"{path}: too short for a safetensors file")
    (n,) = struct.unpack("<Q", buf[:8])
    if n > len(buf) - 8:
        raise ValueError(f"{path}: header of {n} bytes does not fit the file")
    header = json.loads(buf[8:8 + n].decode("utf-8"))
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        if info["dtype"] not in _DTYPES:
            raise ValueError(f"{path}: tensor {name!r} has unsupported dtype {info['dtype']}")
        dt, shape = _DTYPES[info["dtype"]], tuple(info["shape"])
        begin, end = info["data_offsets"]
        count = 1
        for d in shape:
            count *= d
        if begin < 0 or end - begin != count * dt.itemsize or 8 + n + end > len(buf):
            raise ValueError(f"{path}: tensor {name!r} has inconsistent offsets")
        if count == 0:
            out[name] = torch.empty(shape, dtype=dt)
        elif (8 + n + begin) % dt.itemsize:
            out[name] = torch.frombuffer(bytearray(buf[8 + n + begin:8 + n + end]), dtype=dt).reshape(shape)
        else:
            out[name] = torch.frombuffer(buf, dtype=dt, count=count, offset=8 + n + begin).reshape(shape)
    return out
