"""Reader of `.safetensors` files: an 8-byte little-endian header length, that many bytes of JSON
(name -> dtype, shape, data_offsets), then the data. Tensors come back as numpy views of a memory map;
bfloat16 stays in its 16-bit pattern (uint16) and is widened by `as_f32`."""
import json
import struct

import numpy as np

_DTYPES = {"BF16": np.uint16, "F16": np.float16, "F32": np.float32, "I32": np.int32, "I64": np.int64, "U8": np.uint8, "I8": np.int8}


class Tensor:
    def __init__(self, dtype, data):
        self.dtype, self.data = dtype, data

    @property
    def shape(self):
        return self.data.shape

    def as_f32(self):
        if self.dtype == "BF16":
            return (self.data.astype(np.uint32) << np.uint32(16)).view(np.float32)
        return self.data.astype(np.float32)

    def as_bf16(self):
        """The bf16 bit patterns, rounded to nearest even where the tensor is stored in another format."""
        if self.dtype == "BF16":
            return self.data
        u = self.as_f32().view(np.uint32)
        return ((u + np.uint32(0x7FFF) + ((u >> np.uint32(16)) & np.uint32(1))) >> np.uint32(16)).astype(np.uint16)


def read(path):
    """All tensors of a file, by name."""
    raw = np.memmap(path, dtype=np.uint8, mode="r")
    if raw.size < 8:
        raise ValueError(f"{path}: too short for a safetensors file")
    n = struct.unpack("<Q", raw[:8].tobytes())[0]
    if n > raw.size - 8:
        raise ValueError(f"{path}: header longer than the file")
    header = json.loads(raw[8:8 + n].tobytes())
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        if info["dtype"] not in _DTYPES:
            raise ValueError(f"{path}: tensor {name} has dtype {info['dtype']}")
        begin, end = info["data_offsets"]
        dt = np.dtype(_DTYPES[info["dtype"]])
        count = int(np.prod(info["shape"], dtype=np.int64))
        if not 0 <= begin <= end <= raw.size - 8 - n or end - begin != count * dt.itemsize:
            raise ValueError(f"{path}: tensor {name} lies outside the file")
        out[name] = Tensor(info["dtype"], np.frombuffer(raw[8 + n + begin:8 + n + end].tobytes(), dtype=dt).reshape(info["shape"]))
    return out
