"""safetensors container: an 8-byte little-endian header length, a JSON header (name -> dtype, shape,
data_offsets), then the data. Tensors are read lazily from a memory map."""
import json
import struct

import numpy as np

from . import BF16, F16, F32

GGML_TYPE = {"F32": F32, "F16": F16, "BF16": BF16}
ELEM_BYTES = {"F64": 8, "F32": 4, "F16": 2, "BF16": 2, "I64": 8, "I32": 4, "I16": 2, "I8": 1, "U8": 1, "BOOL": 1}


class SafetensorsError(ValueError):
    pass


class SafetensorsFile:
    """`.tensors` {name: (dtype, shape, begin, end)} with offsets into the data section."""

    def __init__(self, path):
        self.path = path
        self.data = np.memmap(path, dtype=np.uint8, mode="r")
        if len(self.data) < 8:
            raise SafetensorsError("not a safetensors file (too short)")
        n = struct.unpack("<Q", bytes(self.data[:8]))[0]
        if 8 + n > len(self.data):
            raise SafetensorsError("the header runs past the end of the file")
        header = json.loads(bytes(self.data[8:8 + n]))
        self.base = 8 + n
        self.tensors = {}
        for name, info in header.items():
            if name == "__metadata__":
                continue
            dtype, shape = info["dtype"], tuple(int(d) for d in info["shape"])
            begin, end = info["data_offsets"]
            if dtype not in ELEM_BYTES:
                raise SafetensorsError(f"tensor {name}: unknown dtype {dtype}")
            if end - begin != int(np.prod(shape, dtype=np.int64)) * ELEM_BYTES[dtype] or self.base + end > len(self.data):
                raise SafetensorsError(f"tensor {name}: {end - begin} bytes at {begin} do not hold {dtype} {list(shape)}")
            self.tensors[name] = (dtype, shape, begin, end)

    def raw(self, name):
        """(ggml type id, shape, bytes) of a floating-point tensor, a view of the memory map."""
        if name not in self.tensors:
            raise SafetensorsError(f"tensor {name} is missing")
        dtype, shape, begin, end = self.tensors[name]
        if dtype not in GGML_TYPE:
            raise SafetensorsError(f"tensor {name}: dtype {dtype} is not a weight type")
        return GGML_TYPE[dtype], shape, self.data[self.base + begin:self.base + end]


def write_safetensors(path, tensors):
    """tensors: [(name, dtype name, shape, bytes-like)]."""
    header, blobs, off = {}, [], 0
    for name, dtype, shape, raw in tensors:
        raw = np.ascontiguousarray(raw).view(np.uint8).reshape(-1)
        header[name] = {"dtype": dtype, "shape": list(shape), "data_offsets": [off, off + raw.size]}
        blobs.append(raw)
        off += raw.size
    head = json.dumps(header).encode()
    head += b" " * (-len(head) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head)
        for b in blobs:
            f.write(b.tobytes())
