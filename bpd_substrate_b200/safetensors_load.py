"""Reader (and writer) of safetensors checkpoints: an 8-byte little-endian length, that many bytes of JSON
(name -> dtype, shape, data_offsets), then the data.  bf16 tensors come back as uint16 bit patterns."""
import json
import mmap
import struct

import numpy as np

DTYPES = {"BF16": np.uint16, "F16": np.float16, "F32": np.float32, "F64": np.float64, "I8": np.int8, "U8": np.uint8, "I16": np.int16,
          "I32": np.int32, "I64": np.int64, "BOOL": np.bool_}


def bf16_to_f32(bits):
    return (np.asarray(bits, np.uint16).astype(np.uint32) << 16).view(np.float32)


def f32_to_bf16(x):
    """Round to nearest even; finite values."""
    u = np.array(x, np.float32, order="C").view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


class SafetensorsFile:
    """Tensor table of a file; tensor bytes are read through a memory map."""

    def __init__(self, path):
        self.path = path
        self._fh = open(path, "rb")
        self._map = mmap.mmap(self._fh.fileno(), 0, access=mmap.ACCESS_READ)
        if len(self._map) < 8:
            raise ValueError(f"{path}: not a safetensors file")
        n = struct.unpack_from("<Q", self._map)[0]
        if 8 + n > len(self._map):
            raise ValueError(f"{path}: header of {n} bytes runs past the end of the file")
        header = json.loads(self._map[8:8 + n].decode("utf-8"))
        header.pop("__metadata__", None)
        self.tensors, self._data = header, 8 + n
        for name, t in header.items():
            if t["dtype"] not in DTYPES:
                raise ValueError(f"{path}: tensor {name} has dtype {t['dtype']}")
            begin, end = t["data_offsets"]
            size = int(np.prod(t["shape"], dtype=np.int64)) * np.dtype(DTYPES[t["dtype"]]).itemsize
            if not 0 <= begin <= end <= len(self._map) - self._data or end - begin != size:
                raise ValueError(f"{path}: tensor {name} does not fit its shape or the file")

    def __contains__(self, name):
        return name in self.tensors

    def shape(self, name):
        if name not in self.tensors:
            raise KeyError(f"{self.path}: no tensor {name}")
        return tuple(self.tensors[name]["shape"])

    def raw(self, name):
        """The tensor as stored (bf16 as uint16)."""
        if name not in self.tensors:
            raise KeyError(f"{self.path}: no tensor {name}")
        t = self.tensors[name]
        begin, end = t["data_offsets"]
        dt = np.dtype(DTYPES[t["dtype"]]).newbyteorder("<")
        return np.frombuffer(self._map, dt, (end - begin) // dt.itemsize, self._data + begin).reshape(t["shape"])

    def f32(self, name):
        a = self.raw(name)
        return bf16_to_f32(a) if self.tensors[name]["dtype"] == "BF16" else a.astype(np.float32)

    def bf16(self, name):
        """bf16 bit patterns (other types are rounded)."""
        return np.array(self.raw(name)) if self.tensors[name]["dtype"] == "BF16" else f32_to_bf16(self.f32(name))

    def close(self):
        try:
            self._map.close()
        except BufferError:
            pass            # arrays returned by raw() still look into the map: it goes when they do
        self._fh.close()


def save_bf16(path, tensors):
    """Writes {name: float array or uint16 bf16 bits} as a bf16 safetensors file (int32 arrays stay int32)."""
    header, blobs, at = {}, [], 0
    for name, a in tensors.items():
        a = np.asarray(a)
        kind = "I32" if a.dtype == np.int32 else "BF16"
        data = (a if a.dtype in (np.uint16, np.int32) else f32_to_bf16(a)).tobytes()
        header[name] = {"dtype": kind, "shape": list(a.shape), "data_offsets": [at, at + len(data)]}
        blobs.append(data)
        at += len(data)
    head = json.dumps(header).encode()
    head += b" " * (-len(head) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(head)))
        f.write(head)
        for b in blobs:
            f.write(b)
