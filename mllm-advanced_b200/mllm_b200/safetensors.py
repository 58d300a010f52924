"""Reader of safetensors files (8-byte little-endian header length, a JSON header, the data), memory-mapped."""
import json
import mmap
import os

import numpy as np

_NUMPY = {"F64": np.float64, "F32": np.float32, "F16": np.float16, "I64": np.int64, "I32": np.int32, "I16": np.int16,
          "I8": np.int8, "U8": np.uint8, "BOOL": np.bool_, "BF16": np.uint16}


def bf16_to_f32(bits):
    return (np.asarray(bits, np.uint16).astype(np.uint32) << 16).view(np.float32)  # (a scalar for a tensor of no dimensions)


def f32_to_bf16(x):
    """Bits of the nearest bf16 (ties to even) of finite numbers."""
    u = np.asarray(x, np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


class Tensors:
    """The tensors of a folder's *.safetensors files by name."""

    def __init__(self, folder):
        self._entries, self._maps = {}, []
        files = sorted(f for f in os.listdir(folder) if f.endswith(".safetensors"))
        if not files:
            raise FileNotFoundError(f"no .safetensors file in {folder}")
        for f in files:
            with open(os.path.join(folder, f), "rb") as fh:
                m = mmap.mmap(fh.fileno(), 0, access=mmap.ACCESS_READ)
            self._maps.append(m)
            n = int.from_bytes(m[:8], "little")
            for name, e in json.loads(m[8:8 + n]).items():
                if name != "__metadata__":
                    lo, hi = e["data_offsets"]
                    self._entries[name] = (m, e["dtype"], tuple(e["shape"]), 8 + n + lo, hi - lo)

    def __contains__(self, name):
        return name in self._entries

    def names(self):
        return list(self._entries)

    def shape(self, name):
        return self._entries[name][2]

    def raw(self, name):
        """(dtype name, array); bf16 as its bits in uint16."""
        if name not in self._entries:
            raise KeyError(f"tensor {name!r} is missing")
        m, dt, shape, at, nbytes = self._entries[name]
        t = np.dtype(_NUMPY[dt])
        return dt, np.frombuffer(m, t, nbytes // t.itemsize, at).reshape(shape)

    def f32(self, name):
        dt, a = self.raw(name)
        return bf16_to_f32(a) if dt == "BF16" else a.astype(np.float32)

    def bf16(self, name):
        dt, a = self.raw(name)
        return a if dt == "BF16" else f32_to_bf16(a)


def save(path, tensors):
    """Writes {name: (dtype name, array)} (bf16 as uint16 bits)."""
    header, blobs, at = {}, [], 0
    for name, (dt, a) in tensors.items():
        b = np.asarray(a).tobytes()
        header[name] = {"dtype": dt, "shape": list(np.shape(a)), "data_offsets": [at, at + len(b)]}
        blobs.append(b)
        at += len(b)
    h = json.dumps(header).encode()
    h += b" " * (-len(h) % 8)
    with open(path, "wb") as f:
        f.write(len(h).to_bytes(8, "little") + h)
        for b in blobs:
            f.write(b)
