"""Reader of .safetensors files: an 8-byte little-endian length, that many bytes of JSON (name -> dtype,
shape, data_offsets), then the data."""
import json
import mmap
import struct

import torch

_DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64, "I64": torch.int64,
           "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}


def read_safetensors(path):
    """name -> CPU tensor (copies of the file's data)."""
    with open(path, "rb") as f:
        size = f.seek(0, 2)
        if size < 8:
            raise ValueError(f"{path}: not a safetensors file")
        f.seek(0)
        (n,) = struct.unpack("<Q", f.read(8))
        if n > size - 8:
            raise ValueError(f"{path}: header of {n} bytes in a file of {size}")
        header = json.loads(f.read(n))
        base, tensors = 8 + n, {}
        with mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ) as data:
            for name, info in header.items():
                if name == "__metadata__":
                    continue
                dtype, shape = _DTYPES[info["dtype"]], info["shape"]
                begin, end = info["data_offsets"]
                count = 1
                for s in shape:
                    count *= s
                if not 0 <= begin <= end <= size - base or end - begin != count * dtype.itemsize:
                    raise ValueError(f"{path}: {name} has data_offsets {begin}..{end} for {count} x {info['dtype']}")
                raw = bytearray(data[base + begin:base + end])
                tensors[name] = torch.frombuffer(raw, dtype=dtype).view(shape) if count else torch.empty(shape, dtype=dtype)
    return tensors


def write_safetensors(path, tensors):
    """The inverse, for contiguous CPU tensors."""
    names = {v: k for k, v in _DTYPES.items()}
    header, at = {}, 0
    for name, t in tensors.items():
        n = t.numel() * t.element_size()
        header[name] = {"dtype": names[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + n]}
        at += n
    text = json.dumps(header).encode()
    text += b" " * (-len(text) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(text)) + text)
        for t in tensors.values():
            f.write(t.contiguous().view(-1).view(torch.uint8).numpy().tobytes())
