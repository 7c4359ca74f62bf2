"""Reader and writer of .safetensors files: an 8-byte little-endian header length, that many bytes of JSON
(name -> dtype, shape, data_offsets), then the tensors' bytes."""
import json
import struct

import numpy as np
import torch

_DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64, "I32": torch.int32,
           "I64": torch.int64, "I8": torch.int8, "U8": torch.uint8, "I16": torch.int16, "BOOL": torch.bool}
_NAMES = {v: k for k, v in _DTYPES.items()}


def read_safetensors(path):
    """{name: CPU tensor}; the tensors share one buffer."""
    with open(path, "rb") as f:
        raw = f.read(8)
        if len(raw) != 8:
            raise ValueError(f"{path}: not a safetensors file")
        n = struct.unpack("<Q", raw)[0]
        try:
            head = json.loads(f.read(n))
        except ValueError as e:
            raise ValueError(f"{path}: not a safetensors file") from e
        data = np.frombuffer(f.read(), np.uint8).copy()
    out = {}
    for name, info in head.items():
        if name == "__metadata__":
            continue
        if info["dtype"] not in _DTYPES:
            raise NotImplementedError(f"{path}: tensor {name} has type {info['dtype']}")
        dt = _DTYPES[info["dtype"]]
        a, b = info["data_offsets"]
        size = int(np.prod(info["shape"], dtype=np.int64)) * dt.itemsize
        if not 0 <= a <= b <= data.size or b - a != size:
            raise ValueError(f"{path}: tensor {name} has bad offsets")
        t = torch.from_numpy(data[a:b].copy()).view(dt) if size else torch.empty(0, dtype=dt)
        out[name] = t.reshape(info["shape"])
    return out


def write_safetensors(path, tensors):
    head, blobs, off = {}, [], 0
    for name, t in tensors.items():
        t = t.detach().cpu().contiguous()
        b = t.reshape(-1).view(torch.uint8).numpy().tobytes()
        head[name] = {"dtype": _NAMES[t.dtype], "shape": list(t.shape), "data_offsets": [off, off + len(b)]}
        blobs.append(b)
        off += len(b)
    h = json.dumps(head).encode()
    h += b" " * (-len(h) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h)
        for b in blobs:
            f.write(b)
