"""Reading a model folder: config.json and the tensors of its safetensors files."""
from __future__ import annotations

import json
import mmap
import struct
from pathlib import Path

import torch

_DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64,
           "I64": torch.int64, "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8,
           "BOOL": torch.bool}


def read_config(folder) -> dict:
    with open(Path(folder) / "config.json") as f:
        return json.load(f)


def read_safetensors(path) -> dict[str, torch.Tensor]:
    """name -> CPU tensor.  The file is an 8-byte little-endian length, that much JSON (name -> dtype, shape,
    data_offsets) and the data the offsets count from."""
    out = {}
    with open(path, "rb") as f:
        data = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ)
        (n,) = struct.unpack("<Q", data[:8])
        if n > len(data) - 8:
            raise ValueError(f"{path}: header of {n} bytes in a file of {len(data)}")
        for name, d in json.loads(data[8:8 + n]).items():
            if name == "__metadata__":
                continue
            if d["dtype"] not in _DTYPES:
                raise ValueError(f"{path}: tensor {name} has dtype {d['dtype']}")
            lo, hi = d["data_offsets"]
            raw = bytearray(data[8 + n + lo:8 + n + hi])
            t = torch.frombuffer(raw, dtype=_DTYPES[d["dtype"]]) if raw else torch.empty(0, dtype=_DTYPES[d["dtype"]])
            out[name] = t.view(d["shape"])
    return out


def read_tensors(folder) -> dict[str, torch.Tensor]:
    """Every tensor of the folder's *.safetensors files."""
    out = {}
    files = sorted(Path(folder).glob("*.safetensors"))
    if not files:
        raise FileNotFoundError(f"no .safetensors file in {folder}")
    for f in files:
        out.update(read_safetensors(f))
    return out


def write_safetensors(path, tensors) -> None:
    """The inverse of read_safetensors for bf16, fp32 and int32 tensors (tests, synthetic checkpoints)."""
    names = {v: k for k, v in _DTYPES.items()}
    head, at, blobs = {}, 0, []
    for name, t in tensors.items():
        t = t.detach().cpu().contiguous()
        raw = t.reshape(-1).view(torch.uint8).numpy().tobytes()
        head[name] = {"dtype": names[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        at += len(raw)
        blobs.append(raw)
    text = json.dumps(head).encode()
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(text)) + text + b"".join(blobs))
