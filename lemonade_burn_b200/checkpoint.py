"""Checkpoints of the bf16 families: a folder with config.json and model.safetensors."""
from __future__ import annotations

import json
import struct
from pathlib import Path
from typing import Dict

import numpy as np

FILE_NAME = "model.safetensors"


def bf16_bits(a: np.ndarray) -> np.ndarray:
    """float32 -> bf16 bits, round to nearest even."""
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def bf16_values(bits: np.ndarray) -> np.ndarray:
    return (bits.astype(np.uint32) << 16).view(np.float32)


def save_checkpoint(directory, cfg: dict, tensors: Dict[str, np.ndarray]) -> None:
    """config.json + model.safetensors; `tensors` are bf16 bits (uint16)."""
    directory = Path(directory)
    directory.mkdir(parents=True, exist_ok=True)
    (directory / "config.json").write_text(json.dumps(cfg))
    head, off = {}, 0
    for name, t in tensors.items():
        head[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [off, off + 2 * t.size]}
        off += 2 * t.size
    text = json.dumps(head).encode()
    text += b" " * (-len(text) % 8)
    with open(directory / FILE_NAME, "wb") as f:
        f.write(struct.pack("<Q", len(text)))
        f.write(text)
        for t in tensors.values():
            f.write(np.ascontiguousarray(t, dtype="<u2").tobytes())
