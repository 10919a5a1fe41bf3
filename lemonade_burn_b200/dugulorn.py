"""The Dugulorn family: a decoder whose layers each have one of three mixers (latent attention with rotated key parts
and YaRN-scaled frequencies, lightning attention, a gated delta rule with a decay per key channel) and a squared-relu
feed-forward with biases or none; only the sublayers' outputs are normed. The compute is in liblbk.so
(csrc/lbk_dugulorn.cu); this module holds the Python class, the configuration helpers and random checkpoints.

config.json: {"architecture": "Dugulorn", "vocab", "width", "norm": {"eps"}, "layers": [{"type", "mixer", "mlp"}]} with
"mlp" null or {"kind": "dense", "ff"} and, by type, the mixer's sizes:
    latent_attention  heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot {base, dims, scaling: null | {factor,
                      original, fast, slow}}, and optionally kv_from, the layer whose cached latents it reads
    lightning         heads, dim, vdim, decay (one per head)
    channel_delta     heads, kv_heads, dim, vdim, conv (taps of the short convolutions)
model.safetensors: bfloat16; names and shapes in tensor_shapes. Layer and model norm weights are stored around zero.
"""
from __future__ import annotations

from typing import Dict, Iterator, Optional, Sequence, Tuple

import numpy as np

from .checkpoint import FILE_NAME, bf16_bits, bf16_values, save_checkpoint  # noqa: F401
from .runtime import NativeModel, register

ARCHITECTURE = "Dugulorn"


class NativeDugulorn(NativeModel):
    """A Dugulorn model on the GPU. dtype "bfloat16" is how it is served; "float32" computes everything in 32-bit."""


register(ARCHITECTURE, NativeDugulorn)


def yarn(factor: float, original: int, fast: float = 32.0, slow: float = 1.0) -> dict:
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def latent_layer(heads: int, dim: int, rot_dim: int, vdim: int, q_rank: int, kv_rank: int, scale: Optional[float] = None, base: float = 10000.0,
                 scaling: Optional[dict] = None, kv_from: Optional[int] = None, ff: Optional[int] = None) -> dict:
    """One entry of config["layers"]: latent attention."""
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
             "scale": scale if scale is not None else (dim + rot_dim) ** -0.5, "rot": {"base": base, "dims": rot_dim, "scaling": scaling}}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": mixer, "mlp": dense_mlp(ff)}


def lightning_layer(heads: int, dim: int, vdim: int, decay: Sequence[float], ff: Optional[int] = None) -> dict:
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}, "mlp": dense_mlp(ff)}


def delta_layer(heads: int, kv_heads: int, dim: int, vdim: int, conv: int, ff: Optional[int] = None) -> dict:
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": dense_mlp(ff)}


def dense_mlp(ff: Optional[int]) -> Optional[dict]:
    return {"kind": "dense", "ff": ff} if ff else None


def make_config(vocab: int, width: int, layers: list, eps: float = 1e-6) -> dict:
    return {"architecture": ARCHITECTURE, "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


def tensor_shapes(cfg: dict, low_rank: int = 16) -> Iterator[Tuple[str, Tuple[int, ...]]]:
    """(name, shape) of every tensor of a model, in file order. low_rank: inner size of the delta rule's two-step
    projections, which the configuration does not fix."""
    V, W = cfg["vocab"], cfg["width"]
    yield "embed", (V, W)
    yield "embed.norm", (W,)
    for i, layer in enumerate(cfg["layers"]):
        p, mx, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        for n in ("norm1",) + (("norm2",) if mlp else ()):
            yield p + n, (W,)
        H, d, vd = mx["heads"], mx["dim"], mx["vdim"]
        if layer["type"] == "latent_attention":
            r, qr, kr = mx["rot_dim"], mx["q_rank"], mx["kv_rank"]
            yield p + "mix.dq", (qr, W)
            yield p + "mix.dq.norm", (qr,)
            yield p + "mix.uq", (H * (d + r), qr)
            if mx.get("kv_from") is None:
                yield p + "mix.dkv", (kr + r, W)
                yield p + "mix.dkv.norm", (kr,)
            yield p + "mix.uk", (H * d, kr)
            yield p + "mix.uv", (H * vd, kr)
            yield p + "mix.g", (H, W)
        elif layer["type"] == "lightning":
            for n, rows in (("q", H * d), ("k", H * d), ("v", H * vd), ("g", H * vd)):
                yield p + "mix." + n, (rows, W)
            yield p + "mix.norm", (H * vd,)
        else:
            for n, rows in (("q", mx["kv_heads"] * d), ("k", mx["kv_heads"] * d), ("v", H * vd)):
                yield p + "mix." + n, (rows, W)
                yield p + "mix." + n + ".conv", (rows, mx["conv"])
            yield p + "mix.b", (H, W)
            yield p + "mix.A_log", (H,)
            yield p + "mix.norm", (vd,)
            yield p + "mix.a1", (low_rank, W)
            yield p + "mix.a2", (H * d, low_rank)
            yield p + "mix.dt_bias", (H * d,)
            yield p + "mix.g1", (low_rank, W)
            yield p + "mix.g2", (H * vd, low_rank)
        yield p + "mix.o", (W, H * vd)
        if mlp:
            yield p + "mlp.up", (mlp["ff"], W)
            yield p + "mlp.up.b", (mlp["ff"],)
            yield p + "mlp.down", (W, mlp["ff"])
            yield p + "mlp.down.b", (W,)
    yield "final.norm", (W,)


def random_checkpoint(cfg: dict, seed: int = 0, low_rank: int = 16) -> Dict[str, np.ndarray]:
    """Random weights as bf16 bits: matrices N(0, 1 / columns), embedding N(0, 1), norm weights near their neutral value,
    decays of the delta rule between none and strong."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg, low_rank):
        a = rng.standard_normal(shape, dtype=np.float32)
        if name.endswith((".norm1", ".norm2")) or name in ("embed.norm", "final.norm"):
            a *= 0.1
        elif name.endswith(".norm"):
            a = 1.0 + 0.1 * a
        elif name.endswith(".b") and len(shape) == 1:
            a *= 0.3
        elif name.endswith("A_log"):
            a *= 0.7
        elif name.endswith("dt_bias"):
            a = 1.5 * a - 2.0
        elif name != "embed":
            a *= shape[1] ** -0.5
        out[name] = bf16_bits(a)
    return out
