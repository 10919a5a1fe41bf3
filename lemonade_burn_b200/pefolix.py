"""The Pefolix family: a decoder with layer norms before and after each sublayer, attention under a sliding window
with kept first tokens and a distance bias, gated or mixture-of-experts feed-forwards. The compute is in liblbk.so
(csrc/lbk_pefolix.cu); this module holds the Python class, the configuration helpers and random checkpoints.

config.json: {"architecture": "Pefolix", "vocab", "width", "norm": {"eps"}, "layers": [{"type": "attention",
"mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "mask": {"size", "keep_first"}}, "mlp": null |
{"kind": "dense", "ff"} | {"kind": "moe", "router": {"experts", "top"}, "expert": {"ff"}, "shared": {"ff"} | null}}]}
model.safetensors: bfloat16; embed, head [vocab, width], final.norm, and per layer l<i>.norm1, norm1b, norm2, norm2b,
mix.q, mix.k, mix.v, mix.o, mlp.gate, up, down, or mlp.router, e<k>.up, e<k>.down, shared.up, shared.down, shared.sg.
"""
from __future__ import annotations

from typing import Dict, Iterator, Optional, Tuple

import numpy as np

from .checkpoint import FILE_NAME, bf16_bits, bf16_values, save_checkpoint  # noqa: F401
from .runtime import NativeModel, register

ARCHITECTURE = "Pefolix"


class NativePefolix(NativeModel):
    """A Pefolix model on the GPU. dtype "bfloat16" is how it is served; "float32" computes everything in 32-bit."""


register(ARCHITECTURE, NativePefolix)


def attention_layer(heads: int, kv_heads: int, dim: int, vdim: Optional[int] = None, window: Optional[int] = None, keep_first: int = 0,
                    scale: Optional[float] = None, mlp: Optional[dict] = None) -> dict:
    """One entry of config["layers"]."""
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim or dim, "scale": scale if scale is not None else dim ** -0.5}
    if window is not None:
        mixer["mask"] = {"size": window, "keep_first": keep_first}
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def dense_mlp(ff: int) -> dict:
    return {"kind": "dense", "ff": ff}


def moe_mlp(experts: int, top: int, ff: int, shared_ff: Optional[int] = None) -> dict:
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff},
            "shared": {"ff": shared_ff} if shared_ff else None}


def make_config(vocab: int, width: int, layers: list, eps: float = 1e-6) -> dict:
    return {"architecture": ARCHITECTURE, "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


def tensor_shapes(cfg: dict) -> Iterator[Tuple[str, Tuple[int, ...]]]:
    """(name, shape) of every tensor of a model, in file order."""
    V, W = cfg["vocab"], cfg["width"]
    yield "embed", (V, W)
    for i, layer in enumerate(cfg["layers"]):
        p, mx, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if mlp else ()):
            yield p + n, (W,)
        yield p + "mix.q", (mx["heads"] * mx["dim"], W)
        yield p + "mix.k", (mx["kv_heads"] * mx["dim"], W)
        yield p + "mix.v", (mx["kv_heads"] * mx["vdim"], W)
        yield p + "mix.o", (W, mx["heads"] * mx["vdim"])
        if not mlp:
            continue
        if mlp["kind"] == "dense":
            yield p + "mlp.gate", (mlp["ff"], W)
            yield p + "mlp.up", (mlp["ff"], W)
            yield p + "mlp.down", (W, mlp["ff"])
            continue
        for e in range(mlp["router"]["experts"]):
            yield f"{p}mlp.e{e}.up", (mlp["expert"]["ff"], W)
            yield f"{p}mlp.e{e}.down", (W, mlp["expert"]["ff"])
        yield p + "mlp.router", (mlp["router"]["experts"], W)
        if mlp.get("shared"):
            yield p + "mlp.shared.up", (mlp["shared"]["ff"], W)
            yield p + "mlp.shared.down", (W, mlp["shared"]["ff"])
            yield p + "mlp.shared.sg", (1, W)
    yield "final.norm", (W,)
    yield "head", (V, W)


def random_checkpoint(cfg: dict, seed: int = 0) -> Dict[str, np.ndarray]:
    """Random weights as bf16 bits: matrices N(0, 1 / columns), norm weights near 1, embedding N(0, 1)."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg):
        a = rng.standard_normal(shape, dtype=np.float32)
        if len(shape) == 1:
            a = 1.0 + 0.1 * a
        elif name != "embed":
            a *= shape[1] ** -0.5
        out[name] = bf16_bits(a)
    return out
