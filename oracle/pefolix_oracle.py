"""Plain numpy restatement of the Pefolix decoder (test infrastructure; float64 by default, nothing shared with the
product path). One function per mechanism, whole sequences at once, no cache:

    layer_norm         (x - mean) / sqrt(var + eps) * w, var = mean of the squared deviations
    slopes             head h of H: 2^(-8 (h + 1) / H)
    visible            which keys a query position sees: a sliding window plus kept first tokens
    attention          grouped heads, scores * scale - slope * distance, softmax over the visible keys
    gelu_tanh, relu2   the two activations
    dense_ff           down(gelu_tanh(gate h) * (up h))
    route              softmax over all experts, the `top` largest, their scores as weights
    expert, moe_ff     down(relu2(up h)); weighted sum of the chosen experts + sigmoid(sg h) * shared
    forward            x += norm1b(mixer(norm1 x)); x += norm2b(ff(norm2 x)); logits = head norm(x)

`cfg` is the dictionary of config.json, `w` maps tensor names to float arrays.
"""
from __future__ import annotations

import json
import struct
from pathlib import Path
from typing import Dict, Optional

import numpy as np


def layer_norm(x, w, eps):
    mean = x.mean(-1, keepdims=True)
    d = x - mean
    return d / np.sqrt((d * d).mean(-1, keepdims=True) + eps) * w


def slopes(heads: int) -> np.ndarray:
    return np.array([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)])


def visible(qpos, kpos, mask: Optional[dict]) -> np.ndarray:
    """[len(qpos), len(kpos)] booleans."""
    i, j = np.asarray(qpos)[:, None], np.asarray(kpos)[None, :]
    causal = j <= i
    if not mask:
        return causal
    return causal & ((i - j < mask["size"]) | (j < mask.get("keep_first", 0)))


def attention(q, k, v, scale, mask, qpos, kpos) -> np.ndarray:
    """q [n, H, dim], k [m, G, dim], v [m, G, vdim] -> [n, H, vdim]."""
    H, G = q.shape[1], k.shape[1]
    see = visible(qpos, kpos, mask)
    dist = (np.asarray(qpos)[:, None] - np.asarray(kpos)[None, :]).astype(q.dtype)
    out = np.empty((q.shape[0], H, v.shape[2]), dtype=q.dtype)
    for h, slope in enumerate(slopes(H)):
        g = h // (H // G)
        s = q[:, h] @ k[:, g].T * scale - slope * dist
        s = np.where(see, s, -np.inf)
        p = np.exp(s - s.max(-1, keepdims=True))
        out[:, h] = (p / p.sum(-1, keepdims=True)) @ v[:, g]
    return out


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def relu2(z):
    r = np.maximum(z, 0.0)
    return r * r


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def dense_ff(h, gate, up, down):
    return (gelu_tanh(h @ gate.T) * (h @ up.T)) @ down.T


def expert(h, up, down):
    return relu2(h @ up.T) @ down.T


def route(h, router, top):
    """(ids [n, top], weights [n, top]): the scores of the chosen experts, not renormalised."""
    z = h @ router.T
    e = np.exp(z - z.max(-1, keepdims=True))
    s = e / e.sum(-1, keepdims=True)
    ids = np.argsort(-s, axis=-1, kind="stable")[:, :top]
    return ids, np.take_along_axis(s, ids, axis=-1)


def moe_ff(h, w, prefix, mlp):
    ids, wt = route(h, w[prefix + "router"], mlp["router"]["top"])
    y = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(ids[t], wt[t]):
            y[t] += s * expert(h[t], w[f"{prefix}e{e}.up"], w[f"{prefix}e{e}.down"])
    if mlp.get("shared"):
        y += sigmoid(h @ w[prefix + "shared.sg"].T) * expert(h, w[prefix + "shared.up"], w[prefix + "shared.down"])
    return y


def mixer(h, w, prefix, mx, pos):
    n = h.shape[0]
    q = (h @ w[prefix + "q"].T).reshape(n, mx["heads"], mx["dim"])
    k = (h @ w[prefix + "k"].T).reshape(n, mx["kv_heads"], mx["dim"])
    v = (h @ w[prefix + "v"].T).reshape(n, mx["kv_heads"], mx["vdim"])
    return attention(q, k, v, mx["scale"], mx.get("mask"), pos, pos).reshape(n, -1) @ w[prefix + "o"].T


def forward(cfg: dict, w: Dict[str, np.ndarray], tokens, layers_out: Optional[list] = None) -> np.ndarray:
    """Logits [n, vocab] of every position of one sequence."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)]
    pos = np.arange(len(tokens))
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + layer_norm(mixer(layer_norm(x, w[p + "norm1"], eps), w, p + "mix.", layer["mixer"], pos), w[p + "norm1b"], eps)
        mlp = layer.get("mlp")
        if mlp:
            h = layer_norm(x, w[p + "norm2"], eps)
            if mlp["kind"] == "dense":
                y = dense_ff(h, w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"])
            else:
                y = moe_ff(h, w, p + "mlp.", mlp)
            x = x + layer_norm(y, w[p + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return layer_norm(x, w["final.norm"], eps) @ w["head"].T


def load(directory, dtype=np.float64):
    """config.json and the bf16 tensors of model.safetensors as `dtype`."""
    directory = Path(directory)
    cfg = json.loads((directory / "config.json").read_text())
    raw = (directory / "model.safetensors").read_bytes()
    n = struct.unpack("<Q", raw[:8])[0]
    head = json.loads(raw[8:8 + n])
    w = {}
    for name, e in head.items():
        if name == "__metadata__":
            continue
        a, b = e["data_offsets"]
        bits = np.frombuffer(raw, dtype=np.uint16, count=(b - a) // 2, offset=8 + n + a).astype(np.uint32) << 16
        w[name] = bits.view(np.float32).reshape(e["shape"]).astype(dtype)
    return cfg, w
