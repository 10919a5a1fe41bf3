"""Plain numpy restatement of the Dugulorn decoder (test infrastructure; float64 by default, nothing shared with the
product path). One function per mechanism, whole sequences at once, token loops where the design is a recurrence:

    rms_norm            x / sqrt(mean(x^2) + eps) * w
    frequencies         angle per position of each rotated pair, with the YaRN ramp, and the factor on cos and sin
    rotate              neighbouring dimensions (2i, 2i + 1) turned by position * frequency
    latent_kv           the normed latent and the rotated key part that a position caches
    latent_attention    causal softmax attention on keys and values expanded from the latents, a gate per head
    short_conv          causal convolution per channel over the last `taps` inputs
    lightning           S = decay S + k v^T, o = S^T q; all heads normed together, gated
    channel_delta       S = g S; u = beta (v - S^T k); S += k u^T; o = S^T q; each head normed, gated
    dense_ff            down(relu2(up h + b)) + b
    forward             x += norm1(mixer(x)); x += norm2(ff(x)); logits = embed norm(x)

`cfg` is the dictionary of config.json, `w` maps tensor names to float arrays. Layer and model norms multiply by
1 + the stored weight; the norms inside mixers by the weight itself.
"""
from __future__ import annotations

import math
from typing import Dict, Optional

import numpy as np


def rms_norm(x, w, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def relu2(z):
    r = np.maximum(z, 0.0)
    return r * r


def frequencies(rot: dict):
    """(frequency of each pair [dims / 2], factor on cos and sin)."""
    dims, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    out = np.empty(dims // 2)
    for i in range(dims // 2):
        out[i] = base ** (-2.0 * i / dims)
    if not sc:
        return out, 1.0

    def at(turns):
        return dims * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo, hi = max(math.floor(at(sc["fast"])), 0), min(math.ceil(at(sc["slow"])), dims - 1)
    for i in range(dims // 2):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out[i] = out[i] / sc["factor"] * ramp + out[i] * (1.0 - ramp)
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, pos, rot):
    """x [n, ..., dims] at positions pos [n]."""
    f, m = frequencies(rot)
    a = np.asarray(pos, dtype=np.float64).reshape((-1,) + (1,) * (x.ndim - 1)) * f
    c, s = (np.cos(a) * m).astype(x.dtype), (np.sin(a) * m).astype(x.dtype)
    u, v = x[..., 0::2], x[..., 1::2]
    y = np.empty_like(x)
    y[..., 0::2] = u * c - v * s
    y[..., 1::2] = v * c + u * s
    return y


def latent_kv(h, w, p, mx, pos, eps):
    kv = h @ w[p + "dkv"].T
    r = mx["kv_rank"]
    return rms_norm(kv[:, :r], w[p + "dkv.norm"], eps), rotate(kv[:, r:], pos, mx["rot"])


def latent_attention(h, w, p, mx, pos, eps, latents) -> np.ndarray:
    """`latents`: (c, k_rot) of the layer whose cache this one reads."""
    n, H, d, r, vd = h.shape[0], mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"]
    c, kr = latents
    q = (rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T).reshape(n, H, d + r)
    qr = rotate(q[..., d:], pos, mx["rot"])
    k = (c @ w[p + "uk"].T).reshape(n, H, d)
    v = (c @ w[p + "uv"].T).reshape(n, H, vd)
    gate = sigmoid(h @ w[p + "g"].T)
    out = np.empty((n, H, vd), dtype=h.dtype)
    see = np.arange(n)[:, None] >= np.arange(n)[None, :]
    for i in range(H):
        s = np.where(see, (q[:, i, :d] @ k[:, i].T + qr[:, i] @ kr.T) * mx["scale"], -np.inf)
        e = np.exp(s - s.max(-1, keepdims=True))
        out[:, i] = e / e.sum(-1, keepdims=True) @ v[:, i] * gate[:, i:i + 1]
    return out.reshape(n, -1) @ w[p + "o"].T


def short_conv(x, taps):
    """x [n, channels], taps [channels, T]: column T - 1 meets the token itself, zeros before the start."""
    T = taps.shape[1]
    y = np.zeros_like(x)
    for j in range(T):
        back = T - 1 - j
        y[back:] += x[:len(x) - back] * taps[:, j] if back else x * taps[:, j]
    return y


def lightning_core(q, k, v, decay):
    """q, k [n, H, d], v [n, H, vd], decay [H] -> o [n, H, vd]."""
    n, H, d = q.shape
    S = np.zeros((H, d, v.shape[2]), dtype=q.dtype)
    out = np.empty_like(v)
    a = np.asarray(decay, dtype=q.dtype)[:, None, None]
    for t in range(n):
        S = a * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hdv,hd->hv", S, q[t])
    return out


def lightning(h, w, p, mx, eps):
    n, H = h.shape[0], mx["heads"]
    q, k = (silu(h @ w[p + t].T).reshape(n, H, mx["dim"]) for t in ("q", "k"))
    v = silu(h @ w[p + "v"].T).reshape(n, H, mx["vdim"])
    o = lightning_core(q, k, v, mx["decay"]).reshape(n, -1)
    return (rms_norm(o, w[p + "norm"], eps) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def delta_core(q, k, v, g, beta):
    """q, k, g [n, H, d], v [n, H, vd], beta [n, H] -> o [n, H, vd]."""
    n, H, d = q.shape
    S = np.zeros((H, d, v.shape[2]), dtype=q.dtype)
    out = np.empty_like(v)
    for t in range(n):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - np.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = np.einsum("hdv,hd->hv", S, q[t])
    return out


def unit(x):
    return x / np.sqrt((x * x).sum(-1, keepdims=True) + 1e-6)


def delta_inputs(h, w, p, mx):
    """(q, k, v, g, beta) as they enter the recurrence."""
    n, H, G, d, vd = h.shape[0], mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q, k, v = (silu(short_conv(h @ w[p + t].T, w[p + t + ".conv"])) for t in ("q", "k", "v"))
    of = np.arange(H) // (H // G)
    q = (unit(q.reshape(n, G, d)) * d ** -0.5)[:, of]
    k = unit(k.reshape(n, G, d))[:, of]
    beta = sigmoid(h @ w[p + "b"].T)
    step = softplus((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]).reshape(n, H, d)
    g = np.exp(-np.exp(w[p + "A_log"])[:, None] * step)
    return q, k, v.reshape(n, H, vd), g, beta


def channel_delta(h, w, p, mx, eps):
    n, H, vd = h.shape[0], mx["heads"], mx["vdim"]
    o = rms_norm(delta_core(*delta_inputs(h, w, p, mx)), w[p + "norm"], eps)
    gate = sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T).reshape(n, H, vd)
    return (o * gate).reshape(n, -1) @ w[p + "o"].T


def dense_ff(h, w, p):
    return relu2(h @ w[p + "up"].T + w[p + "up.b"]) @ w[p + "down"].T + w[p + "down.b"]


def forward(cfg: dict, w: Dict[str, np.ndarray], tokens, layers_out: Optional[list] = None) -> np.ndarray:
    """Logits [n, vocab] of every position of one sequence."""
    eps = cfg["norm"]["eps"]
    pos = np.arange(len(tokens))
    x = rms_norm(w["embed"][np.asarray(tokens)], 1.0 + w["embed.norm"], eps)
    latents = {}
    for i, layer in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", layer["mixer"]
        m = p + "mix."
        if layer["type"] == "latent_attention":
            src = mx.get("kv_from")
            if src is None:
                src = i
                latents[i] = latent_kv(x, w, m, mx, pos, eps)
            y = latent_attention(x, w, m, mx, pos, eps, latents[src])
        elif layer["type"] == "lightning":
            y = lightning(x, w, m, mx, eps)
        else:
            y = channel_delta(x, w, m, mx, eps)
        x = x + rms_norm(y, 1.0 + w[p + "norm1"], eps)
        if layer.get("mlp"):
            x = x + rms_norm(dense_ff(x, w, p + "mlp."), 1.0 + w[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return rms_norm(x, 1.0 + w["final.norm"], eps) @ w["embed"].T
