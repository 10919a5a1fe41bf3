"""The native model runtime (lbk_model_*, lbk_batcher_*) from Python, without a tensor framework: numpy in,
numpy out. A model family is chosen by the "architecture" of its config.json; `load_model` returns the class
registered for it (files without that key are BitNet's).
"""
from __future__ import annotations

import ctypes as C
import json
from pathlib import Path
from typing import Callable, Dict, Optional

import numpy as np

from . import _lib
from .ternary import Context, default_context

COMPUTE = {"bfloat16": 0, "float32": 1}
_FAMILIES: Dict[str, Callable] = {}


def register(architecture: str, cls) -> None:
    _FAMILIES[architecture] = cls


def architecture_of(directory) -> str:
    return json.loads((Path(directory) / "config.json").read_text()).get("architecture", "")


def load_model(directory, ctx: Optional[Context] = None, dtype: str = "bfloat16") -> "NativeModel":
    """The model in `directory`, whatever family it is. dtype: "bfloat16" (what the family is served in) or
    "float32" (families that have it)."""
    if dtype not in COMPUTE:
        raise ValueError(f"dtype must be one of {sorted(COMPUTE)}")
    arch = architecture_of(directory)
    if arch == "" and arch not in _FAMILIES:
        from . import model  # noqa: F401  (registers BitNet; needs torch)
    elif arch not in _FAMILIES:
        from . import dugulorn, pefolix  # noqa: F401
    if arch not in _FAMILIES:
        raise ValueError(f"no model family for architecture {arch!r} (known: {sorted(_FAMILIES)})")
    if arch == "":
        if dtype != "bfloat16":
            raise ValueError("the BitNet family computes in its own precisions only")
        return _FAMILIES[arch](directory, ctx)
    return _FAMILIES[arch](directory, ctx, dtype)


class _ModelConfig(C.Structure):
    _fields_ = [(n, C.c_size_t) for n in ("hidden_size", "intermediate_size", "num_attention_heads", "num_key_value_heads",
                                          "num_hidden_layers", "vocab_size", "max_position_embeddings")] + \
               [("rms_norm_eps", C.c_float), ("rope_theta", C.c_float), ("bos_token_id", C.c_int)]


class _LoadStats(C.Structure):
    _fields_ = [("seconds", C.c_double), ("bytes_read", C.c_size_t), ("bytes_to_device", C.c_size_t), ("staging_bytes", C.c_size_t)]


class NativeModel:
    """A model loaded by liblbk.so, its caches, prompt passes and decode steps; only marshals pointers."""

    def __init__(self, directory, ctx: Optional[Context] = None, dtype: str = "bfloat16"):
        self.ctx = ctx or default_context()
        self._lib = self.ctx._lib
        self.dtype = dtype
        h = C.c_void_p()
        _lib.check(self._load(directory, C.byref(h)))
        self.handle = h
        self.cfg = _ModelConfig()
        _lib.check(self._lib.lbk_model_get_config(h, C.byref(self.cfg)))
        self._caches = []

    def _load(self, directory, out) -> int:
        return self._lib.lbk_model_load_compute(self.ctx.handle, str(directory).encode(), COMPUTE[self.dtype], out)

    @property
    def architecture(self) -> str:
        return self._lib.lbk_model_architecture(self.handle).decode()

    def load_stats(self) -> dict:
        """Seconds, bytes read, bytes copied to the device and pinned staging bytes of the load."""
        s = _LoadStats()
        _lib.check(self._lib.lbk_model_load_stats(self.handle, C.byref(s)))
        return {"seconds": s.seconds, "bytes_read": s.bytes_read, "bytes_to_device": s.bytes_to_device, "staging_bytes": s.staging_bytes}

    def new_cache(self, b: int = 1, cap: int = 0):
        c = C.c_void_p()
        _lib.check(self._lib.lbk_model_new_cache(self.handle, b, cap, C.byref(c)))
        self._caches.append(c)
        return c

    def cache_len(self, cache) -> int:
        return int(self._lib.lbk_kv_cache_len(cache))

    def set_prefill_rows(self, rows: int) -> None:
        """Rows a prompt pass takes at once (default 4096)."""
        _lib.check(self._lib.lbk_model_set_prefill_rows(self.handle, rows))

    def reset_cache(self, cache) -> None:
        """Back to an empty sequence; the buffers and the recorded step are kept."""
        _lib.check(self._lib.lbk_kv_cache_reset(cache))

    def reset_seq(self, cache, seq: int) -> None:
        """One sequence of a cache gives its positions back."""
        _lib.check(self._lib.lbk_kv_cache_reset_seq(cache, seq))

    def forward(self, tokens, cache, all_logits: bool = False) -> np.ndarray:
        """model.rs:305: logits [n, vocab] (all_logits) or [vocab] of the last token, on the host."""
        toks = np.ascontiguousarray(tokens, dtype=np.uint32)
        out = np.empty((len(toks) if all_logits else 1, self.cfg.vocab_size), dtype=np.float32)
        _lib.check(self._lib.lbk_model_forward(self.handle, cache, toks.ctypes.data_as(C.c_void_p), len(toks), int(all_logits),
                                               out.ctypes.data_as(C.c_void_p)))
        return out if all_logits else out[0]

    def forward_rows(self, tokens, cache, want, seq: int = 0) -> np.ndarray:
        """The next tokens of sequence `seq`: logits [len(want), vocab] of the wanted places among them."""
        toks = np.ascontiguousarray(tokens, dtype=np.uint32)
        places = np.ascontiguousarray(want, dtype=np.uint32)
        out = np.empty((len(places), self.cfg.vocab_size), dtype=np.float32)
        _lib.check(self._lib.lbk_model_forward_rows(self.handle, cache, seq, toks.ctypes.data_as(C.c_void_p), len(toks),
                                                    places.ctypes.data_as(C.c_void_p), len(places), out.ctypes.data_as(C.c_void_p)))
        return out

    def decode(self, tokens_dev, cache):
        """One token per sequence (int32 CUDA tensor); returns (logits [b, vocab], greedy next tokens [b]) on the device."""
        import torch
        b = tokens_dev.shape[0]
        logits = torch.empty((b, self.cfg.vocab_size), dtype=torch.float32, device=tokens_dev.device)
        nxt = torch.empty(b, dtype=torch.int32, device=tokens_dev.device)
        _lib.check(self._lib.lbk_model_decode(self.handle, cache, C.c_void_p(tokens_dev.data_ptr()), C.c_void_p(logits.data_ptr()),
                                              C.c_void_p(nxt.data_ptr()), C.c_void_p(torch.cuda.current_stream().cuda_stream)))
        return logits, nxt

    def batcher(self, slots: int, capacity: int = 0) -> "Batcher":
        return Batcher(self, slots, capacity)

    def close(self):
        if getattr(self, "handle", None):
            for bt in list(getattr(self, "_batchers", [])):
                bt.close()
            for c in self._caches:
                self._lib.lbk_kv_cache_free(c)
            self._caches = []
            self._lib.lbk_model_free(self.handle)
            self.handle = None

    def __del__(self):
        try:
            self.close()
        except Exception:
            pass


class Batcher:
    """Continuous batching in front of the batched decode step (lbk_batcher_*): requests queue up, take
    free slots of one shared cache (prompt pass into the slot), advance together one greedy token per
    step, and leave as soon as they finish. The reference's server runs its requests one at a time
    (crates/lb-server/src/main.rs:92-166)."""

    def __init__(self, net: NativeModel, slots: int, capacity: int = 0):
        self.net = net
        self._lib = net._lib
        h = C.c_void_p()
        _lib.check(self._lib.lbk_batcher_create(net.handle, slots, capacity, C.byref(h)))
        self.handle = h
        if not hasattr(net, "_batchers"):
            net._batchers = []
        net._batchers.append(self)

    def submit(self, prompt, max_new_tokens: int, eos: int = -1) -> int:
        toks = np.ascontiguousarray(prompt, dtype=np.uint32)
        rid = C.c_uint64()
        _lib.check(self._lib.lbk_batcher_submit(self.handle, toks.ctypes.data_as(C.c_void_p), len(toks), max_new_tokens, eos, C.byref(rid)))
        return int(rid.value)

    def step(self) -> int:
        """One scheduling step; returns how many requests are still queued or running."""
        pending = C.c_size_t()
        _lib.check(self._lib.lbk_batcher_step(self.handle, C.byref(pending)))
        return int(pending.value)

    def poll(self, rid: int):
        """(tokens generated so far, finished?)"""
        n, done = C.c_size_t(), C.c_int()
        _lib.check(self._lib.lbk_batcher_poll(self.handle, rid, None, 0, C.byref(n), C.byref(done)))
        out = np.empty(n.value, dtype=np.uint32)
        _lib.check(self._lib.lbk_batcher_poll(self.handle, rid, out.ctypes.data_as(C.c_void_p), len(out), C.byref(n), C.byref(done)))
        return out.tolist(), bool(done.value)

    def forget(self, rid: int) -> None:
        _lib.check(self._lib.lbk_batcher_forget(self.handle, rid))

    def run(self, max_steps: int = 1 << 30) -> int:
        """Steps until nothing is queued or running; returns the number of steps."""
        steps = 0
        while steps < max_steps:
            steps += 1
            if self.step() == 0:
                break
        return steps

    def close(self):
        if getattr(self, "handle", None):
            self._lib.lbk_batcher_destroy(self.handle)
            self.handle = None
            if self in getattr(self.net, "_batchers", []):
                self.net._batchers.remove(self)

    def __del__(self):
        try:
            self.close()
        except Exception:
            pass
