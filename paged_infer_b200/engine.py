"""The C++ engine loop (``include/paged_infer_engine.hpp``) from Python: continuous batching over the paged KV pool and the
state slots, greedy generation, and feeding of given tokens.  Works with every model of the registry."""
from __future__ import annotations

import ctypes as C
import os

import numpy as np

from . import _lib

_HERE = os.path.dirname(os.path.abspath(__file__))
LIB_PATH = os.path.join(_HERE, "libpaged_infer_engine.so")

_P, _SZ, _I, _L, _U64 = C.c_void_p, C.c_size_t, C.c_int, C.c_long, C.c_uint64
SIGNATURES = {
    "pie_create": (_P, [_P, _P, _SZ, _SZ, _SZ, _SZ, C.c_uint32, _I, _I, _SZ]),
    "pie_destroy": (None, [_P]),
    "pie_error": (C.c_char_p, [_P]),
    "pie_add_request": (_L, [_P, _U64, _P, _SZ, _SZ, _SZ]),
    "pie_step": (_L, [_P]),
    "pie_next_finished": (_L, [_P, _P, _P, _P, _SZ]),
    "pie_feed": (_L, [_P, _I, _P, _P, _P, _P, _P, _P]),
    "pie_end": (_L, [_P, _U64]),
    "pie_stats": (None, [_P, _P]),
}
_shim = None
FINISH_REASONS = ("none", "eos", "length", "out_of_memory")


def lib() -> C.CDLL:
    global _shim
    if _shim is None:
        if not os.path.exists(LIB_PATH):
            raise ImportError(f"{LIB_PATH} is missing: build it with `python -m paged_infer_b200.build`")
        _lib.lib()   # the device library it calls
        L = C.CDLL(LIB_PATH)
        for name, (res, args) in SIGNATURES.items():
            fn = getattr(L, name)
            fn.restype = res
            fn.argtypes = args
        _shim = L
    return _shim


class EngineError(RuntimeError):
    pass


class Engine:
    """``mixed_batches``: portions of prompts ride beside decoded tokens (default); otherwise a prompt is prefilled at its
    admission.  ``state_slots``: live sequences of a model with recurrent state (0: ``max_batch``)."""

    def __init__(self, ctx, model, num_blocks: int, block_size: int = 16, max_batch: int | None = None, prefill_chunk: int = 512,
                 eos: int | None = None, prefix_cache: bool = True, mixed_batches: bool = True, state_slots: int = 0):
        self.ctx, self.model = ctx, model
        self.handle = lib().pie_create(ctx.handle, model.handle, block_size, num_blocks, max_batch or model.max_batch, prefill_chunk,
                                       0xFFFFFFFF if eos is None else eos, int(prefix_cache), int(mixed_batches), state_slots)
        if not self.handle:
            raise EngineError(lib().pie_error(None).decode())

    def close(self):
        if getattr(self, "handle", None) and _shim is not None:
            _shim.pie_destroy(self.handle)
            self.handle = None

    __del__ = close

    def _check(self, status: int) -> int:
        if status < 0:
            raise EngineError(lib().pie_error(self.handle).decode())
        return int(status)

    def add_request(self, request_id: int, tokens, max_tokens: int, samples: int = 1):
        t = np.ascontiguousarray(tokens, np.uint32)
        self._check(lib().pie_add_request(self.handle, request_id, t.ctypes.data, t.size, max_tokens, samples))

    def step(self) -> bool:
        """One engine step; True while there is work left."""
        return self._check(lib().pie_step(self.handle)) == 1

    def finished(self) -> list:
        """[(request id, generated tokens, reason)] of the sequences that have finished since the last call."""
        out = []
        rid, why = C.c_uint64(), C.c_int()
        while True:
            n = lib().pie_next_finished(self.handle, None, None, None, 0)
            if n < 0:
                return out
            t = np.empty(max(n, 1), np.uint32)
            lib().pie_next_finished(self.handle, C.byref(rid), C.byref(why), t.ctypes.data, n)
            out.append((int(rid.value), t[:n].tolist(), FINISH_REASONS[why.value]))

    def generate(self, prompts, max_tokens: int = 16) -> list:
        """Greedy continuations of ``prompts`` (lists of token ids), in their order."""
        for i, p in enumerate(prompts):
            self.add_request(i, p, max_tokens)
        done = {}
        while True:
            more = self.step()
            for rid, tokens, _ in self.finished():
                done[rid] = tokens
            if not more:
                return [done[i] for i in range(len(prompts))]

    def feed(self, entries) -> np.ndarray:
        """One batch of given tokens.  ``entries``: [(id, tokens, wanted places)]; logits [total wanted, vocab].  An unknown id
        starts a new sequence, :meth:`end` gives back what it holds."""
        ids = np.array([e[0] for e in entries], np.uint64)
        counts = np.array([len(e[1]) for e in entries], np.int32)
        wants = np.array([len(e[2]) for e in entries], np.int32)
        tokens = np.concatenate([np.asarray(e[1], np.uint32).reshape(-1) for e in entries] + [np.empty(0, np.uint32)])
        want = np.concatenate([np.asarray(e[2], np.int32).reshape(-1) for e in entries] + [np.empty(0, np.int32)])
        tokens, want = np.ascontiguousarray(tokens, np.uint32), np.ascontiguousarray(want, np.int32)
        out = np.empty((int(wants.sum()), self.model.vocab_size()), np.float32)
        self._check(lib().pie_feed(self.handle, len(entries), ids.ctypes.data, counts.ctypes.data, tokens.ctypes.data, wants.ctypes.data,
                                   want.ctypes.data, out.ctypes.data))
        return out

    def end(self, sequence_id: int):
        self._check(lib().pie_end(self.handle, sequence_id))

    def stats(self) -> dict:
        out = (C.c_uint64 * 7)()
        lib().pie_stats(self.handle, out)
        keys = ("steps", "requests", "prompt_tokens", "prompt_tokens_prefilled", "generated_tokens", "free_blocks", "free_state_slots")
        return {k: int(v) for k, v in zip(keys, out)}
