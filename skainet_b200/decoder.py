"""Decoders over dense weights (skn_decoder_*): what the models share on the host -- weights, slots, the step function.

A decoder keeps `max_seqs` sequences of any lengths in slots; forward() advances one slot, or a range of them by the same
number of tokens.  A model supplies its configuration, its native decoder and the loading of its checkpoint."""
from __future__ import annotations

import ctypes
from typing import List, Sequence

import numpy as np

from . import _ffi
from .tensor import Context, DenseTensor, SKN_OK, _check, _raise


def loop_runs(n: int, loop) -> List[int]:
    """Layer index of every layer run, the loop (start, stop, times) unrolled."""
    if not loop:
        return list(range(n))
    a, b, times = loop
    return list(range(a)) + list(range(a, b)) * times + list(range(b, n))


class DenseDecoder:
    """Owns the dense weights and the native decoder.  dtype "bfloat16" serves with bf16 operands and fp32 accumulation,
    "float32" computes everything in fp32.  `cfg` has width, vocab and runs."""

    DTYPES = {"float32": 0, "bfloat16": 1}

    def __init__(self, ctx: Context, cfg, max_seqs: int = 1, max_tokens: int = 512, max_ctx: int = 4096, dtype: str = "bfloat16"):
        if dtype not in self.DTYPES:
            raise ValueError(f"dtype must be one of {sorted(self.DTYPES)}")
        self.ctx, self.cfg, self.dtype = ctx, cfg, dtype
        self.max_seqs, self.max_tokens, self.max_ctx = max_seqs, max(max_tokens, max_seqs), max_ctx
        self._tensors: List[DenseTensor] = []
        self._h = ctypes.c_void_p()
        create, spec, keep = self._native_spec()
        rc = create(ctx.handle, ctypes.byref(spec), max_seqs, self.max_tokens, max_ctx, self.DTYPES[dtype], ctypes.byref(self._h))
        del keep
        if rc != SKN_OK:
            self._h = ctypes.c_void_p()
            _raise(ctx.handle, rc)

    def _native_spec(self):
        """(the model's create function, its filled specification, what the specification points at)"""
        raise NotImplementedError

    @property
    def handle(self):
        return self._h

    @property
    def vocab(self) -> int:
        return self.cfg.vocab

    def _up(self, bits: np.ndarray) -> DenseTensor:
        t = DenseTensor(self.ctx, bits)
        self._tensors.append(t)
        return t

    def reset(self, seq: int = -1):
        """Forget the tokens of one sequence (-1: of all); its slot can be used again at once."""
        _check(self.ctx.handle, _ffi.lib().skn_decoder_reset(self._h, seq))

    def position(self, seq: int = 0) -> int:
        return int(_ffi.lib().skn_decoder_position(self._h, seq))

    def forward(self, tokens, seq: int = 0, want: Sequence[int] = (), want_next: bool = True):
        """tokens [T] (one sequence) or [n, T] (the slots seq .. seq + n - 1); None with want_next: feed back the last
        greedy id of slot `seq`.  Longer prompts than a step holds are run in portions.  Returns (next ids [n] or None,
        logits [len(want), vocab] or None); want counts the rows of [n, T] flattened."""
        if tokens is None:
            return self._step(None, seq, 1, 1, list(want), want_next)
        t = np.ascontiguousarray(tokens, dtype=np.int32)
        t = t.reshape(1, -1) if t.ndim == 1 else t
        n, T = t.shape
        want = [int(x) for x in want]
        if n < 1 or T < 1 or any(x < 0 or x >= n * T for x in want):
            raise ValueError("Shapes do not align.")
        per = self.max_tokens // n
        logits = np.empty((len(want), self.vocab), dtype=np.float32) if want else None
        nxt = None
        for a in range(0, T, per):
            b = min(T, a + per)
            here = [(k, (x // T) * (b - a) + x % T - a) for k, x in enumerate(want) if a <= x % T < b]
            nxt, lg = self._step(np.ascontiguousarray(t[:, a:b]), seq, n, b - a, [r for _, r in here], want_next and b == T)
            if here:
                logits[[k for k, _ in here]] = lg
        return nxt, logits

    def _step(self, t, seq, n, T, rows, want_next):
        nxt = np.empty(n, dtype=np.int32) if want_next else None
        want = np.asarray(rows, dtype=np.int32)
        logits = np.empty((len(rows), self.vocab), dtype=np.float32) if len(rows) else None
        _check(self.ctx.handle, _ffi.lib().skn_decoder_forward(
            self._h, seq, n, None if t is None else t.ctypes.data, T, len(rows), want.ctypes.data if len(rows) else None,
            None if logits is None else logits.ctypes.data, None if nxt is None else nxt.ctypes.data))
        return nxt, logits

    def forward_dev(self, tokens_dev=None, T: int = 1, seq: int = 0, n: int = 1, head: bool = True):
        """Enqueue one step: tokens_dev is a device address or tensor of [n, T] int32, None feeds back the greedy ids."""
        ptr = None if tokens_dev is None else (tokens_dev.data_ptr() if hasattr(tokens_dev, "data_ptr") else tokens_dev)
        _check(self.ctx.handle, _ffi.lib().skn_decoder_forward_dev(self._h, seq, n, ptr, T, 1 if head else 0))

    def trace_layers(self, on: bool):
        """Record the residual stream after every layer run of the steps that follow (layer_outputs)."""
        _check(self.ctx.handle, _ffi.lib().skn_decoder_trace(self._h, 1 if on else 0, 0, None))

    def layer_outputs(self, rows: int) -> np.ndarray:
        """[layer runs, rows, width] of the last step."""
        out = np.empty((len(self.cfg.runs), rows, self.cfg.width), dtype=np.float32)
        _check(self.ctx.handle, _ffi.lib().skn_decoder_trace(self._h, 1, rows, out.ctypes.data))
        return out

    def close(self):
        if self._h:
            _ffi.lib().skn_decoder_destroy(self._h)
            self._h = ctypes.c_void_p()
        for t in self._tensors:
            t.close()
        self._tensors = []

    def __del__(self):
        try:
            self.close()
        except Exception:
            pass
