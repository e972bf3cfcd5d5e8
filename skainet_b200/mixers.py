"""Token mixers on their own: a position-addressed KV cache with chunked or windowed softmax attention, and recurrent states with
retention (skn_chunk_attn, skn_retention).  The decoders over dense weights run the same kernels inside their steps."""
from __future__ import annotations

import ctypes

import numpy as np

from . import _ffi
from .tensor import Context, SKN_OK, _check, _raise


def _rows(a, *shape):
    a = np.ascontiguousarray(a, dtype=np.float32)
    if a.shape != shape:
        raise ValueError("Shapes do not align.")
    return a


class PositionCache:
    """K and V of `batch` sequences; position p of a sequence occupies slot p % capacity.  The caller keeps the lengths."""

    DTYPES = {"f32": 0, "bf16": 3}

    def __init__(self, ctx: Context, batch: int, kv_heads: int, dim: int, vdim: int, capacity: int, dtype: str = "bf16"):
        if dtype not in self.DTYPES:
            raise ValueError("dtype must be 'f32' or 'bf16'")
        self.ctx, self.batch, self.kv_heads, self.dim, self.vdim, self.capacity = ctx, batch, kv_heads, dim, vdim, capacity
        self._h = ctypes.c_void_p()
        rc = _ffi.lib().skn_kv_create_by_position(ctx.handle, batch, kv_heads, dim, vdim, capacity, self.DTYPES[dtype], ctypes.byref(self._h))
        if rc != SKN_OK:
            self._h = ctypes.c_void_p()
            _raise(ctx.handle, rc)

    @property
    def handle(self):
        return self._h

    def attend(self, q, k, v, pos, scale: float, *, seq: int = 0, chunk: int = 0, window: int = 0, softcap: float = 0.0,
               rot_dims: int = 0, rot_base: float = 10000.0, q_gain=None, k_gain=None, sink=None, eps: float = 1e-5,
               max_ctx: int = 1 << 20) -> np.ndarray:
        """q [n, T, heads, dim], k [n, T, kv_heads, dim], v [n, T, kv_heads, vdim] (raw heads) of the sequences seq ..,
        pos[n] tokens having come before; returns [n, T, heads, vdim].  A query sees the earlier keys of its own chunk, or the
        last `window` ones, or all; sink [heads] joins the softmax denominators."""
        n, T, H, D = np.shape(q)
        q, k, v = _rows(q, n, T, H, D), _rows(k, n, T, self.kv_heads, D), _rows(v, n, T, self.kv_heads, self.vdim)
        pos = np.ascontiguousarray(pos, dtype=np.int32).reshape(n)
        gains = [None if g is None else _rows(g, D) for g in (q_gain, k_gain)]
        spec = _ffi.AttnSpec(H, self.kv_heads, D, self.vdim, rot_dims, chunk, rot_base, scale, softcap, eps, window)
        sinks = None if sink is None else _rows(sink, H)
        out = np.empty((n, T, H, self.vdim), dtype=np.float32)
        _check(self.ctx.handle, _ffi.lib().skn_chunk_attn(
            self._h, ctypes.byref(spec), seq, n, T, pos.ctypes.data, max_ctx, *[None if g is None else g.ctypes.data for g in gains],
            q.ctypes.data, k.ctypes.data, v.ctypes.data, None if sinks is None else sinks.ctypes.data, out.ctypes.data))
        return out

    def close(self):
        if self._h:
            _ffi.lib().skn_kv_destroy(self._h)
            self._h = ctypes.c_void_p()

    def __del__(self):
        try:
            self.close()
        except Exception:
            pass


class RecurrentState:
    """fp32 states [heads, dim, vdim] of `slots` sequences; a sequence at position 0 starts from zero."""

    def __init__(self, ctx: Context, slots: int, heads: int, dim: int, vdim: int):
        self.ctx, self.slots, self.heads, self.dim, self.vdim = ctx, slots, heads, dim, vdim
        self._h = ctypes.c_void_p()
        rc = _ffi.lib().skn_state_create(ctx.handle, slots, heads, dim, vdim, ctypes.byref(self._h))
        if rc != SKN_OK:
            self._h = ctypes.c_void_p()
            _raise(ctx.handle, rc)

    @property
    def handle(self):
        return self._h

    def retain(self, q, k, v, g, pos, decay, *, seq: int = 0, rot_dims: int = 0, rot_base: float = 10000.0, eps: float = 1e-5,
               max_ctx: int = 1 << 20, exact: bool = False) -> np.ndarray:
        """q, k [n, T, heads, dim], v, g [n, T, heads, vdim]; returns the normalised, gated outputs [n, T, heads, vdim].
        exact: fp32 products only."""
        n, T, H, D = np.shape(q)
        q, k = _rows(q, n, T, self.heads, self.dim), _rows(k, n, T, self.heads, self.dim)
        v, g = _rows(v, n, T, self.heads, self.vdim), _rows(g, n, T, self.heads, self.vdim)
        pos = np.ascontiguousarray(pos, dtype=np.int32).reshape(n)
        if len(decay) != self.heads:
            raise ValueError("Shapes do not align.")
        d = (ctypes.c_double * self.heads)(*[float(x) for x in decay])
        spec = _ffi.RetentionSpec(H, D, self.vdim, rot_dims, rot_base, ctypes.cast(d, _ffi.P(ctypes.c_double)), eps, int(exact))
        out = np.empty((n, T, H, self.vdim), dtype=np.float32)
        _check(self.ctx.handle, _ffi.lib().skn_retention(self._h, ctypes.byref(spec), seq, n, T, pos.ctypes.data, max_ctx, q.ctypes.data,
                                                        k.ctypes.data, v.ctypes.data, g.ctypes.data, out.ctypes.data))
        return out

    def read(self, slot: int) -> np.ndarray:
        out = np.empty((self.heads, self.dim, self.vdim), dtype=np.float32)
        _check(self.ctx.handle, _ffi.lib().skn_state_read(self._h, slot, out.ctypes.data))
        return out

    def close(self):
        if self._h:
            _ffi.lib().skn_state_destroy(self._h)
            self._h = ctypes.c_void_p()

    def __del__(self):
        try:
            self.close()
        except Exception:
            pass
