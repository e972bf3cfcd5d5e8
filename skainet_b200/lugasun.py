"""Host side of the Lugasun decoder (skn_lugasun_*): configuration, weight loading and the step function.

A layer runs chunked softmax attention and retention side by side on one normalised input (`parallel` mixer), then an
optional squared-relu feed-forward, then a token side input; a range of layers may be looped with a cache and a state
per pass.  The decoder keeps `max_seqs` sequences of any lengths in slots; forward() advances one slot, or a range of
them by the same number of tokens."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import List, Optional, Sequence

import numpy as np

from . import _ffi
from .registry import register
from .tensor import Context, DenseTensor, SKN_OK, _check, _raise, from_bf16_bits


@dataclass
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float = 0.0        # 0: scores are not capped
    chunk: int = 0              # positions of a chunk; 0: every earlier key is visible
    rot_dims: int = 0
    rot_base: float = 10000.0

    @classmethod
    def from_dict(cls, d: dict) -> "AttentionConfig":
        rot, mask = d.get("rot") or {}, d.get("mask") or {}
        return cls(heads=int(d["heads"]), kv_heads=int(d["kv_heads"]), dim=int(d["dim"]), vdim=int(d["vdim"]), scale=float(d["scale"]),
                   softcap=float(d.get("softcap") or 0.0), chunk=int(mask.get("size") or 0), rot_dims=int(rot.get("dims") or 0),
                   rot_base=float(rot.get("base") or 10000.0))


@dataclass
class RetentionConfig:
    heads: int
    dim: int
    vdim: int
    decay: List[float]
    rot_dims: int = 0
    rot_base: float = 10000.0

    @classmethod
    def from_dict(cls, d: dict) -> "RetentionConfig":
        rot = d.get("rot") or {}
        decay = [float(x) for x in d["decay"]]
        if len(decay) != int(d["heads"]):
            raise ValueError(f"{len(decay)} decays for {d['heads']} heads")
        return cls(heads=int(d["heads"]), dim=int(d["dim"]), vdim=int(d["vdim"]), decay=decay, rot_dims=int(rot.get("dims") or 0),
                   rot_base=float(rot.get("base") or 10000.0))


@dataclass
class LugasunLayerConfig:
    left: AttentionConfig
    right: RetentionConfig
    left_scale: float
    right_scale: float
    ff: int = 0                 # 0: no feed-forward

    @classmethod
    def from_dict(cls, d: dict) -> "LugasunLayerConfig":
        if d.get("type") != "parallel":
            raise ValueError(f"unknown mixer {d.get('type')!r}")
        m, mlp = d["mixer"], d.get("mlp")
        if mlp and mlp.get("kind", "dense") != "dense":
            raise ValueError(f"unknown feed-forward {mlp.get('kind')!r}")
        return cls(left=AttentionConfig.from_dict(m["left"]), right=RetentionConfig.from_dict(m["right"]),
                   left_scale=float(m["left_scale"]), right_scale=float(m["right_scale"]), ff=int(mlp["ff"]) if mlp else 0)

    @property
    def in_rows(self) -> int:
        a, r = self.left, self.right
        return a.heads * a.dim + a.kv_heads * (a.dim + a.vdim) + 2 * r.heads * (r.dim + r.vdim)

    @property
    def out_cols(self) -> int:
        return self.left.heads * self.left.vdim + self.right.heads * self.right.vdim


@dataclass
class LugasunConfig:
    vocab: int
    width: int
    layers: List[LugasunLayerConfig]
    eps: float = 1e-5
    side_dim: int = 0           # 0: no token side input
    loop: Optional[tuple] = None  # (start, stop, times)

    @classmethod
    def from_dict(cls, d: dict) -> "LugasunConfig":
        loop, side = d.get("loop"), d.get("token_side")
        return cls(vocab=int(d["vocab"]), width=int(d["width"]), layers=[LugasunLayerConfig.from_dict(x) for x in d["layers"]],
                   eps=float(d["norm"]["eps"]), side_dim=int(side["dim"]) if side else 0,
                   loop=(int(loop["start"]), int(loop["stop"]), int(loop["times"])) if loop else None)

    @property
    def runs(self) -> List[int]:
        """Layer index of every layer run, the loop unrolled."""
        n = len(self.layers)
        if not self.loop:
            return list(range(n))
        a, b, times = self.loop
        return list(range(a)) + list(range(a, b)) * times + list(range(b, n))

    def tensor_shapes(self) -> dict:
        """name -> shape of every tensor of a checkpoint."""
        w = self.width
        out = {"embed": (self.vocab, w), "final.norm": (w,)}
        if self.loop:
            out["loop.in"] = (w, 2 * w)
        if self.side_dim:
            out["side.embed"] = (self.vocab, len(self.layers) * self.side_dim)
        for i, l in enumerate(self.layers):
            a, r, p = l.left, l.right, f"l{i}."
            out.update({p + "norm1": (w,), p + "mix.left.q": (a.heads * a.dim, w), p + "mix.left.k": (a.kv_heads * a.dim, w),
                        p + "mix.left.v": (a.kv_heads * a.vdim, w), p + "mix.left.q.norm": (a.dim,), p + "mix.left.k.norm": (a.dim,),
                        p + "mix.left.o": (w, a.heads * a.vdim), p + "mix.right.q": (r.heads * r.dim, w),
                        p + "mix.right.k": (r.heads * r.dim, w), p + "mix.right.v": (r.heads * r.vdim, w),
                        p + "mix.right.g": (r.heads * r.vdim, w), p + "mix.right.o": (w, r.heads * r.vdim)})
            if l.ff:
                out.update({p + "norm2": (w,), p + "mlp.up": (l.ff, w), p + "mlp.down": (w, l.ff)})
            if self.side_dim:
                out.update({p + "side.gate": (self.side_dim, w), p + "side.proj": (w, self.side_dim), p + "side.norm": (w,)})
        return out


class LugasunDecoder:
    """Owns the dense weights and the native decoder.  dtype "bfloat16" serves with bf16 operands and fp32 accumulation,
    "float32" computes everything in fp32."""

    DTYPES = {"float32": 0, "bfloat16": 1}

    def __init__(self, ctx: Context, cfg: LugasunConfig, max_seqs: int = 1, max_tokens: int = 512, max_ctx: int = 4096,
                 dtype: str = "bfloat16"):
        if dtype not in self.DTYPES:
            raise ValueError(f"dtype must be one of {sorted(self.DTYPES)}")
        self.ctx, self.cfg, self.dtype = ctx, cfg, dtype
        self.max_seqs, self.max_tokens, self.max_ctx = max_seqs, max(max_tokens, max_seqs), max_ctx
        self._tensors: List[DenseTensor] = []
        self._h = ctypes.c_void_p()
        decays = [(ctypes.c_double * len(l.right.decay))(*l.right.decay) for l in cfg.layers]
        layers = (_ffi.LugasunLayer * len(cfg.layers))()
        for l, c, d in zip(layers, cfg.layers, decays):
            a, r = c.left, c.right
            l.left = _ffi.AttnSpec(a.heads, a.kv_heads, a.dim, a.vdim, a.rot_dims, a.chunk, a.rot_base, a.scale, a.softcap, cfg.eps, 0)
            l.right = _ffi.RetentionSpec(r.heads, r.dim, r.vdim, r.rot_dims, r.rot_base, ctypes.cast(d, _ffi.P(ctypes.c_double)), cfg.eps, 0)
            l.left_scale, l.right_scale, l.ff = c.left_scale, c.right_scale, c.ff
        start, stop, times = cfg.loop or (0, 0, 0)
        spec = _ffi.LugasunSpec(len(cfg.layers), cfg.width, cfg.vocab, cfg.side_dim, start, stop, times, cfg.eps, layers)
        rc = _ffi.lib().skn_lugasun_create(ctx.handle, ctypes.byref(spec), max_seqs, self.max_tokens, max_ctx, self.DTYPES[dtype],
                                           ctypes.byref(self._h))
        if rc != SKN_OK:
            self._h = ctypes.c_void_p()
            _raise(ctx.handle, rc)

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

    def load(self, get) -> "LugasunDecoder":
        """get(name, shape) -> bf16 bit patterns (uint16) of a checkpoint tensor (SafetensorsFile.bf16_bits).  The
        projections that share an input are stacked, the two output projections sit side by side."""
        c, S = self.cfg, self.cfg.tensor_shapes()

        def w(name):
            return np.ascontiguousarray(get(name, S[name]))

        def gain(name):
            return from_bf16_bits(w(name))

        for i, l in enumerate(c.layers):
            p = f"l{i}."
            w_in = self._up(np.concatenate([w(p + "mix." + n) for n in ("left.q", "left.k", "left.v", "right.q", "right.k", "right.v", "right.g")]))
            w_out = self._up(np.concatenate([w(p + "mix.left.o"), w(p + "mix.right.o")], axis=1))
            t = {"w_in": w_in, "w_out": w_out}
            g = {"norm1": gain(p + "norm1"), "q_gain": gain(p + "mix.left.q.norm"), "k_gain": gain(p + "mix.left.k.norm")}
            if l.ff:
                t.update(up=self._up(w(p + "mlp.up")), down=self._up(w(p + "mlp.down")))
                g["norm2"] = gain(p + "norm2")
            if c.side_dim:
                t.update(side_gate=self._up(w(p + "side.gate")), side_proj=self._up(w(p + "side.proj")))
                g["side_norm"] = gain(p + "side.norm")
            ws = _ffi.LugasunWeights(**{k: v.handle.value for k, v in t.items()}, **{k: v.ctypes.data for k, v in g.items()})
            _check(self.ctx.handle, _ffi.lib().skn_lugasun_set_layer(self._h, i, ctypes.byref(ws)))
        embed, norm = self._up(w("embed")), gain("final.norm")
        loop_in = self._up(w("loop.in")) if c.loop else None
        side = self._up(w("side.embed")) if c.side_dim else None
        _check(self.ctx.handle, _ffi.lib().skn_lugasun_set_head(self._h, embed.handle, norm.ctypes.data, loop_in and loop_in.handle,
                                                               side and side.handle))
        return self

    def reset(self, seq: int = -1):
        """Forget the tokens of one sequence (-1: of all); its slot can be used again at once."""
        _check(self.ctx.handle, _ffi.lib().skn_lugasun_reset(self._h, seq))

    def position(self, seq: int = 0) -> int:
        return int(_ffi.lib().skn_lugasun_position(self._h, seq))

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
        _check(self.ctx.handle, _ffi.lib().skn_lugasun_forward(
            self._h, seq, n, None if t is None else t.ctypes.data, T, len(rows), want.ctypes.data if len(rows) else None,
            None if logits is None else logits.ctypes.data, None if nxt is None else nxt.ctypes.data))
        return nxt, logits

    def forward_dev(self, tokens_dev=None, T: int = 1, seq: int = 0, n: int = 1, head: bool = True):
        """Enqueue one step: tokens_dev is a device address or tensor of [n, T] int32, None feeds back the greedy ids."""
        ptr = None if tokens_dev is None else (tokens_dev.data_ptr() if hasattr(tokens_dev, "data_ptr") else tokens_dev)
        _check(self.ctx.handle, _ffi.lib().skn_lugasun_forward_dev(self._h, seq, n, ptr, T, 1 if head else 0))

    def trace_layers(self, on: bool):
        """Record the residual stream after every layer run of the steps that follow (layer_outputs)."""
        _check(self.ctx.handle, _ffi.lib().skn_lugasun_trace(self._h, 1 if on else 0, 0, None))

    def layer_outputs(self, rows: int) -> np.ndarray:
        """[layer runs, rows, width] of the last step."""
        out = np.empty((len(self.cfg.runs), rows, self.cfg.width), dtype=np.float32)
        _check(self.ctx.handle, _ffi.lib().skn_lugasun_trace(self._h, 1, rows, out.ctypes.data))
        return out

    def close(self):
        if self._h:
            _ffi.lib().skn_lugasun_destroy(self._h)
            self._h = ctypes.c_void_p()
        for t in self._tensors:
            t.close()
        self._tensors = []

    def __del__(self):
        try:
            self.close()
        except Exception:
            pass


@register("Lugasun", family="lugasun")
def load_lugasun(ctx: Context, config: dict, weights, **kw) -> LugasunDecoder:
    return LugasunDecoder(ctx, LugasunConfig.from_dict(config), **kw).load(weights.bf16_bits)
