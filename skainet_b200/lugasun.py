"""Host side of the Lugasun decoder (skn_lugasun_*): configuration and weight loading.

A layer runs chunked softmax attention and retention side by side on one normalised input (`parallel` mixer), then an
optional squared-relu feed-forward, then a token side input; a range of layers may be looped with a cache and a state
per pass."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import List, Optional

import numpy as np

from . import _ffi
from .decoder import DenseDecoder, loop_runs
from .registry import register
from .tensor import Context, _check, from_bf16_bits


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
        return loop_runs(len(self.layers), self.loop)

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


class LugasunDecoder(DenseDecoder):
    def _native_spec(self):
        cfg = self.cfg
        decays = [(ctypes.c_double * len(l.right.decay))(*l.right.decay) for l in cfg.layers]
        layers = (_ffi.LugasunLayer * len(cfg.layers))()
        for l, c, d in zip(layers, cfg.layers, decays):
            a, r = c.left, c.right
            l.left = _ffi.AttnSpec(a.heads, a.kv_heads, a.dim, a.vdim, a.rot_dims, a.chunk, a.rot_base, a.scale, a.softcap, cfg.eps, 0)
            l.right = _ffi.RetentionSpec(r.heads, r.dim, r.vdim, r.rot_dims, r.rot_base, ctypes.cast(d, _ffi.P(ctypes.c_double)), cfg.eps, 0)
            l.left_scale, l.right_scale, l.ff = c.left_scale, c.right_scale, c.ff
        start, stop, times = cfg.loop or (0, 0, 0)
        spec = _ffi.LugasunSpec(len(cfg.layers), cfg.width, cfg.vocab, cfg.side_dim, start, stop, times, cfg.eps, layers)
        return _ffi.lib().skn_lugasun_create, spec, (layers, decays)

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


@register("Lugasun", family="lugasun")
def load_lugasun(ctx: Context, config: dict, weights, **kw) -> LugasunDecoder:
    return LugasunDecoder(ctx, LugasunConfig.from_dict(config), **kw).load(weights.bf16_bits)
