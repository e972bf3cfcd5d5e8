"""Host side of the Tutezen decoder (skn_tutezen_*): configuration and weight loading.

A layer adds residual_mult * (mixer(h) + feed-forward(h)) to the residual stream, h being the one norm of it that both read.  The
mixer is a selective state space (`mamba2`) or `latent_attention`, the feed-forward dense, a mixture of experts, or absent;
a range of layers may be looped with a cache or state per pass."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import List, Optional, Union

import numpy as np

from . import _ffi
from .decoder import DenseDecoder, loop_runs
from .registry import register
from .tensor import Context, _check, from_bf16_bits


def up8(n: int) -> int:
    return (n + 7) // 8 * 8


@dataclass
class SsmConfig:
    heads: int
    vdim: int
    state: int
    groups: int
    taps: int
    norm_groups: int

    @classmethod
    def from_dict(cls, d: dict) -> "SsmConfig":
        c = cls(heads=int(d["heads"]), vdim=int(d["vdim"]), state=int(d["state"]), groups=int(d["groups"]), taps=int(d["conv"]),
                norm_groups=int(d["norm_groups"]))
        if c.heads % c.groups or c.inner % c.norm_groups:
            raise ValueError(f"{c.heads} heads of {c.vdim} do not divide into {c.groups} groups and {c.norm_groups} norm groups")
        return c

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        return self.inner + 2 * self.groups * self.state

    def tensor_shapes(self, p: str, width: int) -> dict:
        H = self.heads
        return {p + "in": (self.inner + self.channels + H, width), p + "conv": (self.channels, self.taps), p + "conv.b": (self.channels,),
                p + "dt_bias": (H,), p + "A_log": (H,), p + "D": (H,), p + "norm": (self.inner,), p + "o": (width, self.inner)}


@dataclass
class LatentConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    window: int = 0             # 0: every earlier key is visible
    rot_dims: int = 0
    rot_base: float = 10000.0

    @classmethod
    def from_dict(cls, d: dict) -> "LatentConfig":
        rot, mask = d.get("rot") or {}, d.get("mask") or {}
        return cls(heads=int(d["heads"]), dim=int(d["dim"]), rot_dim=int(d["rot_dim"]), vdim=int(d["vdim"]), q_rank=int(d["q_rank"]),
                   kv_rank=int(d["kv_rank"]), scale=float(d["scale"]), window=int(mask.get("size") or 0), rot_dims=int(rot.get("dims") or 0),
                   rot_base=float(rot.get("base") or 10000.0))

    @property
    def rot_pad(self) -> int:
        """Rotated dimensions, padded so that a head is a multiple of 16."""
        return (up8(self.dim) + self.rot_dim + 15) // 16 * 16 - up8(self.dim)

    def tensor_shapes(self, p: str, width: int) -> dict:
        H = self.heads
        return {p + "dq": (self.q_rank, width), p + "dq.norm": (self.q_rank,), p + "uq": (H * (self.dim + self.rot_dim), self.q_rank),
                p + "dkv": (self.kv_rank + self.rot_dim, width), p + "dkv.norm": (self.kv_rank,), p + "uk": (H * self.dim, self.kv_rank),
                p + "uv": (H * self.vdim, self.kv_rank), p + "sink": (H,), p + "g": (H * self.vdim, width), p + "o": (width, H * self.vdim)}


@dataclass
class MoeConfig:
    experts: int
    top: int
    ff: int
    shared_ff: int = 0          # 0: no shared expert

    @classmethod
    def from_dict(cls, d: dict) -> "MoeConfig":
        r, shared = d["router"], d.get("shared")
        return cls(experts=int(r["experts"]), top=int(r["top"]), ff=int(d["expert"]["ff"]), shared_ff=int(shared["ff"]) if shared else 0)


MIXERS = {"mamba2": SsmConfig, "latent_attention": LatentConfig}


@dataclass
class TutezenLayerConfig:
    mixer: Union[SsmConfig, LatentConfig]
    ff: int = 0                 # width of a dense feed-forward
    moe: Optional[MoeConfig] = None

    @classmethod
    def from_dict(cls, d: dict) -> "TutezenLayerConfig":
        if d.get("type") not in MIXERS:
            raise ValueError(f"unknown mixer {d.get('type')!r}")
        mlp = d.get("mlp")
        kind = mlp.get("kind", "dense") if mlp else None
        if kind not in (None, "dense", "moe"):
            raise ValueError(f"unknown feed-forward {kind!r}")
        return cls(mixer=MIXERS[d["type"]].from_dict(d["mixer"]), ff=int(mlp["ff"]) if kind == "dense" else 0,
                   moe=MoeConfig.from_dict(mlp) if kind == "moe" else None)

    def tensor_shapes(self, p: str, width: int) -> dict:
        out = {p + "norm1": (width,), **self.mixer.tensor_shapes(p + "mix.", width)}
        gated = {}
        if self.ff:
            out.update({p + "mlp.up": (self.ff, width), p + "mlp.down": (width, self.ff)})
        if self.moe:
            out[p + "mlp.router"] = (self.moe.experts, width)
            gated = {f"{p}mlp.e{e}.": self.moe.ff for e in range(self.moe.experts)}
            if self.moe.shared_ff:
                gated[p + "mlp.shared."] = self.moe.shared_ff
        for q, f in gated.items():
            out.update({q + "gate": (f, width), q + "up": (f, width), q + "down": (width, f)})
        return out


@dataclass
class TutezenConfig:
    vocab: int
    width: int
    layers: List[TutezenLayerConfig]
    eps: float = 1e-5
    residual_mult: float = 1.0
    loop: Optional[tuple] = None  # (start, stop, times)

    @classmethod
    def from_dict(cls, d: dict) -> "TutezenConfig":
        loop = d.get("loop")
        return cls(vocab=int(d["vocab"]), width=int(d["width"]), layers=[TutezenLayerConfig.from_dict(x) for x in d["layers"]],
                   eps=float(d["norm"]["eps"]), residual_mult=float(d["residual_mult"]),
                   loop=(int(loop["start"]), int(loop["stop"]), int(loop["times"])) if loop else None)

    @property
    def runs(self) -> List[int]:
        return loop_runs(len(self.layers), self.loop)

    def tensor_shapes(self) -> dict:
        """name -> shape of every tensor of a checkpoint."""
        out = {"embed": (self.vocab, self.width), "final.norm": (self.width,)}
        if self.loop:
            out["loop.step"] = (self.loop[2], self.width)
        for i, l in enumerate(self.layers):
            out.update(l.tensor_shapes(f"l{i}.", self.width))
        return out


def pad_blocks(a: np.ndarray, size: int, to: int) -> np.ndarray:
    """Blocks of `size` rows, each padded with zero rows to `to`."""
    if size == to:
        return a
    out = np.zeros((a.shape[0] // size, to) + a.shape[1:], a.dtype)
    out[:, :size] = a.reshape(-1, size, *a.shape[1:])
    return out.reshape(-1, *a.shape[1:])


def pad_rows(a: np.ndarray) -> np.ndarray:
    return pad_blocks(a, a.shape[0], up8(a.shape[0]))


def pair_rows(gate: np.ndarray, up: np.ndarray) -> np.ndarray:
    """Rows gate 0, up 0, gate 1, up 1 .. (zero rows up to a multiple of 8 pairs)."""
    gate, up = pad_rows(gate), pad_rows(up)
    return np.stack([gate, up], axis=1).reshape(-1, gate.shape[1])


class TutezenDecoder(DenseDecoder):
    def _native_spec(self):
        cfg = self.cfg
        layers = (_ffi.TutezenLayer * len(cfg.layers))()
        for l, c in zip(layers, cfg.layers):
            m, x = c.mixer, c.moe or MoeConfig(0, 0, 0)
            l.ff, l.experts, l.top, l.expert_ff, l.shared_ff = c.ff, x.experts, x.top, x.ff, x.shared_ff
            if isinstance(m, SsmConfig):
                l.mixer = 0
                l.ssm = _ffi.SsmSpec(m.heads, m.vdim, m.state, m.groups, m.taps, m.norm_groups, cfg.eps, 0)
            else:
                l.mixer = 1
                l.latent = _ffi.LatentSpec(m.heads, m.dim, m.rot_dim, m.vdim, m.q_rank, m.kv_rank, m.rot_dims, m.window, m.rot_base, m.scale, cfg.eps)
        start, stop, times = cfg.loop or (0, 0, 0)
        spec = _ffi.TutezenSpec(len(cfg.layers), cfg.width, cfg.vocab, start, stop, times, cfg.eps, cfg.residual_mult, layers)
        return _ffi.lib().skn_tutezen_create, spec, layers

    def load(self, get) -> "TutezenDecoder":
        """get(name, shape) -> bf16 bit patterns (uint16) of a checkpoint tensor (SafetensorsFile.bf16_bits).  What reads the layer's
        normalised input is stacked, what adds to the residual stream sits side by side, heads padded to multiples of 8."""
        S = self.cfg.tensor_shapes()

        def w(name):
            a = np.ascontiguousarray(get(name, S[name]))
            if a.shape != S[name]:               # (padding would hide it from the native check)
                raise ValueError(f"{name} is {list(a.shape)}, expected {list(S[name])}")
            return a

        def vec(name):
            return from_bf16_bits(w(name))

        for i, l in enumerate(self.cfg.layers):
            p = f"l{i}."
            rows, cols, t, v = (self._ssm if isinstance(l.mixer, SsmConfig) else self._latent)(l.mixer, p + "mix.", w, vec)
            if l.moe:
                q, n = p + "mlp.", l.moe.experts
                rows.append(pad_rows(w(q + "router")))
                if l.moe.shared_ff:
                    rows.append(pair_rows(w(q + "shared.gate"), w(q + "shared.up")))
                    cols.append(pad_rows(w(q + "shared.down").T).T)
                t["e_in"] = np.concatenate([pair_rows(w(f"{q}e{e}.gate"), w(f"{q}e{e}.up")) for e in range(n)])
                t["e_out"] = np.concatenate([pad_rows(w(f"{q}e{e}.down").T).T for e in range(n)])
            elif l.ff:
                rows.append(pad_rows(w(p + "mlp.up")))
                cols.append(pad_rows(w(p + "mlp.down").T).T)
            t.update(w_in=np.concatenate(rows), w_out=np.concatenate(cols, axis=1))
            v["norm"] = vec(p + "norm1")
            v = {k: np.ascontiguousarray(a, np.float32) for k, a in v.items()}
            ws = _ffi.TutezenWeights(**{k: self._up(a).handle.value for k, a in t.items()}, **{k: a.ctypes.data for k, a in v.items()})
            _check(self.ctx.handle, _ffi.lib().skn_tutezen_set_layer(self._h, i, ctypes.byref(ws)))
        step = vec("loop.step") if self.cfg.loop else None
        norm, embed = vec("final.norm"), self._up(w("embed"))
        _check(self.ctx.handle, _ffi.lib().skn_tutezen_set_head(self._h, embed.handle, norm.ctypes.data, None if step is None else step.ctypes.data))
        return self

    @staticmethod
    def _ssm(m: SsmConfig, p: str, w, vec):
        H, V, G, N = m.heads, m.vdim, m.groups, m.state

        def xbc(a):
            """x | B | C, heads and groups padded"""
            x, b, c = np.split(a, [m.inner, m.inner + G * N])
            return np.concatenate([pad_blocks(x, V, up8(V)), pad_blocks(b, N, up8(N)), pad_blocks(c, N, up8(N))])

        z, mid, dt = np.split(w(p + "in"), [m.inner, m.inner + m.channels])
        rows = [pad_blocks(z, V, up8(V)), xbc(mid), pad_rows(dt)]
        cols = [pad_blocks(np.ascontiguousarray(w(p + "o").T), V, up8(V)).T]
        return rows, cols, {}, {"conv": xbc(vec(p + "conv")), "conv_b": xbc(vec(p + "conv.b")), "dt_bias": vec(p + "dt_bias"), "a_log": vec(p + "A_log"),
                                "d": vec(p + "D"), "out_norm": pad_blocks(vec(p + "norm"), V, up8(V))}

    @staticmethod
    def _latent(m: LatentConfig, p: str, w, vec):
        H, D, R, V = m.heads, m.dim, m.rot_dim, m.vdim
        dkv, uq = w(p + "dkv"), w(p + "uq").reshape(H, D + R, m.q_rank)

        def rotated(a):
            """the rotated part, padded"""
            return pad_blocks(a, R, m.rot_pad) if R else np.zeros((a.shape[0] + m.rot_pad, a.shape[1]), a.dtype)

        rows = [pad_rows(w(p + "dq")), pad_rows(dkv[:m.kv_rank]), rotated(dkv[m.kv_rank:]), pad_blocks(w(p + "g"), V, up8(V))]
        cols = [pad_blocks(np.ascontiguousarray(w(p + "o").T), V, up8(V)).T]
        t = {"uq": np.concatenate([np.concatenate([pad_rows(uq[h, :D]), rotated(uq[h, D:])]) for h in range(H)]),
             "ukv": np.concatenate([pad_blocks(w(p + "uk"), D, up8(D)), pad_blocks(w(p + "uv"), V, up8(V))])}
        return rows, cols, t, {"q_gain": vec(p + "dq.norm"), "kv_gain": vec(p + "dkv.norm"), "sink": vec(p + "sink")}


@register("Tutezen", family="tutezen")
def load_tutezen(ctx: Context, config: dict, weights, **kw) -> TutezenDecoder:
    return TutezenDecoder(ctx, TutezenConfig.from_dict(config), **kw).load(weights.bf16_bits)
