"""Small random Lugasun models for the tests: configurations, bf16 weights, and their fp64 values for the oracle."""
import copy

import numpy as np

from skainet_b200.lugasun import LugasunConfig
from skainet_b200.tensor import from_bf16_bits, to_bf16_bits


def layer(heads=3, kv_heads=1, dim=48, vdim=40, chunk=19, softcap=30.0, scale=0.2, rot=32, base=5000.0, rheads=2, rdim=24, rvdim=36,
          rrot=16, rbase=700.0, decay=None, ff=104, left_scale=0.7, right_scale=0.4):
    decay = decay or [1.0 - 2.0 ** -(3 + 2 * h) for h in range(rheads)]
    return {"type": "parallel", "mlp": {"ff": ff, "kind": "dense"} if ff else None,
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": softcap,
                               "mask": {"size": chunk} if chunk else None, "rot": {"base": base, "dims": rot} if rot else None},
                      "right": {"heads": rheads, "dim": rdim, "vdim": rvdim, "decay": decay,
                                "rot": {"base": rbase, "dims": rrot} if rrot else None},
                      "left_scale": left_scale, "right_scale": right_scale}}


def config(layers, width=72, vocab=90, side=12, loop=None, eps=1e-5):
    return {"architecture": "Lugasun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": copy.deepcopy(layers),
            "token_side": {"dim": side} if side else None,
            "loop": {"start": loop[0], "stop": loop[1], "times": loop[2]} if loop else None}


def weights(cfg, seed):
    """name -> bf16 bit patterns.  Gains are away from 1 and matrices keep activations near unit size."""
    g = np.random.default_rng(seed)
    out = {}
    for name, shape in LugasunConfig.from_dict(cfg).tensor_shapes().items():
        if len(shape) == 1:
            a = 1.0 + 0.3 * g.standard_normal(shape)
        else:
            a = g.standard_normal(shape) * (1.0 if "embed" in name else 1.3 / np.sqrt(shape[1]))
        out[name] = to_bf16_bits(a.astype(np.float32))
    return out


def floats(bits):
    return {k: from_bf16_bits(v).astype(np.float64) for k, v in bits.items()}


def getter(bits):
    def get(name, shape):
        assert bits[name].shape == tuple(shape), name
        return bits[name]
    return get


def errors(got, want):
    """Per row: root mean square difference of mean-free logits over the root mean square of the wanted ones."""
    d = np.asarray(got, np.float64) - want
    d -= d.mean(-1, keepdims=True)
    w = want - want.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / np.sqrt((w * w).mean())


def error(got, want):
    return float(errors(got, want).max())


TOL = {"float32": 3e-5, "bfloat16": 4e-2}
