"""Small random Tutezen models for the tests: configurations, bf16 weights, and their fp64 values for the oracle."""
import copy

import numpy as np

from skainet_b200.tensor import to_bf16_bits
from skainet_b200.tutezen import TutezenConfig
from tests.lugasun_models import error, errors, floats, getter  # noqa: F401  (shared helpers)


def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=24, shared=40):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}, "shared": {"ff": shared} if shared else None}


def ssm(heads=6, vdim=16, state=24, groups=2, conv=4, norm_groups=3, mlp=None):
    return {"type": "mamba2", "mlp": mlp, "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}}


def latent(heads=3, dim=24, rot_dim=8, vdim=40, q_rank=56, kv_rank=48, scale=0.21, window=17, base=900.0, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
                      "mask": {"size": window} if window else None, "rot": {"base": base, "dims": rot_dim}}}


def config(layers, width=64, vocab=90, loop=None, eps=1e-5, mult=0.4):
    return {"architecture": "Tutezen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "layers": copy.deepcopy(layers),
            "loop": {"start": loop[0], "stop": loop[1], "times": loop[2]} if loop else None}


def weights(cfg, seed):
    """name -> bf16 bit patterns.  Gains are away from 1, matrices keep activations near unit size, heads forget at different rates."""
    g = np.random.default_rng(seed)
    out = {}
    for name, shape in TutezenConfig.from_dict(cfg).tensor_shapes().items():
        last = name.split(".")[-1]
        if last == "A_log":
            a = g.uniform(-3.0, 1.5, shape)
        elif last == "dt_bias":
            a = g.uniform(-4.0, 0.5, shape)
        elif last == "sink":
            a = g.uniform(-1.0, 2.0, shape)
        elif last == "router":
            a = 4.0 * g.standard_normal(shape) / np.sqrt(shape[1])
        elif last == "step":
            a = 0.5 * g.standard_normal(shape)
        elif last == "b":
            a = 0.3 * g.standard_normal(shape)
        elif last == "conv":
            a = g.standard_normal(shape) / np.sqrt(shape[1])
        elif len(shape) == 1:
            a = 1.0 + 0.3 * g.standard_normal(shape)
        else:
            a = g.standard_normal(shape) * (1.0 if name == "embed" else 1.3 / np.sqrt(shape[1]))
        out[name] = to_bf16_bits(np.asarray(a, np.float32))
    return out


TOL = {"float32": 3e-5, "bfloat16": 4e-2}
