"""Host-side parts of the Lugasun decoder (no GPU): oracle self-checks, configuration, safetensors reader, registry,
generation loop against a stand-in model, and what a one-family build compiles."""
import json
import os

import numpy as np
import pytest

from oracle import lugasun as plain
from skainet_b200 import build, registry
from skainet_b200.generate import generate
from skainet_b200.lugasun import LugasunConfig
from skainet_b200.safetensors import SafetensorsFile, write_safetensors
from skainet_b200.tensor import from_bf16_bits, to_bf16_bits
from tests import lugasun_models as lm


# ---- the oracle against second formulations ---------------------------------------------------------------
def test_retention_recurrence_equals_its_sum():
    g = np.random.default_rng(0)
    q, k, v = (g.standard_normal((9, 2, d)) for d in (5, 5, 3))
    decay = [0.5, 0.97]
    o, S = plain.retention(q, k, v, decay)
    for h in range(2):
        for t in range(9):
            want = sum(decay[h] ** (t - j) * (q[t, h] @ k[j, h]) * v[j, h] for j in range(t + 1))
            np.testing.assert_allclose(o[t, h], want, rtol=1e-12, atol=1e-12)
    o2, S2 = plain.retention(q[4:], k[4:], v[4:], decay, plain.retention(q[:4], k[:4], v[:4], decay)[1])
    np.testing.assert_allclose(o2, o[4:], rtol=1e-12)
    np.testing.assert_allclose(S2, S, rtol=1e-12)


def test_rotation_keeps_lengths_and_depends_on_distance_only():
    g = np.random.default_rng(1)
    x, y = g.standard_normal((1, 1, 10)), g.standard_normal((1, 1, 10))
    rot = {"dims": 6, "base": 50.0}
    at = lambda a, p: plain.rotate_half(a, rot, p)[0, 0]
    assert np.isclose(np.linalg.norm(at(x, 7)), np.linalg.norm(x))
    assert np.isclose(at(x, 12) @ at(y, 5), at(x, 7) @ at(y, 0))
    np.testing.assert_array_equal(at(x, 9)[6:], x[0, 0, 6:])
    # dimension i turns with i + dims / 2
    e = np.zeros((1, 1, 10))
    e[0, 0, 1] = 1.0
    assert set(np.nonzero(at(e, 3))[0]) == {1, 4}


def test_chunk_visibility_edges():
    vis = lambda i, size: [j for j in range(30) if plain.chunk_visible(i, j, size)]
    assert vis(9, 5) == [5, 6, 7, 8, 9] and vis(10, 5) == [10] and vis(14, 5) == [10, 11, 12, 13, 14]
    assert vis(3, None) == [0, 1, 2, 3]


def test_loop_order():
    cfg = lm.config([lm.layer()] * 4, loop=(1, 3, 2))
    assert plain.layer_runs(cfg) == [(0, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    assert LugasunConfig.from_dict(cfg).runs == [0, 1, 2, 1, 2, 3]


# ---- configuration and weights -------------------------------------------------------------------------------
def test_config_reads_every_size_and_optional_part():
    cfg = LugasunConfig.from_dict(lm.config([lm.layer(heads=6, kv_heads=2, ff=0, rot=0), lm.layer(chunk=0, softcap=None, rrot=0)], side=0, loop=(0, 1, 3)))
    a, b = cfg.layers
    assert (a.left.heads, a.left.kv_heads, a.ff, a.left.rot_dims, a.left.chunk) == (6, 2, 0, 0, 19)
    assert (b.left.chunk, b.left.softcap, b.right.rot_dims, b.ff) == (0, 0.0, 0, 104)
    assert cfg.side_dim == 0 and cfg.loop == (0, 1, 3)
    names = cfg.tensor_shapes()
    assert "l0.mlp.up" not in names and "l0.norm2" not in names and "l1.mlp.up" in names and "side.embed" not in names
    assert names["loop.in"] == (72, 144) and names["l0.mix.left.o"] == (72, 6 * 40)


def test_config_rejects_what_it_does_not_know():
    bad = lm.config([lm.layer()])
    bad["layers"][0]["type"] = "serial"
    with pytest.raises(ValueError, match="unknown mixer"):
        LugasunConfig.from_dict(bad)
    bad = lm.config([lm.layer()])
    bad["layers"][0]["mlp"]["kind"] = "sparse"
    with pytest.raises(ValueError, match="unknown feed-forward"):
        LugasunConfig.from_dict(bad)
    bad = lm.config([lm.layer()])
    bad["layers"][0]["mixer"]["right"]["decay"] = [0.5]
    with pytest.raises(ValueError, match="decays"):
        LugasunConfig.from_dict(bad)


def test_bf16_bits_round_to_nearest_even():
    x = np.array([1.0, 1.0 + 2.0 ** -8, 1.0 + 3 * 2.0 ** -8, -2.5, 3.0e38], np.float32)
    y = from_bf16_bits(to_bf16_bits(x))
    np.testing.assert_array_equal(y[:4], np.array([1.0, 1.0, 1.0 + 2.0 ** -6, -2.5], np.float32))


def test_safetensors_round_trip_and_bounds(tmp_path):
    p = str(tmp_path / "w.safetensors")
    t = {"a": np.arange(6, dtype=np.uint16).reshape(2, 3), "b": np.array([1, -2], np.int32), "c": np.ones((3, 1), np.float32)}
    write_safetensors(p, t)
    f = SafetensorsFile(p)
    assert f.tensors == {"a": ("BF16", (2, 3)), "b": ("I32", (2,)), "c": ("F32", (3, 1))}
    for k in t:
        np.testing.assert_array_equal(f.get(k), t[k])
    np.testing.assert_array_equal(f.bf16_bits("a", (2, 3)), t["a"])
    with pytest.raises(ValueError, match="expected"):
        f.bf16_bits("a", (3, 2))
    with pytest.raises(ValueError, match="BF16"):
        f.bf16_bits("c", (3, 1))
    with pytest.raises(KeyError):
        f.get("d")
    raw = open(p, "rb").read()
    open(p, "wb").write(raw[:-8])
    with pytest.raises(ValueError, match="do not hold"):
        SafetensorsFile(p)


def test_registry_names_the_architecture(tmp_path):
    assert registry.architecture_of({"architecture": "Lugasun"}).family == "lugasun"
    with pytest.raises(ValueError, match="unknown architecture 'Other'"):
        registry.architecture_of({"architecture": "Other"})
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Lugasun"}))
    assert registry.read_config(str(tmp_path))["architecture"] == "Lugasun"


def test_family_build_compiles_a_part_of_the_library():
    part, whole = build.sources("lugasun"), build.sources()
    assert set(part) < set(whole) and all(os.path.exists(f) for f in part)
    assert not any("matvec_mma" in f or "gguf" in f for f in part)


# ---- generation loop -------------------------------------------------------------------------------------------
class Echo:
    """Stand-in decoder: the next id is the sum of the sequence so far modulo 50."""
    max_seqs = 2

    def __init__(self):
        self.seqs = {0: [], 1: []}
        self.steps = []

    def reset(self, seq):
        self.seqs[seq] = []

    def forward(self, tokens, seq=0, want=(), want_next=True):
        t = np.asarray(tokens, np.int32)
        t = t.reshape(1, -1) if t.ndim == 1 else t
        self.steps.append((seq, t.shape))
        ids = []
        for i in range(t.shape[0]):
            self.seqs[seq + i] += t[i].tolist()
            ids.append(sum(self.seqs[seq + i]) % 50)
        lg = np.zeros((len(want), 50), np.float32)
        for r in range(len(want)):
            lg[r, ids[r if t.shape[1] == 1 else 0]] = 9.0
        return np.array(ids), lg


@pytest.mark.parametrize("temperature", [0.0, 0.01])
def test_generate_shares_slots_between_prompts(temperature):
    prompts = [[1, 2, 3], [7], [4, 4], [30, 1, 2, 9]]

    def alone(p, n):
        s = list(p)
        for _ in range(n):
            s.append(sum(s) % 50)
        return s[len(p):]

    m = Echo()
    assert generate(m, prompts, 5, temperature) == [alone(p, 5) for p in prompts]
    assert (0, (2, 1)) in m.steps                      # two sequences decoded in one step
    stop = alone(prompts[0], 5)[2]
    got = generate(Echo(), prompts[:1], 5, stop=stop)[0]
    assert got == alone(prompts[0], 5)[:alone(prompts[0], 5).index(stop) + 1]
    assert generate(Echo(), prompts, 0) == [[], [], [], []]
