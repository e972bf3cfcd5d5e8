"""The Lugasun decoder and its mechanisms on the GPU against the plain fp64 restatement (oracle/lugasun.py).

float32: everything is fp32, so a wrong key, edge or state shows far above TOL.  bfloat16: bf16 operands; tests whose
fault would hide among random keys plant one key whose score stands out."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import skainet_b200 as skn
from oracle import lugasun as plain
from skainet_b200.lugasun import LugasunConfig, LugasunDecoder
from skainet_b200.mixers import PositionCache, RecurrentState
from skainet_b200.safetensors import write_safetensors
from skainet_b200.tensor import from_bf16_bits, to_bf16_bits
from tests import lugasun_models as lm

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = ["float32", "bfloat16"]


def rel(a, b):
    return float(np.abs(np.asarray(a, np.float64) - b).max() / np.abs(b).max())


# ---- linear layers ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("N,K", [(30, 37), (130, 100), (257, 520), (64, 8), (1000, 2056)])
@pytest.mark.parametrize("M", [1, 2, 3, 4, 5, 17, 64, 300])
def test_dense_linear(ctx, N, K, M):
    g = np.random.default_rng(N + M)
    w = to_bf16_bits(g.standard_normal((N, K)).astype(np.float32))
    x = g.standard_normal((M, K)).astype(np.float32)
    bias = g.standard_normal(N).astype(np.float32)
    t = skn.DenseTensor(ctx, w)
    wf = from_bf16_bits(w).astype(np.float64)
    exact = x.astype(np.float64) @ wf.T + bias
    y = t.matmul_t(x, bias)
    if M < 64:
        assert rel(y, exact) < 2e-6
    else:                                    # tensor cores: exact in the bf16-rounded activations
        xb = from_bf16_bits(to_bf16_bits(x)).astype(np.float64)
        assert rel(y, xb @ wf.T + bias) < 2e-6
    t.close()


def test_dense_tensor_is_refused_where_blocks_are_expected(ctx):
    t = skn.DenseTensor(ctx, np.ones((8, 256), np.float32))
    with pytest.raises(skn.SknError):
        skn.QuantTensor.dequantize(t)
    with pytest.raises(skn.SknError):
        skn.ffn_swiglu(ctx, t, t, t, np.ones(256, np.float32))
    t.close()


# ---- chunked attention ------------------------------------------------------------------------------------------------
def attention_reference(q, k, v, qg, kg, scale, softcap, chunk, rot, eps):
    q, k, v = (a.astype(np.float64) for a in (q, k, v))
    if qg is not None:
        q, k = plain.rms_norm(q, qg.astype(np.float64), eps), plain.rms_norm(k, kg.astype(np.float64), eps)
    return plain.chunked_attention(plain.rotate_half(q, rot), plain.rotate_half(k, rot), v, scale, softcap, chunk)


def run_attention(cache, cuts, q, k, v, **kw):
    out, at = [], 0
    for n in cuts:
        out.append(cache.attend(q[None, at:at + n], k[None, at:at + n], v[None, at:at + n], [at], **kw)[0])
        at += n
    return np.concatenate(out)


SHAPES = [(4, 1, 64, 64), (3, 3, 48, 80), (6, 2, 40, 24), (8, 1, 128, 128), (5, 1, 20, 12), (2, 2, 256, 192), (2, 1, 320, 288)]


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("H,G,D,V", SHAPES)
@pytest.mark.parametrize("chunk,softcap", [(0, 0.0), (50, 15.0), (129, 0.0)])
def test_chunked_attention(ctx, dtype, H, G, D, V, chunk, softcap):
    g = np.random.default_rng(D)
    T, scale, rot = 171, D ** -0.5 * 1.7, {"dims": D // 4 * 2, "base": 300.0}
    q, k, v = (g.standard_normal((T, h, d)).astype(np.float32) for h, d in ((H, D), (G, D), (G, V)))
    qg, kg = (1 + 0.3 * g.standard_normal(D)).astype(np.float32), (1 + 0.3 * g.standard_normal(D)).astype(np.float32)
    want = attention_reference(q, k, v, qg, kg, scale, softcap, chunk, rot, 1e-4)
    kw = dict(scale=scale, chunk=chunk, softcap=softcap, rot_dims=rot["dims"], rot_base=rot["base"], q_gain=qg, k_gain=kg, eps=1e-4, max_ctx=200)
    tol = 3e-6 if dtype == "f32" else 2e-2
    for cuts in ([T], [2, 1, 47, 1, 2, 70, 48], [100] + [1] * 71):
        cap = min(200, (chunk or 200) + max(cuts))
        cache = PositionCache(ctx, 1, G, D, V, cap, dtype)
        assert rel(run_attention(cache, cuts, q, k, v, **kw), want) < tol, cuts
        cache.close()


def test_attention_without_norm_or_rotation(ctx):
    g = np.random.default_rng(5)
    q, k, v = (g.standard_normal((33, h, 24)).astype(np.float32) for h in (4, 2, 2))
    want = attention_reference(q, k, v, None, None, 0.2, None, None, None, 0.0)
    cache = PositionCache(ctx, 1, 2, 24, 24, 64, "f32")
    for cuts in ([33], [1] * 33):
        assert rel(run_attention(cache, cuts, q, k, v, scale=0.2, max_ctx=64), want) < 3e-6
    cache.close()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("chunk", [16, 64, 100, 128, 200])
def test_chunk_edges_show(ctx, dtype, decode, chunk):
    """One key near each chunk edge answers every query: seen by its own chunk only, from the first to the last position."""
    D = 32
    T = 3 * chunk + 2
    g = np.random.default_rng(chunk)
    q = np.tile(np.eye(1, D, dtype=np.float32), (T, 1, 1)) * 8
    k = 0.01 * g.standard_normal((T, 1, D)).astype(np.float32)
    v = 0.1 * g.standard_normal((T, 1, D)).astype(np.float32)
    for j in (0, chunk - 1, chunk, 2 * chunk - 1, 2 * chunk, 3 * chunk - 1):
        k[j, 0, 0], v[j, 0] = 1.0 + 0.2 * (j % chunk == 0), 5.0 + j
    want = attention_reference(q, k, v, None, None, 1.0, None, chunk, None, 0.0)
    cuts = [2] + [1] * (T - 2) if decode else [chunk - 1, 2, chunk - 1, 1, T - 2 * chunk - 1]
    cache = PositionCache(ctx, 1, 1, D, D, chunk + max(cuts), dtype)
    got = run_attention(cache, cuts, q, k, v, scale=1.0, chunk=chunk, max_ctx=T)
    cache.close()
    err = np.abs(got - want).max(axis=(1, 2)) / np.abs(want).max(axis=(1, 2))
    assert err.max() < (1e-5 if dtype == "f32" else 3e-2), int(err.argmax())


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_far_key_shows_without_chunks(ctx, dtype):
    """One key at the start among hundreds stands out for the last queries, through the split and the tile kernels."""
    D, T = 64, 700
    g = np.random.default_rng(3)
    q, k, v = (g.standard_normal((T, h, D)).astype(np.float32) for h in (4, 1, 1))
    k[3, 0] = q[690, 1] * 3
    v[3, 0] = 40.0
    ref = np.zeros((4, D))
    for h in range(4):
        s = k[:691, 0].astype(np.float64) @ q[690, h] * 0.125
        p = np.exp(s - s.max())
        ref[h] = (p / p.sum()) @ v[:691, 0]
    assert ref[1].mean() > 20                 # the planted key dominates
    for cuts in ([T], [600] + [1] * 100):
        cache = PositionCache(ctx, 1, 1, D, D, T, dtype)
        got = run_attention(cache, cuts, q, k, v, scale=0.125, max_ctx=T)[690]
        cache.close()
        assert rel(got, ref) < (1e-5 if dtype == "f32" else 2e-2)


def test_attention_sequences_and_reused_slots(ctx):
    """Three sequences at unequal positions share a step; a slot is taken over without clearing."""
    D, G, H, chunk = 16, 1, 2, 12
    g = np.random.default_rng(9)
    cache = PositionCache(ctx, 3, G, D, D, chunk + 30, "f32")
    kw = dict(scale=0.3, chunk=chunk, max_ctx=100)
    seqs = [[g.standard_normal((40, h, D)).astype(np.float32) for h in (H, G, G)] for _ in range(3)]
    want = [attention_reference(*s, None, None, 0.3, None, chunk, None, 0.0) for s in seqs]
    pos = [5, 29, 14]
    for b, s in enumerate(seqs):
        got = cache.attend(*(a[None, :pos[b]] for a in s), [0], seq=b, **kw)[0]
        assert rel(got, want[b][:pos[b]]) < 3e-6
    for _ in range(4):
        got = cache.attend(*(np.stack([s[i][p:p + 1] for s, p in zip(seqs, pos)]) for i in range(3)), pos, **kw)
        for b in range(3):
            assert rel(got[b, 0], want[b][pos[b]]) < 3e-6
        pos = [p + 1 for p in pos]
    got = cache.attend(*(np.stack([s[i][p:p + 3] for s, p in zip(seqs[:2], pos)]) for i in range(3)), pos[:2], **kw)
    for b in range(2):
        assert rel(got[b], want[b][pos[b]:pos[b] + 3]) < 3e-6
    new = [g.standard_normal((15, h, D)).astype(np.float32) for h in (H, G, G)]
    want1 = attention_reference(*new, None, None, 0.3, None, chunk, None, 0.0)
    got = np.concatenate([cache.attend(*(a[None, i:i + 1] for a in new), [i], seq=1, **kw)[0] for i in range(15)])
    assert rel(got, want1) < 3e-6
    cache.close()


def test_attention_refuses_bad_calls(ctx):
    cache = PositionCache(ctx, 1, 1, 16, 16, 8, "f32")
    x = np.zeros((1, 4, 1, 16), np.float32)
    with pytest.raises(ValueError):
        cache.attend(x, x, x, [0], 1.0, chunk=16, max_ctx=64)      # a chunk and a step do not fit
    with pytest.raises(ValueError):
        cache.attend(x, x, x, [6], 1.0, max_ctx=8)                 # past the context
    with pytest.raises(skn.SknError):
        cache.attend(x, x, x, [0], 1.0, seq=1, max_ctx=8)
    cache.close()


# ---- retention ------------------------------------------------------------------------------------------------------
def retention_reference(q, k, v, gate, decay, rot, eps):
    q, k, v, gate = (a.astype(np.float64) for a in (q, k, v, gate))
    o, S = plain.retention(plain.rotate_half(q, rot), plain.rotate_half(k, rot) * q.shape[2] ** -0.5, v, decay)
    return plain.rms_unit(o, eps) * plain.silu(gate), S


@pytest.mark.parametrize("exact", [False, True])
@pytest.mark.parametrize("H,D,V", [(2, 32, 32), (3, 24, 40), (1, 128, 128), (2, 20, 13), (1, 70, 260), (5, 8, 64), (1, 200, 136)])
def test_retention(ctx, H, D, V, exact):
    g = np.random.default_rng(D + V)
    T, rot, decay = 200, {"dims": D // 4 * 2, "base": 90.0}, [0.999, 0.5, 0.97, 1.0, 0.9][:H]
    q, k, v, gate = (g.standard_normal((T, H, d)).astype(np.float32) for d in (D, D, V, V))
    want, S = retention_reference(q, k, v, gate, decay, rot, 1e-5)
    for cuts in ([T], [2, 3, 63, 1, 64, 2, 65], [1] * T, [130] + [1] * 70):
        st = RecurrentState(ctx, 1, H, D, V)
        out, at = [], 0
        for n in cuts:
            out.append(st.retain(*(a[None, at:at + n] for a in (q, k, v, gate)), [at], decay, rot_dims=rot["dims"], rot_base=rot["base"], exact=exact)[0])
            at += n
        assert rel(np.concatenate(out), want) < 2e-5, cuts
        assert rel(st.read(0), S) < 2e-5, cuts
        st.close()


def test_retention_far_token_and_reused_slots(ctx):
    """A large token far back stays visible through a slow decay, across chunks of the kernel; slots start from zero again."""
    g = np.random.default_rng(2)
    T, D = 180, 16
    q, k, v, gate = (g.standard_normal((T, 1, D)).astype(np.float32) for _ in range(4))
    k[3], v[3] = 30 * q[170], 20.0
    want, _ = retention_reference(q, k, v, gate, [0.9995], None, 1e-5)
    st = RecurrentState(ctx, 3, 1, D, D)
    for seq in (0, 2, 2):
        a = st.retain(*(x[None, :150] for x in (q, k, v, gate)), [0], [0.9995], seq=seq)[0]
        b = [st.retain(*(x[None, i:i + 1] for x in (q, k, v, gate)), [i], [0.9995], seq=seq)[0] for i in range(150, T)]
        assert rel(np.concatenate([a] + b), want) < 2e-5
    # unequal sequences in one step
    pos = [20, 0, 90]
    for s, p in enumerate(pos):
        if p:
            st.retain(*(x[None, :p] for x in (q, k, v, gate)), [0], [0.9995], seq=s)
    got = st.retain(*(np.stack([x[p:p + 1] for p in pos]) for x in (q, k, v, gate)), pos, [0.9995])
    for s, p in enumerate(pos):
        assert rel(got[s, 0], want[p]) < 2e-5
    st.close()


# ---- the decoder -------------------------------------------------------------------------------------------------------
MODELS = {
    "plain": lm.config([lm.layer()], side=0),
    "side": lm.config([lm.layer(), lm.layer(ff=0)], side=12),
    "loop": lm.config([lm.layer(chunk=7), lm.layer(heads=4, kv_heads=4, dim=16, vdim=64, rot=16, chunk=33), lm.layer(ff=40)], loop=(1, 2, 3), side=20),
    "loop_all": lm.config([lm.layer(dim=64, vdim=64, rot=64, rdim=32, rvdim=32, rrot=32)] * 2, width=128, loop=(0, 2, 2), side=8, vocab=161),
    "mixed": lm.config([lm.layer(heads=8, kv_heads=2, dim=20, rot=8, chunk=0, softcap=None, rheads=5, rdim=10, rvdim=6, rrot=0),
                        lm.layer(heads=2, kv_heads=1, rot=0, chunk=64, scale=0.05, ff=301, left_scale=-0.3, right_scale=1.5)], width=101, vocab=97, side=5),
    "wide": lm.config([lm.layer(heads=2, kv_heads=1, dim=320, vdim=300, chunk=40, rot=100, rheads=1, rdim=260, rvdim=270, rrot=40, ff=520)], width=264, side=30),
}
_built = {}


def model(name):
    """(config dict, bf16 weights, token ids, oracle logits) of one of MODELS; computed once."""
    if name not in _built:
        cfg = MODELS[name]
        bits = lm.weights(cfg, seed=len(name))
        tokens = np.random.default_rng(1).integers(0, cfg["vocab"], size=110)
        _built[name] = (cfg, bits, tokens, plain.forward(cfg, lm.floats(bits), tokens))
    return _built[name]


def decoder(ctx, cfg, bits, dtype, **kw):
    kw = {"max_seqs": 1, "max_tokens": 128, "max_ctx": 256, **kw}
    return LugasunDecoder(ctx, LugasunConfig.from_dict(cfg), dtype=dtype, **kw).load(lm.getter(bits))


def in_portions(dec, tokens, cuts, seq=0):
    out, at = [], 0
    for n in cuts:
        out.append(dec.forward(tokens[at:at + n], seq=seq, want=range(n), want_next=False)[1])
        at += n
    assert at == len(tokens) and dec.position(seq) == at
    return np.concatenate(out)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(MODELS))
def test_prompt_portions_and_decoding(ctx, name, dtype):
    cfg, bits, tokens, want = model(name)
    n = len(tokens)
    dec = decoder(ctx, cfg, bits, dtype)
    for cuts in ([n], [1] * n, [2, 3, 2, 40, 5, 58], [64, 4] + [1] * 42):
        dec.reset()
        e = lm.errors(in_portions(dec, tokens, cuts), want)
        assert np.quantile(e, 0.98) < lm.TOL[dtype], cuts
        # a retention output is divided by its size: where q . k nearly cancels, bf16 rounding of q and k grows with it
        assert e.max() < lm.TOL[dtype] * (1 if dtype == "float32" else 8), cuts
    dec.close()


def test_layers_match_one_by_one(ctx):
    cfg, bits, tokens, _ = model("loop")
    runs = []
    plain.forward(cfg, lm.floats(bits), tokens[:30], lambda r, x: runs.append(x))
    dec = decoder(ctx, cfg, bits, "float32")
    dec.trace_layers(True)
    dec.forward(tokens[:30], want_next=False)
    got = dec.layer_outputs(30)
    assert got.shape[0] == len(runs) == 5
    for r, x in enumerate(runs):
        assert rel(got[r], x) < 1e-5, r
    dec.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_step_longer_than_the_buffers_runs_in_portions(ctx, dtype):
    cfg, bits, tokens, want = model("loop")
    dec = decoder(ctx, cfg, bits, dtype, max_tokens=16)
    picks = [109, 0, 15, 16, 63]
    nxt, lg = dec.forward(tokens, want=picks)
    assert lm.error(lg, want[picks]) < lm.TOL[dtype]
    assert int(nxt[0]) == int(lg[0].argmax())
    dec.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_sequences_together_and_reused_slots(ctx, dtype):
    """Six sequences of unequal lengths decode in shared steps as each does alone; a slot is freed and used again."""
    cfg, bits, tokens, _ = model("loop")
    w = lm.floats(bits)
    g = np.random.default_rng(4)
    seqs = [g.integers(0, cfg["vocab"], size=n + 9) for n in (1, 13, 32, 33, 7, 50)]
    want = [plain.forward(cfg, w, s) for s in seqs]
    dec = decoder(ctx, cfg, bits, dtype, max_seqs=6)
    for i, s in enumerate(seqs):
        got = dec.forward(s[:-9], seq=i, want=[len(s) - 10], want_next=False)[1]
        assert lm.error(got, want[i][[len(s) - 10]]) < lm.TOL[dtype]
    for t in range(9):
        lo, n = (0, 6) if t % 3 else (1, 4)            # all six, or a range of them (the others wait)
        idx = [dec.position(i) for i in range(lo, lo + n)]
        ids = np.array([seqs[i][p] for i, p in zip(range(lo, lo + n), idx)])[:, None]
        got = dec.forward(ids, seq=lo, want=range(n), want_next=False)[1]
        for r, i in enumerate(range(lo, lo + n)):
            assert lm.error(got[[r]], want[i][[idx[r]]]) < lm.TOL[dtype], (t, i)
    other = g.integers(0, cfg["vocab"], size=40)
    dec.reset(2)
    assert dec.position(2) == 0 and dec.position(3) > 0
    assert lm.error(in_portions(dec, other, [37, 1, 1, 1], seq=2), plain.forward(cfg, w, other)) < lm.TOL[dtype]
    # two sequences prefill in one step
    dec.reset(4); dec.reset(5)
    got = dec.forward(np.stack([other[:21], tokens[:21]]), seq=4, want=range(42), want_next=False)[1]
    assert lm.error(got[:21], plain.forward(cfg, w, other[:21])) < lm.TOL[dtype]
    assert lm.error(got[21:], plain.forward(cfg, w, tokens[:21])) < lm.TOL[dtype]
    dec.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_past_the_ring(ctx, dtype):
    """The caches hold a chunk and one step: hundreds of decoded tokens pass over them several times."""
    cfg = lm.config([lm.layer(chunk=19, ff=48, heads=2), lm.layer(chunk=32, ff=0, heads=2)], width=48, side=0, loop=(0, 1, 2))
    bits = lm.weights(cfg, 8)
    tokens = np.random.default_rng(6).integers(0, cfg["vocab"], size=330)
    want = plain.forward(cfg, lm.floats(bits), tokens)
    dec = decoder(ctx, cfg, bits, dtype, max_tokens=5, max_ctx=330)
    got = np.concatenate([dec.forward(tokens[i:i + 1], want=[0], want_next=False)[1] for i in range(330)])
    assert lm.error(got, want) < lm.TOL[dtype]
    with pytest.raises(ValueError, match="exceeded"):
        dec.forward([1], want_next=False)
    dec.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cuts", [[23, 1, 1, 1, 1, 1, 1, 1], [20, 4, 2, 2, 2], [30]])
def test_chunk_edge_of_the_whole_model(ctx, cuts, dtype):
    """Attention that is nearly even over the visible keys, and alone in the layer: one key more or less shows."""
    cfg = lm.config([lm.layer(heads=1, kv_heads=1, dim=16, vdim=16, chunk=24, softcap=None, scale=0.02, rot=0, right_scale=0.0, left_scale=3.0, ff=0)], width=32, side=0)
    bits = lm.weights(cfg, 3)
    tokens = np.random.default_rng(11).integers(0, cfg["vocab"], size=30)
    w = lm.floats(bits)
    want = plain.forward(cfg, w, tokens)
    wrong = copy_with_chunk(cfg, 25)
    assert lm.error(plain.forward(wrong, w, tokens)[[24]], want[[24]]) > 0.5    # the edge matters here
    dec = decoder(ctx, cfg, bits, dtype, max_tokens=32)
    assert lm.error(in_portions(dec, tokens, cuts), want) < lm.TOL[dtype]
    dec.close()


def copy_with_chunk(cfg, size):
    c = json.loads(json.dumps(cfg))
    for l in c["layers"]:
        l["mixer"]["left"]["mask"]["size"] = size
    return c


def test_result_does_not_depend_on_slot_or_neighbours(ctx):
    cfg, bits, tokens, _ = model("loop")
    dec = decoder(ctx, cfg, bits, "bfloat16", max_seqs=3)
    a = dec.forward(tokens[:40], seq=0, want=range(40), want_next=False)[1]
    dec.forward(tokens[40:90], seq=1, want_next=False)
    b = dec.forward(tokens[:40], seq=2, want=range(40), want_next=False)[1]
    assert np.array_equal(a, b)
    dec.close()


# ---- generation, commands -------------------------------------------------------------------------------------------------
def greedy(cfg, w, prompt, n):
    s = list(prompt)
    for _ in range(n):
        s.append(int(plain.forward(cfg, w, s)[-1].argmax()))
    return s[len(prompt):]


PROMPTS = [[5, 17, 3], [1], [44, 2, 9, 9, 31, 60, 7], [12, 13]]


def test_greedy_generation(ctx):
    cfg, bits, _, _ = model("loop")
    w = lm.floats(bits)
    want = [greedy(cfg, w, p, 12) for p in PROMPTS]
    dec = decoder(ctx, cfg, bits, "float32", max_seqs=2)
    assert skn.generate(dec, PROMPTS, 12) == want
    # ids fed back on the device
    dec.reset()
    ids = [int(dec.forward(PROMPTS[0], seq=1)[0][0])]
    for _ in range(11):
        ids.append(int(dec.forward(None, seq=1)[0][0]))
    assert ids == want[0]
    dec.close()


def test_captured_step_replays(ctx):
    torch = pytest.importorskip("torch")
    cfg, bits, _, _ = model("side")
    dec = decoder(ctx, cfg, bits, "bfloat16", max_seqs=2)
    prompt = np.array([[5, 17, 3], [8, 1, 2]])

    dec.forward(prompt)
    for _ in range(8):
        dec.forward_dev(None, 1, n=2)
    ctx.sync()
    want_last = dec.forward(None)[0]
    stream = torch.cuda.Stream()
    graph = torch.cuda.CUDAGraph()
    dec.reset()
    try:
        with torch.cuda.stream(stream):
            ctx.set_stream(stream.cuda_stream)
            with torch.cuda.graph(graph, stream=stream):
                dec.forward_dev(None, 1, n=2)
        dec.reset()
        dec.forward(prompt)
        with torch.cuda.stream(stream):
            for _ in range(8):
                graph.replay()
        torch.cuda.synchronize()
    finally:
        ctx.set_stream(None)
    # the next eager step continues from the replayed positions
    assert np.array_equal(dec.forward(None)[0], want_last)
    del graph
    dec.close()


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    cfg, bits, _, _ = model("loop")
    d = tmp_path_factory.mktemp("model")
    (d / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(d / "model.safetensors"), bits)
    return str(d)


def test_generate_command(ctx, folder):
    cfg, bits, _, _ = model("loop")
    args = sum((["--prompt", ",".join(map(str, p))] for p in PROMPTS), [])
    r = subprocess.run([sys.executable, "-m", "skainet_b200.generate", "--model", folder, "--dtype", "float32", "--max-new", "6", *args],
                       cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    w = lm.floats(bits)
    assert [list(map(int, l.split(","))) for l in r.stdout.splitlines()] == [greedy(cfg, w, p, 6) for p in PROMPTS]


@pytest.mark.parametrize("dtype", DTYPES)
def test_replay_command(ctx, folder, tmp_path, dtype):
    cfg, bits, tokens, want = model("loop")
    t = tokens.tolist()
    steps = [{"entries": [{"id": "a", "tokens": t[:50], "want": [0, 49]}], "end": []},
             {"entries": [{"id": "a", "tokens": t[50:52], "want": []}], "end": []},
             {"entries": [{"id": "b", "tokens": t[:3], "want": [1]}], "end": ["b"]},
             {"entries": [{"id": "a", "tokens": t[52:53], "want": [0]}], "end": ["a"]},
             {"entries": [{"id": "c", "tokens": t[:1], "want": [0]}], "end": ["c"]}]
    lines = "".join(json.dumps({"step": i, **s}) + "\n" for i, s in enumerate(steps))
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "64"],
                       input=lines, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(5)]
    for i, rows in ((0, [0, 49]), (2, [1]), (3, [52]), (4, [0])):
        got = np.fromfile(tmp_path / f"{i}.f32", "<f4").reshape(-1, cfg["vocab"])
        assert lm.error(got, want[rows]) < lm.TOL[dtype], i
    assert not (tmp_path / "1.f32").exists()


def test_weights_of_the_wrong_shape_are_refused(ctx):
    cfg, bits, _, _ = model("plain")
    bad = dict(bits)
    bad["l0.mix.left.q"] = bits["l0.mix.left.q"][:-1]
    dec = LugasunDecoder(ctx, LugasunConfig.from_dict(cfg), max_tokens=8, max_ctx=8)
    with pytest.raises(ValueError):
        dec.load(lambda name, shape: bad[name])
    dec.close()
    with pytest.raises(skn.SknError):
        LugasunDecoder(ctx, LugasunConfig.from_dict({**cfg, "loop": {"start": 0, "stop": 5, "times": 1}}), max_tokens=8, max_ctx=8)
