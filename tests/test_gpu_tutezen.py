"""The Tutezen decoder and its mechanisms on the GPU against the plain fp64 restatement (oracle/tutezen.py).

float32: everything is fp32, so a wrong key, edge or state shows far above TOL.  bfloat16: bf16 operands; tests whose fault would hide
among random keys plant one that stands out, and tokens whose choice of experts is a close call are left out."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import skainet_b200 as skn
from oracle import tutezen as plain
from skainet_b200.mixers import PositionCache
from skainet_b200.safetensors import write_safetensors
from skainet_b200.tensor import from_bf16_bits, to_bf16_bits
from skainet_b200.tutezen import TutezenConfig, TutezenDecoder
from tests import tutezen_models as tm

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = ["float32", "bfloat16"]


def rel(a, b):
    return float(np.abs(np.asarray(a, np.float64) - b).max() / np.abs(b).max())


def oracle(cfg, w, tokens, on_layer=None):
    """(logits, margin): margin[t] is the smallest gap between a token's last chosen and first unchosen router logit, over all layer runs"""
    margin, real, at = np.full(len(tokens), np.inf), plain.route, [0]

    def watched(z, top):
        s = np.sort(z)[::-1]
        if top < len(s):
            t = at[0] % len(tokens)
            margin[t] = min(margin[t], s[top - 1] - s[top])
        at[0] += 1
        return real(z, top)

    plain.route = watched
    try:
        return plain.forward(cfg, w, tokens, on_layer), margin
    finally:
        plain.route = real


def check(got, want, margin, dtype, what=None):
    e = tm.errors(got, want)
    if dtype == "float32":
        assert e.max() < tm.TOL[dtype], (what, int(e.argmax()), float(e.max()))
        return
    clear = margin > 0.08
    assert clear.mean() > 0.4
    e = e[clear]
    # a row that follows a close call feels its neighbour's other expert through state and keys
    assert np.quantile(e, 0.95) < tm.TOL[dtype], (what, float(np.quantile(e, 0.95)))
    assert e.max() < 8 * tm.TOL[dtype], (what, float(e.max()))


def decoder(ctx, cfg, bits, dtype, **kw):
    kw = {"max_seqs": 1, "max_tokens": 160, "max_ctx": 400, **kw}
    return TutezenDecoder(ctx, TutezenConfig.from_dict(cfg), dtype=dtype, **kw).load(tm.getter(bits))


def in_portions(dec, tokens, cuts, seq=0):
    out, at = [], 0
    for n in cuts:
        out.append(dec.forward(tokens[at:at + n], seq=seq, want=range(n), want_next=False)[1])
        at += n
    assert at == len(tokens) and dec.position(seq) == at
    return np.concatenate(out)


# ---- sliding window and sink on their own --------------------------------------------------------------------------
def window_reference(q, k, v, scale, window, sink):
    q, k, v = (a.astype(np.float64) for a in (q, k, v))
    rep = q.shape[1] // k.shape[1]
    return plain.window_attention(q, np.repeat(k, rep, axis=1), np.repeat(v, rep, axis=1), scale, window, None if sink is None else sink.astype(np.float64))


def run_attention(cache, cuts, q, k, v, **kw):
    out, at = [], 0
    for n in cuts:
        out.append(cache.attend(q[None, at:at + n], k[None, at:at + n], v[None, at:at + n], [at], **kw)[0])
        at += n
    return np.concatenate(out)


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("window", [1, 2, 31, 64, 129, 0])
@pytest.mark.parametrize("H,G,D,V,sinks", [(4, 1, 48, 32, True), (3, 3, 20, 44, False), (8, 2, 128, 128, True)])
def test_window_and_sink(ctx, dtype, window, H, G, D, V, sinks):
    g = np.random.default_rng(window + D)
    T = 300
    q, k, v = (g.standard_normal((T, h, d)).astype(np.float32) for h, d in ((H, D), (G, D), (G, V)))
    sink = g.uniform(-1, 4, H).astype(np.float32) if sinks else None
    want = window_reference(q, k, v, D ** -0.5, window, sink)
    for cuts in ([T], [2, 1, 64, 63, 2, 100, 68], [150] + [1] * 150):
        cap = min(T, (window or T) + max(cuts))
        cache = PositionCache(ctx, 1, G, D, V, cap, dtype)
        got = run_attention(cache, cuts, q, k, v, scale=D ** -0.5, window=window, sink=sink, max_ctx=T)
        cache.close()
        assert rel(got, want) < (3e-6 if dtype == "f32" else 2e-2), cuts


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("window", [16, 64, 100, 128, 200])
def test_window_edges_show(ctx, dtype, decode, window):
    """Single keys answer every query that sees them: the query `window` - 1 later is the last one."""
    D, T = 32, 3 * window + 2
    g = np.random.default_rng(window)
    q = np.tile(np.eye(1, D, dtype=np.float32), (T, 1, 1)) * 8
    k = 0.01 * g.standard_normal((T, 1, D)).astype(np.float32)
    v = 0.1 * g.standard_normal((T, 1, D)).astype(np.float32)
    for j in (0, 5, window, 2 * window - 1, 2 * window + 1):
        k[j, 0, 0], v[j, 0] = 1.0 + 0.1 * j / window, 5.0 + j
    want = window_reference(q, k, v, 1.0, window, None)
    cuts = [2] + [1] * (T - 2) if decode else [window - 1, 2, window - 1, 1, T - 2 * window - 1]
    cache = PositionCache(ctx, 1, 1, D, D, window + max(cuts), dtype)
    got = run_attention(cache, cuts, q, k, v, scale=1.0, window=window, max_ctx=T)
    cache.close()
    err = np.abs(got - want).max(axis=(1, 2)) / np.abs(want).max(axis=(1, 2))
    assert err.max() < (1e-5 if dtype == "f32" else 3e-2), int(err.argmax())


def test_chunk_and_window_together_are_refused(ctx):
    cache = PositionCache(ctx, 1, 1, 16, 16, 64, "f32")
    x = np.zeros((1, 4, 1, 16), np.float32)
    with pytest.raises(skn.SknError):
        cache.attend(x, x, x, [0], 1.0, chunk=8, window=8, max_ctx=64)
    cache.close()


# ---- one mechanism at a time: a single layer, the other parts silent -------------------------------------------------
def silent(bits, *names):
    out = dict(bits)
    for n in names:
        out[n] = np.zeros_like(bits[n])
    return out


SSMS = {
    "one_head": tm.ssm(heads=1, vdim=16, state=16, groups=1, norm_groups=1),
    "groups": tm.ssm(heads=6, vdim=24, state=40, groups=3, norm_groups=2, conv=3),
    "odd": tm.ssm(heads=5, vdim=13, state=21, groups=1, norm_groups=1, conv=6),
    "cut_heads": tm.ssm(heads=6, vdim=10, state=12, groups=2, norm_groups=4, conv=2),     # a norm part ends inside a head
    "no_history": tm.ssm(heads=4, vdim=16, state=16, groups=4, norm_groups=4, conv=1),
    "wide_head": tm.ssm(heads=2, vdim=128, state=128, groups=1, norm_groups=1),
    "wide_state": tm.ssm(heads=2, vdim=40, state=200, groups=2, norm_groups=1, conv=5),
    "too_wide_for_chunks": tm.ssm(heads=1, vdim=200, state=48, groups=1, norm_groups=1),
    "deep_state": tm.ssm(heads=1, vdim=64, state=400, groups=1, norm_groups=1),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(SSMS))
def test_state_space_alone(ctx, name, dtype):
    cfg = tm.config([SSMS[name]], width=56, mult=1.0)
    bits = tm.weights(cfg, 3)
    tokens = np.random.default_rng(1).integers(0, 90, size=150)
    want, margin = oracle(cfg, tm.floats(bits), tokens)
    dec = decoder(ctx, cfg, bits, dtype)
    for cuts in ([150], [1] * 150, [2, 3, 2, 63, 64, 1, 15], [129] + [1] * 21, [33, 2, 31, 32, 52]):
        dec.reset()
        check(in_portions(dec, tokens, cuts), want, margin, dtype, cuts)
    dec.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_token_lives_in_the_state(ctx, dtype):
    """Heads that hardly forget: what stands at position 3 is seen 200 tokens on, across chunks and portions."""
    cfg = tm.config([tm.ssm(heads=2, vdim=16, state=16, groups=1, norm_groups=1)], width=48, mult=2.0)
    bits = tm.weights(cfg, 4)
    bits["l0.mix.A_log"] = to_bf16_bits(np.full(2, -9.0, np.float32))
    bits["l0.mix.D"] = np.zeros_like(bits["l0.mix.D"])
    big = from_bf16_bits(bits["embed"])
    g = np.random.default_rng(2)
    tokens = g.integers(1, 90, size=220)
    tokens[3] = 0
    # token 0 opens dt wide, the others hardly
    p = from_bf16_bits(bits["l0.mix.in"]).copy()
    p[-2:] = 0.4 * big[0] / np.linalg.norm(big[0]) * 6
    bits["l0.mix.in"] = to_bf16_bits(p)
    bits["l0.mix.dt_bias"] = to_bf16_bits(np.full(2, -6.0, np.float32))
    w = tm.floats(bits)
    want, margin = oracle(cfg, w, tokens)
    other = tokens.copy()
    other[3] = 7
    assert np.median(tm.errors(oracle(cfg, w, other)[0][200:], want[200:])) > 0.3
    dec = decoder(ctx, cfg, bits, dtype, max_tokens=256)
    for cuts in ([220], [4, 2, 150] + [1] * 64, [100, 100, 20]):
        dec.reset()
        check(in_portions(dec, tokens, cuts), want, margin, dtype, cuts)
    dec.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_many_heads_share_a_block(ctx, dtype):
    """Enough chunks and heads that several heads run in one block of the chunk kernels."""
    cfg = tm.config([tm.ssm(heads=64, vdim=8, state=8, groups=4, norm_groups=8)], width=40, mult=1.0)
    bits = tm.weights(cfg, 5)
    tokens = np.random.default_rng(3).integers(0, 90, size=1100)
    want, margin = oracle(cfg, tm.floats(bits), tokens)
    dec = decoder(ctx, cfg, bits, dtype, max_tokens=1100, max_ctx=1100)
    check(dec.forward(tokens, want=range(1100), want_next=False)[1], want, margin, dtype)
    dec.close()


LATENTS = {
    "plain": tm.latent(),
    "odd": tm.latent(heads=5, dim=20, rot_dim=6, vdim=13, q_rank=29, kv_rank=37, window=33),
    "no_window": tm.latent(heads=2, window=0, dim=16, rot_dim=32, vdim=8),
    "narrow": tm.latent(heads=9, window=1, dim=8, rot_dim=2, vdim=8, q_rank=8, kv_rank=16),
    "wide": tm.latent(heads=4, dim=128, rot_dim=64, vdim=128, q_rank=200, kv_rank=264, window=70, scale=0.07),
    "too_wide_for_tiles": tm.latent(heads=2, dim=260, rot_dim=16, vdim=72, kv_rank=120, window=50, scale=0.05),
    "values_wide": tm.latent(heads=2, dim=40, rot_dim=24, vdim=250, kv_rank=512, window=129, scale=0.1),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(LATENTS))
def test_latent_attention_alone(ctx, name, dtype):
    cfg = tm.config([LATENTS[name]], width=56, mult=1.0)
    bits = tm.weights(cfg, 3)
    tokens = np.random.default_rng(1).integers(0, 90, size=190)
    want, margin = oracle(cfg, tm.floats(bits), tokens)
    dec = decoder(ctx, cfg, bits, dtype, max_tokens=100)
    for cuts in ([100, 90], [1] * 190, [2, 3, 2, 31, 32, 64, 1, 55], [99] + [1] * 91):
        dec.reset()
        check(in_portions(dec, tokens, cuts), want, margin, dtype, cuts)
    dec.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_sink_weighs_in_the_model(ctx, dtype):
    cfg = tm.config([tm.latent(heads=2, window=9)], width=48, mult=2.0)
    bits = tm.weights(cfg, 6)
    bits["l0.mix.sink"] = to_bf16_bits(np.array([3.0, -2.0], np.float32))
    tokens = np.random.default_rng(1).integers(0, 90, size=60)
    w = tm.floats(bits)
    want, margin = oracle(cfg, w, tokens)
    w["l0.mix.sink"] = np.full(2, -np.inf)
    assert np.median(tm.errors(oracle(cfg, w, tokens)[0], want)) > 0.1
    dec = decoder(ctx, cfg, bits, dtype)
    for cuts in ([60], [1] * 60, [2, 40, 18]):
        dec.reset()
        check(in_portions(dec, tokens, cuts), want, margin, dtype, cuts)
    dec.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cuts", [[23] + [1] * 17, [20, 4, 2, 14], [40], [3, 33, 2, 2]])
def test_window_edge_of_the_whole_model(ctx, cuts, dtype):
    """Nearly even attention over the window: one key more or less shows, also where the window passes over the start."""
    layer = tm.latent(heads=1, dim=16, rot_dim=2, vdim=16, q_rank=16, kv_rank=16, scale=0.02, window=6)
    cfg = tm.config([layer], width=32, mult=3.0)
    bits = tm.weights(cfg, 3)
    tokens = np.random.default_rng(11).integers(0, 90, size=40)
    w = tm.floats(bits)
    want, margin = oracle(cfg, w, tokens)
    for size in (5, 7):
        wrong = json.loads(json.dumps(cfg))
        wrong["layers"][0]["mixer"]["mask"]["size"] = size
        assert np.median(tm.errors(plain.forward(wrong, w, tokens)[7:], want[7:])) > 0.1
    dec = decoder(ctx, cfg, bits, dtype, max_tokens=40)
    e = tm.errors(in_portions(dec, tokens, cuts), want)
    assert e.max() < tm.TOL[dtype], int(e.argmax())
    dec.close()


MOES = {
    "plain": tm.moe(), "one_of_many": tm.moe(experts=40, top=1, ff=16, shared=0), "all": tm.moe(experts=5, top=5, ff=9, shared=17),
    "single": tm.moe(experts=1, top=1, ff=33, shared=8), "wide": tm.moe(experts=8, top=3, ff=150, shared=200),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(MOES))
def test_experts_alone(ctx, name, dtype):
    cfg = tm.config([tm.ssm(heads=2, norm_groups=1, mlp=MOES[name])], width=136, mult=1.0)
    bits = silent(tm.weights(cfg, 7), "l0.mix.o")
    tokens = np.random.default_rng(1).integers(0, 90, size=400)
    want, margin = oracle(cfg, tm.floats(bits), tokens)
    dec = decoder(ctx, cfg, bits, dtype, max_tokens=400)
    for cuts in ([400], [1, 2, 3, 4, 5, 17, 2, 33, 1, 65, 67] + [1] * 200, [2] * 200):
        dec.reset()
        check(in_portions(dec, tokens, cuts), want, margin, dtype, cuts[:3])
    dec.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_favoured_expert_takes_most_tokens(ctx, dtype):
    """Groups of very unequal sizes, empty ones among them: the router follows one direction of the embedding."""
    cfg = tm.config([tm.ssm(heads=2, norm_groups=1, mlp=tm.moe(experts=7, top=2, ff=24, shared=0))], width=64, mult=1.0)
    bits = silent(tm.weights(cfg, 8), "l0.mix.o")
    r = from_bf16_bits(bits["l0.mlp.router"]).copy()
    emb = from_bf16_bits(bits["embed"]).copy()
    emb[:, 0] = 4.0                                        # a direction that all tokens share
    r[:, 0] = [0, 30, -30, 20, -30, -30, -20]
    bits["embed"], bits["l0.mlp.router"] = to_bf16_bits(emb), to_bf16_bits(r)
    tokens = np.random.default_rng(1).integers(0, 90, size=300)
    want, margin = oracle(cfg, tm.floats(bits), tokens)
    dec = decoder(ctx, cfg, bits, dtype, max_tokens=300)
    check(in_portions(dec, tokens, [300]), want, margin, dtype)
    dec.reset()
    check(in_portions(dec, tokens[:60], [5, 1, 1, 2, 51]), want[:60], margin[:60], dtype)
    dec.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("ff", [8, 75, 300])
def test_dense_feed_forward_alone(ctx, ff, dtype):
    cfg = tm.config([tm.latent(heads=1, mlp=tm.dense(ff))], width=72, mult=0.7)
    bits = silent(tm.weights(cfg, 9), "l0.mix.o")
    tokens = np.random.default_rng(1).integers(0, 90, size=70)
    want, margin = oracle(cfg, tm.floats(bits), tokens)
    dec = decoder(ctx, cfg, bits, dtype)
    for cuts in ([70], [1] * 70, [2, 3, 65]):
        dec.reset()
        check(in_portions(dec, tokens, cuts), want, margin, dtype, cuts)
    dec.close()


# ---- the decoder -------------------------------------------------------------------------------------------------------
MODELS = {
    "loop": tm.config([tm.ssm(mlp=tm.dense()), tm.latent(mlp=tm.moe()), tm.ssm(groups=1, conv=2, mlp=tm.moe(shared=0)), tm.latent(window=40)], loop=(1, 3, 3)),
    "loop_all": tm.config([tm.latent(heads=8, dim=16, rot_dim=16, vdim=16, mlp=tm.dense(128)), tm.ssm(heads=4, vdim=32, state=16, groups=1, norm_groups=1)] * 2, width=128,
                          loop=(0, 4, 2), vocab=161),
    "once": tm.config([tm.ssm(mlp=tm.moe(experts=4, top=4)), tm.latent(mlp=tm.dense(33))], loop=(0, 1, 1), width=101, eps=1e-3),
    "no_loop": tm.config([tm.latent(window=0), tm.ssm(heads=5, vdim=13, state=21, groups=5, norm_groups=5, mlp=tm.dense(31)),
                          tm.latent(heads=5, dim=20, rot_dim=6, vdim=13, q_rank=29, kv_rank=37, window=33, mlp=tm.moe(experts=9, top=3, ff=11, shared=5))], width=100, vocab=97),
}
_built = {}


def model(name):
    """(config dict, bf16 weights, token ids, oracle logits, routing margins) of one of MODELS; computed once."""
    if name not in _built:
        cfg = MODELS[name]
        bits = tm.weights(cfg, seed=len(name))
        tokens = np.random.default_rng(1).integers(0, cfg["vocab"], size=130)
        _built[name] = (cfg, bits, tokens, *oracle(cfg, tm.floats(bits), tokens))
    return _built[name]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(MODELS))
def test_prompt_portions_and_decoding(ctx, name, dtype):
    cfg, bits, tokens, want, margin = model(name)
    n = len(tokens)
    dec = decoder(ctx, cfg, bits, dtype)
    for cuts in ([n], [1] * n, [2, 3, 2, 40, 5, 78], [64, 4] + [1] * 62, [2] * (n // 2)):
        dec.reset()
        check(in_portions(dec, tokens, cuts), want, margin, dtype, cuts[:6])
    dec.close()


def test_layers_match_one_by_one(ctx):
    cfg, bits, tokens, _, _ = model("loop")
    runs = []
    plain.forward(cfg, tm.floats(bits), tokens[:30], lambda r, x: runs.append(x))
    dec = decoder(ctx, cfg, bits, "float32")
    dec.trace_layers(True)
    dec.forward(tokens[:30], want_next=False)
    got = dec.layer_outputs(30)
    assert got.shape[0] == len(runs) == 8
    for r, x in enumerate(runs):
        assert rel(got[r], x) < 1e-5, r
    dec.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_step_longer_than_the_buffers_runs_in_portions(ctx, dtype):
    cfg, bits, tokens, want, margin = model("loop")
    dec = decoder(ctx, cfg, bits, dtype, max_tokens=16)
    picks = [129, 0, 15, 16, 63]
    nxt, lg = dec.forward(tokens, want=picks)
    if dtype == "float32":
        assert tm.error(lg, want[picks]) < tm.TOL[dtype]
    else:
        assert np.median(tm.errors(lg, want[picks])) < tm.TOL[dtype]
    assert int(nxt[0]) == int(lg[0].argmax())
    dec.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_sequences_together_and_reused_slots(ctx, dtype):
    """Six sequences of unequal lengths decode in shared steps as each does alone; a slot is freed and used again."""
    cfg, bits, tokens, _, _ = model("loop")
    w = tm.floats(bits)
    g = np.random.default_rng(4)
    seqs = [g.integers(0, cfg["vocab"], size=n + 9) for n in (1, 13, 32, 33, 7, 50)]
    want, margin = zip(*[oracle(cfg, w, s) for s in seqs])
    dec = decoder(ctx, cfg, bits, dtype, max_seqs=6)
    got = [[] for _ in seqs]
    for i, s in enumerate(seqs):
        got[i].append(dec.forward(s[:-9], seq=i, want=range(len(s) - 9), want_next=False)[1])
    for t in range(9):
        lo, n = (0, 6) if t % 3 else (1, 4)            # all six, or a range of them (the others wait)
        ids = np.array([seqs[i][dec.position(i)] for i in range(lo, lo + n)])[:, None]
        lg = dec.forward(ids, seq=lo, want=range(n), want_next=False)[1]
        for r, i in enumerate(range(lo, lo + n)):
            got[i].append(lg[[r]])
    rows = [np.concatenate(x) for x in got]
    cat = lambda parts: np.concatenate([p[:len(r)] for p, r in zip(parts, rows)])
    check(np.concatenate(rows), cat(want), cat(margin), dtype)
    other = g.integers(0, cfg["vocab"], size=40)
    want_o, margin_o = oracle(cfg, w, other)
    dec.reset(2)
    assert dec.position(2) == 0 and dec.position(3) > 0
    check(in_portions(dec, other, [37, 1, 1, 1], seq=2), want_o, margin_o, dtype)
    dec.reset(1)
    check(in_portions(dec, other, [1] * 40, seq=1), want_o, margin_o, dtype)
    # two sequences prefill in one step, by steps of tokens and in chunks
    for n in (21, 40):
        dec.reset(4)
        dec.reset(5)
        lg = dec.forward(np.stack([other[:n], tokens[:n]]), seq=4, want=range(2 * n), want_next=False)[1]
        check(lg[:n], want_o[:n], margin_o[:n], dtype)
        check(lg[n:], *(a[:n] for a in oracle(cfg, w, tokens[:n])), dtype)
        if dtype == "float32":                         # and the second goes on from there
            more = dec.forward(tokens[n:n + 2], seq=5, want=[0, 1], want_next=False)[1]
            check(more, *(a[n:] for a in oracle(cfg, w, tokens[:n + 2])), dtype)
    dec.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_past_the_ring(ctx, dtype):
    """The latent caches hold a window and one step: hundreds of decoded tokens pass over them several times."""
    cfg = tm.config([tm.latent(heads=2, window=19, mlp=tm.dense(48)), tm.ssm(heads=2, norm_groups=1), tm.latent(heads=2, window=32)], width=48, loop=(0, 2, 2))
    bits = tm.weights(cfg, 8)
    tokens = np.random.default_rng(6).integers(0, cfg["vocab"], size=400)
    want, margin = oracle(cfg, tm.floats(bits), tokens)
    dec = decoder(ctx, cfg, bits, dtype, max_tokens=5, max_ctx=400)
    got = np.concatenate([dec.forward(tokens[i:i + 1], want=[0], want_next=False)[1] for i in range(400)])
    check(got, want, margin, dtype)
    with pytest.raises(ValueError, match="exceeded"):
        dec.forward([1], want_next=False)
    dec.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_portions_wrap_around_the_ring(ctx, dtype):
    """Portions of every size from 2 to the step's limit, the ring's end falling inside them."""
    cfg = tm.config([tm.latent(heads=2, window=30)], width=48, mult=1.0)
    bits = tm.weights(cfg, 8)
    tokens = np.random.default_rng(6).integers(0, cfg["vocab"], size=390)
    want, margin = oracle(cfg, tm.floats(bits), tokens)
    dec = decoder(ctx, cfg, bits, dtype, max_tokens=45, max_ctx=400)
    for cuts in ([45] * 8 + [30], [2, 44, 3, 43, 33, 12, 45, 2, 2, 45, 32, 31, 45, 41, 10], [38] * 10 + [10]):
        dec.reset()
        check(in_portions(dec, tokens, cuts), want, margin, dtype, cuts)
    dec.close()


def test_result_does_not_depend_on_slot_or_neighbours(ctx):
    cfg, bits, tokens, _, _ = model("loop")
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
    cfg, bits, _, _, _ = model("loop")
    w = tm.floats(bits)
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


@pytest.mark.parametrize("n", [1, 3])
def test_captured_step_replays(ctx, n):
    torch = pytest.importorskip("torch")
    cfg, bits, _, _, _ = model("loop")
    dec = decoder(ctx, cfg, bits, "bfloat16", max_seqs=n)
    prompt = np.array([[5, 17, 3], [8, 1, 2], [4, 4, 9]])[:n]
    dec.forward(prompt)
    for _ in range(8):
        dec.forward_dev(None, 1, n=n)
    ctx.sync()
    want_last = dec.forward(None)[0]
    stream = torch.cuda.Stream()
    graph = torch.cuda.CUDAGraph()
    dec.reset()
    try:
        with torch.cuda.stream(stream):
            ctx.set_stream(stream.cuda_stream)
            with torch.cuda.graph(graph, stream=stream):
                dec.forward_dev(None, 1, n=n)
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
    cfg, bits, _, _, _ = model("loop")
    d = tmp_path_factory.mktemp("model")
    (d / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(d / "model.safetensors"), bits)
    return str(d)


def test_generate_command(ctx, folder):
    cfg, bits, _, _, _ = model("loop")
    args = sum((["--prompt", ",".join(map(str, p))] for p in PROMPTS), [])
    r = subprocess.run([sys.executable, "-m", "skainet_b200.generate", "--model", folder, "--dtype", "float32", "--max-new", "6", *args],
                       cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    w = tm.floats(bits)
    assert [list(map(int, l.split(","))) for l in r.stdout.splitlines()] == [greedy(cfg, w, p, 6) for p in PROMPTS]


@pytest.mark.parametrize("dtype", DTYPES)
def test_replay_command(ctx, folder, tmp_path, dtype):
    cfg, bits, tokens, want, margin = model("loop")
    t = tokens.tolist()
    steps = [{"entries": [{"id": "a", "tokens": t[:50], "want": list(range(50))}], "end": []},
             {"entries": [{"id": "a", "tokens": t[50:52], "want": []}], "end": []},
             {"entries": [{"id": "b", "tokens": t[:33], "want": list(range(33))}], "end": ["b"]},
             {"entries": [{"id": "a", "tokens": t[52:], "want": list(range(78))}], "end": ["a"]},
             {"entries": [{"id": "c", "tokens": t[:20], "want": list(range(20))}], "end": ["c"]}]
    lines = "".join(json.dumps({"step": i, **s}) + "\n" for i, s in enumerate(steps))
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "140"],
                       input=lines, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(5)]
    for i, a, b in ((0, 0, 50), (2, 0, 33), (3, 52, 130), (4, 0, 20)):
        got = np.fromfile(tmp_path / f"{i}.f32", "<f4").reshape(-1, cfg["vocab"])
        check(got, want[a:b], margin[a:b], dtype, i)
    assert not (tmp_path / "1.f32").exists()


def test_weights_and_shapes_that_do_not_fit_are_refused(ctx):
    cfg, bits, _, _, _ = model("no_loop")
    bad = dict(bits)
    bad["l0.mix.dq"] = bits["l0.mix.dq"][:-1]
    dec = TutezenDecoder(ctx, TutezenConfig.from_dict(cfg), max_tokens=8, max_ctx=8)
    with pytest.raises(ValueError):
        dec.load(lambda name, shape: bad[name])
    with pytest.raises(skn.SknError):
        dec.forward([1])                                 # a layer has no weights
    dec.close()
    for c in (tm.config([tm.ssm()], loop=(0, 5, 1)), tm.config([tm.ssm(mlp=tm.moe(experts=2, top=3))])):
        with pytest.raises(skn.SknError):
            TutezenDecoder(ctx, TutezenConfig.from_dict(c), max_tokens=8, max_ctx=8)
