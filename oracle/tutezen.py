"""Plain fp64 restatement of the Tutezen decoder, one function per mechanism, loops where a loop is the definition.  It
shares no code with the product path: weights are a dict name -> array [out, in], `cfg` is the parsed configuration
(plain dicts and lists), and every function takes whole sequences from position 0.

Notation: x is the residual stream [T, width], h the normalised input that a layer's mixer and feed-forward share."""
import numpy as np


def rms_norm(x, w, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


# ---- selective state space -------------------------------------------------------------------------------------
def causal_conv(u, w, b):
    """u [T, channels], w [channels, taps]: y_t = b + sum over k of w_k u_(t - taps + 1 + k), with u = 0 ahead of the sequence."""
    T, taps = u.shape[0], w.shape[1]
    y = np.zeros_like(u)
    for t in range(T):
        y[t] = b
        for k in range(taps):
            j = t - (taps - 1) + k
            if j >= 0:
                y[t] += w[:, k] * u[j]
    return y


def selective_scan(x, B, C, dt, A_log, D, state=None):
    """x [T, H, V], B, C [T, G, N], dt [T, H] (positive): S <- exp(-exp(A_log) dt) S + dt B x^T, y = S^T C + D x.
    Returns (y [T, H, V], S [H, N, V])."""
    T, H, V = x.shape
    G, N = B.shape[1:]
    S = np.zeros((H, N, V)) if state is None else state.copy()
    y = np.zeros_like(x)
    for t in range(T):
        for h in range(H):
            g = h // (H // G)
            S[h] = np.exp(-np.exp(A_log[h]) * dt[t, h]) * S[h] + dt[t, h] * np.outer(B[t, g], x[t, h])
            y[t, h] = S[h].T @ C[t, g] + D[h] * x[t, h]
    return y, S


def grouped_rms_norm(y, w, parts, eps):
    T, n = y.shape
    u = y.reshape(T, parts, n // parts)
    return (u / np.sqrt((u * u).mean(-1, keepdims=True) + eps)).reshape(T, n) * w


def mamba2_mixer(w, p, m, h, eps):
    T = h.shape[0]
    H, V, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * V
    u = h @ w[p + "in"].T
    z, xbc, dt = u[:, :inner], u[:, inner:2 * inner + 2 * G * N], u[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, w[p + "conv"], w[p + "conv.b"]))
    x, B, C = xbc[:, :inner].reshape(T, H, V), xbc[:, inner:inner + G * N].reshape(T, G, N), xbc[:, inner + G * N:].reshape(T, G, N)
    y, _ = selective_scan(x, B, C, softplus(dt + w[p + "dt_bias"]), w[p + "A_log"], w[p + "D"])
    y = y.reshape(T, inner) * silu(z)
    return grouped_rms_norm(y, w[p + "norm"], m["norm_groups"], eps) @ w[p + "o"].T


# ---- latent attention --------------------------------------------------------------------------------------------
def rotate_pairs(x, rot, pos0=0):
    """x [T, heads, dim]: dimensions 2i and 2i + 1 of the first `dims` turn by position * base^(-2i / dims)."""
    if not rot or not rot.get("dims"):
        return x
    dims, base = int(rot["dims"]), float(rot["base"])
    y = x.copy()
    for t in range(x.shape[0]):
        for i in range(dims // 2):
            a = (pos0 + t) * base ** (-2.0 * i / dims)
            u, v = x[t, :, 2 * i], x[t, :, 2 * i + 1]
            y[t, :, 2 * i] = u * np.cos(a) - v * np.sin(a)
            y[t, :, 2 * i + 1] = v * np.cos(a) + u * np.sin(a)
    return y


def window_visible(i, j, size):
    return 0 <= i - j and (not size or i - j < size)


def sink_softmax(s, sink):
    """Weights of the scores s when one more score, `sink`, shares the denominator."""
    top = max(s.max(), sink)
    e = np.exp(s - top)
    return e / (e.sum() + np.exp(sink - top))


def window_attention(q, k, v, scale, size=None, sink=None):
    """q, k [T, H, dim], v [T, H, vdim], sink [H] or None -> [T, H, vdim]."""
    T, H = q.shape[:2]
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        js = [j for j in range(i + 1) if window_visible(i, j, size)]
        for h in range(H):
            s = (k[js, h] @ q[i, h]) * scale
            out[i, h] = sink_softmax(s, -np.inf if sink is None else sink[h]) @ v[js, h]
    return out


def latent_attention_mixer(w, p, m, h, eps):
    T = h.shape[0]
    H, D, R, V, K = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    c_q = rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps)
    q = (c_q @ w[p + "uq"].T).reshape(T, H, D + R)
    u = h @ w[p + "dkv"].T
    c = rms_norm(u[:, :K], w[p + "dkv.norm"], eps)
    k_rot = rotate_pairs(u[:, K:].reshape(T, 1, R), m.get("rot"))
    q = np.concatenate([q[:, :, :D], rotate_pairs(q[:, :, D:], m.get("rot"))], axis=2)
    k = np.concatenate([(c @ w[p + "uk"].T).reshape(T, H, D), np.repeat(k_rot, H, axis=1)], axis=2)
    v = (c @ w[p + "uv"].T).reshape(T, H, V)
    o = window_attention(q, k, v, m["scale"], (m.get("mask") or {}).get("size"), w[p + "sink"]).reshape(T, H * V)
    return (o * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---- feed-forward ----------------------------------------------------------------------------------------------
def dense_ff(w, p, h):
    return gelu_tanh(h @ w[p + "up"].T) @ w[p + "down"].T


def gated_ff(w, p, h):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(z, top):
    """Router logits of one token -> (chosen experts, their weights)."""
    e = np.exp(z - z.max())
    s = e / e.sum()
    chosen = np.argsort(-s, kind="stable")[:top]
    return chosen, s[chosen] / (s[chosen].sum() + 1e-20)


def moe_ff(w, p, mlp, h):
    out = np.zeros((h.shape[0], w[p + "e0.down"].shape[0]))
    z = h @ w[p + "router"].T
    for t in range(h.shape[0]):
        for e, weight in zip(*route(z[t], mlp["router"]["top"])):
            out[t] += weight * gated_ff(w, f"{p}e{e}.", h[t])
    if mlp.get("shared"):
        out += gated_ff(w, p + "shared.", h)
    return out


MIXERS = {"mamba2": mamba2_mixer, "latent_attention": latent_attention_mixer}


def layer_runs(cfg):
    """(layer index, number of the pass that begins before it or None) in the order the layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    once = [[(i, t if i == a else None) for i in range(a, b)] for t in range(loop["times"])]
    return [(i, None) for i in range(a)] + sum(once, []) + [(i, None) for i in range(b, n)]


def forward(cfg, w, tokens, on_layer=None):
    """Logits [T, vocab] of a whole sequence; on_layer(run, x) sees the residual stream after every layer run."""
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x0 = w["embed"][np.asarray(tokens)]
    x = x0
    for run, (i, begins) in enumerate(layer_runs(cfg)):
        if begins is not None:
            x = x + (x0 if begins else 0.0) + w["loop.step"][begins]
        p, layer = f"l{i}.", cfg["layers"][i]
        h = rms_norm(x, w[p + "norm1"], eps)
        y = MIXERS[layer["type"]](w, p + "mix.", layer["mixer"], h, eps)
        mlp = layer.get("mlp")
        if mlp:
            y = y + (moe_ff(w, p + "mlp.", mlp, h) if mlp["kind"] == "moe" else dense_ff(w, p + "mlp.", h))
        x = x + mult * y
        if on_layer:
            on_layer(run, x)
    return rms_norm(x, w["final.norm"], eps) @ w["embed"].T
