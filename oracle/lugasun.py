"""Plain fp64 restatement of the Lugasun decoder, one function per mechanism, loops where a loop is the
definition.  It shares no code with the product path: weights are a dict name -> array [out, in], `cfg` is the
parsed configuration (plain dicts and lists), and every function takes whole sequences from position 0.

Notation: x is the residual stream [T, width], h a mixer's input, heads are split out as [T, heads, dim]."""
import numpy as np


def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) along the last axis."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return rms_unit(x, eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z / (1.0 + np.exp(-z))


def relu_squared(z):
    return np.maximum(z, 0.0) ** 2


def rotate_half(x, rot, pos0=0):
    """x [T, heads, dim]: dimensions i and i + dims/2 of the first `dims` form a pair turned by pos * base^(-2i/dims)."""
    if not rot or not rot.get("dims"):
        return x
    dims, base = int(rot["dims"]), float(rot["base"])
    half = dims // 2
    y = x.copy()
    for t in range(x.shape[0]):
        for i in range(half):
            a = (pos0 + t) * base ** (-2.0 * i / dims)
            u, v = x[t, :, i], x[t, :, i + half]
            y[t, :, i] = u * np.cos(a) - v * np.sin(a)
            y[t, :, i + half] = v * np.cos(a) + u * np.sin(a)
    return y


def chunk_visible(i, j, size):
    """Key j is visible to query i: not in the future and, with a chunk size, in the same chunk."""
    return j <= i and (not size or i // size == j // size)


def chunked_attention(q, k, v, scale, softcap=None, size=None):
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim] -> [T, H, vdim]."""
    T, H = q.shape[:2]
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        js = [j for j in range(i + 1) if chunk_visible(i, j, size)]
        for h in range(H):
            g = h // (H // G)
            s = (k[js, g] @ q[i, h]) * scale
            if softcap:
                s = softcap * np.tanh(s / softcap)
            p = np.exp(s - s.max())
            out[i, h] = (p / p.sum()) @ v[js, g]
    return out


def retention(q, k, v, decay, state=None):
    """q, k [T, H, dim], v [T, H, vdim]; S <- decay S + k v^T, o = S^T q.  Returns (o [T, H, vdim], S)."""
    T, H, D = q.shape
    S = np.zeros((H, D, v.shape[2])) if state is None else state.copy()
    o = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        for h in range(H):
            S[h] = decay[h] * S[h] + np.outer(k[t, h], v[t, h])
            o[t, h] = S[h].T @ q[t, h]
    return o, S


def attention_mixer(w, p, m, h, eps):
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).reshape(T, H, D)
    k = (h @ w[p + "k"].T).reshape(T, G, D)
    v = (h @ w[p + "v"].T).reshape(T, G, V)
    q, k = rms_norm(q, w[p + "q.norm"], eps), rms_norm(k, w[p + "k.norm"], eps)
    q, k = rotate_half(q, m.get("rot")), rotate_half(k, m.get("rot"))
    o = chunked_attention(q, k, v, m["scale"], m.get("softcap"), (m.get("mask") or {}).get("size"))
    return o.reshape(T, H * V) @ w[p + "o"].T


def retention_mixer(w, p, m, h, eps):
    T = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q = rotate_half((h @ w[p + "q"].T).reshape(T, H, D), m.get("rot"))
    k = rotate_half((h @ w[p + "k"].T).reshape(T, H, D), m.get("rot")) * D ** -0.5
    v = (h @ w[p + "v"].T).reshape(T, H, V)
    o, _ = retention(q, k, v, m["decay"])
    o = rms_unit(o, eps).reshape(T, H * V)
    return (o * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def parallel_mixer(w, p, m, h, eps):
    return (m["left_scale"] * attention_mixer(w, p + "left.", m["left"], h, eps)
            + m["right_scale"] * retention_mixer(w, p + "right.", m["right"], h, eps))


def dense_ff(w, p, h):
    return relu_squared(h @ w[p + "up"].T) @ w[p + "down"].T


def token_side(w, p, x, e, eps):
    g = gelu_tanh(x @ w[p + "gate"].T) * e
    return x + rms_norm(g @ w[p + "proj"].T, w[p + "norm"], eps)


def layer_runs(cfg):
    """(layer index, first layer of a pass of the loop) in the order the layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    once = [(i, i == a) for i in range(a, b)]
    return [(i, False) for i in range(a)] + once * loop["times"] + [(i, False) for i in range(b, n)]


def forward(cfg, w, tokens, on_layer=None):
    """Logits [T, vocab] of a whole sequence; on_layer(run, x) sees the residual stream after every layer run."""
    tokens = np.asarray(tokens)
    eps = cfg["norm"]["eps"]
    x0 = w["embed"][tokens]
    x = x0
    side = cfg.get("token_side")
    for run, (i, first) in enumerate(layer_runs(cfg)):
        if first:
            x = np.concatenate([x, x0], axis=1) @ w["loop.in"].T
        p, layer = f"l{i}.", cfg["layers"][i]
        x = x + parallel_mixer(w, p + "mix.", layer["mixer"], rms_norm(x, w[p + "norm1"], eps), eps)
        if layer.get("mlp"):
            x = x + dense_ff(w, p + "mlp.", rms_norm(x, w[p + "norm2"], eps))
        if side:
            d = side["dim"]
            x = token_side(w, p + "side.", x, w["side.embed"][tokens][:, i * d:(i + 1) * d], eps)
        if on_layer:
            on_layer(run, x)
    return rms_norm(x, w["final.norm"], eps) @ w["embed"].T
