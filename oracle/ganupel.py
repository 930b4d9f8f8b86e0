"""Plain, slow restatement of the Ganupel decoder in float64 numpy, one function per mechanism.

TEST INFRASTRUCTURE ONLY, like the rest of ``oracle/``: nothing here is shared with the library.  Every function takes
whole sequences from position 0 (there is no cache), so portions and token-by-token decoding are questions for the library
alone; the answer it has to give is the row this file computes.

``forward(config, tensors, tokens)`` -> (logits [tokens, vocab], residual stream after every layer).
``config`` is the parsed config.json dictionary, ``tensors`` maps names to arrays.
"""
import numpy as np


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm_around_zero(x, w, eps):
    """RMS norm whose weight is stored as its distance from one."""
    return rms(x, eps) * (1.0 + w)


def sigmoid(x):
    return 0.5 * (1.0 + np.tanh(0.5 * x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return np.logaddexp(0.0, x)


def gelu_tanh(x):
    return 0.5 * x * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (x + 0.044715 * x ** 3)))


# ---- windowed attention whose weights are sigmoids ---------------------------------------------------
def rotate_halves(x, rot):
    """x [tokens, heads, dim]: dimension i of the first dims / 2 turns together with dimension i + dims / 2."""
    if not rot or not rot["dims"]:
        return x
    half = rot["dims"] // 2
    f = float(rot["base"]) ** (-2.0 * np.arange(half) / rot["dims"])
    angle = np.arange(x.shape[0])[:, None] * f[None, :]
    c, s = np.cos(angle)[:, None, :], np.sin(angle)[:, None, :]
    u, v = x[:, :, :half], x[:, :, half:2 * half]
    return np.concatenate([u * c - v * s, v * c + u * s, x[:, :, 2 * half:]], axis=2)


def sigmoid_attend(q, k, v, scale, bias, window):
    """Every visible key counts with sigmoid(score + bias of the head); nothing is normalised over keys."""
    length, heads = q.shape[:2]
    per = heads // k.shape[1]
    lag = np.arange(length)[:, None] - np.arange(length)[None, :]
    seen = (lag >= 0) & (lag < window)
    out = np.zeros((length, heads, v.shape[2]))
    for h in range(heads):
        s = (q[:, h] @ k[:, h // per].T) * scale + bias[h]
        out[:, h] = np.where(seen, sigmoid(s), 0.0) @ v[:, h // per]
    return out


def windowed_attention(h, m, t):
    length = h.shape[0]
    q = rotate_halves((h @ t["q"].T).reshape(length, m["heads"], m["dim"]), m.get("rot"))
    k = rotate_halves((h @ t["k"].T).reshape(length, m["kv_heads"], m["dim"]), m.get("rot"))
    v = (h @ t["v"].T).reshape(length, m["kv_heads"], m["vdim"])
    o = sigmoid_attend(q, k, v, m["scale"], t["pb"], m["mask"]["size"])
    return o.reshape(length, -1) @ t["o"].T


# ---- gated linear attention (HGRN2) --------------------------------------------------------------------
def gated_scan(q, f, v):
    """q, f [t, heads, dim], v [t, heads, vdim]: what a channel forgets is what it writes, token by token."""
    length, heads, dim = q.shape
    out = np.zeros_like(v)
    for h in range(heads):
        s = np.zeros((dim, v.shape[2]))
        for i in range(length):
            s = f[i, h][:, None] * s + np.outer(1.0 - f[i, h], v[i, h])
            out[i, h] = s.T @ q[i, h]
    return out


def hgrn2(h, m, t, eps):
    length, heads = h.shape[0], m["heads"]
    q = silu(h @ t["q"].T).reshape(length, heads, m["dim"])
    v = (h @ t["v"].T).reshape(length, heads, m["vdim"])
    f = t["lower"] + (1.0 - t["lower"]) * sigmoid(h @ t["f"].T + t["f.b"])
    o = gated_scan(q, f.reshape(length, heads, m["dim"]), v)
    return (rms(o, eps) * t["norm"]).reshape(length, -1) @ t["o"].T


def under(tensors, prefix):
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def parallel_mixer(h, m, t, eps):
    left = windowed_attention(h, m["left"], under(t, "left."))
    right = hgrn2(h, m["right"], under(t, "right."), eps)
    return m["left_scale"] * left + m["right_scale"] * right


# ---- real-gated linear recurrent unit ------------------------------------------------------------------
def causal_conv(u, w, b):
    """y[t, c] = b[c] + sum_j w[c, j] u[t - taps + 1 + j, c], zeros before the start."""
    length, channels = u.shape
    taps = w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, channels)), u], axis=0)
    return b + sum(padded[j:j + length] * w[:, j] for j in range(taps))


def block_diagonal(u, w, b):
    """u [t, blocks * n], w [blocks, n, n] (out, in), b [blocks, n]."""
    parts = u.reshape(u.shape[0], w.shape[0], w.shape[2])
    return (np.einsum("tbi,boi->tbo", parts, w) + b).reshape(u.shape[0], -1)


def linear_unit_scan(u, r, i, lam):
    log_a = -8.0 * r * softplus(lam)
    a, gain = np.exp(log_a), np.sqrt(-np.expm1(2.0 * log_a))
    out, s = np.zeros_like(u), np.zeros(u.shape[1])
    for n in range(u.shape[0]):
        s = a[n] * s + gain[n] * i[n] * u[n]
        out[n] = s
    return out


def rglru_mixer(h, m, t, eps):
    y = gelu_tanh(h @ t["y"].T + t["y.b"])
    u = causal_conv(h @ t["x"].T + t["x.b"], t["conv"], t["conv.b"])
    r = sigmoid(block_diagonal(u, t["ra"], t["ra.b"].reshape(t["ra"].shape[:2])))
    i = sigmoid(block_diagonal(u, t["ri"], t["ri.b"].reshape(t["ri"].shape[:2])))
    return (linear_unit_scan(u, r, i, t["lam"]) * y) @ t["o"].T


# ---- feed-forwards ---------------------------------------------------------------------------------------
def poly_norm(z, act, eps):
    a, b, c, e = act
    return a * rms(z, eps) + b * rms(z ** 2, eps) + c * rms(z ** 3, eps) + e


def dense_feed_forward(h, m, t, eps):
    return poly_norm(h @ t["up"].T, t["act"], eps) @ t["down"].T


def route(h, router, w, correction):
    """Chosen experts [t, top] (largest corrected score first) and their weights."""
    z = h @ w.T
    s = np.exp(z - z.max(axis=1, keepdims=True))
    s = s / s.sum(axis=1, keepdims=True)
    chosen = np.argsort(-(s + correction), axis=1, kind="stable")[:, :router["top"]]
    w = np.take_along_axis(s, chosen, axis=1)
    return chosen, w / (w.sum(axis=1, keepdims=True) + 1e-20) * router["scale"]


def mixture(h, m, t, eps):
    router = m["router"]
    chosen, weights = route(h, router, t["router"], t["correction"])
    out = np.zeros_like(h)
    for i in range(h.shape[0]):
        for e, w in zip(chosen[i], weights[i]):
            if e >= router["experts"]:
                out[i] += w * h[i]                                   # an identity expert
            else:
                out[i] += w * (np.maximum(h[i] @ t[f"e{e}.up"].T, 0.0) ** 2 @ t[f"e{e}.down"].T)
    return out


MIXERS = {"parallel": parallel_mixer, "rglru": rglru_mixer}
FEED_FORWARDS = {"dense": dense_feed_forward, "moe": mixture}


def forward(config, tensors, tokens):
    get = {k: np.asarray(v, dtype=np.float64) for k, v in tensors.items()}
    eps = config["norm"]["eps"]
    x = get["embed"][np.asarray(tokens)]
    after = []
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        h = norm_around_zero(x, get[p + "norm1"], eps)
        x = x + MIXERS[layer["type"]](h, layer["mixer"], under(get, p + "mix."), eps) * get[p + "ls1"]
        if layer.get("mlp"):
            h = norm_around_zero(x, get[p + "norm2"], eps)
            x = x + FEED_FORWARDS[layer["mlp"]["kind"]](h, layer["mlp"], under(get, p + "mlp."), eps) * get[p + "ls2"]
        after.append(x)
    return norm_around_zero(x, get["final.norm"], eps) @ get["head"].T, np.stack(after)
