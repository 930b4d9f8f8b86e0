"""Plain, slow restatement of the Bolonex decoder in float64 numpy, one function per mechanism.

TEST INFRASTRUCTURE ONLY, like the rest of ``oracle/``: nothing here is shared with the library.  Every function takes
whole sequences from position 0 (there is no cache), so "prompt in portions" and "token by token" are questions only for
the library; the answer it has to give is the row this file computes.

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


def causal_conv(u, w):
    """y[t, c] = sum_j w[c, j] * u[t - taps + 1 + j, c], zeros before the start."""
    length, channels = u.shape
    taps = w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, channels)), u], axis=0)
    out = np.zeros_like(u)
    for j in range(taps):
        out += padded[j:j + length] * w[:, j]
    return out


def rotation_frequencies(rot):
    """Angular frequencies of the dims/2 pairs, with the wavelength-dependent scaling when ``rot.scaling`` is given."""
    f = float(rot["base"]) ** (-2.0 * np.arange(rot["dims"] // 2) / rot["dims"])
    scaling = rot.get("scaling")
    if not scaling:
        return f
    out = f.copy()
    for i, fi in enumerate(f):
        wavelength = 2.0 * np.pi / fi
        turns = scaling["original"] / wavelength
        if wavelength < scaling["original"] / scaling["high"]:
            continue
        if wavelength > scaling["original"] / scaling["low"]:
            out[i] = fi / scaling["factor"]
        else:
            s = (turns - scaling["low"]) / (scaling["high"] - scaling["low"])
            out[i] = (1.0 - s) * fi / scaling["factor"] + s * fi
    return out


def rotate_interleaved(x, rot):
    """x [tokens, heads, dim]: pairs (2i, 2i + 1) of the first rot.dims dimensions turn by position * frequency."""
    f = rotation_frequencies(rot)
    angle = np.arange(x.shape[0])[:, None] * f[None, :]
    c, s = np.cos(angle)[:, None, :], np.sin(angle)[:, None, :]
    out = x.copy()
    u, v = x[:, :, 0:rot["dims"]:2], x[:, :, 1:rot["dims"]:2]
    out[:, :, 0:rot["dims"]:2] = u * c - v * s
    out[:, :, 1:rot["dims"]:2] = v * c + u * s
    return out


def attend(q, k, v, scale, softcap):
    """Causal softmax attention, grouped heads, capped scores: q [t, H, dim], k [t, G, dim], v [t, G, vdim]."""
    length, heads = q.shape[:2]
    per = heads // k.shape[1]
    out = np.zeros((length, heads, v.shape[2]))
    hidden = np.triu(np.ones((length, length), dtype=bool), 1)
    for h in range(heads):
        s = (q[:, h] @ k[:, h // per].T) * scale
        if softcap:
            s = softcap * np.tanh(s / softcap)
        s = np.where(hidden, -np.inf, s)
        p = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = (p / p.sum(axis=1, keepdims=True)) @ v[:, h // per]
    return out


def attention_mixer(h, m, t, eps):
    length = h.shape[0]

    def project(name, heads, width):
        u = h @ t[name].T + t[name + ".b"]
        return causal_conv(u, t[name + ".conv"]).reshape(length, heads, width)

    q = project("q", m["heads"], m["dim"])
    k = project("k", m["kv_heads"], m["dim"])
    v = project("v", m["kv_heads"], m["vdim"])
    q = rotate_interleaved(rms(q, eps) * t["q.norm"], m["rot"])
    k = rotate_interleaved(rms(k, eps) * t["k.norm"], m["rot"])
    o = attend(q, k, v, m["scale"], m.get("softcap"))
    o = o * sigmoid(h @ t["g"].T)[:, :, None]
    return o.reshape(length, -1) @ t["o"].T


def state_space_scan(x, b, c, dt, a_log, d):
    """x [t, heads, vdim], b / c [t, groups, N], dt [t, heads] (after softplus): the recurrence token by token."""
    length, heads, vdim = x.shape
    per = heads // b.shape[1]
    y = np.zeros_like(x)
    for h in range(heads):
        s = np.zeros((b.shape[2], vdim))
        for i in range(length):
            s = np.exp(-np.exp(a_log[h]) * dt[i, h]) * s + dt[i, h] * np.outer(b[i, h // per], x[i, h])
            y[i, h] = s.T @ c[i, h // per] + d[h] * x[i, h]
    return y


def gated_group_norm(y, z, weight, groups, eps):
    length, inner = y.shape
    g = (y * silu(z)).reshape(length, groups, inner // groups)
    return rms(g, eps).reshape(length, inner) * weight


def mamba2_mixer(h, m, t, eps):
    length = h.shape[0]
    inner, gn = m["heads"] * m["vdim"], m["groups"] * m["state"]
    u = h @ t["in"].T
    z, xbc, dt = u[:, :inner], u[:, inner:2 * inner + 2 * gn], u[:, 2 * inner + 2 * gn:]
    xbc = silu(causal_conv(xbc, t["conv"]) + t["conv.b"])
    x = xbc[:, :inner].reshape(length, m["heads"], m["vdim"])
    b = xbc[:, inner:inner + gn].reshape(length, m["groups"], m["state"])
    c = xbc[:, inner + gn:].reshape(length, m["groups"], m["state"])
    y = state_space_scan(x, b, c, softplus(dt + t["dt_bias"]), t["A_log"], t["D"])
    return gated_group_norm(y.reshape(length, inner), z, t["norm"], m["norm_groups"], eps) @ t["o"].T


def dense_feed_forward(h, t):
    return gelu_tanh(h @ t["up"].T) @ t["down"].T


MIXERS = {"attention": attention_mixer, "mamba2": mamba2_mixer}


def owner_of(layers, i):
    while layers[i].get("weights_of") is not None:
        i = layers[i]["weights_of"]
    return i


def forward(config, tensors, tokens):
    get = {k: np.asarray(v, dtype=np.float64) for k, v in tensors.items()}
    eps = config["norm"]["eps"]

    def under(prefix):
        return {k[len(prefix):]: v for k, v in get.items() if k.startswith(prefix)}

    x = get["embed"][np.asarray(tokens)] * config["embedding"]["scale"]
    after = []
    for i, layer in enumerate(config["layers"]):
        p = f"l{owner_of(config['layers'], i)}."
        h = norm_around_zero(x, get[p + "norm1"], eps)
        delta = MIXERS[layer["type"]](h, layer["mixer"], under(p + "mix."), eps)
        if layer.get("mlp"):
            delta = delta + dense_feed_forward(h, under(p + "mlp."))
        x = x + delta
        after.append(x)
    return norm_around_zero(x, get["final.norm"], eps) @ get["head"].T, np.stack(after)
