"""Plain numpy statement of the Supevik decoder: one function per mechanism, float64 by default. Slow on purpose; shares
no code with the package.

A model is `cfg` (the dictionary of config.json) and `t` (tensor name -> array). A sequence is run from its first token
every time: no cache, no portions.
"""
import math

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rms_unit(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def tanh_norm(x, alpha, w, b):
    """Element by element: no mean, no variance."""
    return np.tanh(alpha * x) * w + b


def frequencies(rot):
    """(angle per position of every pair, factor on cosine and sine) of a rotation over rot["dims"] dimensions."""
    dims, base = rot["dims"], rot["base"]
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    s = rot.get("scaling")
    if not s:
        return f, 1.0

    def at(turns):           # the (fractional) dimension whose pair makes `turns` turns over the original context
        return dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(at(s["fast"])), 0)
    hi = min(math.ceil(at(s["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / s["factor"] * r + fi * (1.0 - r))
    return np.array(out), 0.1 * math.log(s["factor"]) + 1.0


def rotate_halves(x, pos, rot):
    """x [..., tokens, n]: dimension i turns with dimension i + dims/2, the ones from dims on stay."""
    d = rot["dims"]
    f, mag = frequencies(rot)
    a = np.asarray(pos, np.float64)[:, None] * f[None, :]
    c, s = (np.cos(a) * mag).astype(x.dtype), (np.sin(a) * mag).astype(x.dtype)
    u, v = x[..., :d // 2], x[..., d // 2:d]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., d:]], axis=-1)


def window_mask(n, size):
    """[query, key]: the query itself and the size - 1 tokens before it."""
    gap = np.arange(n)[:, None] - np.arange(n)[None, :]
    return (gap >= 0) & (gap < size)


def attention(h, m, p, eps):
    """h [T, width]; m: mixer sizes; p(name): tensor of this mixer."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ p("q").T + p("q.b")).reshape(T, H, D).transpose(1, 0, 2)
    k = (h @ p("k").T + p("k.b")).reshape(T, G, D).transpose(1, 0, 2)
    v = (h @ p("v").T + p("v.b")).reshape(T, G, V).transpose(1, 0, 2)
    pos = np.arange(T)
    q = rotate_halves(rms_unit(q, eps) * p("q.norm"), pos, m["rot"])
    k = rotate_halves(rms_unit(k, eps) * p("k.norm"), pos, m["rot"])
    see = window_mask(T, m["mask"]["size"])
    out = np.empty((T, H, V), h.dtype)
    for i in range(H):
        j = i // (H // G)
        s = np.where(see, q[i] @ k[j].T * m["scale"], -np.inf)
        w = np.exp(s - s.max(axis=-1, keepdims=True))
        out[:, i] = w / w.sum(axis=-1, keepdims=True) @ v[j]
    return (out.reshape(T, H * V) * sigmoid(h @ p("g").T)) @ p("o").T


def dense(h, p):
    return (gelu_tanh(h @ p("gate").T) * (h @ p("up").T)) @ p("down").T


MIXERS = {"attention": attention}


def schedule(cfg):
    """Layer runs in order: (layer, True where a pass of the loop begins)."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, z = loop["start"], loop["stop"]
    out = [(i, False) for i in range(a)]
    for _ in range(loop["times"]):
        out += [(i, i == a) for i in range(a, z)]
    return out + [(i, False) for i in range(z, n)]


def run(cfg, t, tokens, dtype=np.float64):
    """Logits [T, vocab] and the residual stream after every layer run [runs, T, width]."""
    t = {k: np.asarray(a, dtype) for k, a in t.items()}
    eps = cfg["norm"]["eps"]

    def norm(name, x):
        return tanh_norm(x, t[name + ".alpha"], t[name], t[name + ".b"])
    x0 = x = t["embed"][np.asarray(tokens)] * dtype(cfg["embedding"]["scale"])
    trail = []
    for i, enter in schedule(cfg):
        layer, pre = cfg["layers"][i], "l%d." % i
        if enter:
            x = np.concatenate([x, x0], axis=-1) @ t["loop.in"].T
        y = MIXERS[layer["type"]](norm(pre + "norm1", x), layer["mixer"], lambda n: t[pre + "mix." + n], eps)
        x = x + norm(pre + "norm1b", y)
        if layer.get("mlp") is not None:
            assert layer["mlp"]["kind"] == "dense"
            y = dense(norm(pre + "norm2", x), lambda n: t[pre + "mlp." + n])
            x = x + norm(pre + "norm2b", y)
        trail.append(x)
    return norm("final.norm", x) @ t["head"].T, np.stack(trail)
