"""Plain numpy statement of the Ripidra decoder: one function per mechanism, float64 by default, token loops where
the mechanism is a recurrence. Slow on purpose; shares no code with the package.

A model is `cfg` (the dictionary of config.json) and `t` (tensor name -> array). A sequence is run from its first
token every time: no cache, no portions.
"""
import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def rms_unit(x, eps):
    """x over the root of its mean square along the last axis (eps under the root)."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm_about_one(x, w, eps):
    """RMS norm whose stored weight is the deviation from one."""
    return rms_unit(x, eps) * (1.0 + w)


def rotate_pairs(x, pos, base):
    """Neighbouring components (2i, 2i+1) of the last axis turned by pos * base^(-2i/n). x [..., tokens, n]; the
    token axis is the last but one and pos lists the tokens' positions."""
    n = x.shape[-1]
    a = np.asarray(pos, x.dtype)[:, None] * (base ** (-np.arange(0, n, 2) / n)).astype(x.dtype)[None, :]
    c, s = np.cos(a), np.sin(a)
    out = np.empty_like(x)
    out[..., 0::2] = x[..., 0::2] * c - x[..., 1::2] * s
    out[..., 1::2] = x[..., 1::2] * c + x[..., 0::2] * s
    return out


def causal_conv(x, w):
    """Depthwise convolution along time: y[t, c] = sum_j w[c, taps-1-j] x[t-j, c], zeros before the start."""
    T, taps = x.shape[0], w.shape[1]
    xp = np.concatenate([np.zeros((taps - 1, x.shape[1]), x.dtype), x])
    return sum(xp[j:j + T] * w[:, j] for j in range(taps))


def unit_heads(x, tiny=1e-6):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + tiny)


def delta_recurrence(q, k, v, g, beta):
    """Per head: the rows of S decay by g, the value is corrected by what S returns for k, the outer product of k
    and the corrected value is written, q reads. q, k, g [T, H, D], v [T, H, V], beta [T, H] -> o [T, H, V]."""
    T, H, D = k.shape
    S = np.zeros((H, D, v.shape[-1]), v.dtype)
    out = np.zeros_like(v)
    for t in range(T):
        for h in range(H):
            S[h] *= g[t, h][:, None]
            u = beta[t, h] * (v[t, h] - S[h].T @ k[t, h])
            S[h] += np.outer(k[t, h], u)
            out[t, h] = S[h].T @ q[t, h]
    return out


def channel_delta(h, m, p, eps):
    """h [T, width]; m: mixer sizes; p(name): tensor of this mixer."""
    T, H, KH, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ p(n).T, p(n + ".conv"))) for n in ("q", "k", "v"))
    q = unit_heads(q.reshape(T, KH, D)) * D ** -0.5
    k = unit_heads(k.reshape(T, KH, D))
    rep = H // KH
    q, k = np.repeat(q, rep, axis=1), np.repeat(k, rep, axis=1)
    beta = sigmoid(h @ p("b").T)
    a = (h @ p("a1").T @ p("a2").T + p("dt_bias")).reshape(T, H, D)
    g = np.exp(-np.exp(p("A_log"))[None, :, None] * softplus(a))
    o = delta_recurrence(q, k, v.reshape(T, H, V), g, beta)
    gate = sigmoid(h @ p("g1").T @ p("g2").T).reshape(T, H, V)
    o = rms_unit(o, eps) * p("norm") * gate
    return o.reshape(T, H * V) @ p("o").T


def latent_attention(h, m, p, eps):
    T, H, D, R, V, C = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(T)
    q = (h @ p("q").T).reshape(T, H, D + R).transpose(1, 0, 2)
    qn, qr = q[..., :D], rotate_pairs(q[..., D:], pos, m["rot"]["base"])
    d = h @ p("dkv").T
    c = rms_unit(d[:, :C], eps) * p("dkv.norm")
    kr = rotate_pairs(d[:, C:], pos, m["rot"]["base"])
    kn = (c @ p("uk").T).reshape(T, H, D).transpose(1, 0, 2)
    v = (c @ p("uv").T).reshape(T, H, V).transpose(1, 0, 2)
    s = (qn @ kn.transpose(0, 2, 1) + qr @ kr.T) * m["scale"]
    s = np.where(np.tril(np.ones((T, T), bool)), s, -np.inf)
    w = np.exp(s - s.max(axis=-1, keepdims=True))
    w /= w.sum(axis=-1, keepdims=True)
    o = w @ v * sigmoid(h @ p("g").T).T[:, :, None]
    return o.transpose(1, 0, 2).reshape(T, H * V) @ p("o").T


def dense(h, up, down):
    return np.maximum(h @ up.T, 0.0) ** 2 @ down.T


MIXERS = {"channel_delta": channel_delta, "latent_attention": latent_attention}


def owner(layers, i):
    while layers[i].get("weights_of") is not None:
        i = layers[i]["weights_of"]
    return i


def run(cfg, t, tokens, dtype=np.float64):
    """Logits [T, vocab] and the residual stream after every layer [layers, T, width]."""
    t = {k: np.asarray(a, dtype) for k, a in t.items()}
    eps = cfg["norm"]["eps"]
    x = t["embed"][np.asarray(tokens)]
    trail = []
    for i, layer in enumerate(cfg["layers"]):
        pre = "l%d." % owner(cfg["layers"], i)
        y = MIXERS[layer["type"]](x, layer["mixer"], lambda n: t[pre + "mix." + n], eps)
        x = x + norm_about_one(y, t[pre + "norm1"], eps)
        if layer.get("mlp") is not None:
            assert layer["mlp"]["kind"] == "dense"
            x = x + norm_about_one(dense(x, t[pre + "mlp.up"], t[pre + "mlp.down"]), t[pre + "norm2"], eps)
        trail.append(x)
    return norm_about_one(x, t["final.norm"], eps) @ t["embed"].T, np.stack(trail)
