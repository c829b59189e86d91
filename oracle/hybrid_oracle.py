"""Plain restatement, in numpy, of the mechanisms of the layered decoders (Nerulorn): one function per
mechanism, token by token, no chunking, no caches, fp64 by default.  Test infrastructure only; it shares
no code with the product path.

Weights come as a dict name -> array under the checkpoint's tensor names; `cfg` is the parsed config.json.
"""
from __future__ import annotations

import math

import numpy as np


def sigmoid(z):
    z = np.asarray(z)
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0 / (1.0 + e), e / (1.0 + e))


def silu(z):
    return z * sigmoid(z)


def layer_norm(x, w, eps):
    """(x - mean) / sqrt(var + eps) * w over the last axis; var is the mean of the squared deviations."""
    d = x - x.mean(-1, keepdims=True)
    return d / np.sqrt((d * d).mean(-1, keepdims=True) + eps) * w


def rms_norm(x, w, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


def rope_frequencies(dims, base, scaling=None):
    """(frequencies of the dims/2 pairs, factor on cos and sin); scaling: YaRN parameters or None."""
    f = np.array([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)])
    if not scaling:
        return f, 1.0

    def turns_dim(t):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))
    lo = max(math.floor(turns_dim(scaling["fast"])), 0)
    hi = min(math.ceil(turns_dim(scaling["slow"])), dims - 1)
    out = np.empty_like(f)
    for i in range(dims // 2):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out[i] = f[i] / scaling["factor"] * ramp + f[i] * (1.0 - ramp)
    return out, 0.1 * math.log(scaling["factor"]) + 1.0


def rotate(x, positions, rot):
    """x (T, ..., D): the first rot['dims'] entries of the last axis, as pairs (2i, 2i + 1), are turned by
    position * frequency_i."""
    f, m = rope_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    y = x.copy()
    for i in range(rot["dims"] // 2):
        a = positions * f[i]
        c, s = np.cos(a) * m, np.sin(a) * m
        shape = (len(positions),) + (1,) * (x.ndim - 2)
        c, s = c.reshape(shape), s.reshape(shape)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i] = u * c - v * s
        y[..., 2 * i + 1] = v * c + u * s
    return y


def windowed_attention(q, k, v, scale, window):
    """q, k (T, H, D), v (T, H, V): query i attends to keys j with 0 <= i - j < window (window None: all)."""
    T, H, _ = q.shape
    out = np.zeros((T, H, v.shape[-1]), q.dtype)
    for i in range(T):
        j0 = 0 if window is None else max(0, i - window + 1)
        for h in range(H):
            s = k[j0:i + 1, h] @ q[i, h] * scale
            p = np.exp(s - s.max())
            out[i, h] = (p / p.sum()) @ v[j0:i + 1, h]
    return out


def exact(x):
    return x


def linear(x, weight, cast=exact):
    """W x; `cast` rounds what goes into the product and what comes out of it (a model of 16-bit activations)."""
    return cast(cast(x) @ weight.T)


def latent_attention(h, w, p, mix, eps, shared=None, cast=exact):
    """h (T, C) -> (output (T, C), (latents, rotated key part)).  `shared`: the pair of another layer."""
    T = h.shape[0]
    H, dim, rd, vd, rank = mix["heads"], mix["dim"], mix["rot_dim"], mix["vdim"], mix["kv_rank"]
    pos = np.arange(T)
    cq = rms_norm(linear(h, w[p + "dq"], cast), w[p + "dq.norm"], eps)
    q = linear(cq, w[p + "uq"], cast).reshape(T, H, dim + rd)
    if shared is None:
        kv = linear(h, w[p + "dkv"], cast)
        c = cast(rms_norm(kv[:, :rank], w[p + "dkv.norm"], eps))
        kr = cast(rotate(kv[:, rank:], pos, mix["rot"]))
    else:
        c, kr = shared
    qr = cast(rotate(q[..., dim:], pos, mix["rot"]))
    k = linear(c, w[p + "uk"], cast).reshape(T, H, dim)
    v = linear(c, w[p + "uv"], cast).reshape(T, H, vd)
    qq = np.concatenate([q[..., :dim], qr], -1)
    kk = np.concatenate([k, np.repeat(kr[:, None, :], H, 1)], -1)
    o = windowed_attention(qq, kk, v, mix["scale"], mix["mask"]["size"])
    o = o * sigmoid(linear(h, w[p + "g"], cast))[..., None]
    return linear(o.reshape(T, H * vd), w[p + "o"], cast), (c, kr)


def gla_recurrence(q, k, v, alpha, state=None):
    """q, k, alpha (T, H, D), v (T, H, V): S <- diag(alpha) S + k v^T, o = S^T q; returns (o, S)."""
    T, H, D = q.shape
    S = np.zeros((H, D, v.shape[-1]), q.dtype) if state is None else state.copy()
    o = np.zeros((T, H, v.shape[-1]), q.dtype)
    for t in range(T):
        for h in range(H):
            S[h] = alpha[t, h][:, None] * S[h] + np.outer(k[t, h], v[t, h])
            o[t, h] = S[h].T @ q[t, h]
    return o, S


def gla(h, w, p, mix, eps, cast=exact):
    T = h.shape[0]
    H, D, V = mix["heads"], mix["dim"], mix["vdim"]
    q = linear(h, w[p + "q"], cast).reshape(T, H, D) * D ** -0.5
    k = linear(h, w[p + "k"], cast).reshape(T, H, D)
    v = linear(h, w[p + "v"], cast).reshape(T, H, V)
    z = linear(h, w[p + "a1"], cast) @ w[p + "a2"].T + w[p + "a2.b"]
    alpha = (sigmoid(z) ** (1.0 / mix["tau"])).reshape(T, H, D)
    o, _ = gla_recurrence(q, k, v, alpha)
    o = rms_norm(o, w[p + "norm"], eps).reshape(T, H * V)
    return linear(o * silu(linear(h, w[p + "g"], cast)), w[p + "o"], cast)


def dense_ffn(h, w, p, cast=exact):
    a = silu(linear(h, w[p + "gate"], cast) + w[p + "gate.b"]) * (linear(h, w[p + "up"], cast) + w[p + "up.b"])
    return linear(a, w[p + "down"], cast) + w[p + "down.b"]


def forward(cfg, w, tokens, dtype=np.float64, cast=exact):
    """(logits (T, V), residual stream after every layer (L, T, C)) of one sequence."""
    w = {n: np.asarray(a, dtype) for n, a in w.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    kept, stream = {}, []
    for i, layer in enumerate(cfg["layers"]):
        p, mix = f"l{i}.", layer["mixer"]
        h = layer_norm(x, w[p + "norm1"], eps)
        if layer["type"] == "gla":
            y = gla(h, w, p + "mix.", mix, eps, cast)
        elif layer["type"] == "latent_attention":
            src = mix.get("kv_from")
            y, kv = latent_attention(h, w, p + "mix.", mix, eps, None if src is None else kept[src], cast)
            kept[i] = kv
        else:
            raise ValueError(layer["type"])
        x = x + layer_norm(y, w[p + "norm1b"], eps)
        if layer["mlp"] is not None:
            y = dense_ffn(layer_norm(x, w[p + "norm2"], eps), w, p + "mlp.", cast)
            x = x + layer_norm(y, w[p + "norm2b"], eps)
        stream.append(x)
    return cast(layer_norm(x, w["final.norm"], eps)) @ w["head"].T, np.stack(stream)
