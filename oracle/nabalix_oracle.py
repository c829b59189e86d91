"""Plain restatement, in numpy, of the mechanisms of Nabalix models: one function per mechanism, token by token, no
chunking, no caches, fp64 by default.  Test infrastructure only; it shares no code with the product path.

Weights come as a dict name -> array under the checkpoint's tensor names; `cfg` is the parsed config.json.  `cast`
rounds what goes into a matrix product and what comes out of it (a model of 16-bit activations).
"""
from __future__ import annotations

import numpy as np

from .hybrid_oracle import exact, linear, rms_norm, sigmoid, silu


def distance_penalty(r1, r2, distance):
    """What a head with numbers r1, r2 takes off the score of a key `distance` tokens back."""
    return r1 * np.log(1.0 + r2 * distance)


def mixed_head_attention(q, k, v, scale, softcap, r1, r2, talk, window):
    """q (T, H, D), k (T, G, D), v (T, G, V) -> (T, H, V).  Per pair (i, j): the H capped and penalised scores become H
    mixed ones through `talk` (H, H), and each head's softmax runs over its mixed scores.  Query i sees the `window` keys
    i - window + 1 .. i."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[-1]), q.dtype)
    group = np.arange(H) // (H // G)                         # key/value head of every query head
    for i in range(T):
        j0 = max(0, i - window + 1)
        dist = np.arange(i - j0, -1, -1).astype(q.dtype)
        s = np.empty((H, i - j0 + 1), q.dtype)
        for h in range(H):
            z = k[j0:i + 1, group[h]] @ q[i, h] * scale
            s[h] = softcap * np.tanh(z / softcap) - distance_penalty(r1[h], r2[h], dist)
        s = talk @ s
        for h in range(H):
            p = np.exp(s[h] - s[h].max())
            out[i, h] = (p / p.sum()) @ v[j0:i + 1, group[h]]
    return out


def attention(h, w, p, mix, cast=exact):
    """The attention half of a parallel mixer, up to and with its output projection."""
    T, H, G, D, V = h.shape[0], mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    q = linear(h, w[p + "q"], cast).reshape(T, H, D)
    k = linear(h, w[p + "k"], cast).reshape(T, G, D)
    v = linear(h, w[p + "v"], cast).reshape(T, G, V)
    dt = h.dtype.type
    o = mixed_head_attention(q, k, v, dt(mix["scale"]), dt(mix["softcap"]), w[p + "r1"], w[p + "r2"], w[p + "talk"], mix["mask"]["size"])
    return linear(o.reshape(T, H * V) * sigmoid(linear(h, w[p + "g"], cast)), w[p + "o"], cast)


def forget_gate(z, lower):
    """f = lower + (1 - lower) sigmoid(z), and what it lets in, 1 - f = (1 - lower) sigmoid(-z)."""
    return lower + (1 - lower) * sigmoid(z), (1 - lower) * sigmoid(-z)


def forget_recurrence(q, v, f, write, state=None):
    """q, f, write (T, H, D), v (T, H, V): S <- diag(f) S + write v^T, o = S^T q; returns (o, S)."""
    T, H, D = q.shape
    S = np.zeros((H, D, v.shape[-1]), q.dtype) if state is None else state.copy()
    o = np.zeros((T, H, v.shape[-1]), q.dtype)
    for t in range(T):
        S = f[t][:, :, None] * S + write[t][:, :, None] * v[t][:, None, :]
        o[t] = (S * q[t][:, :, None]).sum(1)
    return o, S


def hgrn2(h, w, p, mix, eps, cast=exact):
    """The recurrent half of a parallel mixer, up to and with its output projection."""
    T, H, D, V = h.shape[0], mix["heads"], mix["dim"], mix["vdim"]
    q = silu(linear(h, w[p + "q"], cast)).reshape(T, H, D)
    v = linear(h, w[p + "v"], cast).reshape(T, H, V)
    f, write = forget_gate(linear(h, w[p + "f"], cast) + w[p + "f.b"], w[p + "lower"])
    o, _ = forget_recurrence(q, v, f.reshape(T, H, D), write.reshape(T, H, D))
    return linear(rms_norm(o, w[p + "norm"], eps).reshape(T, H * V), w[p + "o"], cast)


def parallel(h, w, p, mix, eps, cast=exact):
    a = attention(h, w, p + "left.", mix["left"], cast)
    b = hgrn2(h, w, p + "right.", mix["right"], eps, cast)
    return (rms_norm(a, w[p + "left.out"], eps) + rms_norm(b, w[p + "right.out"], eps)) / 2


def clamped_glu(gate, up, limit):
    g = np.minimum(gate, limit)
    return g * sigmoid(1.702 * g) * (np.clip(up, -limit, limit) + 1)


def feed_forward(h, w, p, limit, cast=exact):
    return linear(clamped_glu(linear(h, w[p + "gate"], cast), linear(h, w[p + "up"], cast), h.dtype.type(limit)), w[p + "down"], cast)


def connect(streams, w, p, sublayer):
    """One sublayer over the streams (s, T, C): it reads a weighted sum of them; every new stream is a mixture of the old
    ones plus its share of the result."""
    read, share, mix = w[p + "in"], w[p + "out"], w[p + "mix"]
    y = sublayer(np.tensordot(read, streams, 1))
    return np.tensordot(mix.T, streams, 1) + share[:, None, None] * y


def forward(cfg, w, tokens, dtype=np.float64, cast=exact):
    """(logits (T, V), sum of the streams after every layer (L, T, C)) of one sequence."""
    w = {n: np.asarray(a, dtype) for n, a in w.items()}
    eps = cfg["norm"]["eps"]
    x = np.repeat(w["embed"][np.asarray(tokens)][None], cfg["streams"], 0)
    kept = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        if layer["type"] != "parallel":
            raise ValueError(layer["type"])

        def mixer(u):
            return w[p + "ls1"] * parallel(rms_norm(u, 1 + w[p + "norm1"], eps), w, p + "mix.", layer["mixer"], eps, cast)

        def ffn(u):
            return w[p + "ls2"] * feed_forward(rms_norm(u, 1 + w[p + "norm2"], eps), w, p + "mlp.", layer["mlp"]["limit"], cast)
        x = connect(x, w, p + "hc1.", mixer)
        if layer["mlp"] is not None:
            x = connect(x, w, p + "hc2.", ffn)
        kept.append(x.sum(0))
    return cast(rms_norm(x.sum(0), 1 + w["final.norm"], eps)) @ w["head"].T, np.stack(kept)
