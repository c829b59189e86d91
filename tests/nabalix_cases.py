"""Small Nabalix configurations and random weights for the tests.  Sizes are odd on purpose: no two of a layer's sizes are
equal, several are no multiple of 8, and windows are short enough to slide many times."""
import copy

import numpy as np
import torch


def layer(left, right, ff=None, limit=1.5):
    """left: (heads, kv_heads, dim, vdim, window, scale, softcap); right: (heads, dim, vdim)."""
    H, G, D, V, window, scale, cap = left
    return {"type": "parallel", "mlp": {"kind": "dense", "ff": ff, "limit": limit} if ff else None,
            "mixer": {"left": {"heads": H, "kv_heads": G, "dim": D, "vdim": V, "mask": {"size": window}, "scale": scale, "softcap": cap},
                      "right": dict(zip(("heads", "dim", "vdim"), right))}}


def config(layers, width=72, vocab=131, eps=1e-5, streams=3):
    return {"architecture": "Nabalix", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps}, "layers": copy.deepcopy(layers)}


# name -> configuration
CASES = {
    "mixed": config([layer((6, 2, 20, 28, 7, 0.3, 9.0), (3, 12, 36), 100), layer((4, 4, 16, 24, 19, 0.2, 30.0), (5, 20, 12)),
                     layer((8, 4, 24, 12, 64, 0.25, 15.0), (2, 28, 20), 68, 0.7)]),
    # a layer without a feed-forward first, one head, odd sizes, a window of one, one wider than the sequence, one stream
    "order": config([layer((1, 1, 7, 9, 33, 0.5, 6.0), (7, 5, 11)), layer((3, 1, 10, 6, 1, 0.4, 12.0), (1, 13, 50), 37, 3.0),
                     layer((2, 2, 9, 15, 500, 0.3, 25.0), (2, 6, 7), 60, 0.4)], width=50, vocab=77, eps=1e-3, streams=1),
    # sizes that take the wide code paths: 16-byte copies, several tiles of channels and values, more heads than one register tile
    "wide": config([layer((12, 3, 64, 136, 70, 0.12, 20.0), (2, 96, 136), 264), layer((18, 6, 32, 40, 130, 0.2, 50.0), (4, 136, 40), 136, 5.0),
                    layer((5, 5, 40, 72, 64, 0.15, 10.0), (3, 64, 80))], width=264, vocab=300, streams=4),
}


def weights(cfg, seed=0, sharp=1.0):
    """Random weights under the checkpoint's names (torch, bf16), made without the product's initialiser.  sharp > 1 makes
    softmax weights peaked, so that single keys and window edges show in the logits."""
    r = np.random.default_rng(seed)
    out = {}

    def put(name, a):
        out[name] = torch.from_numpy(np.asarray(a, np.float32)).bfloat16()

    def mat(name, n, k, g=1.0):
        put(name, r.standard_normal((n, k)) * g / np.sqrt(k))

    def vec(name, n, mean, std):
        put(name, mean + std * r.standard_normal(n))
    C, V, S = cfg["width"], cfg["vocab"], cfg["streams"]
    mat("embed", V, C, np.sqrt(C))
    mat("head", V, C)
    vec("final.norm", C, 0.0, 0.2)
    for i, spec in enumerate(cfg["layers"]):
        p, a, b = f"l{i}.", spec["mixer"]["left"], spec["mixer"]["right"]
        H, G, D, VD = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
        m = p + "mix.left."
        mat(m + "q", H * D, C, sharp)
        mat(m + "k", G * D, C)
        mat(m + "v", G * VD, C)
        mat(m + "g", H * VD, C)
        mat(m + "o", C, H * VD)
        put(m + "r1", r.uniform(0.0, 1.5, H))
        put(m + "r2", r.uniform(0.05, 0.6, H))
        put(m + "talk", np.eye(H) + 0.4 * r.standard_normal((H, H)))
        H, D, VD = b["heads"], b["dim"], b["vdim"]
        m = p + "mix.right."
        mat(m + "q", H * D, C)
        mat(m + "f", H * D, C)
        vec(m + "f.b", H * D, 1.5, 1.5)
        lower = r.uniform(-0.3, 0.95, H * D)
        put(m + "lower", np.maximum(lower, 0.0))                    # some channels have no lower bound at all
        mat(m + "v", H * VD, C)
        vec(m + "norm", VD, 1.0, 0.2)
        mat(m + "o", C, H * VD)
        for side in ("left", "right"):
            vec(f"{p}mix.{side}.out", C, 1.0, 0.3)
        if spec["mlp"]:
            F = spec["mlp"]["ff"]
            for n, rows, k in (("gate", F, C), ("up", F, C), ("down", C, F)):
                mat(f"{p}mlp.{n}", rows, k, 1.5)
        for q in (1, 2) if spec["mlp"] else (1,):
            vec(f"{p}norm{q}", C, 0.0, 0.2)
            vec(f"{p}ls{q}", C, 0.6, 0.3)
            put(f"{p}hc{q}.in", r.uniform(-0.2, 1.0, S) if S > 1 else r.uniform(0.5, 1.0, 1))
            put(f"{p}hc{q}.out", r.uniform(0.5, 1.4, S))
            put(f"{p}hc{q}.mix", 0.9 * np.eye(S) + 0.25 * r.standard_normal((S, S)) if S > 1 else [[0.9]])
    return out


def as_numpy(w):
    return {k: v.float().numpy().astype(np.float64) for k, v in w.items()}


def tokens(cfg, n, seed=0):
    return np.random.default_rng(2000 + seed).integers(0, cfg["vocab"], n)
