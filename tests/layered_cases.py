"""Small configurations and random weights for the layered-decoder tests.  Sizes are odd on purpose: no two of a layer's
sizes are equal, several are no multiple of 8, and windows are short enough to slide many times."""
import copy

import numpy as np
import torch

YARN = {"factor": 6.0, "original": 64, "fast": 4.0, "slow": 0.5}


def gla(heads=3, dim=20, vdim=28, tau=4.0):
    return {"type": "gla", "mlp": None, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}}


def latent(heads=3, dim=20, rot=12, vdim=28, rank=36, q_rank=44, window=7, ff=100, yarn=True, kv_from=None, base=300.0, scale=0.3):
    r = {"dims": rot, "base": base}
    if yarn:
        r["scaling"] = dict(YARN)
    mix = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank, "mask": {"size": window},
           "rot": r, "scale": scale}
    if kv_from is not None:
        mix["kv_from"] = kv_from
    return {"type": "latent_attention", "mlp": {"kind": "dense", "ff": ff} if ff else None, "mixer": mix}


def config(layers, width=72, vocab=131, eps=1e-5, scale=1.7):
    return {"architecture": "Nerulorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "layers": copy.deepcopy(layers)}


# name -> configuration
CASES = {
    "mixed": config([gla(), latent(), gla(heads=2, dim=12, vdim=36, tau=1.0), latent(heads=5, dim=16, vdim=20, q_rank=30, window=19, kv_from=1), gla()]),
    # attention first and last, a feed-forward behind a recurrent layer, none behind an attention layer, one head, no scaling
    "order": config([latent(heads=1, dim=40, rot=4, vdim=9, rank=17, q_rank=13, window=33, ff=0, yarn=False),
                     dict(gla(heads=7, dim=5, vdim=11, tau=16.0), mlp={"kind": "dense", "ff": 37}),
                     latent(heads=2, dim=6, rot=4, vdim=50, rank=17, q_rank=70, window=1, ff=60, yarn=False, kv_from=0),
                     latent(heads=4, dim=24, rot=8, vdim=16, rank=48, q_rank=24, window=200)], width=50, vocab=77, eps=1e-3, scale=0.6),
    # sizes that take the wide code paths: 16-byte copies, several tiles of channels and values
    "wide": config([gla(heads=2, dim=96, vdim=136), latent(heads=2, dim=128, rot=32, vdim=136, rank=136, q_rank=160, window=70, ff=264),
                    latent(heads=3, dim=64, rot=32, vdim=72, rank=136, q_rank=88, window=130, ff=0, kv_from=1), gla(heads=4, dim=136, vdim=40, tau=2.0)],
                   width=264, vocab=300),
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
    C, V = cfg["width"], cfg["vocab"]
    mat("embed", V, C, np.sqrt(C))
    mat("head", V, C)
    vec("final.norm", C, 1.0, 0.2)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        H, D, VD = m["heads"], m["dim"], m["vdim"]
        for n in ["norm1", "norm1b"] + (["norm2", "norm2b"] if layer["mlp"] else []):
            vec(p + n, C, 1.0, 0.2)
        if layer["type"] == "gla":
            ra = 6 + i
            for n, rows in (("q", H * D), ("k", H * D), ("v", H * VD), ("g", H * VD), ("a1", ra)):
                mat(p + "mix." + n, rows, C)
            mat(p + "mix.a2", H * D, ra, 2.0)
            vec(p + "mix.a2.b", H * D, 1.0, 1.5)
            vec(p + "mix.norm", VD, 1.0, 0.2)
        else:
            R, Q, rd = m["kv_rank"], m["q_rank"], m["rot_dim"]
            mat(p + "mix.dq", Q, C)
            vec(p + "mix.dq.norm", Q, sharp, 0.2)
            mat(p + "mix.uq", H * (D + rd), Q)
            mat(p + "mix.uk", H * D, R)
            mat(p + "mix.uv", H * VD, R)
            mat(p + "mix.g", H, C)
            if m.get("kv_from") is None:
                mat(p + "mix.dkv", R + rd, C)
                vec(p + "mix.dkv.norm", R, 1.0, 0.2)
        mat(p + "mix.o", C, H * VD)
        if layer["mlp"]:
            F = layer["mlp"]["ff"]
            for n, rows, k in (("gate", F, C), ("up", F, C), ("down", C, F)):
                mat(p + "mlp." + n, rows, k)
                vec(p + "mlp." + n + ".b", rows, 0.0, 0.3)
    return out


def as_numpy(w):
    return {k: v.float().numpy().astype(np.float64) for k, v in w.items()}


def tokens(cfg, n, seed=0):
    return np.random.default_rng(1000 + seed).integers(0, cfg["vocab"], n)
