"""Prefill and decode throughput of Nabalix layers (random weights) beside Nerulorn's at equal width, feed-forward, heads,
window and vocabulary, and every kernel of both against its roofline.  Run by `bench.py --nabalix`.

One Nabalix layer (attention and recurrence side by side, a feed-forward) stands against two Nerulorn layers (a recurrence
without a feed-forward, attention with one).  Kernel times as in bench_layered.py."""
from __future__ import annotations

import json

import torch

from . import bench_layered as BL
from . import layer_ops as L
from . import nabalix, nerulorn
from .bench_layered import SIZES, VOCAB, WINDOW, graph_us, peaks, throughput

STREAMS = 2


def config(width: int, ff: int, n_layers: int, window: int = WINDOW) -> dict:
    heads = width // 128
    mixer = {"left": {"heads": heads, "kv_heads": heads // 4, "dim": 128, "vdim": 128, "mask": {"size": window}, "scale": 128 ** -0.5,
                      "softcap": 30.0}, "right": {"heads": heads, "dim": 128, "vdim": 128}}
    return {"architecture": "Nabalix", "vocab": VOCAB, "width": width, "streams": STREAMS, "norm": {"eps": 1e-6},
            "layers": [{"type": "parallel", "mixer": mixer, "mlp": {"kind": "dense", "ff": ff, "limit": 7.0}} for _ in range(n_layers)]}


def kernels(width: int, ff: int, T: int, window: int, only: str = "") -> list[dict]:
    """Every kernel of a layer: microseconds and the fraction of its roofline (the larger of bytes over HBM bandwidth and
    FLOPs over the bf16 tensor peak); `like`: Nerulorn's kernel of the same kind."""
    dev = torch.device("cuda")
    pk = peaks()
    rows = []

    def add(name, like, fns, nbytes, flops=0.0):
        us = graph_us(fns)
        floor = max(nbytes / (pk["hbm_gbs"] * 1e3), flops / (pk["bf16_tflops"] * 1e6))
        rows.append({"kernel": name, "like": like, "us": round(us, 2), "floor_us": round(floor, 3), "frac": round(floor / us, 4)})

    def copies(nbytes):
        return min(160, max(2, int(400e6 / nbytes) + 1))
    model = nabalix.random_init(config(width, ff, 2, window), 0, torch.bfloat16, T + 64, dev)
    layer = model.layers[1]
    mix, ffn = layer.mixer, layer.ffn
    att, rec = mix.branches
    H, G, hd, C, F, S = att.heads, att.kv_heads, 128, width, ff, STREAMS
    bf, f32 = dict(dtype=torch.bfloat16, device=dev), dict(dtype=torch.float32, device=dev)
    from .layered import Span
    span = Span(1, T, 0, torch.bfloat16, dev)

    def wanted(name):
        return not only or only in name

    # ---- prompts
    for nm, n, k, dt, act in (("in", mix.n_in, C, bf, L.PLAIN), ("gate|up, clamped", 2 * F, C, bf, ffn.act), ("down", C, F, f32, L.PLAIN),
                              ("out", C, H * hd, f32, L.PLAIN)):
        if not wanted("linear"):
            continue
        cols, size = n // 2 if act.kind else n, 4 if dt is f32 else 2
        sets = [(torch.randn(T, k, **bf), torch.randn(n, k, **bf) * 0.02, torch.empty(T, cols, **dt))
                for _ in range(copies(2 * (n * k + T * k) + size * T * cols))]
        add(f"linear_bf16 {T}x{n}x{k} ({nm})", "linear_bf16", [lambda s=s: L.linear(s[0], s[1], k, n, s[2], act=act) for s in sets],
            2 * (n * k + T * k) + size * T * cols, 2.0 * T * n * k)
        del sets
    proj = [torch.randn(T, mix.n_in, **bf) for _ in range(copies(T * mix.n_in * 2))]
    caches = [att.new_cache(1, T + 64, torch.bfloat16, dev) for _ in proj]
    row = caches[0].rows.shape[2]
    if wanted("cache_append"):
        add(f"cache_append {T} rows", "latent_prepare", [lambda a=a, c=c: L.cache_append(a, att.k_off, att.kv_cols, c.rows, 1, T, 0)
                                                        for a, c in zip(proj, caches)], T * row * 4.0)
    seen = sum(min(i + 1, window) for i in range(T))
    if wanted("talk_attention"):
        outs = torch.empty(T, H * hd, **bf)
        for a, c in zip(proj, caches):
            L.cache_append(a, att.k_off, att.kv_cols, c.rows, 1, T, 0)
        add(f"talk_attention {T} tokens, {H} heads, window {window} (scores, values)", "latent_attention",
            [lambda a=a, c=c: L.talk_attention(dev, q=L._ptr(a, att.q_off), gate=L._ptr(a, att.g_off), out=outs.data_ptr(), dtype=2, B=1, T=T,
                                               ldq=a.stride(0), ldg=a.stride(0), ldo=outs.stride(0), pos0=0, **att._sizes(c))
             for a, c in zip(proj, caches)], T * (row + 3 * H * hd) * 2.0, 2.0 * seen * H * (2 * hd))
    if wanted("gla_prefill"):
        st = rec.new_cache(1, 0, torch.bfloat16, dev)
        o = torch.empty(T, H * hd, **bf)
        ws = torch.empty(L.gla_workspace_bytes(1, T, H, hd, hd), dtype=torch.uint8, device=dev)
        fl = 2.0 * T * H * (2 * hd * hd + 64 * hd / 2 + 64 * hd / 2)
        add(f"gla_prefill, forget gate, {T} tokens, {H} heads", "gla_prefill",
            [lambda a=a: L.gla_prefill(ws, **rec._args(a, a.stride(0), o, o.stride(0), st, torch.bfloat16, 1, T)) for a in proj],
            T * 4 * H * hd * 2.0, fl)
    del proj, caches
    coef, w = model.coefs[1], torch.ones(C, device=dev)
    for nb, post_norm in ((2, L.NORM_RMS), (1, None)):
        if not wanted("stream_norm"):
            continue
        nbytes = T * C * (8.0 * S + 4 * nb + 2)
        sets = [(torch.randn(T, S, C, device=dev), [torch.randn(T, C, device=dev) for _ in range(nb)], torch.empty(T, C, **bf))
                for _ in range(copies(nbytes))]
        add(f"stream_norm {T}x{S}x{C}, {nb} result{'s' if nb > 1 else ''}", "residual_norm",
            [lambda s=s: L.stream_norm(s[0], s[1], [w] * nb, post_norm, coef, L.NORM_RMS, 1e-6, w, s[2]) for s in sets], nbytes)
        del sets

    # ---- decode
    for nm, n, k, act, nb in (("in", mix.n_in, C, L.PLAIN, 1), ("gate|up, clamped", 2 * F, C, ffn.act, 2), ("head", VOCAB, C, L.PLAIN, 1)):
        if not wanted("matvec_streams"):
            continue
        ws = [torch.randn(n, k, **bf) * 0.02 for _ in range(copies(2 * n * k))]
        x, x2 = torch.randn(S, C, device=dev), torch.empty(S, C, device=dev)
        ys, y = [torch.randn(C, device=dev) for _ in range(nb)], torch.empty(n, device=dev)
        add(f"matvec_streams {n}x{k} ({nm})", "matvec_bf16",
            [lambda m=m: L.matvec_streams(m, n, k, y, x, x2, ys, [w] * nb, L.NORM_RMS if nb == 2 else None, coef, L.NORM_RMS, 1e-6, w, act=act)
             for m in ws], 2.0 * n * k + 4 * (n + (2 * S + nb) * C))
        del ws
    if wanted("matvec_pair"):
        ws = [(torch.randn(C, H * hd, **bf), torch.randn(C, H * hd, **bf)) for _ in range(copies(4 * C * H * hd))]
        x, ya, yb = torch.randn(H * hd, device=dev), torch.empty(C, device=dev), torch.empty(C, device=dev)
        add(f"matvec_pair 2x{C}x{H * hd} (out)", "matvec_bf16", [lambda m=m: L.matvec_pair((m[0], C, H * hd, x, ya), (m[1], C, H * hd, x, yb)) for m in ws],
            4.0 * C * H * hd + 8 * (C + H * hd))
        del ws
    if wanted("matvec_bf16"):
        ws = [torch.randn(C, F, **bf) * 0.02 for _ in range(copies(2 * C * F))]
        x, y = torch.randn(F, device=dev), torch.empty(C, device=dev)
        add(f"matvec_bf16 {C}x{F} (down)", "matvec_bf16", [lambda m=m: L.matvec(m, C, F, x, y) for m in ws], 2.0 * C * F + 4 * (C + F))
        del ws
    p, o = torch.randn(mix.n_in, device=dev), torch.empty(H * hd, device=dev)
    pos = torch.full((1,), T, dtype=torch.long, device=dev)
    keys = min(window, T + 1)
    if wanted("talk_decode"):
        cs = [att.new_cache(1, T + 64, torch.bfloat16, dev) for _ in range(copies(keys * row * 2))]
        for c in cs:
            c.rows.normal_()
        add(f"talk_decode {H} heads, {keys} keys", "latent_decode",
            [lambda c=c: L.talk_decode(p=p.data_ptr(), pos=pos.data_ptr(), out=o.data_ptr(), cache_dtype=2, B=1, ldp=p.numel(), q_off=att.q_off,
                                       k_off=att.k_off, g_off=att.g_off, ldo=o.numel(), **att._sizes(c)) for c in cs], keys * row * 2.0)
        del cs
    if wanted("gla_decode"):
        sts = [rec.new_cache(1, 0, torch.bfloat16, dev) for _ in range(copies(H * hd * hd * 4))]
        add(f"gla_decode, forget gate, {H} heads", "gla_decode",
            [lambda s=s: L.gla_decode(**rec._args(p, p.numel(), o, o.numel(), s, torch.float32, 1, 1)) for s in sts], H * hd * hd * 8.0)
    return rows


def run(args) -> None:
    dev = torch.device("cuda", 0)
    torch.cuda.set_device(dev)
    from bench import ClockSampler
    sampler = ClockSampler(0)
    sampler.start()
    line = {"nabalix": {}, "peaks": peaks()}
    if args.nabalix_only:                    # one kernel's rows (tuning, profiles)
        width, ff, _ = SIZES[args.layered_sizes.split(",")[-1]]
        print(json.dumps({"kernels": kernels(width, ff, 2048, WINDOW, args.nabalix_only), "clocks": sampler.stop()}))
        return
    for name in args.layered_sizes.split(","):
        width, ff, n = SIZES[name]
        ctx = max(args.layered_prompts) + 256
        res = {"window": WINDOW}
        for family, module, cfg in (("nabalix", nabalix, config(width, ff, n // 2)), ("nerulorn", nerulorn, BL.config(width, ff, n))):
            model = module.random_init(cfg, 0, torch.bfloat16, ctx, dev)
            res[family] = {"layers": len(cfg["layers"]), **throughput(model, args.layered_prompts, 64)}
            del model
            torch.cuda.empty_cache()
        line["nabalix"][name] = res
    if not args.no_layered_kernels:
        width, ff, _ = SIZES[args.layered_sizes.split(",")[-1]]
        line["kernels"] = kernels(width, ff, 2048, WINDOW)
        line["nerulorn_kernels"] = [r for r in BL.kernels(width, ff, 2048, WINDOW) if r["like"] != "itself"]
    line["clocks"] = sampler.stop()
    print(json.dumps(line))
