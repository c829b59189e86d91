"""Prefill and decode throughput of the layered decoder (Nerulorn layers, random weights) beside the packed decoder at
equal width, feed-forward and vocabulary, and every kernel of both against its roofline.  Run by `bench.py --layered`.

Two layers of the layered model (gated linear attention without a feed-forward, latent attention with one) stand against
one block of the packed model, so both have the same number of feed-forwards.  Kernel times: CUDA events around a CUDA graph
of many launches over distinct weights, caches or activations that together exceed the 126 MB L2."""
from __future__ import annotations

import json
import os

import torch

from . import generate as G
from . import layer_ops as L
from . import nerulorn, ops, synthetic
from .packed_linear import PackedLinear

SIZES = {"1024": (1024, 2816, 8), "2048": (2048, 5632, 8), "2560": (2560, 6912, 12)}   # width: (width, ff, layers)
VOCAB, WINDOW = 32000, 1024


def config(width: int, ff: int, n_layers: int, window: int = WINDOW) -> dict:
    heads = width // 128
    rot = {"dims": 64, "base": 500000.0, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}
    layers = []
    for i in range(n_layers):
        if i % 2 == 0:
            layers.append({"type": "gla", "mlp": None, "mixer": {"heads": heads, "dim": 128, "vdim": 128, "tau": 16.0}})
        else:
            mix = {"heads": heads, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "q_rank": width * 3 // 8,
                   "mask": {"size": window}, "rot": rot, "scale": 192 ** -0.5}
            if i % 4 == 3:
                mix["kv_from"] = i - 2
            layers.append({"type": "latent_attention", "mlp": {"kind": "dense", "ff": ff}, "mixer": mix})
    return {"architecture": "Nerulorn", "vocab": VOCAB, "width": width, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0}, "layers": layers}


def event_ms(fn, reps: int) -> float:
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    a.record()
    for _ in range(reps):
        fn()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / reps


def graph_us(fns: list, reps: int = 10) -> float:
    """Mean microseconds of one of `fns`, captured one after another in a CUDA graph."""
    st = torch.cuda.Stream()
    st.wait_stream(torch.cuda.current_stream())
    with torch.cuda.stream(st):
        for f in fns[:2]:
            f()
        st.synchronize()
        g = torch.cuda.CUDAGraph()
        with torch.cuda.graph(g, stream=st):
            for f in fns:
                f()
    torch.cuda.current_stream().wait_stream(st)
    for _ in range(3):
        g.replay()
    return event_ms(g.replay, reps) / len(fns) * 1e3


def throughput(model, prompts, n_decode: int) -> dict:
    out = {}
    dev = model.embedding.device
    sess = model.session(1)
    for T in prompts:
        p = torch.randint(0, VOCAB, (1, T), device=dev)
        for _ in range(3):
            sess.prefill(p)
        ms = event_ms(lambda: sess.prefill(p), 5)
        for _ in range(3):
            sess.step()
        d = event_ms(sess.step, n_decode)
        out[f"T{T}"] = {"prefill_ms": round(ms, 3), "prefill_tok_s": round(T / ms * 1e3), "decode_ms_per_token": round(d, 4),
                        "decode_tok_s": round(1e3 / d, 1)}
    sess.check()
    del sess
    torch.cuda.empty_cache()
    return out


def peaks() -> dict:
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "MEASURED_PEAKS.json")
    if os.path.exists(path):
        d = json.load(open(path))
        return {"hbm_gbs": d["hbm_gbs"], "bf16_tflops": d["bf16_tflops"], "source": "measured"}
    return {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}


def kernels(width: int, ff: int, T: int, window: int) -> list[dict]:
    """Every kernel of both models at one size: microseconds and the fraction of its roofline (the larger of bytes over
    HBM bandwidth and FLOPs over the bf16 tensor peak)."""
    dev = torch.device("cuda")
    pk = peaks()
    rows = []

    def add(name, like, us, nbytes, flops=0.0):
        floor = max(nbytes / (pk["hbm_gbs"] * 1e3), flops / (pk["bf16_tflops"] * 1e6))
        rows.append({"kernel": name, "like": like, "us": round(us, 2), "floor_us": round(floor, 3), "frac": round(floor / us, 4)})
    cfg = config(width, ff, 4, window)
    model = nerulorn.random_init(cfg, 0, torch.bfloat16, T + 64, dev)
    gla, att, ffn = model.layers[0].mixer, model.layers[1].mixer, model.layers[1].ffn
    H, hd, C, F = width // 128, 128, width, ff
    bf = dict(dtype=torch.bfloat16, device=dev)
    from .layered import LatentCache, RecurrentState, Span
    span = Span(1, T, 0, torch.bfloat16, dev)
    tabs = model.tables(att)

    # ---- prompts: matrix products
    for nm, n, k in (("gla in", gla.n_in, C), ("latent in", att.n_in, C), ("gate|up", 2 * F, C), ("down", C, F)):
        copies = max(2, int(400e6 / (2 * (n * k + T * k + T * n))) + 1)
        xs = [torch.randn(T, k, **bf) for _ in range(copies)]
        ws = [torch.randn(n, k, **bf) * 0.02 for _ in range(copies)]
        ys = [torch.empty(T, n, **bf) for _ in range(copies)]
        us = graph_us([lambda x=x, w=w, y=y: L.linear(x, w, k, n, y) for x, w, y in zip(xs, ws, ys)])
        add(f"linear_bf16 {T}x{n}x{k} ({nm})", "packed prompt linear", us, 2 * (n * k + T * k + T * n), 2.0 * T * n * k)
        del xs, ws, ys
    for nm, n, k in (("gate_up", 2 * F, C), ("down", C, F)):
        p2, c2 = synthetic.synthetic_packed(n, k, 3, seed=1, device=dev)
        lin = PackedLinear(p2, c2, n, k, bits=3)
        x = torch.randn(T, k, dtype=torch.float32, device=dev)
        us = graph_us([lambda: lin(x)] * 4)
        add(f"packed prompt linear {T}x{n}x{k} ({nm}, fp32 rows)", "itself", us, n * k * 0.5 + 4 * T * (k + n), 2.0 * T * n * k)
        del lin, p2, c2, x

    # ---- prompts: mixers
    copies = max(2, int(300e6 / (T * H * 192 * 2 * 3)) + 1)
    sets = []
    for _ in range(copies):
        cache = LatentCache(1, T + 64, 576, torch.bfloat16, dev)
        cache.rows.normal_()
        sets.append((torch.randn(T, H * 192, **bf), torch.randn(T, att.n_kv, **bf), cache, torch.empty(T, H * 128, **bf), torch.randn(T, att.n_in, **bf)))

    def run_att(s):
        q, kv, cache, o, a = s
        L.latent_attention(q=q.data_ptr(), kv=kv.data_ptr(), gate=L._ptr(a, att.g_off), out=o.data_ptr(), dtype=2, B=1, T=T, ldq=q.stride(0),
                           ldkv=kv.stride(0), v_off=att.v_off, kv_rows=T, kv_pos0=0, ldg=a.stride(0), ldo=o.stride(0), pos0=0,
                           **att._sizes(cache, tabs))
    seen = sum(min(i + 1, window) for i in range(T))
    us = graph_us([lambda s=s: run_att(s) for s in sets])
    add(f"latent_attention {T} tokens, {H} heads, window {window}", "prefill_attention", us, T * H * (192 + 256 + 128) * 2, 2.0 * seen * H * (192 + 128))
    cqs = torch.empty(T, att.q_rank, **bf)

    def run_prep(s):
        L.latent_prepare(a=s[4].data_ptr(), cq=cqs.data_ptr(), cache=s[2].rows.data_ptr(), q_norm=att.q_norm.data_ptr(),
                         kv_norm=att.kv_norm.data_ptr(), cos2=tabs[0].data_ptr(), sin2=tabs[1].data_ptr(), eps=1e-6, dtype=2, B=1, T=T,
                         lda=s[4].stride(0), q_off=att.q_off, q_rank=att.q_rank, ldcq=att.q_rank, kv_off=att.kv_off, rank=512, rot=64,
                         ctx=T + 64, ldc=s[2].rows.shape[2], pos0=0)
    us = graph_us([lambda s=s: run_prep(s) for s in sets])
    add(f"latent_prepare {T} rows", "add_rmsnorm", us, T * 2.0 * (att.q_rank + 576) * 2)
    del sets
    ps = [torch.randn(T, gla.n_in, **bf) for _ in range(max(2, int(300e6 / (T * gla.n_in * 2)) + 1))]
    o, st = torch.empty(T, H * hd, **bf), RecurrentState(1, H, hd, hd, dev)
    ws = torch.empty(L.gla_workspace_bytes(1, T, H, hd, hd), dtype=torch.uint8, device=dev)
    us = graph_us([lambda p=p: L.gla_prefill(ws, **gla._args(p, p.stride(0), o, o.stride(0), st, torch.bfloat16, 1, T)) for p in ps])
    # per chunk of 64 tokens and head: the two products with the state, the scores and their product with the values
    fl = 2.0 * T * H * (2 * hd * hd + 64 * hd / 2 + 64 * hd / 2)
    add(f"gla_prefill {T} tokens, {H} heads (5 launches)", "prefill_attention", us, T * gla.n_in * 2 + T * H * hd * 2, fl)
    del ps, ws
    cs = torch.randn(T + 64, hd, device=dev)
    qkv = [torch.randn(T, 3 * C, device=dev) for _ in range(max(2, int(300e6 / (T * 12 * C)) + 1))]
    kc, vc = torch.zeros(1, H, T + 64, hd, device=dev), torch.zeros(1, H, T + 64, hd, device=dev)
    oo = torch.empty(T, C, device=dev)
    us = graph_us([lambda x=x: ops.prefill_attention(x, T, cs, cs, 0, kc, vc, oo, 0) for x in qkv], 3)
    add(f"prefill_attention {T} tokens, {H} heads (fp32, all keys)", "itself", us, T * C * 4 * 6, 2.0 * T * (T + 1) / 2 * H * 2 * hd)
    del qkv

    # ---- prompts: norms
    n = max(2, int(300e6 / (T * C * 10)) + 1)
    xs = [(torch.randn(T, C, device=dev), torch.randn(T, C, device=dev), torch.empty(T, C, **bf), torch.empty(T, C, device=dev)) for _ in range(n)]
    w = torch.ones(C, device=dev)
    us = graph_us([lambda s=s: L.residual_norm(s[0], s[1], w, w, L.NORM_LAYER, 1e-6, s[2]) for s in xs])
    add(f"residual_norm {T}x{C}", "add_rmsnorm", us, T * C * 14.0)
    us = graph_us([lambda s=s: ops.add_rmsnorm(s[0], s[1], w, 1e-6, s[3]) for s in xs])
    add(f"add_rmsnorm {T}x{C}", "itself", us, T * C * 16.0)
    few = int(T * (att.q_rank + 576) * 4 / (C * 16))             # as many bytes as latent_prepare moves
    us = graph_us([lambda s=s: ops.add_rmsnorm(s[0][:few], s[1][:few], w, 1e-6, s[3][:few]) for s in xs])
    add(f"add_rmsnorm {few}x{C}", "itself", us, few * C * 16.0)
    del xs

    # ---- decode: matvecs
    for nm, n, k, kw in (("gla in", gla.n_in, C, "chain"), ("uq", att.n_q, att.q_rank, "rms"), ("out", C, H * 128, None), ("gate|up", 2 * F, C, "ffn"),
                         ("down", C, F, None), ("head", VOCAB, C, "chain")):
        copies = max(2, int(400e6 / (2 * n * k)) + 1)
        ws = [torch.randn(n, k, **bf) * 0.02 for _ in range(copies)]
        x, d, x2, wn = (torch.randn(k, device=dev) for _ in range(4))
        y, bias = torch.empty(n, device=dev), torch.zeros(n, device=dev)
        opt = dict(norm=L.NORM_LAYER, eps=1e-6, norm_w=wn, delta=d, delta_w=wn, x_out=x2) if kw in ("chain", "ffn") else \
            dict(norm=L.NORM_RMS, eps=1e-6, norm_w=wn) if kw == "rms" else {}
        if kw == "ffn":
            opt.update(bias=bias, act=L.SWIGLU)
        us = graph_us([lambda w=w: L.matvec(w, n, k, x, y, **opt) for w in ws])
        add(f"matvec_bf16 {n}x{k} ({nm})", "lm_head" if nm == "head" else "gemv_stream", us, 2.0 * n * k + 4 * (n + k))
        del ws
    for nm, n, k, pro in (("qkv", 3 * C, C, ops.PRO_ADD_RMSNORM), ("out_proj", C, C, ops.PRO_NONE), ("gate_up", 2 * F, C, ops.PRO_ADD_RMSNORM),
                          ("down", C, F, ops.PRO_NONE)):
        copies = max(2, int(300e6 / (0.625 * n * k)) + 1)
        p2, c2 = synthetic.synthetic_packed(n, k, 3, seed=1, device=dev)
        w0 = PackedLinear(p2, c2, n, k, bits=3).stream_weight()
        ws = [w0.clone() for _ in range(copies)]
        x, d, x2, wn = (torch.randn(k, device=dev) for _ in range(4))
        y = torch.empty(n, device=dev)
        opt = dict(delta=d, norm_weight=wn, eps=1e-6, x_out=x2) if pro == ops.PRO_ADD_RMSNORM else {}
        us = graph_us([lambda w=w: ops.gemv_stream(pro, x, w, 3, n, k, y, **opt) for w in ws])
        add(f"gemv_stream {n}x{k} ({nm}, 3-bit)", "itself", us, 0.5 * n * k + 4 * (n + k))
        del ws, w0
    table = [torch.randn(VOCAB, C, **bf) for _ in range(4)]
    if ops.lm_head_supported(table[0]):
        x, d, wn = (torch.randn(C, device=dev) for _ in range(3))
        lg, tok, pos = torch.empty(1, VOCAB, device=dev), torch.zeros(1, 1, dtype=torch.long, device=dev), torch.zeros(1, dtype=torch.long, device=dev)
        us = graph_us([lambda t=t: ops.lm_head(x.view(1, -1), d.view(1, -1), wn, 1e-6, t, 30.0, lg, tok, pos) for t in table])
        add(f"lm_head {VOCAB}x{C} (two launches)", "itself", us, 2.0 * VOCAB * C)
    del table

    # ---- decode: mixers, at position T with cold caches
    pos = torch.full((1,), T, dtype=torch.long, device=dev)
    n = max(2, int(300e6 / (min(window, T) * 576 * 2)) + 1)
    layers = [(LatentCache(1, T + 64, 576, torch.bfloat16, dev), att.w_ukv.clone()) for _ in range(min(n, 160))]
    a, q, o = torch.randn(att.n_in, device=dev), torch.randn(att.n_q, device=dev), torch.empty(H * 128, device=dev)

    def run_ld(s):
        cache, ukv = s
        L.latent_decode(q=q.data_ptr(), a=a.data_ptr(), uk=ukv.data_ptr(), uv=L._ptr(ukv, att.v_off * ukv.stride(0)),
                        kv_norm=att.kv_norm.data_ptr(), pos=pos.data_ptr(), out=o.data_ptr(), eps=1e-6, cache_dtype=2, B=1, ldq=q.numel(),
                        lda=a.numel(), kv_off=att.kv_off, g_off=att.g_off, ldu=ukv.stride(0), ldo=o.numel(), **att._sizes(cache, tabs))
    us = graph_us([lambda s=s: run_ld(s) for s in layers])
    keys = min(window, T + 1)
    add(f"latent_decode {H} heads, {keys} keys", "decode_attention_rope", us, keys * 576 * 2.0 + 2.0 * att.n_kv * 512)
    del layers
    sts = [RecurrentState(1, H, hd, hd, dev) for _ in range(int(300e6 / (H * hd * hd * 4)) + 1)]
    p, o = torch.randn(gla.n_in, device=dev), torch.empty(H * hd, device=dev)
    us = graph_us([lambda s=s: L.gla_decode(**gla._args(p, p.numel(), o, o.numel(), s, torch.float32, 1, 1)) for s in sts])
    add(f"gla_decode {H} heads", "decode_attention_rope", us, H * hd * hd * 8.0)
    del sts
    kvs = [(torch.zeros(1, H, T + 64, hd, device=dev), torch.zeros(1, H, T + 64, hd, device=dev)) for _ in range(max(2, int(300e6 / (T * C * 8)) + 1))]
    qkv1, o1 = torch.randn(1, 3 * C, device=dev), torch.empty(1, C, device=dev)
    us = graph_us([lambda s=s: ops.decode_attention_rope(qkv1, cs, cs, pos, s[0], s[1], o1, 0) for s in kvs])
    add(f"decode_attention_rope {H} heads, {T + 1} keys", "itself", us, (T + 1) * C * 8.0)
    # the same kernel over as many bytes as the two mixers above move
    for keys in (int((min(window, T + 1) * 576 * 2.0 + 2.0 * att.n_kv * 512) / (C * 8)), int(H * hd * hd / C)):
        few = torch.full((1,), keys - 1, dtype=torch.long, device=dev)
        us = graph_us([lambda s=s: ops.decode_attention_rope(qkv1, cs, cs, few, s[0], s[1], o1, 0) for s in kvs])
        add(f"decode_attention_rope {H} heads, {keys} keys", "itself", us, keys * C * 8.0)
    return rows


def run(args) -> None:
    dev = torch.device("cuda", 0)
    torch.cuda.set_device(dev)
    from bench import ClockSampler
    sampler = ClockSampler(0)
    sampler.start()
    line = {"layered": {}, "peaks": peaks()}
    for name in args.layered_sizes.split(","):
        width, ff, n = SIZES[name]
        ctx = max(args.layered_prompts) + 256
        model = nerulorn.random_init(config(width, ff, n), 0, torch.bfloat16, ctx, dev)
        res = {"layers": n, "window": WINDOW, "parameters": sum(t.numel() for t in _tensors(model)), "layered": throughput(model, args.layered_prompts, 64)}
        del model
        torch.cuda.empty_cache()
        cfg = G.ModelConfig(vocab_size=VOCAB, n_layers=n // 2, n_embd=width, n_head=width // 128, ffn_hidden=ff, context_len=ctx)
        packed = G.PackedGPT.random_init(cfg, seed=0, device=dev)
        res["packed"] = throughput(packed, args.layered_prompts, 64)
        del packed
        torch.cuda.empty_cache()
        line["layered"][name] = res
    if not args.no_layered_kernels:
        width, ff, _ = SIZES[args.layered_sizes.split(",")[-1]]
        line["kernels"] = kernels(width, ff, 2048, WINDOW)
    line["clocks"] = sampler.stop()
    print(json.dumps(line))


def _tensors(model):
    seen = []
    for layer in model.layers:
        for part in (layer.mixer, layer.ffn):
            seen += [t for k, t in vars(part).items() if k.startswith("w_")] if part is not None else []
    return seen + [model.embedding, model.head]
