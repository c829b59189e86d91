"""Nabalix: every mixer runs two branches on one input, attention with scores mixed across heads over a sliding window and
the HGRN2 recurrence, joined as half the sum of their RMS-normed results; a clamped gated feed-forward or none;
hyper-connections with a scale per channel on every sublayer's result; norm weights stored around zero.  This file reads
its config.json and tensor names into the layers of layered.py."""
from __future__ import annotations

import torch

from .layer_ops import ACT_CLAMPED_GLU_PAIRS, Act, pad_matrix
from .layered import BranchMixer, DenseFFN, ForgetLinearAttention, Layer, LayeredDecoder, Link, MixedHeadAttention
from .weights import load_checkpoint

GATE_SLOPE = 1.702             # of the feed-forward's sigmoid


def _attention(get, mix: dict, width: int, context_len: int) -> MixedHeadAttention:
    H, G, dim, vd = (int(mix[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
    return MixedHeadAttention(heads=H, kv_heads=G, dim=dim, vdim=vd, window=int(mix["mask"]["size"]), scale=float(mix["scale"]),
                              softcap=float(mix["softcap"]), context_len=context_len, w_q=get("q", (H * dim, width)),
                              w_k=get("k", (G * dim, width)), w_v=get("v", (G * vd, width)), w_gate=get("g", (H * vd, width)),
                              r1=get("r1", (H,)), r2=get("r2", (H,)), talk=get("talk", (H, H)), w_out=get("o", (width, H * vd)))


def _hgrn2(get, mix: dict, width: int, eps: float) -> ForgetLinearAttention:
    H, dim, vd = (int(mix[k]) for k in ("heads", "dim", "vdim"))
    return ForgetLinearAttention(heads=H, dim=dim, vdim=vd, eps=eps, w_q=get("q", (H * dim, width)), w_f=get("f", (H * dim, width)),
                                 f_bias=get("f.b", (H * dim,)), lower=get("lower", (H * dim,)), w_v=get("v", (H * vd, width)),
                                 norm_w=get("norm", (vd,)), w_out=get("o", (width, H * vd)))


def _ffn(get, mlp: dict | None, width: int) -> DenseFFN | None:
    if mlp is None:
        return None
    if mlp["kind"] != "dense":
        raise ValueError(f"feed-forward kind {mlp['kind']!r}")
    F = int(mlp["ff"])
    return DenseFFN(w_gate=get("gate", (F, width)), w_up=get("up", (F, width)), w_down=get("down", (width, F)),
                    act=Act(ACT_CLAMPED_GLU_PAIRS, GATE_SLOPE, float(mlp["limit"])))


def build(config: dict, tensor, dtype: torch.dtype, context_len: int) -> LayeredDecoder:
    """tensor(name, shape) -> the weight of that name on the device."""
    C, V, S, eps = int(config["width"]), int(config["vocab"]), int(config["streams"]), float(config["norm"]["eps"])

    def vector(name):
        return tensor(name, (C,)).float()

    def link(layer, q, post, post_norm=None):
        hc = f"{layer}hc{q}."
        return Link(1.0 + vector(f"{layer}norm{q}"), post, post_norm, read=tensor(hc + "in", (S,)).float(), share=tensor(hc + "out", (S,)).float(),
                    mix=tensor(hc + "mix", (S, S)).float())
    layers = []
    for i, spec in enumerate(config["layers"]):
        if spec["type"] != "parallel":
            raise ValueError(f"layer {i} has the unknown mixer {spec['type']!r}")
        at, mix = f"l{i}.", spec["mixer"]
        mixer = BranchMixer("parallel", [_attention(lambda n, s: tensor(f"{at}mix.left.{n}", s), mix["left"], C, context_len),
                                         _hgrn2(lambda n, s: tensor(f"{at}mix.right.{n}", s), mix["right"], C, eps)])
        scale = 0.5 * vector(at + "ls1")
        link1 = link(at, 1, [scale * vector(f"{at}mix.{side}.out") for side in ("left", "right")], "rms")
        ffn = _ffn(lambda n, s: tensor(f"{at}mlp.{n}", s), spec["mlp"], C)
        extra = {} if ffn is None else {"ffn": ffn, "link2": link(at, 2, [vector(at + "ls2")])}
        layers.append(Layer(mixer, link1, **extra))
    ones = torch.ones(S, dtype=torch.float32, device=layers[0].link1.read.device)
    return LayeredDecoder(tensor("embed", (V, C)), 1.0, layers, Link(1.0 + vector("final.norm"), read=ones), pad_matrix(tensor("head", (V, C))),
                          "rms", eps, dtype, context_len, streams=S)


def load(folder: str, config: dict, dtype: torch.dtype, context_len: int, device) -> LayeredDecoder:
    # a layer without a feed-forward may carry the connection of one
    spare = tuple(f"l{i}.{n}" for i, spec in enumerate(config["layers"]) if spec["mlp"] is None for n in ("norm2", "ls2", "hc2."))
    return load_checkpoint(folder, device, lambda tensor: build(config, tensor, dtype, context_len), spare)


def random_tensors(config: dict, seed: int, device) -> dict[str, torch.Tensor]:
    """Random-init weights of a configuration under the checkpoint's names (benchmarks and tests): matrices
    ~ N(0, 1 / fan-in), norm weights around their neutral value, talk and mix near the identity, embeddings ~ N(0, 1)."""
    g = torch.Generator(device=device).manual_seed(seed)
    C, V, S = int(config["width"]), int(config["vocab"]), int(config["streams"])
    out: dict[str, torch.Tensor] = {}

    def mat(name, n, k, std=None):
        out[name] = (torch.randn(n, k, device=device, generator=g) * (k ** -0.5 if std is None else std)).bfloat16()

    def vec(name, n, mean, std):
        out[name] = (mean + std * torch.randn(n, device=device, generator=g)).bfloat16()

    def near_identity(name, n, std):
        out[name] = (torch.eye(n, device=device) + std * torch.randn(n, n, device=device, generator=g)).bfloat16()

    def uniform(name, n, lo, hi):
        out[name] = (lo + (hi - lo) * torch.rand(n, device=device, generator=g)).bfloat16()
    mat("embed", V, C, 1.0)
    mat("head", V, C)
    vec("final.norm", C, 0.0, 0.1)
    for i, spec in enumerate(config["layers"]):
        p, a, r = f"l{i}.", spec["mixer"]["left"], spec["mixer"]["right"]
        H, G, dim, vd = (a[k] for k in ("heads", "kv_heads", "dim", "vdim"))
        for n, rows, k in (("q", H * dim, C), ("k", G * dim, C), ("v", G * vd, C), ("g", H * vd, C), ("o", C, H * vd)):
            mat(f"{p}mix.left.{n}", rows, k)
        uniform(p + "mix.left.r1", H, 0.0, 2.0)
        uniform(p + "mix.left.r2", H, 0.05, 0.5)
        near_identity(p + "mix.left.talk", H, 0.3)
        H, dim, vd = (r[k] for k in ("heads", "dim", "vdim"))
        for n, rows, k in (("q", H * dim, C), ("f", H * dim, C), ("v", H * vd, C), ("o", C, H * vd)):
            mat(f"{p}mix.right.{n}", rows, k)
        vec(p + "mix.right.f.b", H * dim, 1.5, 1.5)
        uniform(p + "mix.right.lower", H * dim, 0.0, 0.9)
        vec(p + "mix.right.norm", vd, 1.0, 0.1)
        for side in ("left", "right"):
            vec(f"{p}mix.{side}.out", C, 1.0, 0.1)
        if spec["mlp"] is not None:
            F = spec["mlp"]["ff"]
            for n, rows, k in (("gate", F, C), ("up", F, C), ("down", C, F)):
                mat(f"{p}mlp.{n}", rows, k)
        for q in (1, 2) if spec["mlp"] is not None else (1,):
            vec(f"{p}norm{q}", C, 0.0, 0.1)
            vec(f"{p}ls{q}", C, 0.5, 0.1)
            vec(f"{p}hc{q}.in", S, 1.0 / S, 0.2)
            vec(f"{p}hc{q}.out", S, 1.0, 0.2)
            near_identity(f"{p}hc{q}.mix", S, 0.15)
    return out


def random_init(config: dict, seed: int = 0, dtype: torch.dtype = torch.bfloat16, context_len: int = 4096, device="cuda") -> LayeredDecoder:
    w = random_tensors(config, seed, torch.device(device))
    model = build(config, lambda n, s: w[n], dtype, context_len)
    torch.cuda.synchronize(device)
    return model
