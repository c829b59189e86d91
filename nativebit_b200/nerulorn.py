"""Nerulorn: latent attention over a sliding window (with an output gate per head, some layers reading another layer's
cache) interleaved with gated linear attention, LayerNorm before and after every sublayer, SwiGLU feed-forward with
biases on some layers.  This file reads its config.json and tensor names into the layers of layered.py."""
from __future__ import annotations

import torch

from .layered import DenseFFN, GatedLinearAttention, LatentAttention, Layer, LayeredDecoder, Link, Rotation, Yarn
from .layer_ops import pad_matrix
from .weights import load_checkpoint


def _rotation(rot: dict) -> Rotation:
    s = rot.get("scaling")
    yarn = Yarn(float(s["factor"]), float(s["original"]), float(s["fast"]), float(s["slow"])) if s else None
    return Rotation(int(rot["dims"]), float(rot["base"]), yarn)


def _latent_attention(get, mix: dict, width: int, eps: float) -> LatentAttention:
    H, dim, rd, vd, rank, qr = (int(mix[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank"))
    rot = _rotation(mix["rot"])
    if rot.dims != rd:
        raise ValueError(f"the rotation covers {rot.dims} dimensions, the rotated part has {rd}")
    src = mix.get("kv_from")
    own = {} if src is not None else {"w_dkv": get("dkv", (rank + rd, width)), "kv_norm": get("dkv.norm", (rank,))}
    return LatentAttention(heads=H, dim=dim, rot=rot, vdim=vd, kv_rank=rank, window=int(mix["mask"]["size"]), scale=float(mix["scale"]),
                           eps=eps, w_dq=get("dq", (qr, width)), q_norm=get("dq.norm", (qr,)), w_uq=get("uq", (H * (dim + rd), qr)),
                           w_uk=get("uk", (H * dim, rank)), w_uv=get("uv", (H * vd, rank)), w_gate=get("g", (H, width)),
                           w_out=get("o", (width, H * vd)), kv_from=None if src is None else int(src), **own)


def _gla(get, mix: dict, width: int, eps: float) -> GatedLinearAttention:
    H, dim, vd = (int(mix[k]) for k in ("heads", "dim", "vdim"))
    return GatedLinearAttention(heads=H, dim=dim, vdim=vd, tau=float(mix["tau"]), eps=eps, w_q=get("q", (H * dim, width)),
                                w_k=get("k", (H * dim, width)), w_v=get("v", (H * vd, width)), w_gate=get("g", (H * vd, width)),
                                w_a1=get("a1", (None, width)), w_a2=get("a2", (H * dim, None)), a2_bias=get("a2.b", (H * dim,)),
                                norm_w=get("norm", (vd,)), w_out=get("o", (width, H * vd)))


MIXERS = {"latent_attention": _latent_attention, "gla": _gla}


def _ffn(get, mlp: dict | None, width: int) -> DenseFFN | None:
    if mlp is None:
        return None
    if mlp["kind"] != "dense":
        raise ValueError(f"feed-forward kind {mlp['kind']!r}")
    F = int(mlp["ff"])
    return DenseFFN(w_gate=get("gate", (F, width)), b_gate=get("gate.b", (F,)), w_up=get("up", (F, width)), b_up=get("up.b", (F,)),
                    w_down=get("down", (width, F)), b_down=get("down.b", (width,)))


def build(config: dict, tensor, dtype: torch.dtype, context_len: int) -> LayeredDecoder:
    """tensor(name, shape) -> the weight of that name on the device."""
    C, V, eps = int(config["width"]), int(config["vocab"]), float(config["norm"]["eps"])
    layers = []
    for i, spec in enumerate(config["layers"]):
        if spec["type"] not in MIXERS:
            raise ValueError(f"layer {i} has the unknown mixer {spec['type']!r}")
        norm = lambda name: tensor(f"l{i}.{name}", (C,)).float()                                        # noqa: E731
        mixer = MIXERS[spec["type"]](lambda n, s: tensor(f"l{i}.mix.{n}", s), spec["mixer"], C, eps)
        ffn = _ffn(lambda n, s: tensor(f"l{i}.mlp.{n}", s), spec["mlp"], C)
        extra = {} if ffn is None else {"ffn": ffn, "link2": Link(norm("norm2"), [norm("norm2b")])}
        layers.append(Layer(mixer, Link(norm("norm1"), [norm("norm1b")]), **extra))
    return LayeredDecoder(tensor("embed", (V, C)), float(config["embedding"]["scale"]), layers, Link(tensor("final.norm", (C,)).float()),
                          pad_matrix(tensor("head", (V, C))), "layer", eps, dtype, context_len)


def load(folder: str, config: dict, dtype: torch.dtype, context_len: int, device) -> LayeredDecoder:
    return load_checkpoint(folder, device, lambda tensor: build(config, tensor, dtype, context_len))


def random_tensors(config: dict, seed: int, device) -> dict[str, torch.Tensor]:
    """Random-init weights of a configuration under the checkpoint's names (benchmarks and tests): matrices
    ~ N(0, 1 / fan-in), norm weights around 1, biases ~ N(0, 0.1), embeddings ~ N(0, 1)."""
    g = torch.Generator(device=device).manual_seed(seed)
    C, V = int(config["width"]), int(config["vocab"])
    out: dict[str, torch.Tensor] = {}

    def mat(name, n, k, std=None):
        out[name] = (torch.randn(n, k, device=device, generator=g) * (k ** -0.5 if std is None else std)).bfloat16()

    def vec(name, n, mean, std):
        out[name] = (mean + std * torch.randn(n, device=device, generator=g)).bfloat16()
    mat("embed", V, C, 1.0)
    mat("head", V, C)
    vec("final.norm", C, 1.0, 0.1)
    for i, spec in enumerate(config["layers"]):
        p, m = f"l{i}.", spec["mixer"]
        H, dim, vd = m["heads"], m["dim"], m["vdim"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if spec["mlp"] is not None else ()):
            vec(p + n, C, 1.0, 0.1)
        if spec["type"] == "gla":
            ra = m.get("a_rank", 16)
            for n, rows in (("q", H * dim), ("k", H * dim), ("v", H * vd), ("g", H * vd), ("a1", ra)):
                mat(p + "mix." + n, rows, C)
            mat(p + "mix.a2", H * dim, ra)
            vec(p + "mix.a2.b", H * dim, 1.0, 1.0)
            vec(p + "mix.norm", vd, 1.0, 0.1)
        else:
            rank, qr, rd = m["kv_rank"], m["q_rank"], m["rot_dim"]
            for n, rows, k in (("dq", qr, C), ("uq", H * (dim + rd), qr), ("uk", H * dim, rank), ("uv", H * vd, rank), ("g", H, C)):
                mat(p + "mix." + n, rows, k)
            vec(p + "mix.dq.norm", qr, 1.0, 0.1)
            if m.get("kv_from") is None:
                mat(p + "mix.dkv", rank + rd, C)
                vec(p + "mix.dkv.norm", rank, 1.0, 0.1)
        mat(p + "mix.o", C, H * vd)
        if spec["mlp"] is not None:
            F = spec["mlp"]["ff"]
            for n, rows, k in (("gate", F, C), ("up", F, C), ("down", C, F)):
                mat(p + "mlp." + n, rows, k)
                vec(p + "mlp." + n + ".b", rows, 0.0, 0.1)
    return out


def random_init(config: dict, seed: int = 0, dtype: torch.dtype = torch.bfloat16, context_len: int = 4096, device="cuda") -> LayeredDecoder:
    w = random_tensors(config, seed, torch.device(device))
    model = build(config, lambda n, s: w[n], dtype, context_len)
    torch.cuda.synchronize(device)
    return model
