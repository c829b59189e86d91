"""Layered decoders: models that list their layers one by one, each with its own mixer (latent attention over a
sliding window, gated linear attention, several branches side by side) and feed-forward or none, and a residual of one
of two kinds: a norm before and after every sublayer,

    x <- x + post(sublayer(pre(x))),

or hyper-connections, several streams that every sublayer reads as a weighted sum and leaves mixed (`Link`).

A model family describes its layers with the classes below (see nerulorn.py, nabalix.py); this file runs them:
`LayeredDecoder` takes prompts and portions of prompts through the matrix-product kernels, `LayeredSession` decodes single
tokens through the fused matvec chain in a CUDA graph.  The activation dtype is bf16 or fp32; the residual stream, norms,
positions, attention scores and weights, decays and recurrent states are fp32 in both, and a single sequence's decode
step has fp32 activations throughout (only the latent cache follows the dtype)."""
from __future__ import annotations

import math
from dataclasses import dataclass, field

import torch

from . import layer_ops as L
from .session import Session

NORMS = {"rms": L.NORM_RMS, "layer": L.NORM_LAYER}


@dataclass(frozen=True)
class Yarn:
    """YaRN: frequencies below `slow` turns over the original context are divided by `factor`, those above `fast` stay,
    a ramp in between; cos and sin grow by 0.1 ln(factor) + 1."""
    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class Rotation:
    """Rotary positions on interleaved pairs (2i, 2i + 1) of `dims` dimensions."""
    dims: int
    base: float
    yarn: Yarn | None = None

    def frequencies(self) -> tuple[torch.Tensor, float]:
        """(fp64 frequency of every pair, factor on cos and sin)"""
        i = torch.arange(self.dims // 2, dtype=torch.float64)
        f = torch.pow(torch.tensor(float(self.base), dtype=torch.float64), -2.0 * i / self.dims)
        if self.yarn is None:
            return f, 1.0
        y = self.yarn

        def at(turns: float) -> float:
            return self.dims * math.log(y.original / (2 * math.pi * turns)) / (2 * math.log(self.base))
        lo, hi = max(math.floor(at(y.fast)), 0), min(math.ceil(at(y.slow)), self.dims - 1)
        ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
        return f / y.factor * ramp + f * (1 - ramp), 0.1 * math.log(y.factor) + 1.0

    def tables(self, max_len: int, device) -> tuple[torch.Tensor, torch.Tensor]:
        """cos and sin, (max_len, dims) fp32, every pair's entry twice; the angles are formed in fp64."""
        f, m = self.frequencies()
        a = torch.outer(torch.arange(max_len, dtype=torch.float64), f)
        return tuple((t * m).float().repeat_interleave(2, dim=1).contiguous().to(device) for t in (a.cos(), a.sin()))


# ---------------------------------------------------------------------- caches and states
class LatentCache:
    """One latent and one rotated key part per position, (B, context, row) of the activation dtype; layers may share it."""

    def __init__(self, batch: int, context_len: int, width: int, dtype: torch.dtype, device):
        self.rows = torch.zeros(batch, context_len, L.pad8(width), dtype=dtype, device=device)

    def reset(self) -> None:
        """Rows past the position are never read: nothing to clear."""

    def carried(self) -> list[torch.Tensor]:
        return []


class KeyValueCache:
    """Keys of a layer's key/value heads, then their values, one row per position: (B, context, row) of the activation dtype."""

    def __init__(self, batch: int, context_len: int, keys: int, values: int, dtype: torch.dtype, device):
        self.v_off = L.pad8(keys)
        self.rows = torch.zeros(batch, context_len, self.v_off + L.pad8(values), dtype=dtype, device=device)

    def reset(self) -> None:
        """Rows past the position are never read: nothing to clear."""

    def carried(self) -> list[torch.Tensor]:
        return []


class RecurrentState:
    """(B, heads, dim, padded vdim) fp32, carried from token to token."""

    def __init__(self, batch: int, heads: int, dim: int, vdim: int, device):
        self.s = torch.zeros(batch, heads, dim, (vdim + 3) // 4 * 4, dtype=torch.float32, device=device)

    def reset(self) -> None:
        self.s.zero_()

    def carried(self) -> list[torch.Tensor]:
        """What a step changes in place."""
        return [self.s]


class BranchCaches:
    """One cache or state per branch of a mixer."""

    def __init__(self, parts: list):
        self.parts = parts

    def reset(self) -> None:
        for p in self.parts:
            p.reset()

    def carried(self) -> list[torch.Tensor]:
        return [t for p in self.parts for t in p.carried()]


# ---------------------------------------------------------------------- pieces of a layer
@dataclass
class Span:
    """What a portion of a prompt brings: B sequences x T tokens at positions pos0 .."""
    B: int
    T: int
    pos0: int
    dtype: torch.dtype
    device: torch.device

    @property
    def rows(self) -> int:
        return self.B * self.T

    def empty(self, cols: int) -> torch.Tensor:
        return L.rows_empty(self.rows, cols, self.dtype, self.device)


class LatentAttention:
    """Queries through a latent of their own, keys and values as linear maps of one cached latent per position plus a
    rotated key part shared by the heads, a sliding window, a sigmoid gate per head.  With `kv_from` the layer reads
    another layer's cache and has no key/value projection of its own."""
    kind = "latent_attention"

    def __init__(self, *, heads: int, dim: int, rot: Rotation, vdim: int, kv_rank: int, window: int, scale: float, eps: float,
                 w_dq, q_norm, w_uq, w_uk, w_uv, w_gate, w_out, w_dkv=None, kv_norm=None, kv_from: int | None = None):
        self.heads, self.dim, self.rot, self.vdim, self.rank = heads, dim, rot, vdim, kv_rank
        self.window, self.scale, self.eps, self.kv_from = window, scale, eps, kv_from
        self.q_rank, self.width = w_dq.shape
        if (w_dkv is None) != (kv_from is not None):
            raise ValueError("a layer has either its own key/value projection or another layer's cache")
        mats = [w_dq, w_gate] + ([w_dkv] if w_dkv is not None else [])
        self.w_in, offs = L.stack_rows(mats)
        self.n_in, self.q_off, self.g_off, self.kv_off = self.w_in.shape[0], offs[0], offs[1], offs[2] if len(offs) > 2 else -1
        self.w_uq, self.n_q = L.pad_matrix(w_uq), w_uq.shape[0]
        self.w_ukv, (_, self.v_off) = L.stack_rows([w_uk, w_uv])
        self.n_kv = self.w_ukv.shape[0]
        self.w_out, self.n_out = L.pad_matrix(w_out), w_out.shape[0]
        self.q_norm, self.kv_norm = q_norm.float(), None if kv_norm is None else kv_norm.float()
        want = {"uq": (heads * (dim + rot.dims), self.q_rank), "uk": (heads * dim, kv_rank), "uv": (heads * vdim, kv_rank),
                "out": (self.n_out, heads * vdim)}
        for name, w in (("uq", w_uq), ("uk", w_uk), ("uv", w_uv), ("out", w_out)):
            if tuple(w.shape) != want[name]:
                raise ValueError(f"{name} has shape {tuple(w.shape)}, the layer's sizes want {want[name]}")

    def new_cache(self, batch: int, context_len: int, dtype, device) -> LatentCache:
        return LatentCache(batch, context_len, self.rank + self.rot.dims, dtype, device)

    def _sizes(self, cache: LatentCache, cos_sin) -> dict:
        return dict(H=self.heads, dim=self.dim, rot=self.rot.dims, vdim=self.vdim, rank=self.rank, ctx=cache.rows.shape[1],
                    ldc=cache.rows.shape[2], cos2=cos_sin[0].data_ptr(), sin2=cos_sin[1].data_ptr(), scale=self.scale, window=self.window,
                    cache=cache.rows.data_ptr())

    def prompt(self, h: torch.Tensor, span: Span, cache: LatentCache, cos_sin) -> list[torch.Tensor]:
        H, tag = self.heads, L._DTYPE[span.dtype]
        a = span.empty(self.n_in)
        L.linear(h, self.w_in, self.width, self.n_in, a)
        cq = span.empty(self.q_rank)
        rows = cache.rows
        L.latent_prepare(a=a.data_ptr(), cq=cq.data_ptr(), cache=rows.data_ptr(), q_norm=self.q_norm.data_ptr(),
                         kv_norm=L._ptr(self.kv_norm), cos2=cos_sin[0].data_ptr(), sin2=cos_sin[1].data_ptr(), eps=self.eps, dtype=tag,
                         B=span.B, T=span.T, lda=a.stride(0), q_off=self.q_off, q_rank=self.q_rank, ldcq=cq.stride(0), kv_off=self.kv_off,
                         rank=self.rank, rot=self.rot.dims, ctx=rows.shape[1], ldc=rows.shape[2], pos0=span.pos0)
        q = span.empty(self.n_q)
        L.linear(cq, self.w_uq, self.q_rank, self.n_q, q)
        # keys and values of every position the portion can see, up-projected from the cache
        lo = max(0, span.pos0 - self.window + 1) if self.window > 0 else 0
        n = span.pos0 + span.T - lo
        kv = L.rows_empty(span.B * n, self.n_kv, span.dtype, span.device)
        for b in range(span.B):
            L.linear(rows[b, lo:lo + n], self.w_ukv, self.rank, self.n_kv, kv[b * n:(b + 1) * n])
        att = span.empty(H * self.vdim)
        L.latent_attention(q=q.data_ptr(), kv=kv.data_ptr(), gate=L._ptr(a, self.g_off), out=att.data_ptr(), dtype=tag, B=span.B, T=span.T,
                           ldq=q.stride(0), ldkv=kv.stride(0), v_off=self.v_off, kv_rows=n, kv_pos0=lo, ldg=a.stride(0), ldo=att.stride(0),
                           pos0=span.pos0, **self._sizes(cache, cos_sin))
        y = torch.empty(span.rows, self.n_out, dtype=torch.float32, device=span.device)
        L.linear(att, self.w_out, H * self.vdim, self.n_out, y)
        return [y]

    def buffers(self) -> dict[str, int]:
        """fp32 scratch of the decode step, in elements."""
        return {"a": self.n_in, "q": self.n_q, "o": self.heads * self.vdim, "y": self.n_out}

    def decode(self, chain, s: "LayeredSession", cache: LatentCache, cos_sin) -> list[torch.Tensor]:
        a, q, o, y = s.buf["a"], s.buf["q"], s.buf["o"], s.buf["y"]
        chain(self.w_in, self.n_in, self.width, a)
        L.matvec(self.w_uq, self.n_q, self.q_rank, a, q, norm=L.NORM_RMS, eps=self.eps, norm_w=self.q_norm, x_offset=self.q_off)
        L.latent_decode(q=q.data_ptr(), a=a.data_ptr(), uk=self.w_ukv.data_ptr(), uv=L._ptr(self.w_ukv, self.v_off * self.w_ukv.stride(0)),
                        kv_norm=L._ptr(self.kv_norm), pos=s.pos.data_ptr(), out=o.data_ptr(), eps=self.eps,
                        cache_dtype=L._DTYPE[cache.rows.dtype], B=1, ldq=q.numel(), lda=a.numel(), kv_off=self.kv_off, g_off=self.g_off,
                        ldu=self.w_ukv.stride(0), ldo=o.numel(), **self._sizes(cache, cos_sin))
        L.matvec(self.w_out, self.n_out, self.heads * self.vdim, o, y)
        return [y]


class GatedLinearAttention:
    """A (dim x vdim) fp32 state per head that decays per key channel, sigmoid(z)^(1 / tau) with z from a low-rank
    projection; the heads' outputs are RMS-normed and gated by silu."""
    kind = "gla"

    def __init__(self, *, heads: int, dim: int, vdim: int, tau: float, eps: float, w_q, w_k, w_v, w_gate, w_a1, w_a2, a2_bias, norm_w, w_out):
        self.heads, self.dim, self.vdim, self.tau, self.eps = heads, dim, vdim, float(tau), eps
        self.width, self.a_rank = w_q.shape[1], w_a1.shape[0]
        self.w_in, (self.q_off, self.k_off, self.v_off, self.g_off, self.a_off) = L.stack_rows([w_q, w_k, w_v, w_gate, w_a1])
        self.n_in = self.w_in.shape[0]
        self.w_a2, self.a2_bias, self.norm_w = L.pad_matrix(w_a2), a2_bias.float(), norm_w.float()
        self.w_out, self.n_out = L.pad_matrix(w_out), w_out.shape[0]
        for name, w, want in (("q", w_q, (heads * dim, self.width)), ("k", w_k, (heads * dim, self.width)),
                              ("v", w_v, (heads * vdim, self.width)), ("g", w_gate, (heads * vdim, self.width)),
                              ("a2", w_a2, (heads * dim, self.a_rank)), ("out", w_out, (self.n_out, heads * vdim)), ("norm", norm_w, (vdim,))):
            if tuple(w.shape) != want:
                raise ValueError(f"{name} has shape {tuple(w.shape)}, the layer's sizes want {want}")

    def new_cache(self, batch: int, context_len: int, dtype, device) -> RecurrentState:
        return RecurrentState(batch, self.heads, self.dim, self.vdim, device)

    def _args(self, p: torch.Tensor, ldp: int, out: torch.Tensor, ldo: int, state: RecurrentState, dtype: torch.dtype, B: int, T: int) -> dict:
        return dict(p=p.data_ptr(), out=out.data_ptr(), state=state.s.data_ptr(), a2=self.w_a2.data_ptr(), a2_b=self.a2_bias.data_ptr(),
                    norm_w=self.norm_w.data_ptr(), tau=self.tau, eps=self.eps, kind=L.GLA_LOW_RANK, dtype=L._DTYPE[dtype], B=B, T=T, H=self.heads, dim=self.dim,
                    vdim=self.vdim, ldp=ldp, q_off=self.q_off, k_off=self.k_off, v_off=self.v_off, g_off=self.g_off, a_off=self.a_off,
                    a_rank=self.a_rank, lda2=self.w_a2.stride(0), lds=state.s.shape[3], ldo=ldo)

    def prompt(self, h: torch.Tensor, span: Span, state: RecurrentState, cos_sin) -> list[torch.Tensor]:
        p = span.empty(self.n_in)
        L.linear(h, self.w_in, self.width, self.n_in, p)
        o = span.empty(self.heads * self.vdim)
        ws = torch.empty(L.gla_workspace_bytes(span.B, span.T, self.heads, self.dim, self.vdim), dtype=torch.uint8, device=span.device)
        L.gla_prefill(ws, **self._args(p, p.stride(0), o, o.stride(0), state, span.dtype, span.B, span.T))
        y = torch.empty(span.rows, self.n_out, dtype=torch.float32, device=span.device)
        L.linear(o, self.w_out, self.heads * self.vdim, self.n_out, y)
        return [y]

    def buffers(self) -> dict[str, int]:
        return {"a": self.n_in, "o": self.heads * self.vdim, "y": self.n_out}

    def decode(self, chain, s: "LayeredSession", state: RecurrentState, cos_sin) -> list[torch.Tensor]:
        p, o, y = s.buf["a"], s.buf["o"], s.buf["y"]
        chain(self.w_in, self.n_in, self.width, p)
        L.gla_decode(**self._args(p, p.numel(), o, o.numel(), state, torch.float32, 1, 1))
        L.matvec(self.w_out, self.n_out, self.heads * self.vdim, o, y)
        return [y]


# ---------------------------------------------------------------------- branches
class MixedHeadAttention:
    """A branch (see `BranchMixer`): grouped attention over a sliding window without a rotation.  Scores pass through a soft
    cap, lose r1_h ln(1 + r2_h distance) and are mixed across the heads by `talk` (heads, heads) before the softmax; the
    heads' outputs are gated element by element by a sigmoid."""

    def __init__(self, *, heads: int, kv_heads: int, dim: int, vdim: int, window: int, scale: float, softcap: float, context_len: int,
                 w_q, w_k, w_v, w_gate, r1, r2, talk, w_out):
        if heads % kv_heads:
            raise ValueError(f"{heads} heads do not share {kv_heads} key/value heads evenly")
        self.heads, self.kv_heads, self.dim, self.vdim, self.window, self.scale, self.softcap = heads, kv_heads, dim, vdim, window, scale, softcap
        width = w_q.shape[1]
        _shapes({"q": (w_q, (heads * dim, width)), "k": (w_k, (kv_heads * dim, width)), "v": (w_v, (kv_heads * vdim, width)),
                 "g": (w_gate, (heads * vdim, width)), "r1": (r1, (heads,)), "r2": (r2, (heads,)), "talk": (talk, (heads, heads)),
                 "o": (w_out, (w_out.shape[0], heads * vdim))})
        # keys and values stand side by side, each from a multiple of eight rows on: the cache's row is a copy of them
        self.w_in = [w_q, w_k, w_v, w_gate]
        self.kv_cols = L.pad8(kv_heads * dim) + kv_heads * vdim
        self.w_out, self.cols = w_out, heads * vdim
        self.talk = talk.float().contiguous()
        n = min(window, context_len) if window > 0 else context_len
        far = torch.arange(n, dtype=torch.float64, device=r1.device)
        self.penalty = (r1.double()[:, None] * torch.log1p(r2.double()[:, None] * far)).float().contiguous()

    def place(self, offsets: list[int]) -> None:
        """Columns of the pieces of w_in in the joint projection."""
        self.q_off, self.k_off, _, self.g_off = offsets

    def new_cache(self, batch: int, context_len: int, dtype, device) -> KeyValueCache:
        return KeyValueCache(batch, context_len, self.kv_heads * self.dim, self.kv_heads * self.vdim, dtype, device)

    def _sizes(self, cache: KeyValueCache) -> dict:
        return dict(cache=cache.rows.data_ptr(), penalty=self.penalty.data_ptr(), talk=self.talk.data_ptr(), scale=self.scale, softcap=self.softcap,
                    H=self.heads, G=self.kv_heads, dim=self.dim, vdim=self.vdim, ctx=cache.rows.shape[1], ldc=cache.rows.shape[2],
                    v_off=cache.v_off, window=self.window, n_pen=self.penalty.shape[1])

    def prompt(self, a: torch.Tensor, span: Span, cache: KeyValueCache) -> torch.Tensor:
        """a: the joint projection of the portion's rows."""
        o = span.empty(self.cols)
        L.cache_append(a, self.k_off, self.kv_cols, cache.rows, span.B, span.T, span.pos0)
        L.talk_attention(span.device, q=L._ptr(a, self.q_off), gate=L._ptr(a, self.g_off), out=o.data_ptr(), dtype=L._DTYPE[span.dtype], B=span.B,
                         T=span.T, ldq=a.stride(0), ldg=a.stride(0), ldo=o.stride(0), pos0=span.pos0, **self._sizes(cache))
        return o

    def decode(self, a: torch.Tensor, o: torch.Tensor, s: "LayeredSession", cache: KeyValueCache) -> None:
        L.talk_decode(p=a.data_ptr(), pos=s.pos.data_ptr(), out=o.data_ptr(), cache_dtype=L._DTYPE[cache.rows.dtype], B=1, ldp=a.numel(),
                      q_off=self.q_off, k_off=self.k_off, g_off=self.g_off, ldo=o.numel(), **self._sizes(cache))


class ForgetLinearAttention:
    """A branch: the HGRN2 recurrence.  Per head a (dim x vdim) fp32 state that decays by f per channel and takes up
    (1 - f) v^T, f = lower + (1 - lower) sigmoid(z); read by silu(q), RMS-normed per head."""

    def __init__(self, *, heads: int, dim: int, vdim: int, eps: float, w_q, w_f, f_bias, lower, w_v, norm_w, w_out):
        self.heads, self.dim, self.vdim, self.eps = heads, dim, vdim, eps
        width = w_q.shape[1]
        _shapes({"q": (w_q, (heads * dim, width)), "f": (w_f, (heads * dim, width)), "f.b": (f_bias, (heads * dim,)),
                 "lower": (lower, (heads * dim,)), "v": (w_v, (heads * vdim, width)), "norm": (norm_w, (vdim,)),
                 "o": (w_out, (w_out.shape[0], heads * vdim))})
        self.w_in = [w_q, w_f, w_v]
        self.w_out, self.cols = w_out, heads * vdim
        self.f_bias, self.lower, self.norm_w = f_bias.float(), lower.float(), norm_w.float()

    def place(self, offsets: list[int]) -> None:
        self.q_off, self.f_off, self.v_off = offsets

    def new_cache(self, batch: int, context_len: int, dtype, device) -> RecurrentState:
        return RecurrentState(batch, self.heads, self.dim, self.vdim, device)

    def _args(self, p: torch.Tensor, ldp: int, out: torch.Tensor, ldo: int, state: RecurrentState, dtype: torch.dtype, B: int, T: int) -> dict:
        return dict(p=p.data_ptr(), out=out.data_ptr(), state=state.s.data_ptr(), a2_b=self.f_bias.data_ptr(), lower=self.lower.data_ptr(),
                    norm_w=self.norm_w.data_ptr(), eps=self.eps, kind=L.GLA_FORGET, dtype=L._DTYPE[dtype], B=B, T=T, H=self.heads, dim=self.dim,
                    vdim=self.vdim, ldp=ldp, q_off=self.q_off, k_off=self.f_off, v_off=self.v_off, g_off=-1, lds=state.s.shape[3], ldo=ldo)

    def prompt(self, a: torch.Tensor, span: Span, state: RecurrentState) -> torch.Tensor:
        o = span.empty(self.cols)
        ws = torch.empty(L.gla_workspace_bytes(span.B, span.T, self.heads, self.dim, self.vdim), dtype=torch.uint8, device=span.device)
        L.gla_prefill(ws, **self._args(a, a.stride(0), o, o.stride(0), state, span.dtype, span.B, span.T))
        return o

    def decode(self, a: torch.Tensor, o: torch.Tensor, s: "LayeredSession", state: RecurrentState) -> None:
        L.gla_decode(**self._args(a, a.numel(), o, o.numel(), state, torch.float32, 1, 1))


class BranchMixer:
    """One or two branches side by side: one product for all their projections, every branch on its columns, an output
    projection each.  The results stay apart; the layer's link weights and adds them."""

    def __init__(self, kind: str, branches: list):
        if not 1 <= len(branches) <= 2:
            raise ValueError(f"{len(branches)} branches")
        self.kind, self.branches = kind, branches
        self.w_in, offs = L.stack_rows([m for b in branches for m in b.w_in])
        self.width, self.n_in = branches[0].w_in[0].shape[1], self.w_in.shape[0]
        for b in branches:
            b.place(offs[:len(b.w_in)])
            offs = offs[len(b.w_in):]
            del b.w_in
            b.w_out, b.n_out = L.pad_matrix(b.w_out), b.w_out.shape[0]

    def new_cache(self, batch: int, context_len: int, dtype, device) -> BranchCaches:
        return BranchCaches([b.new_cache(batch, context_len, dtype, device) for b in self.branches])

    def prompt(self, h: torch.Tensor, span: Span, cache: BranchCaches, cos_sin) -> list[torch.Tensor]:
        a = span.empty(self.n_in)
        L.linear(h, self.w_in, self.width, self.n_in, a)
        ys = []
        for b, c in zip(self.branches, cache.parts):
            o = b.prompt(a, span, c)
            y = torch.empty(span.rows, b.n_out, dtype=torch.float32, device=span.device)
            L.linear(o, b.w_out, b.cols, b.n_out, y)
            ys.append(y)
        return ys

    def buffers(self) -> dict[str, int]:
        out = {"a": self.n_in}
        for i, b in enumerate(self.branches):
            out[f"o{i}"], out[f"y{i}"] = b.cols, b.n_out
        return out

    def decode(self, chain, s: "LayeredSession", cache: BranchCaches, cos_sin) -> list[torch.Tensor]:
        a = s.buf["a"]
        chain(self.w_in, self.n_in, self.width, a)
        jobs = []
        for i, (b, c) in enumerate(zip(self.branches, cache.parts)):
            b.decode(a, s.buf[f"o{i}"], s, c)
            jobs.append((b.w_out, b.n_out, b.cols, s.buf[f"o{i}"], s.buf[f"y{i}"]))
        L.matvec_pair(*jobs) if len(jobs) == 2 else L.matvec(*jobs[0])
        return [j[4] for j in jobs]


def _shapes(want: dict) -> None:
    for name, (w, shape) in want.items():
        if tuple(w.shape) != shape:
            raise ValueError(f"{name} has shape {tuple(w.shape)}, the layer's sizes want {shape}")


class DenseFFN:
    """W_down act(W_gate h + b, W_up h + b) + b with a gated activation (silu(g) * u unless told otherwise; biases may be
    absent); gate and up rows interleaved, so the product's epilogue emits the activation."""

    def __init__(self, *, w_gate, w_up, w_down, b_gate=None, b_up=None, b_down=None, act: L.Act = L.SWIGLU):
        F, self.width = w_gate.shape
        self.hidden, self.n_out, self.act = F, w_down.shape[0], act
        self.w_gu = L.pad_matrix(torch.stack((w_gate, w_up), dim=1).reshape(2 * F, self.width))
        self.b_gu = None if b_gate is None else torch.stack((b_gate.float(), b_up.float()), dim=1).reshape(-1).contiguous()
        self.w_down, self.b_down = L.pad_matrix(w_down), None if b_down is None else b_down.float()

    def prompt(self, h: torch.Tensor, span: Span) -> list[torch.Tensor]:
        act = span.empty(self.hidden)
        L.linear(h, self.w_gu, self.width, 2 * self.hidden, act, bias=self.b_gu, act=self.act)
        y = torch.empty(span.rows, self.n_out, dtype=torch.float32, device=span.device)
        L.linear(act, self.w_down, self.hidden, self.n_out, y, bias=self.b_down)
        return [y]

    def buffers(self) -> dict[str, int]:
        return {"f": self.hidden, "y": self.n_out}

    def decode(self, chain, s: "LayeredSession") -> list[torch.Tensor]:
        f, y = s.buf["f"], s.buf["y"]
        chain(self.w_gu, 2 * self.hidden, self.width, f, bias=self.b_gu, act=self.act)
        L.matvec(self.w_down, self.n_out, self.hidden, f, y, bias=self.b_down)
        return [y]


# ---------------------------------------------------------------------- the residual
@dataclass
class Link:
    """How a sublayer hangs on the residual.  One stream: x <- x + norm(y) * post around h = norm(x) * norm.  Hyper-connections:
    h = norm(sum_s read_s x_s) * norm, y = the sum of the results (each normed by `post_norm`, if given) times their weights
    in `post`, then x_t <- sum_s mix[s, t] x_s + share_t y, all streams at once."""
    norm: torch.Tensor                      # (C) weight of the norm in front
    post: list[torch.Tensor] = field(default_factory=list)       # (C) weight of each result
    post_norm: str | None = None
    read: torch.Tensor | None = None
    share: torch.Tensor | None = None
    mix: torch.Tensor | None = None

    def behind(self, before: "Link | None") -> torch.Tensor:
        """The coefficients of the step from the link `before` to this one (nb_stream_args): what this link reads, expressed in
        the streams in front of `before`'s update and its result."""
        read = self.read.double()
        n = read.numel()
        if before is None:
            read, direct, share, mix = read, read.new_zeros(1), read.new_zeros(n), torch.eye(n, dtype=read.dtype, device=read.device)
        else:
            share, mix = before.share.double(), before.mix.double()
            read, direct = mix @ read, (share @ read).reshape(1)
        return torch.cat([read, direct, share, mix.reshape(-1)]).float()


class PromptResidual:
    """The residual of a portion of a prompt: `enter` applies what the sublayer before left and returns the next one's input."""

    def __init__(self, model: "LayeredDecoder", tokens: torch.Tensor, span: Span):
        self.m, self.span = model, span
        self.x = torch.empty(span.rows, *([model.streams] if model.streams else []), model.width, dtype=torch.float32, device=span.device)
        L.embed_scaled(model.embedding, tokens.contiguous(), model.embedding_scale, self.x)
        self.h = span.empty(model.width)
        self.ys, self.link, self.n = [], None, 0

    def leave(self, link: Link, ys: list[torch.Tensor]) -> None:
        self.ys, self.link = ys, link

    def keep(self, rows: list[int]) -> None:
        """Only these rows go on."""
        if len(rows) == 1:
            pick = slice(rows[0], rows[0] + 1)
            self.x, self.ys = self.x[pick], [y[pick] for y in self.ys]
        else:
            at = torch.tensor(rows, dtype=torch.long, device=self.x.device)
            self.x, self.ys = self.x.index_select(0, at), [y.index_select(0, at) for y in self.ys]
        self.h = L.rows_empty(len(rows), self.m.width, self.span.dtype, self.x.device)

    def enter(self, link: Link) -> torch.Tensor:
        y, post = (self.ys[0], self.link.post[0]) if self.ys else (None, None)
        L.residual_norm(self.x, y, post, link.norm, NORMS[self.m.norm], self.m.eps, self.h)
        return self.h

    def total(self) -> torch.Tensor:
        """The residual after `enter`, (rows, C)."""
        return self.x.clone()


class PromptStreams(PromptResidual):
    """The same with hyper-connections: x (rows, streams, C)."""

    def enter(self, link: Link) -> torch.Tensor:
        L.stream_norm(self.x, self.ys, self.link.post if self.ys else [], self.m.post_norm(self.link), self.m.coefs[self.n], NORMS[self.m.norm],
                      self.m.eps, link.norm, self.h)
        self.n += 1
        return self.h

    def total(self) -> torch.Tensor:
        return self.x.sum(1)


class DecodeResidual:
    """The residual of a decode step of one sequence, in a session's two buffers; `chain` makes the product that follows, with
    the residual's update and the norm folded in."""

    def __init__(self, model: "LayeredDecoder", s: "LayeredSession"):
        self.m, self.xa, self.xb = model, s.buf["x"], s.buf["x2"]
        L.embed_scaled(model.embedding, s.token, model.embedding_scale, self.xa.view(1, *([model.streams] if model.streams else []), model.width))
        self.ys, self.link, self.n = [], None, 0

    def leave(self, link: Link, ys: list[torch.Tensor]) -> None:
        self.ys, self.link = ys, link

    def chain(self, link: Link):
        def run(w, n, k, out, bias=None, act=L.PLAIN):
            opt = dict(bias=bias, act=act, norm=NORMS[self.m.norm], eps=self.m.eps, norm_w=link.norm)
            if not self.ys:
                L.matvec(w, n, k, self.xa, out, **opt)
            else:
                L.matvec(w, n, k, self.xa, out, delta=self.ys[0], delta_w=self.link.post[0], x_out=self.xb, **opt)
                self.xa, self.xb = self.xb, self.xa
        return run


class DecodeStreams(DecodeResidual):
    def chain(self, link: Link):
        def run(w, n, k, out, bias=None, act=L.PLAIN):
            shape = (self.m.streams, self.m.width)
            L.matvec_streams(w, n, k, out, self.xa.view(shape), self.xb.view(shape), self.ys, self.link.post if self.ys else [],
                             self.m.post_norm(self.link), self.m.coefs[self.n], NORMS[self.m.norm], self.m.eps, link.norm, bias, act)
            if self.ys:
                self.xa, self.xb = self.xb, self.xa
            self.n += 1
        return run


# ---------------------------------------------------------------------- model and session
@dataclass
class Layer:
    mixer: LatentAttention | GatedLinearAttention | BranchMixer
    link1: Link                             # around the mixer
    ffn: DenseFFN | None = None
    link2: Link | None = None               # around the feed-forward


@dataclass
class LayeredDecoder:
    """Embedding (scaled) -> layers -> norm -> head.  `context_len` bounds a sequence's positions."""
    embedding: torch.Tensor                 # (V, C) bf16
    embedding_scale: float
    layers: list[Layer]
    final: Link
    head: torch.Tensor                      # (V, C) bf16, padded columns
    norm: str                               # "layer" | "rms"
    eps: float
    dtype: torch.dtype
    context_len: int
    streams: int = 0                        # streams of hyper-connections; 0: one residual with norms behind the sublayers
    _tables: dict = field(default_factory=dict)

    def __post_init__(self):
        for i, layer in enumerate(self.layers):
            src = getattr(layer.mixer, "kv_from", None)
            if src is None:
                continue
            other = self.layers[src].mixer if 0 <= src < i else None
            if not isinstance(other, LatentAttention) or other.kv_from is not None:
                raise ValueError(f"layer {i} reads the cache of layer {src}, which is not an earlier latent-attention layer with its own")
            if (other.rank, other.rot) != (layer.mixer.rank, layer.mixer.rot):
                raise ValueError(f"layer {i} reads the cache of layer {src}, whose latent size or rotation differs")
        links = [k for layer in self.layers for k in (layer.link1, layer.link2) if k is not None] + [self.final]
        self.coefs = [k.behind(links[i - 1] if i else None) for i, k in enumerate(links)] if self.streams else []

    @staticmethod
    def post_norm(link: Link | None) -> int | None:
        return None if link is None or link.post_norm is None else NORMS[link.post_norm]

    @property
    def width(self) -> int:
        return self.embedding.shape[1]

    @property
    def vocab_size(self) -> int:
        return self.embedding.shape[0]

    @property
    def device(self):
        return self.embedding.device

    def session(self, batch_size: int = 1, use_graph: bool = True) -> "LayeredSession":
        return LayeredSession(self, batch_size, use_graph)

    def new_caches(self, batch: int) -> list:
        """One cache or state per layer; layers that share one hold the same object."""
        caches: list = []
        for layer in self.layers:
            src = getattr(layer.mixer, "kv_from", None)
            caches.append(caches[src] if src is not None
                          else layer.mixer.new_cache(batch, self.context_len, self.dtype, self.device))
        return caches

    def tables(self, mixer):
        """The rotary tables of a mixer (layers with one rotation share them)."""
        rot = getattr(mixer, "rot", None)
        if rot is None:
            return None
        if rot not in self._tables:
            self._tables[rot] = rot.tables(self.context_len, self.device)
        return self._tables[rot]

    @torch.no_grad()
    def forward(self, tokens: torch.Tensor, pos0: int, caches: list, want: list[int], trace: list | None = None) -> torch.Tensor:
        """tokens (B, T) at positions pos0 .. -> logits (B, len(want), V) fp32 of the places `want`; caches and states are
        updated.  trace: a list that receives the residual stream (B, T, C) after every layer."""
        B, T = tokens.shape
        span = Span(B, T, pos0, self.dtype, self.device)
        res = (PromptStreams if self.streams else PromptResidual)(self, tokens, span)
        for i, (layer, cache) in enumerate(zip(self.layers, caches)):
            h = res.enter(layer.link1)
            if trace is not None and i:
                trace.append(res.total().view(B, T, -1))
            res.leave(layer.link1, layer.mixer.prompt(h, span, cache, self.tables(layer.mixer)))
            if layer.ffn is not None:
                res.leave(layer.link2, layer.ffn.prompt(res.enter(layer.link2), span))
        some = trace is None and len(want) < T          # the last norm and the head run on the wanted rows only
        if some and not want:
            return torch.empty(B, 0, self.vocab_size, dtype=torch.float32, device=self.device)
        if some:
            res.keep([b * T + w for b in range(B) for w in want])
        h = res.enter(self.final)
        logits = torch.empty(h.shape[0], self.vocab_size, dtype=torch.float32, device=self.device)
        L.linear(h, self.head, self.width, self.vocab_size, logits)
        if trace is not None:
            trace.append(res.total().view(B, T, -1))
        logits = logits.view(B, -1, self.vocab_size)
        return logits if some else logits[:, want, :]


class LayeredSession(Session):
    """Sequences of a LayeredDecoder in lockstep.  One sequence decodes through the matvec chain (every norm folded into
    the matvec behind it) in a CUDA graph; several run the step through the matrix products."""

    def __init__(self, model: LayeredDecoder, batch_size: int = 1, use_graph: bool = True):
        super().__init__(model, batch_size, model.context_len, model.vocab_size, model.device, use_graph)
        self.caches = model.new_caches(batch_size)
        for layer in model.layers:           # tables are built before anything is captured
            model.tables(layer.mixer)
        stream = max(1, model.streams) * model.width
        sizes: dict[str, int] = {"x": stream, "x2": stream}
        for layer in model.layers:
            for part in (layer.mixer, layer.ffn):
                for name, n in (part.buffers() if part is not None else {}).items():
                    sizes[name] = max(sizes.get(name, 0), n)
        self.buf = {name: torch.zeros(n, dtype=torch.float32, device=self.dev) for name, n in sizes.items()}
        if batch_size > 1:
            self.use_graph = False           # the batched step takes its position from the host

    def _on_reset(self) -> None:
        for cache in {id(c): c for c in self.caches}.values():
            cache.reset()

    def _step_state(self) -> list[torch.Tensor]:
        return [t for c in {id(c): c for c in self.caches}.values() for t in c.carried()]

    def _prefill_body(self, prompt: torch.Tensor) -> None:
        self._on_reset()
        logits = self.model.forward(prompt, 0, self.caches, [prompt.shape[1] - 1])
        self.pos.fill_(prompt.shape[1])
        self._take(logits)

    def _take(self, logits: torch.Tensor) -> None:
        self.logits.copy_(logits[:, -1, :])
        L.argmax(self.logits, self.token, None)

    def _extend_body(self, tokens: torch.Tensor, want: list[int]) -> torch.Tensor:
        last = tokens.shape[1] - 1
        all_want = list(want) if last in want else [*want, last]
        logits = self.model.forward(tokens, self.pos_host, self.caches, all_want)
        self._take(logits[:, all_want.index(last):all_want.index(last) + 1, :])
        return logits[:, :len(want), :]

    @torch.no_grad()
    def _step_body(self) -> None:
        m = self.model
        if self.B > 1:
            self._take(m.forward(self.token, self.pos_host, self.caches, [0]))
            self.pos.add_(1)
            return
        res = (DecodeStreams if m.streams else DecodeResidual)(m, self)
        for layer, cache in zip(m.layers, self.caches):
            res.leave(layer.link1, layer.mixer.decode(res.chain(layer.link1), self, cache, m.tables(layer.mixer)))
            if layer.ffn is not None:
                res.leave(layer.link2, layer.ffn.decode(res.chain(layer.link2), self))
        res.chain(m.final)(m.head, m.vocab_size, m.width, self.logits)
        L.argmax(self.logits, self.token, self.pos)

    def check(self) -> None:
        if int(L.linear_status(self.dev).item()) != 0:
            raise RuntimeError("nb_linear_bf16: a bounded wait ran out")
