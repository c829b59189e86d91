"""Thin torch-tensor wrappers over the layered-model kernels (include/nativebit_b200_layered.h): device tensors in,
device tensors out, on torch's current stream.  Weights are bf16 matrices padded by `pad_matrix`; activations are
bf16 or fp32 rows whose stride is a multiple of 8 elements (`rows_empty`)."""
from __future__ import annotations

import ctypes
from typing import NamedTuple

import torch

from . import _lib
from .ops import _DTYPE, _need_cuda, _stream

NORM_RMS, NORM_LAYER = 0, 1
ACT_NONE, ACT_SWIGLU_PAIRS, ACT_CLAMPED_GLU_PAIRS = 0, 1, 2
GLA_LOW_RANK, GLA_FORGET = 0, 1


class Act(NamedTuple):
    """What a product's epilogue does with its columns: an ACT_ constant and the constants of the clamped form."""
    kind: int = ACT_NONE
    alpha: float = 0.0
    limit: float = 0.0


PLAIN, SWIGLU = Act(), Act(ACT_SWIGLU_PAIRS)


def pad8(n: int) -> int:
    return (n + 7) // 8 * 8


def pad_matrix(w: torch.Tensor) -> torch.Tensor:
    """(N, K) -> contiguous (N, pad8(K)) with zero columns at the end."""
    n, k = w.shape
    if k % 8 == 0:
        return w.contiguous()
    out = w.new_zeros(n, pad8(k))
    out[:, :k] = w
    return out


def stack_rows(mats: list[torch.Tensor]) -> tuple[torch.Tensor, list[int]]:
    """Matrices of one input width stacked into one (every one starts at a multiple of 8 rows) and their first rows."""
    k = mats[0].shape[1]
    offs, n = [], 0
    for m in mats:
        offs.append(n)
        n += pad8(m.shape[0])
    out = mats[0].new_zeros(n, k)
    for o, m in zip(offs, mats):
        out[o:o + m.shape[0]] = m
    return pad_matrix(out), offs


def rows_empty(rows: int, cols: int, dtype: torch.dtype, device) -> torch.Tensor:
    """Uninitialised (rows, pad8(cols)) activations."""
    return torch.empty(rows, pad8(cols), dtype=dtype, device=device)


def _call(name: str, *args) -> None:
    l = _lib.layered_lib()
    _lib.check(getattr(l, name)(*args), name, l)


def _ptr(t: torch.Tensor | None, offset: int = 0):
    return None if t is None else t.data_ptr() + offset * t.element_size()


def embed_scaled(table: torch.Tensor, token: torch.Tensor, scale: float, x: torch.Tensor) -> None:
    """x (rows, C) fp32 = table[token] * scale; x (rows, streams, C): once per stream."""
    _need_cuda(table, token, x)
    _call("nb_embed_scaled", table.data_ptr(), token.data_ptr(), x.shape[0], table.shape[0], table.shape[1], scale,
          x.shape[1] if x.dim() == 3 else 1, x.data_ptr(), _stream())


def residual_norm(x: torch.Tensor, y: torch.Tensor | None, wy: torch.Tensor | None, w: torch.Tensor | None, norm: int, eps: float,
                  h: torch.Tensor | None) -> None:
    """x += norm(y) * wy (if y); h = norm(x) * w (if h)."""
    _need_cuda(x)
    _call("nb_residual_norm", x.data_ptr(), _ptr(y), _ptr(wy), _ptr(w), norm, eps, _ptr(h), _DTYPE[h.dtype] if h is not None else 0,
          h.stride(0) if h is not None else 0, x.shape[0], x.shape[1], _stream())


def _stream_args(x: torch.Tensor, x_out: torch.Tensor | None, ys: list, weights: list, y_norm: int | None, coef: torch.Tensor,
                 norm: int, eps: float, norm_w: torch.Tensor) -> "_lib.StreamArgs":
    y, w = [*ys, None, None][:2], [*weights, None, None][:2]
    return _lib.StreamArgs(x.data_ptr(), _ptr(x_out), _ptr(y[0]), _ptr(w[0]), _ptr(y[1]), _ptr(w[1]), coef.data_ptr(), norm_w.data_ptr(),
                           eps, x.shape[-2], x.shape[-1], -1 if y_norm is None else y_norm, norm)


def stream_norm(x: torch.Tensor, ys: list, weights: list, y_norm: int | None, coef: torch.Tensor, norm: int, eps: float, norm_w: torch.Tensor,
                h: torch.Tensor) -> None:
    """Hyper-connections (see nb_stream_args): the streams x (rows, streams, C) take up the results ys (up to two branches) and
    h becomes the norm of what the next sublayer reads."""
    _need_cuda(x, h)
    _call("nb_stream_norm", ctypes.byref(_stream_args(x, x, ys, weights, y_norm, coef, norm, eps, norm_w)), h.data_ptr(), _DTYPE[h.dtype],
          h.stride(0), x.shape[0], _stream())


_status: dict = {}


def linear_status(device: torch.device) -> torch.Tensor:
    """The device word that a tensor-core product sets when one of its bounded waits runs out."""
    key = (device.type, device.index)
    if key not in _status:
        _status[key] = torch.zeros(1, dtype=torch.int32, device=device)
    return _status[key]


def linear(x: torch.Tensor, w: torch.Tensor, k: int, n: int, out: torch.Tensor, bias: torch.Tensor | None = None, act: Act = PLAIN,
           rows: int | None = None) -> None:
    """out[:, :n] (or n / 2 with pairs of gate and up) = x[:, :k] . w[:n, :k]^T; bf16 x on the tensor cores, fp32 x in fp32."""
    m = x.shape[0] if rows is None else rows
    if x.dtype == torch.bfloat16:
        _call("nb_linear_bf16", x.data_ptr(), x.stride(0), w.data_ptr(), w.stride(0), _ptr(bias), *act, m, n, k, out.data_ptr(),
              _DTYPE[out.dtype], out.stride(0), linear_status(x.device).data_ptr(), _stream())
    else:
        if out.dtype != torch.float32:
            raise RuntimeError("an fp32 product has an fp32 result")
        _call("nb_linear_f32", x.data_ptr(), x.stride(0), w.data_ptr(), w.stride(0), _ptr(bias), *act, m, n, k, out.data_ptr(), out.stride(0),
              _stream())


def matvec(w: torch.Tensor, n: int, k: int, x: torch.Tensor, y: torch.Tensor, bias: torch.Tensor | None = None, act: Act = PLAIN,
           norm: int = NORM_RMS, eps: float = 0.0, norm_w: torch.Tensor | None = None, delta: torch.Tensor | None = None,
           delta_w: torch.Tensor | None = None, x_out: torch.Tensor | None = None, x_offset: int = 0) -> None:
    """One row: y = w . act, act = x, norm(x) or norm(x + norm(delta)) (see nb_matvec_bf16)."""
    a = _lib.MatvecArgs(w.data_ptr(), _ptr(bias), y.data_ptr(), _ptr(x, x_offset), _ptr(delta), _ptr(delta_w), _ptr(x_out), _ptr(norm_w),
                        eps, act.alpha, act.limit, n, k, w.stride(0), act.kind, norm)
    _call("nb_matvec_bf16", ctypes.byref(a), _stream())


def _plain_matvec(w, n, k, x, y, bias=None, act: Act = PLAIN) -> "_lib.MatvecArgs":
    return _lib.MatvecArgs(w.data_ptr(), _ptr(bias), y.data_ptr(), _ptr(x), None, None, None, None, 0.0, act.alpha, act.limit, n, k,
                           w.stride(0), act.kind, NORM_RMS)


def matvec_streams(w: torch.Tensor, n: int, k: int, y: torch.Tensor, x: torch.Tensor, x_out: torch.Tensor | None, ys: list, weights: list,
                   y_norm: int | None, coef: torch.Tensor, norm: int, eps: float, norm_w: torch.Tensor, bias: torch.Tensor | None = None,
                   act: Act = PLAIN) -> None:
    """One row behind hyper-connections: y = w . h with the h of `stream_norm`; the streams behind the results go to x_out."""
    s = _stream_args(x, x_out, ys, weights, y_norm, coef, norm, eps, norm_w)
    _call("nb_matvec_streams", ctypes.byref(_plain_matvec(w, n, k, None, y, bias, act)), ctypes.byref(s), _stream())


def matvec_pair(a: tuple, b: tuple) -> None:
    """Two products of one row each, (w, n, k, x, y), in one launch."""
    _call("nb_matvec_pair", ctypes.byref(_plain_matvec(*a)), ctypes.byref(_plain_matvec(*b)), _stream())


def latent_prepare(**kw) -> None:
    _call("nb_latent_prepare", ctypes.byref(_lib.LatentPrepareArgs(**kw)), _stream())


def latent_attention(**kw) -> None:
    _call("nb_latent_attention", ctypes.byref(_lib.LatentAttentionArgs(**kw)), _stream())


def latent_decode(**kw) -> None:
    _call("nb_latent_decode", ctypes.byref(_lib.LatentDecodeArgs(**kw)), _stream())


def gla_prefill(workspace: torch.Tensor, **kw) -> None:
    _call("nb_gla_prefill", ctypes.byref(_lib.GlaArgs(**kw)), workspace.data_ptr(), workspace.numel(), _stream())


def gla_workspace_bytes(b: int, t: int, heads: int, dim: int, vdim: int) -> int:
    return int(_lib.layered_lib().nb_gla_workspace_bytes(b, t, heads, dim, vdim))


def gla_decode(**kw) -> None:
    _call("nb_gla_decode", ctypes.byref(_lib.GlaArgs(**kw)), _stream())


def cache_append(src: torch.Tensor, offset: int, cols: int, cache: torch.Tensor, B: int, T: int, pos0: int) -> None:
    """cache[b, pos0 + t, :cols] = src[b * T + t, offset:offset + cols]."""
    _need_cuda(src, cache)
    _call("nb_cache_append", src.data_ptr(), src.stride(0), offset, cols, cache.data_ptr(), cache.shape[2], _DTYPE[src.dtype], B, T,
          cache.shape[1], pos0, _stream())


TALK_WORKSPACE = 256 << 20             # bytes of mixed scores at a time: fewer, longer launches measured faster than a block that stays in L2


def talk_workspace_bytes(b: int, t: int, heads: int, pos0: int, window: int, tiles: int) -> int:
    return int(_lib.layered_lib().nb_talk_attention_workspace_bytes(b, t, heads, pos0, window, tiles))


def talk_attention_in(workspace: torch.Tensor, args: "_lib.TalkAttentionArgs") -> None:
    _call("nb_talk_attention", ctypes.byref(args), workspace.data_ptr(), workspace.numel(), _stream())


def talk_attention(device, **kw) -> None:
    size = [kw[n] for n in ("B", "T", "H", "pos0", "window")]
    tiles = max(1, TALK_WORKSPACE // max(1, talk_workspace_bytes(*size, 1)))
    talk_attention_in(torch.empty(talk_workspace_bytes(*size, tiles), dtype=torch.uint8, device=device), _lib.TalkAttentionArgs(**kw))


def talk_decode(**kw) -> None:
    _call("nb_talk_decode", ctypes.byref(_lib.TalkDecodeArgs(**kw)), _stream())


def argmax(logits: torch.Tensor, token: torch.Tensor, pos: torch.Tensor | None) -> None:
    """token[b] = index of the largest logit (lowest among equals); pos += 1 if given."""
    _call("nb_argmax", logits.data_ptr(), logits.shape[0], logits.shape[1], token.data_ptr(), _ptr(pos), _stream())
