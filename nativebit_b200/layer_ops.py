"""Thin torch-tensor wrappers over the layered-model kernels (include/nativebit_b200_layered.h): device tensors in,
device tensors out, on torch's current stream.  Weights are bf16 matrices padded by `pad_matrix`; activations are
bf16 or fp32 rows whose stride is a multiple of 8 elements (`rows_empty`)."""
from __future__ import annotations

import ctypes

import torch

from . import _lib
from .ops import _DTYPE, _need_cuda, _stream

NORM_RMS, NORM_LAYER = 0, 1
ACT_NONE, ACT_SWIGLU_PAIRS = 0, 1


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
    """x (rows, C) fp32 = table[token] * scale."""
    _need_cuda(table, token, x)
    _call("nb_embed_scaled", table.data_ptr(), token.data_ptr(), x.shape[0], table.shape[0], table.shape[1], scale, x.data_ptr(), _stream())


def residual_norm(x: torch.Tensor, y: torch.Tensor | None, wy: torch.Tensor | None, w: torch.Tensor | None, norm: int, eps: float,
                  h: torch.Tensor | None) -> None:
    """x += norm(y) * wy (if y); h = norm(x) * w (if h)."""
    _need_cuda(x)
    _call("nb_residual_norm", x.data_ptr(), _ptr(y), _ptr(wy), _ptr(w), norm, eps, _ptr(h), _DTYPE[h.dtype] if h is not None else 0,
          h.stride(0) if h is not None else 0, x.shape[0], x.shape[1], _stream())


_status: dict = {}


def linear_status(device: torch.device) -> torch.Tensor:
    """The device word that a tensor-core product sets when one of its bounded waits runs out."""
    key = (device.type, device.index)
    if key not in _status:
        _status[key] = torch.zeros(1, dtype=torch.int32, device=device)
    return _status[key]


def linear(x: torch.Tensor, w: torch.Tensor, k: int, n: int, out: torch.Tensor, bias: torch.Tensor | None = None, act: int = ACT_NONE,
           rows: int | None = None) -> None:
    """out[:, :n] (or n / 2 with SwiGLU pairs) = x[:, :k] . w[:n, :k]^T; bf16 x on the tensor cores, fp32 x in fp32."""
    m = x.shape[0] if rows is None else rows
    if x.dtype == torch.bfloat16:
        _call("nb_linear_bf16", x.data_ptr(), x.stride(0), w.data_ptr(), w.stride(0), _ptr(bias), act, m, n, k, out.data_ptr(),
              _DTYPE[out.dtype], out.stride(0), linear_status(x.device).data_ptr(), _stream())
    else:
        if out.dtype != torch.float32:
            raise RuntimeError("an fp32 product has an fp32 result")
        _call("nb_linear_f32", x.data_ptr(), x.stride(0), w.data_ptr(), w.stride(0), _ptr(bias), act, m, n, k, out.data_ptr(), out.stride(0),
              _stream())


def matvec(w: torch.Tensor, n: int, k: int, x: torch.Tensor, y: torch.Tensor, bias: torch.Tensor | None = None, act: int = ACT_NONE,
           norm: int = NORM_RMS, eps: float = 0.0, norm_w: torch.Tensor | None = None, delta: torch.Tensor | None = None,
           delta_w: torch.Tensor | None = None, x_out: torch.Tensor | None = None, x_offset: int = 0) -> None:
    """One row: y = w . act, act = x, norm(x) or norm(x + norm(delta)) (see nb_matvec_bf16)."""
    a = _lib.MatvecArgs(w.data_ptr(), _ptr(bias), y.data_ptr(), _ptr(x, x_offset), _ptr(delta), _ptr(delta_w), _ptr(x_out), _ptr(norm_w),
                        eps, n, k, w.stride(0), act, norm)
    _call("nb_matvec_bf16", ctypes.byref(a), _stream())


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


def argmax(logits: torch.Tensor, token: torch.Tensor, pos: torch.Tensor | None) -> None:
    """token[b] = index of the largest logit (lowest among equals); pos += 1 if given."""
    _call("nb_argmax", logits.data_ptr(), logits.shape[0], logits.shape[1], token.data_ptr(), _ptr(pos), _stream())
