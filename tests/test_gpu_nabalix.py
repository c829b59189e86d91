"""Nabalix on the GPU against the plain oracle: every kernel alone, then whole models — prompts, portions, decoding,
batches, sessions used again, greedy generation, the trace runner and the command line."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import nabalix_cases as nc
from gpu_util import BF16, F32, TOL, close, cu, f64, rel, rounded, rounding
from oracle import hybrid_oracle as HO
from oracle import nabalix_oracle as O

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.fixture(scope="module", autouse=True)
def dev():
    if not torch.cuda.is_available():
        pytest.fail("needs a CUDA device")
    from nativebit_b200.build import build_library
    build_library(which="layered")
    return torch.device("cuda:0")


# ---------------------------------------------------------------- dense pieces
def test_embedding_in_streams(dev):
    from nativebit_b200 import layer_ops as L
    table = torch.randn(37, 50, device=dev).bfloat16()
    tok = torch.tensor([0, 36, 5], device=dev)
    x = torch.empty(3, 4, 50, device=dev)
    L.embed_scaled(table, tok, 1.0, x)
    assert torch.equal(x, table[tok].float()[:, None].expand(-1, 4, -1))


@pytest.mark.parametrize("m,n,k", [(1, 8, 8), (70, 130, 72), (130, 300, 264), (513, 264, 100), (3, 50, 50)])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_clamped_glu_epilogue(dev, m, n, k, dtype):
    from nativebit_b200 import layer_ops as L
    r = np.random.default_rng(m + n + k)
    w = rounded(r.standard_normal((n, k)) * 2 / np.sqrt(k), BF16)
    x = rounded(r.standard_normal((m, k)), dtype)
    xt, wt = L.rows_empty(m, k, dtype, dev), L.pad_matrix(cu(w, BF16))
    xt[:, :k] = cu(x, dtype)
    act = L.Act(L.ACT_CLAMPED_GLU_PAIRS, 1.3, 0.9)
    z = x @ w.T
    g, u = np.minimum(z[:, ::2], 0.9), np.clip(z[:, 1::2], -0.9, 0.9)
    ref = g * HO.sigmoid(1.3 * g) * (u + 1)
    assert (z[:, ::2] > 0.9).any() and (np.abs(z[:, 1::2]) > 0.9).any()
    out = L.rows_empty(m, n // 2, dtype, dev)
    L.linear(xt, wt, k, n, out, act=act)
    close(out[:, :n // 2], ref, max(TOL[dtype], 1e-5))
    if dtype == F32:
        y = torch.empty(n // 2, device=dev)
        L.matvec(wt, n, k, xt[0, :k].contiguous(), y, act=act)
        close(y, ref[0], 1e-5)
        assert np.allclose(O.clamped_glu(z[:, ::2], z[:, 1::2], 0.9), np.minimum(z[:, ::2], 0.9) * HO.sigmoid(1.702 * g) * (u + 1))


def stream_case(rows, S, C, branches, normed, seed=0):
    """Inputs of a step of the streams and what it gives: (dict, streams behind it, h)."""
    r = np.random.default_rng(seed + S * C + branches)
    x, ys = r.standard_normal((rows, S, C)).astype(np.float32), (2.0 + r.standard_normal((branches, rows, C))).astype(np.float32)
    ws = r.standard_normal((branches, C)).astype(np.float32)
    share, mix, read = r.standard_normal(S), r.standard_normal((S, S)), r.uniform(0.2, 1, S)
    nw = (1 + 0.3 * r.standard_normal(C)).astype(np.float32)
    y = sum((HO.rms_norm(a.astype(np.float64), 1.0, 1e-5) if normed else a) * w for a, w in zip(ys, ws)) if branches else 0.0
    new = np.einsum("st,rsc->rtc", mix, x.astype(np.float64)) + (share[:, None] * np.asarray(y)[:, None] if branches else 0.0) if branches else x
    u = np.einsum("s,rsc->rc", read, new)
    from nativebit_b200.layered import Link
    t = lambda a: torch.from_numpy(np.asarray(a))                                           # noqa: E731
    coef = Link(None, read=t(read)).behind(Link(None, share=t(share), mix=t(mix)) if branches else None)
    case = dict(x=cu(x), ys=[cu(a) for a in ys], ws=[cu(a) for a in ws], coef=coef.cuda(), nw=cu(nw), y_norm=0 if normed else None)
    return case, new, HO.rms_norm(u, nw, 1e-5)


SIZES = [(1, 50), (2, 72), (3, 264), (4, 1500), (2, 4096), (5, 100), (8, 2052)]


@pytest.mark.parametrize("S,C", SIZES)
@pytest.mark.parametrize("branches,normed", [(0, False), (1, False), (1, True), (2, True), (2, False)])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_stream_norm(dev, S, C, branches, normed, dtype):
    from nativebit_b200 import layer_ops as L
    c, new, ref = stream_case(5, S, C, branches, normed)
    h = L.rows_empty(5, C, dtype, dev)
    L.stream_norm(c["x"], c["ys"], c["ws"], c["y_norm"], c["coef"], L.NORM_RMS, 1e-5, c["nw"], h)
    close(c["x"], new, 1e-5)
    close(h[:, :C], ref, max(TOL[dtype], 1e-5))


@pytest.mark.parametrize("S,C", SIZES)
@pytest.mark.parametrize("branches,normed", [(0, False), (1, False), (2, True)])
@pytest.mark.parametrize("n", [1, 6, 300])
def test_matvec_behind_streams(dev, S, C, branches, normed, n):
    from nativebit_b200 import layer_ops as L
    c, new, h = stream_case(1, S, C, branches, normed, 7)
    r = np.random.default_rng(n)
    w = rounded(r.standard_normal((n, C)) / np.sqrt(C), BF16)
    wt, y, x2 = L.pad_matrix(cu(w, BF16)), torch.empty(n, device=dev), torch.full((S, C), 7.0, device=dev)
    args = (c["x"][0], x2, c["ys"], c["ws"], c["y_norm"], c["coef"], L.NORM_RMS, 1e-5, c["nw"])
    L.matvec_streams(wt, n, C, y, *args)
    ref = w @ h[0]
    scale = np.abs(w).max() * np.abs(h).max() * np.sqrt(C)
    assert np.abs(f64(y) - ref).max() <= 3e-6 * max(scale, np.abs(ref).max())
    if branches:
        close(x2, new[0], 1e-5)
    else:
        assert (x2 == 7.0).all()                                    # nothing to take up: the streams stay where they are
    if n % 2 == 0:
        b, out = cu(r.standard_normal(n)), torch.empty(n // 2, device=dev)
        L.matvec_streams(wt, n, C, out, *args, b, L.Act(L.ACT_CLAMPED_GLU_PAIRS, 1.702, 0.5))
        z = ref + f64(b)
        close(out, O.clamped_glu(z[::2], z[1::2], 0.5), 2e-5)


@pytest.mark.parametrize("a,b", [((50, 72), (131, 50)), ((1, 8), (300, 264)), ((640, 520), (640, 1000)), ((33, 4100), (33, 8)), ((64, 9000), (7, 30))])
def test_matvec_pair(dev, a, b):
    from nativebit_b200 import layer_ops as L
    r = np.random.default_rng(a[0] + b[1])
    jobs, refs = [], []
    for n, k in (a, b):
        w, x = rounded(r.standard_normal((n, k)) / np.sqrt(k), BF16), r.standard_normal(k).astype(np.float32)
        jobs.append((L.pad_matrix(cu(w, BF16)), n, k, cu(x), torch.empty(n, device=dev)))
        refs.append(w @ x.astype(np.float64))
    L.matvec_pair(*jobs)
    for j, ref in zip(jobs, refs):
        assert np.abs(f64(j[4]) - ref).max() <= 1e-5 * max(1.0, np.abs(ref).max())


# ---------------------------------------------------------------- mixed-head attention, alone
SHAPES = [dict(H=6, G=2, D=20, V=28), dict(H=1, G=1, D=7, V=9), dict(H=12, G=3, D=64, V=136), dict(H=5, G=5, D=128, V=64), dict(H=20, G=4, D=32, V=40),
          dict(H=34, G=17, D=16, V=8), dict(H=44, G=4, D=24, V=264), dict(H=8, G=2, D=72, V=200)]


def attention_inputs(shape, B, N, dtype, seed, at, loud):
    """Random q, k, v and constants; the key `loud` would take nearly all the weight of queries that see it (its score's sign
    follows the talk matrix's row sums, which are kept positive)."""
    H, G, D, V = (shape[k] for k in "HGDV")
    r = np.random.default_rng(seed)
    q, k, v = (rounded(r.standard_normal((B, N, n, d)), dtype) for n, d in ((H, D), (G, D), (G, V)))
    q = np.abs(q)
    if loud is not None:
        k[:, loud] = 1.0
    talk = (np.eye(H) + 0.5 / H + 0.2 / np.sqrt(H) * r.standard_normal((H, H))).astype(np.float32)
    r1, r2 = r.uniform(0, 0.5, H).astype(np.float32), r.uniform(0, 0.6, H).astype(np.float32)
    gate = rounded(r.standard_normal((B, N, H * V)), dtype)
    return q, k, v, talk, r1, r2, gate


def penalty_table(r1, r2, n):
    return cu(r1.astype(np.float64)[:, None] * np.log1p(r2.astype(np.float64)[:, None] * np.arange(n))).contiguous()


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("T,pos0,window,tiles", [(5, 0, 3, 1), (64, 0, 64, 1), (65, 0, 64, 1), (150, 0, 63, 2), (2, 70, 9, 1), (70, 33, 40, 9), (33, 100, 1, 1),
                                                 (90, 20, 1000, 1), (200, 61, 129, 3)])
def test_talk_attention(dev, shape, dtype, T, pos0, window, tiles):
    """A portion at pos0 .. of two sequences against the oracle's attention over all positions; one key leaves the window in the
    middle of the portion and dominates until then.  The workspace holds `tiles` query tiles at a time."""
    from nativebit_b200 import _lib
    from nativebit_b200 import layer_ops as L
    H, G, D, V = (shape[k] for k in "HGDV")
    B, N = 2, pos0 + T
    loud = max(0, N - window - T // 2 - 1)
    q, k, v, talk, r1, r2, gate = attention_inputs(shape, B, N, dtype, T + pos0 + D, pos0, loud)
    scale, cap = 4.0 / np.sqrt(D), 8.0
    first = max(0, pos0 - window + 1)
    ref = np.stack([O.mixed_head_attention(q[b, first:], k[b, first:], v[b, first:], scale, cap, r1, r2, talk.astype(np.float64), window)[pos0 - first:]
                    for b in range(B)]).reshape(B * T, H * V)
    ref = ref * HO.sigmoid(gate[:, pos0:].reshape(B * T, H * V))
    ctx = N + 3
    v_off = L.pad8(G * D)
    cols = v_off + G * V
    off = 16
    src = torch.full((B * T, L.pad8(off + cols) + 8), 9.0, dtype=dtype, device=dev)
    cache = torch.full((B, ctx, v_off + L.pad8(G * V)), float("nan"), dtype=dtype, device=dev)
    for dst, lo, hi in ((cache, first, pos0), (src.view(B, T, -1), pos0, N)):               # earlier rows sit in the cache
        at = 0 if dst is cache else off
        rows = dst[:, first:pos0] if dst is cache else dst
        rows[:, :, at:at + G * D] = cu(k[:, lo:hi].reshape(B, hi - lo, G * D), dtype)
        rows[:, :, at + v_off:at + cols] = cu(v[:, lo:hi].reshape(B, hi - lo, G * V), dtype)
    L.cache_append(src, off, cols, cache, B, T, pos0)
    assert torch.equal(cache[:, pos0:N, :G * D], src.view(B, T, -1)[:, :, off:off + G * D])
    assert torch.equal(cache[:, pos0:N, v_off:cols], src.view(B, T, -1)[:, :, off + v_off:off + cols])
    assert cache[:, N:].isnan().all() and cache[:, :first].isnan().all()
    qt, gt, out = (L.rows_empty(B * T, n, dtype, dev) for n in (H * D, H * V, H * V))
    qt[:, :H * D] = cu(q[:, pos0:].reshape(B * T, -1), dtype)
    gt[:, :H * V] = cu(gate[:, pos0:].reshape(B * T, -1), dtype)
    n_pen = min(window, ctx)
    pen, tk = penalty_table(r1, r2, n_pen), cu(talk)
    size = L.talk_workspace_bytes(B, T, H, pos0, window, tiles)
    ws = torch.full((size,), 255, dtype=torch.uint8, device=dev)
    a = _lib.TalkAttentionArgs(q=qt.data_ptr(), cache=cache.data_ptr(), gate=gt.data_ptr(), out=out.data_ptr(), penalty=pen.data_ptr(),
                               talk=tk.data_ptr(), scale=scale, softcap=cap, dtype=L._DTYPE[dtype], B=B, T=T, H=H, G=G, dim=D, vdim=V, ctx=ctx,
                               ldc=cache.shape[2], v_off=v_off, ldq=qt.stride(0), ldg=gt.stride(0), ldo=out.stride(0), pos0=pos0, window=window,
                               n_pen=n_pen)
    L.talk_attention_in(ws, a)
    close(out[:, :H * V], ref, 2e-5 if dtype == F32 else 2.0 ** -7)


def dense_attention(q, k, v, scale, cap, r1, r2, talk, window):
    """O.mixed_head_attention over whole matrices (the oracle's own test holds the two together)."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    i = np.arange(T)
    s = np.einsum("ihd,jhd->hij", q, np.repeat(k, rep, 1), optimize=True) * scale
    far = np.maximum(i[:, None] - i[None], 0)
    s = cap * np.tanh(s / cap) - r1.astype(np.float64)[:, None, None] * np.log1p(r2.astype(np.float64)[:, None, None] * far)
    s = np.tensordot(talk.astype(np.float64), s, 1)
    s[:, (i[None, :] > i[:, None]) | (i[:, None] - i[None, :] >= window)] = -np.inf
    p = np.exp(s - s.max(-1, keepdims=True))
    return np.einsum("hij,jhd->ihd", p / p.sum(-1, keepdims=True), np.repeat(v, rep, 1), optimize=True)


@pytest.mark.parametrize("shape", [SHAPES[0], SHAPES[2], SHAPES[5], dict(H=10, G=5, D=48, V=32), dict(H=9, G=3, D=40, V=24),
                                   dict(H=20, G=4, D=160, V=16)])
@pytest.mark.parametrize("B,T,pos0,window,tiles", [(3, 1400, 30, 700, 99), (1, 330, 100, 290, 2), (3, 1400, 0, 2000, 7)])
def test_talk_attention_over_many_steps(dev, shape, B, T, pos0, window, tiles):
    """Windows of many tiles and enough queries that a CTA walks several steps of keys (one sequence, B times)."""
    from nativebit_b200 import layer_ops as L
    H, G, D, V = (shape[k] for k in "HGDV")
    N = pos0 + T
    q, k, v, talk, r1, r2, gate = attention_inputs(shape, 1, N, BF16, T + D, pos0, max(0, N - window - T // 3))
    scale, cap = 4.0 / np.sqrt(D), 8.0
    ref = np.tile(dense_attention(q[0], k[0], v[0], scale, cap, r1, r2, talk, window)[pos0:].reshape(T, H * V), (B, 1))
    q, k, v, gate = (np.repeat(x, B, 0) for x in (q, k, v, gate))
    ref = ref * HO.sigmoid(gate[:, pos0:].reshape(B * T, H * V))
    v_off = L.pad8(G * D)
    cache = torch.zeros(B, N, v_off + L.pad8(G * V), dtype=BF16, device=dev)
    cache[:, :, :G * D], cache[:, :, v_off:v_off + G * V] = cu(k.reshape(B, N, G * D), BF16), cu(v.reshape(B, N, G * V), BF16)
    qt, gt, out = (L.rows_empty(B * T, n, BF16, dev) for n in (H * D, H * V, H * V))
    qt[:, :H * D], gt[:, :H * V] = cu(q[:, pos0:].reshape(B * T, H * D), BF16), cu(gate[:, pos0:].reshape(B * T, H * V), BF16)
    n_pen = min(window, N)
    pen, tk = penalty_table(r1, r2, n_pen), cu(talk)
    from nativebit_b200 import _lib
    a = _lib.TalkAttentionArgs(q=qt.data_ptr(), cache=cache.data_ptr(), gate=gt.data_ptr(), out=out.data_ptr(), penalty=pen.data_ptr(),
                               talk=tk.data_ptr(), scale=scale, softcap=cap, dtype=L._DTYPE[BF16], B=B, T=T, H=H, G=G, dim=D, vdim=V, ctx=N,
                               ldc=cache.shape[2], v_off=v_off, ldq=qt.stride(0), ldg=gt.stride(0), ldo=out.stride(0), pos0=pos0, window=window,
                               n_pen=n_pen)
    ws = torch.full((L.talk_workspace_bytes(B, T, H, pos0, window, tiles),), 255, dtype=torch.uint8, device=dev)
    L.talk_attention_in(ws, a)
    close(out[:, :H * V], ref, 2.0 ** -7)


def test_talk_attention_without_its_options(dev):
    """No cap, no penalty, no gate, no window, heads not mixed: ordinary grouped attention."""
    from nativebit_b200 import _lib
    from nativebit_b200 import layer_ops as L
    T, H, G, D, V = 100, 4, 2, 24, 16
    for dtype in (F32, BF16):
        r = np.random.default_rng(0)
        q, k, v = (rounded(r.standard_normal((T, n, d)), dtype) for n, d in ((H, D), (G, D), (G, V)))
        ref = HO.windowed_attention(q, np.repeat(k, 2, 1), np.repeat(v, 2, 1), 0.4, None).reshape(T, H * V)
        cache = torch.zeros(1, T, G * (D + V), dtype=dtype, device=dev)
        cache[0, :, :G * D], cache[0, :, G * D:] = cu(k.reshape(T, -1), dtype), cu(v.reshape(T, -1), dtype)
        qt, out, eye = cu(q.reshape(T, -1), dtype), torch.empty(T, H * V, dtype=dtype, device=dev), torch.eye(H, device=dev)
        a = _lib.TalkAttentionArgs(q=qt.data_ptr(), cache=cache.data_ptr(), out=out.data_ptr(), talk=eye.data_ptr(), scale=0.4, softcap=0.0,
                                   dtype=L._DTYPE[dtype], B=1, T=T, H=H, G=G, dim=D, vdim=V, ctx=T, ldc=cache.shape[2], v_off=G * D, ldq=H * D,
                                   ldg=0, ldo=H * V, pos0=0, window=0, n_pen=0)
        L.talk_attention_in(torch.empty(L.talk_workspace_bytes(1, T, H, 0, 0, 2), dtype=torch.uint8, device=dev), a)
        close(out, ref, 1e-5 if dtype == F32 else 2.0 ** -7)


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("pos,window", [(0, 5), (4, 5), (5, 5), (63, 64), (64, 64), (200, 17), (300, 1000), (77, 1), (1500, 1400)])
def test_talk_decode(dev, shape, dtype, pos, window):
    """One position of two sequences: keys and values are appended to the cache and attended to.  The key that just left the
    window would dominate, the one just inside stands out."""
    from nativebit_b200 import layer_ops as L
    H, G, D, V = (shape[k] for k in "HGDV")
    if pos > 1000 and H > 20:
        pytest.skip("large and slow in the oracle")
    B, N = 2, pos + 1
    q, k, v, talk, r1, r2, gate = attention_inputs(shape, B, N, F32, pos + D, pos, None)
    for j, loud in ((pos - window, 3.0), (pos - window + 1, 1.0)):
        if 0 <= j < pos:
            k[:, j] = loud
    raw_k, raw_v = k[:, pos].astype(np.float32), v[:, pos].astype(np.float32)
    k, v = rounded(k, dtype), rounded(v, dtype)
    scale, cap = 3.0 / np.sqrt(D), 7.0
    lo = max(0, pos - window + 1)
    ref = np.stack([O.mixed_head_attention(np.broadcast_to(q[b, pos], (N - lo, H, D)), k[b, lo:], v[b, lo:], scale, cap, r1, r2, talk.astype(np.float64),
                                           window)[-1] for b in range(B)]).reshape(B, H * V) * HO.sigmoid(gate[:, pos])
    ctx = pos + 4
    v_off = L.pad8(G * D)
    cache = torch.zeros(B, ctx, v_off + L.pad8(G * V), dtype=dtype, device=dev)
    cache[:, :N, :G * D], cache[:, :N, v_off:v_off + G * V] = cu(k.reshape(B, N, -1), dtype), cu(v.reshape(B, N, -1), dtype)
    want_row = cache[:, pos].clone()
    cache[:, :lo] = float("nan")                                    # what the window does not cover is not read
    cache[:, pos:] = float("nan")
    k_off = H * D + 3
    g_off = k_off + v_off + G * V + 2
    p = torch.zeros(B, g_off + H * V, device=dev)
    p[:, :H * D], p[:, k_off:k_off + G * D] = cu(q[:, pos].reshape(B, -1)), cu(raw_k.reshape(B, -1))
    p[:, k_off + v_off:k_off + v_off + G * V], p[:, g_off:] = cu(raw_v.reshape(B, -1)), cu(gate[:, pos])
    out, pt = torch.empty(B, H * V, device=dev), torch.tensor([pos], device=dev)
    n_pen = min(window, ctx)
    pen, tk = penalty_table(r1, r2, n_pen), cu(talk)
    torch.cuda.synchronize()                                        # cached rows are requested ahead of the dependency wait
    L.talk_decode(p=p.data_ptr(), cache=cache.data_ptr(), penalty=pen.data_ptr(), talk=tk.data_ptr(), pos=pt.data_ptr(), out=out.data_ptr(), scale=scale,
                  softcap=cap, cache_dtype=L._DTYPE[dtype], B=B, H=H, G=G, dim=D, vdim=V, ctx=ctx, ldc=cache.shape[2], v_off=v_off, ldp=p.shape[1],
                  q_off=0, k_off=k_off, g_off=g_off, ldo=H * V, window=window, n_pen=n_pen)
    close(out, ref, 2e-5 if dtype == F32 else 5e-5)                 # bf16: softmax weights as two bf16 terms
    assert torch.equal(cache[:, pos], want_row) and cache[:, N:].isnan().all()


# ---------------------------------------------------------------- the forget-gate recurrence, alone
@pytest.mark.parametrize("H,D,V", [(3, 20, 28), (2, 96, 136), (1, 5, 11), (4, 136, 40), (2, 64, 64), (1, 40, 264)])
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("bias", [1.5, -30.0, 40.0])
def test_forget_recurrence(dev, H, D, V, dtype, bias):
    """Portions of several sizes (cut inside chunks and sub-blocks) continue one another; gates from closed to wide open.  With
    fp32 activations single tokens go through the decode kernel in between."""
    from nativebit_b200 import layer_ops as L
    from nativebit_b200.layered import BranchMixer, ForgetLinearAttention
    B, T, eps, C = 2, 213, 1e-5, 24
    r = np.random.default_rng(D + V)
    z = lambda n, k: torch.zeros(n, k, dtype=BF16, device=dev)                              # noqa: E731
    fb = (bias + r.standard_normal(H * D) * 2).astype(np.float32)
    lower = np.maximum(r.uniform(-0.5, 0.95, H * D), 0.0).astype(np.float32)
    nw = (1 + 0.2 * r.standard_normal(V)).astype(np.float32)
    rec = ForgetLinearAttention(heads=H, dim=D, vdim=V, eps=eps, w_q=z(H * D, C), w_f=z(H * D, C), f_bias=cu(fb), lower=cu(lower), w_v=z(H * V, C),
                                norm_w=cu(nw), w_out=z(C, H * V))
    n_in = BranchMixer("recurrence", [rec]).n_in
    p, parts = torch.zeros(B, T, n_in, dtype=dtype, device=dev), {}
    for n, off, cols in (("q", rec.q_off, H * D), ("f", rec.f_off, H * D), ("v", rec.v_off, H * V)):
        parts[n] = rounded(r.standard_normal((B, T, cols)), dtype)
        p[:, :, off:off + cols] = cu(parts[n], dtype)

    def oracle(dt):
        outs, ends = [], []
        for b in range(B):
            q, f, v = (parts[n][b].astype(dt) for n in ("q", "f", "v"))
            gate, write = O.forget_gate(f + fb.astype(dt), lower.astype(dt))
            o, S = O.forget_recurrence(HO.silu(q).reshape(T, H, D), v.reshape(T, H, V), gate.reshape(T, H, D), write.reshape(T, H, D))
            assert o.dtype == dt
            outs.append(HO.rms_norm(o, nw, dt(eps)).reshape(T, H * V))
            ends.append(S)
        return np.stack(outs), np.stack(ends)
    ref, ends = oracle(np.float64)
    # outputs are normed, so where q . k cancels the norm shows the rounding: the limit follows the oracle in fp32
    lim_o, lim_s = (rounding(x, y, 1e-5) for x, y in zip((ref, ends), oracle(np.float32)))

    def run(cuts, single=False):
        st = rec.new_cache(B, 0, dtype, dev)
        out, at = torch.empty(B, T, H * V, dtype=dtype, device=dev), 0
        for n in cuts:
            src, dst = p[:, at:at + n].contiguous(), torch.empty(B, n, H * V, dtype=dtype, device=dev)
            if n == 1 and single:
                L.gla_decode(**rec._args(src, n_in, dst, H * V, st, F32, B, 1))
            else:
                ws = torch.full((L.gla_workspace_bytes(B, n, H, D, V),), 255, dtype=torch.uint8, device=dev)
                L.gla_prefill(ws, **rec._args(src, n_in, dst, H * V, st, dtype, B, n))
            out[:, at:at + n] = dst
            at += n
        assert at == T
        close(out, ref, lim_o if dtype == F32 else max(2.0 ** -7, 16 * lim_o))     # bf16: products of two-term operands, bf16 output
        close(st.s[..., :V], ends, lim_s if dtype == F32 else 1e-4)
        assert (st.s[..., V:] == 0).all()
    run([T])
    run([2, 3, 64, 15, 17, 1, 100, 11])
    if dtype == F32:
        run([1] * T, True)
        run([66] + [1] * 40 + [65, 2] + [1] * 40, True)


# ---------------------------------------------------------------- whole models
_built, _refs, _limits = {}, {}, {}
SHARP = 4.0


def model_of(name, dtype, context=400):
    from nativebit_b200 import nabalix
    if (name, dtype, context) not in _built:
        cfg = nc.CASES[name]
        w = nc.weights(cfg, seed=5, sharp=SHARP)
        wd = {k: v.cuda() for k, v in w.items()}
        m = nabalix.build(cfg, lambda n, s: wd[n], dtype, context)
        torch.cuda.synchronize()
        _built[name, dtype, context] = (cfg, nc.as_numpy(w), m)
    return _built[name, dtype, context]


def reference(name, n, seed=0):
    """(tokens, logits, residual stream) of the oracle; also sets the limits of the case.  The weights are made so that scores
    are sharp, which enlarges rounding: the limits are six times what the oracle itself loses in fp32, and three times what
    it loses when the products' inputs and outputs are rounded to bf16."""
    if (name, n, seed) not in _refs:
        cfg = nc.CASES[name]
        w = nc.as_numpy(nc.weights(cfg, seed=5, sharp=SHARP))
        toks = nc.tokens(cfg, n, seed)
        logits, stream = O.forward(cfg, w, toks)
        l32, _ = O.forward(cfg, w, toks, np.float32)
        assert l32.dtype == np.float32
        _refs[name, n, seed] = (toks, logits, stream)
        _limits[name, F32] = max(_limits.get((name, F32), 5e-6), 6 * rel(l32, logits))
        if (name, BF16) not in _limits or n >= 200:
            l16, _ = O.forward(cfg, w, toks, cast=lambda a: rounded(a, BF16))
            _limits[name, BF16] = max(_limits.get((name, BF16), 0.0), 3 * rel(l16, logits))
    return _refs[name, n, seed]


def limit(name, dtype):
    return _limits[name, dtype]


def test_the_reference_shows_faults(dev):
    """The cases' weights are such that a window one off, an unmixed head, a lost state or a missing penalty shows in the oracle's
    logits by far more than the limits."""
    import copy
    cfg, w, _ = model_of("mixed", F32)
    toks, logits, _ = reference("mixed", 210)

    def moved(change_cfg=None, change_w=None):
        c, x = copy.deepcopy(cfg), dict(w)
        if change_cfg:
            change_cfg(c["layers"])
        if change_w:
            x.update(change_w)
        return rel(O.forward(c, x, toks)[0], logits)
    floor = 20 * max(limit("mixed", F32), 1e-4)
    for i in range(3):
        for d in (-1, 1):
            assert moved(lambda ls: ls[i]["mixer"]["left"]["mask"].update(size=cfg["layers"][i]["mixer"]["left"]["mask"]["size"] + d)) > floor
        for n in ("mix.left.talk", "mix.left.r1", "mix.right.lower", "hc1.mix"):
            name = f"l{i}.{n}"
            assert moved(change_w={name: w[name].T if n == "mix.left.talk" else w[name] * 0.5}) > floor, name


@pytest.mark.parametrize("name", sorted(nc.CASES))
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_prompt_and_residual_stream(dev, name, dtype):
    cfg, _, m = model_of(name, dtype)
    toks, logits, stream = reference(name, 210)
    trace = []
    got = m.forward(cu(toks[None], torch.long), 0, m.new_caches(1), list(range(len(toks))), trace=trace)[0]
    assert rel(f64(got), logits) <= limit(name, dtype)
    for i, (a, b) in enumerate(zip(trace, stream)):
        err = np.abs(f64(a[0]) - b).max() / np.abs(b).max()
        assert err <= 4 * limit(name, dtype), (i, err)
    assert len(trace) == len(cfg["layers"])


@pytest.mark.parametrize("name", sorted(nc.CASES))
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("cuts", [[210], [2] * 105, [150] + [1] * 60, [7, 1, 1, 2, 64, 3, 65, 1, 1, 31, 34], [1] * 210])
def test_portions_and_decoding(dev, name, dtype, cuts):
    _, _, m = model_of(name, dtype)
    toks, logits, _ = reference(name, 210)
    s = m.session()
    got, at = [], 0
    for n in cuts:
        got.append(s.extend(cu(toks[None, at:at + n], torch.long), list(range(n)))[0].clone())
        at += n
    assert at == len(toks) and s.pos_host == at and int(s.pos.item()) == at
    assert rel(f64(torch.cat(got)), logits) <= limit(name, dtype)
    s.check()


def test_wanted_places_only(dev):
    _, _, m = model_of("mixed", F32)
    toks, logits, _ = reference("mixed", 210)
    s = m.session()
    t = cu(toks[None], torch.long)
    assert s.extend(t[:, :50], []).shape == (1, 0, 131)
    got = s.extend(t[:, 50:90], [39, 0, 7])[0]
    assert rel(f64(got), logits[[89, 50, 57]]) <= limit("mixed", F32)
    assert int(s.token[0, 0]) == int(logits[89].argmax())           # the last place decides the next token even if it comes first
    assert rel(f64(s.extend(t[:, 90:91], [0])[0]), logits[90:91]) <= limit("mixed", F32)


@pytest.mark.parametrize("name", ["order", "mixed"])
def test_sessions_are_used_again(dev, name):
    """A reset gives the cache and state back: the next request does not see the one before, with or without a captured step."""
    _, _, m = model_of(name, F32)
    s = m.session()
    other = cu(nc.tokens(nc.CASES[name], 300, seed=9)[None], torch.long)
    for seed, n in ((0, 210), (1, 64), (2, 23)):
        toks, logits, _ = reference(name, n, seed)
        t = cu(toks[None], torch.long)
        got = [s.extend(t[:, :n - 9], list(range(n - 9)))[0].clone()] + [s.extend(t[:, i:i + 1], [0])[0].clone() for i in range(n - 9, n)]
        assert rel(f64(torch.cat(got)), logits) <= limit(name, F32)
        s.reset()
        s.extend(other, [0])                                        # fills every row with something else
        s.reset()


def test_batches_equal_single_sequences(dev):
    for dtype in (F32, BF16):
        _, _, m = model_of("mixed", dtype)
        refs = [reference("mixed", 100, seed) for seed in (3, 4, 5)]
        t = cu(np.stack([r[0] for r in refs]), torch.long)
        s, at, got = m.session(3), 0, []
        for n in (64, 7, 1, 1, 2, 24, 1):
            got.append(s.extend(t[:, at:at + n], list(range(n))).clone())
            at += n
        got = f64(torch.cat(got, 1))
        for b, (_, logits, _) in enumerate(refs):
            assert rel(got[b], logits) <= limit("mixed", dtype)


def test_long_decoding_slides_every_window(dev):
    """Hundreds of decoded tokens from a short prompt; the captured step equals the eager one."""
    _, _, m = model_of("mixed", F32)
    toks, logits, _ = reference("mixed", 330, 7)
    t = cu(toks[None], torch.long)
    got = {}
    for graph in (True, False):
        s = m.session(use_graph=graph)
        s.extend(t[:, :3], [2])
        got[graph] = torch.cat([s.extend(t[:, i:i + 1], [0])[0].clone() for i in range(3, 330)])
        assert rel(f64(got[graph]), logits[3:]) <= limit("mixed", F32)
    assert torch.equal(got[True], got[False])


def greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(O.forward(cfg, w, toks)[0][-1].argmax()))
    return toks[len(prompt):]


def test_greedy_generation(dev):
    cfg, w, m = model_of("mixed", F32)
    prompts = [nc.tokens(cfg, 12, s) for s in (0, 1)]
    want = [greedy(cfg, w, p, 14) for p in prompts]
    s = m.session()
    for p, ref in zip(prompts, want):                               # the second prompt replays the captured prefill
        assert s.generate(cu(p[None], torch.long), 14)[0].tolist() == ref
    assert m.session(2).generate(cu(np.stack(prompts), torch.long), 14).tolist() == want
    assert s.generate(cu(prompts[0][None], torch.long), 14)[0].tolist() == want[0]


def test_the_end_of_the_context_is_refused(dev):
    _, _, m = model_of("mixed", F32, context=20)                    # shorter than two of the windows
    toks, logits, _ = reference("mixed", 100, 3)
    s, t = m.session(), cu(toks[None, :20], torch.long)
    s.extend(t[:, :18], [])
    with pytest.raises(RuntimeError):
        s.extend(t[:, :3], [])
    got = torch.cat([s.extend(t[:, i:i + 1], [0])[0].clone() for i in (18, 19)])
    assert rel(f64(got), logits[18:20]) <= limit("mixed", F32)
    with pytest.raises(RuntimeError):
        s.step()


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    from nativebit_b200.weights import write_safetensors
    d = tmp_path_factory.mktemp("model")
    (d / "config.json").write_text(json.dumps(nc.CASES["mixed"]))
    write_safetensors(str(d / "model.safetensors"), nc.weights(nc.CASES["mixed"], seed=5, sharp=SHARP))
    return d


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_runner(dev, folder, tmp_path, dtype):
    """Requests one after the other and two at a time, through the program and its files."""
    a, b = reference("mixed", 100, 3), reference("mixed", 210)
    steps = [({"id": "x", "n": 40, "want": [0, 39]},), ({"id": "x", "n": 1, "want": [0]},), ({"id": "x", "n": 59, "want": []},),
             ({"id": "y", "n": 150, "want": [149, 3]},), ({"id": "z", "n": 100, "want": [99]}, {"id": "y", "n": 2, "want": [1]})]
    data = {"x": a, "y": b, "z": a}
    at, lines, want = {}, [], []
    for i, entries in enumerate(steps):
        out, ref = [], []
        for e in entries:
            lo = at.get(e["id"], 0)
            toks, logits, _ = data[e["id"]]
            out.append({"id": e["id"], "tokens": toks[lo:lo + e["n"]].tolist(), "want": e["want"]})
            ref += [logits[lo + k] for k in e["want"]]
            at[e["id"]] = lo + e["n"]
        lines.append(json.dumps({"step": i, "entries": out, "end": ["x"] if i == 2 else []}))
        want.append(ref)
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(tmp_path),
                        "--max-tokens", "260"], input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(len(steps))]
    for i, ref in enumerate(want):
        path = tmp_path / f"{i}.f32"
        assert path.exists() == bool(ref)
        if ref:
            got = np.fromfile(path, "<f4").reshape(len(ref), -1).astype(np.float64)
            assert rel(got, np.stack(ref)) <= limit("mixed", F32 if dtype == "float32" else BF16)


def test_command_line_generates(dev, folder):
    cfg, w, _ = model_of("mixed", F32)
    p = nc.tokens(cfg, 12, 0)
    r = subprocess.run([sys.executable, "-m", "nativebit_b200", "generate", "--model", str(folder), "--prompt", ",".join(map(str, p)), "--tokens", "9",
                        "--dtype", "float32", "--context", "64"], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [int(x) for x in r.stdout.strip().splitlines()[-1].split(",")] == greedy(cfg, w, p, 9)


def test_unknown_tensors_are_refused(dev, tmp_path):
    from nativebit_b200 import registry
    from nativebit_b200.weights import write_safetensors
    w = nc.weights(nc.CASES["mixed"], seed=5)
    (tmp_path / "config.json").write_text(json.dumps(nc.CASES["mixed"]))
    for extra, known in (("l1.norm2", True), ("l1.hc2.in", True), ("l0.mix.extra", False)):      # layer 1 has no feed-forward
        write_safetensors(str(tmp_path / "model.safetensors"), {**w, extra: torch.zeros(3).bfloat16()})
        if known:
            registry.load_model(str(tmp_path), "float32", 64)
        else:
            with pytest.raises(ValueError):
                registry.load_model(str(tmp_path), "float32", 64)
