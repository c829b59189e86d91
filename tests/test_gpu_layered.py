"""Layered decoders on the GPU against the plain oracle: every kernel alone, then whole models — prompts, portions,
decoding, batches, sessions used again, greedy generation, the trace runner and the command line."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import layered_cases as lc
from gpu_util import BF16, F32, TOL, close, cu, f64, rel, rounded, rounding
from oracle import hybrid_oracle as O

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
def test_embedding(dev):
    from nativebit_b200 import layer_ops as L
    table = torch.randn(37, 50, device=dev).bfloat16()
    tok = torch.tensor([0, 36, 5, 5], device=dev)
    x = torch.empty(4, 50, device=dev)
    L.embed_scaled(table, tok, 0.37, x)
    assert torch.equal(x, table[tok].float() * np.float32(0.37))


@pytest.mark.parametrize("norm", [0, 1])
@pytest.mark.parametrize("C", [50, 72, 1000, 5000])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_residual_norm(dev, norm, C, dtype):
    from nativebit_b200 import layer_ops as L
    r = np.random.default_rng(C + norm)
    # a mean far from zero: a variance taken as E[x^2] - mean^2 would lose it
    x, y = r.standard_normal((5, C)).astype(np.float32), (30.0 + r.standard_normal((5, C))).astype(np.float32)
    wy, w = (1 + 0.2 * r.standard_normal((2, C))).astype(np.float32)
    fn = O.layer_norm if norm else O.rms_norm
    x2 = x + fn(y.astype(np.float64), wy, 1e-5)
    xt, h = cu(x), L.rows_empty(5, C, dtype, dev)
    L.residual_norm(xt, cu(y), cu(wy), cu(w), norm, 1e-5, h)
    close(xt, x2, 1e-5)
    close(h[:, :C], fn(x2, w, 1e-5), max(TOL[dtype], 1e-5))
    L.residual_norm(xt, None, None, cu(w), norm, 1e-5, h)           # no sublayer result: x stays
    close(xt, x2, 1e-5)


@pytest.mark.parametrize("m,n,k", [(1, 8, 8), (3, 50, 50), (70, 131, 72), (130, 300, 264), (200, 40, 17), (64, 1030, 520), (513, 264, 100)])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_linear(dev, m, n, k, dtype):
    from nativebit_b200 import layer_ops as L
    r = np.random.default_rng(m + n + k)
    w = rounded(r.standard_normal((n, k)) / np.sqrt(k), BF16)
    x = rounded(r.standard_normal((m, k)), dtype)
    b = r.standard_normal(n).astype(np.float32)
    xt = L.rows_empty(m, k, dtype, dev)
    xt[:, k:] = float("nan")                                        # padding is never read
    xt[:, :k] = cu(x, dtype)
    wt = L.pad_matrix(cu(w, BF16))
    out = torch.full((m, n + 3), 7.0, dtype=F32, device=dev)
    L.linear(xt, wt, k, n, out, bias=cu(b))
    close(out[:, :n], x @ w.T + b, 3e-6)
    assert (out[:, n:] == 7.0).all()
    L.linear(xt, wt, k, n, out)
    close(out[:, :n], x @ w.T, 3e-6)
    if dtype == BF16:
        o16 = L.rows_empty(m, n, BF16, dev)
        L.linear(xt, wt, k, n, o16)
        close(o16[:, :n], x @ w.T, TOL[BF16])
        assert int(L.linear_status(dev).item()) == 0
    if n % 2 == 0:
        y = x @ w.T + b
        ref = O.silu(y[:, ::2]) * y[:, 1::2]
        act = L.rows_empty(m, n // 2, dtype, dev)
        L.linear(xt, wt, k, n, act, bias=cu(b), act=L.SWIGLU)
        close(act[:, :n // 2], ref, max(TOL[dtype], 1e-5))


@pytest.mark.parametrize("n,k", [(1, 8), (6, 50), (131, 72), (148, 256), (150, 257), (700, 264), (4000, 1000), (3001, 2560), (64, 7000)])
def test_matvec(dev, n, k):
    from nativebit_b200 import layer_ops as L
    r = np.random.default_rng(n + k)
    w = rounded(r.standard_normal((n, k)) / np.sqrt(k), BF16)
    x, d = (r.standard_normal((2, k)) + np.array([[0.0], [3.0]])).astype(np.float32)
    nw, dw = (1 + 0.2 * r.standard_normal((2, k))).astype(np.float32)
    b = r.standard_normal(n).astype(np.float32)
    wt, y = L.pad_matrix(cu(w, BF16)), torch.empty(n, device=dev)
    L.matvec(wt, n, k, cu(x), y)
    close(y, w @ x.astype(np.float64), 3e-6)
    L.matvec(wt, n, k, cu(x), y, bias=cu(b), norm=0, eps=1e-5, norm_w=cu(nw))
    close(y, w @ O.rms_norm(x.astype(np.float64), nw, 1e-5) + b, 5e-6)
    xo = torch.zeros(k, device=dev)
    L.matvec(wt, n, k, cu(x), y, norm=1, eps=1e-5, norm_w=cu(nw), delta=cu(d), delta_w=cu(dw), x_out=xo)
    res = x + O.layer_norm(d.astype(np.float64), dw, 1e-5)
    close(xo, res, 5e-6)
    close(y, w @ O.layer_norm(res, nw, 1e-5), 1e-5)
    again = torch.empty_like(y)
    L.matvec(wt, n, k, cu(x), again, norm=1, eps=1e-5, norm_w=cu(nw), delta=cu(d), delta_w=cu(dw), x_out=xo)
    assert torch.equal(y, again)
    if n % 2 == 0:
        z = w @ x.astype(np.float64) + b
        act = torch.empty(n // 2, device=dev)
        L.matvec(wt, n, k, cu(x), act, bias=cu(b), act=L.SWIGLU)
        close(act, O.silu(z[::2]) * z[1::2], 1e-5)


def test_argmax_takes_the_lowest_of_equals(dev):
    from nativebit_b200 import layer_ops as L
    lg = torch.randn(2, 5000, device=dev)
    lg[0, 4000] = lg[0, 33] = 50.0
    tok, pos = torch.zeros(2, 1, dtype=torch.long, device=dev), torch.tensor([6], device=dev)
    L.argmax(lg, tok, pos)
    assert tok[0, 0] == 33 and tok[1, 0] == lg[1].argmax() and pos[0] == 7


# ---------------------------------------------------------------- latent attention, alone
def rot_tables(rot, n):
    from nativebit_b200.layered import Rotation
    return Rotation(rot, 200.0).tables(n, "cuda:0")


def rot_np(x, pos, rot):
    return O.rotate(x, pos, {"dims": rot, "base": 200.0}) if rot else x


SHAPES = [dict(H=3, dim=20, rot=12, vdim=28, rank=36), dict(H=2, dim=64, rot=32, vdim=72, rank=136), dict(H=1, dim=7, rot=4, vdim=9, rank=17),
          dict(H=2, dim=128, rot=64, vdim=128, rank=64), dict(H=2, dim=96, rot=16, vdim=200, rank=40)]


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("T,pos0,window", [(5, 0, 3), (64, 0, 64), (65, 0, 64), (130, 0, 63), (2, 70, 9), (70, 33, 40), (33, 100, 1), (90, 20, 1000)])
def test_latent_attention(dev, shape, dtype, T, pos0, window):
    """A portion at pos0 .. of two sequences against the oracle's attention over all positions; one key per sequence is made
    to dominate, so the window's edge shows."""
    from nativebit_b200 import layer_ops as L
    H, D, R, V, rank = (shape[k] for k in ("H", "dim", "rot", "vdim", "rank"))
    B, N = 2, pos0 + T
    r = np.random.default_rng(T + pos0 + D)
    q = rounded(r.standard_normal((B, N, H, D + R)), dtype)
    kn, kr, v = (rounded(r.standard_normal((B, N, H, n)), dtype) for n in (D, R, V))
    kr = kr[:, :, 0]
    loud = max(0, N - window - T // 2 - 1)                          # leaves the window in the middle of the portion
    kn[:, loud] = 1.0
    q[..., :D] = np.abs(q[..., :D])
    kr_rot = rounded(np.stack([rot_np(kr[b], np.arange(N), R) for b in range(B)]), dtype)
    scale = 1.5 / np.sqrt(D + R)
    gate = rounded(r.standard_normal((B, T, H)), dtype)
    ref = []
    for b in range(B):
        qq = np.concatenate([q[b, ..., :D], rounded(rot_np(q[b, ..., D:], np.arange(N), R), dtype)], -1)
        kk = np.concatenate([kn[b], np.repeat(kr_rot[b][:, None], H, 1)], -1)
        ref.append(O.windowed_attention(qq, kk, v[b], scale, window)[pos0:] * O.sigmoid(gate[b])[..., None])
    ref = np.stack(ref).reshape(B * T, H * V)

    ctx = N + 5
    cos, sin = rot_tables(R, ctx)
    cache = torch.zeros(B, ctx, L.pad8(rank + R), dtype=dtype, device=dev)
    cache[:, :, :rank] = float("nan")                               # the latents themselves are not read here
    cache[:, N:] = float("nan")                                     # nor rows past the portion
    cache[:, :N, rank:rank + R] = cu(kr_rot, dtype)
    lo = max(0, pos0 - window + 1)
    v_off = L.pad8(H * D)
    kv = torch.full((B, N - lo, L.pad8(v_off + H * V)), float("nan"), dtype=dtype, device=dev)
    kv[:, :, :H * D] = cu(kn[:, lo:].reshape(B, N - lo, H * D), dtype)
    kv[:, :, v_off:v_off + H * V] = cu(v[:, lo:].reshape(B, N - lo, H * V), dtype)
    qt = L.rows_empty(B * T, H * (D + R), dtype, dev)
    qt[:, :H * (D + R)] = cu(q[:, pos0:].reshape(B * T, -1), dtype)
    gt = L.rows_empty(B * T, H, dtype, dev)
    gt[:, :H] = cu(gate.reshape(B * T, H), dtype)
    out = L.rows_empty(B * T, H * V, dtype, dev)
    L.latent_attention(q=qt.data_ptr(), kv=kv.data_ptr(), cache=cache.data_ptr(), gate=gt.data_ptr(), out=out.data_ptr(), cos2=cos.data_ptr(),
                       sin2=sin.data_ptr(), scale=scale, dtype=L._DTYPE[dtype], B=B, T=T, H=H, dim=D, rot=R, vdim=V, rank=rank, ctx=ctx,
                       ldc=cache.shape[2], ldq=qt.stride(0), ldkv=kv.shape[2], v_off=v_off, kv_rows=N - lo, kv_pos0=lo, ldg=gt.stride(0),
                       ldo=out.stride(0), pos0=pos0, window=window)
    close(out[:, :H * V], ref, 1e-5 if dtype == F32 else 2.0 ** -7)


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("pos,window", [(0, 5), (4, 5), (5, 5), (63, 64), (64, 64), (200, 17), (300, 1000), (77, 1)])
@pytest.mark.parametrize("own", [True, False])
def test_latent_decode(dev, shape, dtype, pos, window, own):
    """One position of two sequences: the row is normed, rotated and written (own) or read from the cache, and the absorbed
    form equals attention over up-projected keys and values.  The key that just left the window would dominate."""
    from nativebit_b200 import layer_ops as L
    H, D, R, V, rank = (shape[k] for k in ("H", "dim", "rot", "vdim", "rank"))
    B, r = 2, np.random.default_rng(pos + D)
    uk = rounded(r.standard_normal((H * D, rank)) / np.sqrt(rank), BF16)
    uv = rounded(r.standard_normal((H * V, rank)) / np.sqrt(rank), BF16)
    q = r.standard_normal((B, H, D + R)).astype(np.float32)
    c = r.standard_normal((B, pos + 1, rank))
    kr = r.standard_normal((B, pos + 1, R))
    direction = np.einsum("bhd,hdr->br", q[..., :D], uk.reshape(H, D, rank))
    for j in (pos - window, pos - window + 1):                      # just outside and just inside the window
        if 0 <= j < pos:
            c[:, j] = direction / np.linalg.norm(direction, axis=-1, keepdims=True) * np.sqrt(rank) * (4.0 if j == pos - window else 1.5)
    kv_norm = (1 + 0.2 * r.standard_normal(rank)).astype(np.float32)
    raw = r.standard_normal((B, rank + R)).astype(np.float32)       # this position's projection
    c[:, pos] = O.rms_norm(raw[:, :rank].astype(np.float64), kv_norm, 1e-5)
    kr[:, pos] = np.stack([rot_np(raw[b:b + 1, rank:].astype(np.float64), np.array([pos]), R)[0] for b in range(B)])
    c, kr = rounded(c, dtype), rounded(kr, dtype)
    scale, gate = 1.0 / np.sqrt(D + R), r.standard_normal((B, H)).astype(np.float32)
    ref = np.empty((B, H, V))
    j0 = max(0, pos - window + 1)
    for b in range(B):
        qr = rot_np(q[b, :, D:].astype(np.float64)[None], np.array([pos]), R)[0]
        for h in range(H):
            k = np.concatenate([c[b, j0:] @ uk[h * D:(h + 1) * D].T, kr[b, j0:]], -1)
            s = k @ np.concatenate([q[b, h, :D], qr[h]]) * scale
            p = np.exp(s - s.max())
            ref[b, h] = (p / p.sum()) @ (c[b, j0:] @ uv[h * V:(h + 1) * V].T) * O.sigmoid(gate[b, h])
    ctx = pos + 3
    cos, sin = rot_tables(R, ctx)
    cache = torch.zeros(B, ctx, L.pad8(rank + R), dtype=dtype, device=dev)
    cache[:, :pos + 1, :rank] = cu(c, dtype)
    cache[:, :pos + 1, rank:rank + R] = cu(kr, dtype)
    cache[:, :j0] = float("nan")                                    # what the window does not cover is not read
    want_row = cache[:, pos, :rank + R].clone()
    if own:
        cache[:, pos] = float("nan")
    cache[:, pos + 1:] = float("nan")
    kv_off, g_off = 3, 3 + rank + R
    a = torch.zeros(B, g_off + H, device=dev)
    a[:, kv_off:g_off] = cu(raw)
    a[:, g_off:] = cu(gate)
    ukt, uvt = L.pad_matrix(cu(uk, BF16)), L.pad_matrix(cu(uv, BF16))
    out = torch.empty(B, H * V, device=dev)
    qt, kn, pt = cu(q.reshape(B, -1)), cu(kv_norm), torch.tensor([pos], device=dev)
    torch.cuda.synchronize()                                        # cached rows are requested ahead of the dependency wait
    L.latent_decode(q=qt.data_ptr(), a=a.data_ptr(), cache=cache.data_ptr(), uk=ukt.data_ptr(), uv=uvt.data_ptr(), kv_norm=kn.data_ptr(),
                    cos2=cos.data_ptr(), sin2=sin.data_ptr(), pos=pt.data_ptr(), out=out.data_ptr(), scale=scale, eps=1e-5,
                    cache_dtype=L._DTYPE[dtype], B=B, H=H, dim=D, rot=R, vdim=V, rank=rank, ctx=ctx, ldc=cache.shape[2], ldq=qt.shape[1],
                    lda=a.shape[1], kv_off=kv_off if own else -1, g_off=g_off, ldu=ukt.shape[1], ldo=out.shape[1], window=window)
    # an own bf16 row may round the other way at a tie of the norm's last bit
    close(out, ref.reshape(B, -1), 1e-5 if dtype == F32 else 2e-3 if own else 1e-5)
    close(cache[:, pos, :rank + R], f64(want_row), 1e-5 if dtype == F32 else 2.0 ** -7)


# ---------------------------------------------------------------- gated linear attention, alone
@pytest.mark.parametrize("H,D,V,ra", [(3, 20, 28, 6), (2, 96, 136, 16), (1, 5, 11, 3), (4, 136, 40, 9), (2, 64, 64, 16)])
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("bias", [1.0, -30.0, 40.0])
def test_gla(dev, H, D, V, ra, dtype, bias):
    """Portions of several sizes (cut inside chunks and sub-blocks) continue one another; decays from none to total.  With
    fp32 activations single tokens go through the decode kernel in between."""
    from nativebit_b200 import layer_ops as L
    from nativebit_b200.layered import GatedLinearAttention
    B, T, tau, eps, C = 2, 213, 2.0, 1e-5, 24
    r = np.random.default_rng(D + V)
    w = {n: rounded(r.standard_normal((rows, C)) / np.sqrt(C), BF16) for n, rows in
         (("q", H * D), ("k", H * D), ("v", H * V), ("g", H * V), ("a1", ra), ("o", C))}
    a2 = rounded(r.standard_normal((H * D, ra)) * 2, BF16)
    b2 = (bias + r.standard_normal(H * D) * 3).astype(np.float32)
    nw = (1 + 0.2 * r.standard_normal(V)).astype(np.float32)
    t = {n: cu(x, BF16) for n, x in w.items()}
    mix = GatedLinearAttention(heads=H, dim=D, vdim=V, tau=tau, eps=eps, w_q=t["q"], w_k=t["k"], w_v=t["v"], w_gate=t["g"], w_a1=t["a1"],
                               w_a2=cu(a2, BF16), a2_bias=cu(b2), norm_w=cu(nw), w_out=torch.zeros(C, H * V, dtype=BF16, device=dev))
    p = torch.zeros(B, T, mix.n_in, dtype=dtype, device=dev)
    parts = {}
    for n, off, cols in (("q", mix.q_off, H * D), ("k", mix.k_off, H * D), ("v", mix.v_off, H * V), ("g", mix.g_off, H * V), ("a", mix.a_off, ra)):
        parts[n] = rounded(r.standard_normal((B, T, cols)), dtype)
        p[:, :, off:off + cols] = cu(parts[n], dtype)

    def oracle(dt):
        outs, ends = [], []
        for b in range(B):
            a, q, k, v, g = (parts[n][b].astype(dt) for n in ("a", "q", "k", "v", "g"))
            alpha = O.sigmoid(a @ a2.astype(dt).T + b2) ** dt(1 / tau)
            o, S = O.gla_recurrence(q.reshape(T, H, D) * dt(D ** -0.5), k.reshape(T, H, D), v.reshape(T, H, V), alpha.reshape(T, H, D))
            assert o.dtype == dt
            outs.append(O.rms_norm(o, nw, dt(eps)).reshape(T, H * V) * O.silu(g))
            ends.append(S)
        return np.stack(outs), np.stack(ends)
    ref, ends = oracle(np.float64)
    # outputs are normed, so where q . k cancels the norm shows the rounding: the limit follows the oracle in fp32
    lim_o, lim_s = (rounding(x, y, 1e-5) for x, y in zip((ref, ends), oracle(np.float32)))

    def run(cuts, single=False):
        st = mix.new_cache(B, 0, dtype, dev)
        out, at = torch.empty(B, T, H * V, dtype=dtype, device=dev), 0
        for n in cuts:
            src, dst = p[:, at:at + n].contiguous(), torch.empty(B, n, H * V, dtype=dtype, device=dev)
            if n == 1 and single:
                L.gla_decode(**mix._args(src, mix.n_in, dst, H * V, st, F32, B, 1))
            else:
                ws = torch.full((L.gla_workspace_bytes(B, n, H, D, V),), 255, dtype=torch.uint8, device=dev)
                L.gla_prefill(ws, **mix._args(src, mix.n_in, dst, H * V, st, dtype, B, n))
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
_built = {}


def model_of(name, dtype, context=400, sharp=3.0):
    from nativebit_b200 import nerulorn
    key = (name, dtype, context, sharp)
    if key not in _built:
        cfg = lc.CASES[name]
        w = lc.weights(cfg, seed=5, sharp=sharp)
        wd = {k: v.cuda() for k, v in w.items()}
        m = nerulorn.build(cfg, lambda n, s: wd[n], dtype, context)
        torch.cuda.synchronize()
        _built[key] = (cfg, lc.as_numpy(w), m)
    return _built[key]


_refs, _limits = {}, {}


def reference(name, n, seed=0):
    """(tokens, logits, residual stream) of the oracle; also sets the limits of the case.  The weights are made so that scores
    are sharp, which enlarges rounding: the limits are six times what the oracle itself loses in fp32, and three times what
    it loses when the products' inputs and outputs are rounded to bf16."""
    if (name, n, seed) not in _refs:
        cfg = lc.CASES[name]
        w = lc.as_numpy(lc.weights(cfg, seed=5, sharp=3.0))
        toks = lc.tokens(cfg, n, seed)
        logits, stream = O.forward(cfg, w, toks)
        l32, s32 = O.forward(cfg, w, toks, np.float32)
        assert l32.dtype == np.float32
        _refs[name, n, seed] = (toks, logits, stream)
        _limits[name, F32] = max(_limits.get((name, F32), 5e-6), 6 * rel(l32, logits))
        l16, _ = O.forward(cfg, w, toks, cast=lambda a: rounded(a, BF16))
        _limits[name, BF16] = max(_limits.get((name, BF16), 0.0), 3 * rel(l16, logits))
    return _refs[name, n, seed]


def limit(name, dtype):
    return _limits[name, dtype]


@pytest.mark.parametrize("name", sorted(lc.CASES))
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


@pytest.mark.parametrize("name", sorted(lc.CASES))
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


def test_portions_do_not_change_the_logits(dev):
    """bf16: however a prompt is cut, the logits differ by rounding only."""
    _, _, m = model_of("wide", BF16)
    toks, _, _ = reference("wide", 210)
    out = []
    for cuts in ([210], [100, 110], [2] * 105):
        s, at, got = m.session(), 0, []
        for n in cuts:
            got.append(s.extend(cu(toks[None, at:at + n], torch.long), list(range(n)))[0].clone())
            at += n
        out.append(f64(torch.cat(got)))
    assert rel(out[1], out[0]) <= limit("wide", BF16) / 2 and rel(out[2], out[0]) <= limit("wide", BF16) / 2


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
    with pytest.raises(RuntimeError):
        s.extend(t[:, :3], [3])


def test_sessions_are_used_again(dev):
    """A reset gives the cache and state back: the next request does not see the one before, with or without a captured step."""
    _, _, m = model_of("order", F32)
    s = m.session()
    other = cu(lc.tokens(lc.CASES["order"], 300, seed=9)[None], torch.long)
    for seed, n in ((0, 210), (1, 64), (2, 23)):
        toks, logits, _ = reference("order", n, seed)
        t = cu(toks[None], torch.long)
        got = [s.extend(t[:, :n - 9], list(range(n - 9)))[0].clone()] + [s.extend(t[:, i:i + 1], [0])[0].clone() for i in range(n - 9, n)]
        assert rel(f64(torch.cat(got)), logits) <= limit("order", F32)
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
    _, _, m = model_of("order", F32)
    toks, logits, _ = reference("order", 330, 7)
    t = cu(toks[None], torch.long)
    got = {}
    for graph in (True, False):
        s = m.session(use_graph=graph)
        s.extend(t[:, :3], [2])
        got[graph] = torch.cat([s.extend(t[:, i:i + 1], [0])[0].clone() for i in range(3, 330)])
        assert rel(f64(got[graph]), logits[3:]) <= limit("order", F32)
    assert torch.equal(got[True], got[False])


def greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(O.forward(cfg, w, toks)[0][-1].argmax()))
    return toks[len(prompt):]


def test_greedy_generation(dev):
    cfg, w, m = model_of("mixed", F32)
    prompts = [lc.tokens(cfg, 12, s) for s in (0, 1)]
    want = [greedy(cfg, w, p, 14) for p in prompts]
    s = m.session()
    for p, ref in zip(prompts, want):                               # the second prompt replays the captured prefill
        assert s.generate(cu(p[None], torch.long), 14)[0].tolist() == ref
    assert m.session(2).generate(cu(np.stack(prompts), torch.long), 14).tolist() == want
    assert s.generate(cu(prompts[0][None], torch.long), 14)[0].tolist() == want[0]


def test_the_end_of_the_context_is_refused(dev):
    _, _, m = model_of("mixed", F32, context=20)
    s = m.session()
    t = torch.zeros(1, 18, dtype=torch.long, device=dev)
    s.extend(t, [])
    with pytest.raises(RuntimeError):
        s.extend(t[:, :3], [])
    s.step()
    s.step()
    with pytest.raises(RuntimeError):
        s.step()


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    from nativebit_b200.weights import write_safetensors
    d = tmp_path_factory.mktemp("model")
    (d / "config.json").write_text(json.dumps(lc.CASES["mixed"]))
    write_safetensors(str(d / "model.safetensors"), lc.weights(lc.CASES["mixed"], seed=5, sharp=3.0))
    return d


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_runner(dev, folder, tmp_path, dtype):
    """Two requests one after the other, then two at a time, through the program and its files."""
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
    p = lc.tokens(cfg, 12, 0)
    r = subprocess.run([sys.executable, "-m", "nativebit_b200", "generate", "--model", str(folder), "--prompt", ",".join(map(str, p)), "--tokens", "9",
                        "--dtype", "float32", "--context", "64"], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [int(x) for x in r.stdout.strip().splitlines()[-1].split(",")] == greedy(cfg, w, p, 9)


def test_unknown_tensors_are_refused(dev, folder, tmp_path):
    from nativebit_b200 import registry
    from nativebit_b200.weights import write_safetensors
    w = lc.weights(lc.CASES["mixed"], seed=5)
    w["l0.mix.extra"] = torch.zeros(4, 4).bfloat16()
    (tmp_path / "config.json").write_text(json.dumps(lc.CASES["mixed"]))
    write_safetensors(str(tmp_path / "model.safetensors"), w)
    with pytest.raises(ValueError):
        registry.load_model(str(tmp_path), "float32", 64)
