"""Nabalix on the CPU: the oracle's own mechanisms against independent expressions, reading of configurations and
checkpoints, the registry, and the kernels' argument checks (nothing is launched)."""
import copy
import ctypes

import numpy as np
import pytest
import torch

import nabalix_cases as nc
from oracle import nabalix_oracle as O


# ---------------------------------------------------------------- oracle
def test_oracle_attention_against_whole_matrices():
    r = np.random.default_rng(0)
    T, H, G, D, V = 30, 6, 2, 5, 4
    q, k, v = r.standard_normal((T, H, D)), r.standard_normal((T, G, D)), r.standard_normal((T, G, V))
    r1, r2, talk = r.uniform(0, 2, H), r.uniform(0, 1, H), r.standard_normal((H, H))
    i = np.arange(T)
    for window in (1, 4, 29, 30, 100):
        s = np.einsum("ihd,jhd->hij", q, np.repeat(k, H // G, 1)) * 0.7
        s = 3.0 * np.tanh(s / 3.0) - r1[:, None, None] * np.log1p(r2[:, None, None] * np.maximum(i[:, None] - i[None], 0))
        s = np.einsum("hg,gij->hij", talk, s)
        seen = (i[None, :] <= i[:, None]) & (i[:, None] - i[None, :] < window)
        p = torch.softmax(torch.from_numpy(np.where(seen[None], s, -np.inf)), -1).numpy()
        want = np.einsum("hij,jhd->ihd", p, np.repeat(v, H // G, 1))
        assert np.allclose(O.mixed_head_attention(q, k, v, 0.7, 3.0, r1, r2, talk, window), want)


def test_oracle_talk_reads_rows():
    """Row h of the talk matrix makes head h's score: a row that takes another head's score makes both heads' weights equal."""
    r = np.random.default_rng(1)
    q, k, v = r.standard_normal((9, 2, 4)), r.standard_normal((9, 1, 4)), r.standard_normal((9, 1, 3))
    out = O.mixed_head_attention(q, k, v, 1.0, 50.0, np.zeros(2), np.zeros(2), np.array([[1.0, 0.0], [1.0, 0.0]]), 9)
    own = O.mixed_head_attention(q, k, v, 1.0, 50.0, np.zeros(2), np.zeros(2), np.eye(2), 9)
    assert np.allclose(out[:, 0], own[:, 0]) and np.allclose(out[:, 1], own[:, 0]) and not np.allclose(out[:, 1], own[:, 1])


def test_oracle_recurrence():
    r = np.random.default_rng(2)
    z, lower, q, v = r.standard_normal((20, 2, 4)), r.uniform(0, 1, (2, 4)), r.standard_normal((20, 2, 4)), r.standard_normal((20, 2, 3))
    f, write = O.forget_gate(z, lower)
    assert np.allclose(f + write, 1.0) and (f >= lower).all()
    whole, end = O.forget_recurrence(q, v, f, write)
    first, s = O.forget_recurrence(q[:7], v[:7], f[:7], write[:7])
    second, s = O.forget_recurrence(q[7:], v[7:], f[7:], write[7:], s)
    assert np.allclose(np.concatenate([first, second]), whole) and np.allclose(s, end)
    t = 13
    o = sum(((q[t, 1] * np.prod(f[s + 1:t + 1, 1], 0)) @ write[s, 1]) * v[s, 1] for s in range(t + 1))
    assert np.allclose(o, whole[t, 1])


def test_oracle_streams():
    """mix is indexed [from, to]; all streams are formed from the old ones."""
    x = np.arange(12.0).reshape(2, 2, 3)
    w = {"in": np.array([1.0, 2.0]), "out": np.array([1.0, 10.0]), "mix": np.array([[0.0, 1.0], [0.5, 0.0]])}
    seen = []
    new = O.connect(x, w, "", lambda u: seen.append(u) or np.ones_like(u))
    assert np.array_equal(seen[0], x[0] + 2 * x[1])
    assert np.array_equal(new[0], 0.5 * x[1] + 1) and np.array_equal(new[1], x[0] + 10)


def test_oracle_clamped_glu():
    out = O.clamped_glu(np.array([9.0, -9.0, 1.0]), np.array([9.0, -9.0, 0.5]), 2.0)
    s = lambda z: 1 / (1 + np.exp(-1.702 * z))                                              # noqa: E731
    assert np.allclose(out, [2 * s(2) * 3, -9 * s(-9) * -1, 1 * s(1) * 1.5])


# ---------------------------------------------------------------- configurations, weights, registry
@pytest.mark.parametrize("name", sorted(nc.CASES))
def test_layers_are_read_from_the_configuration(name):
    from nativebit_b200 import nabalix
    cfg = nc.CASES[name]
    w = nc.weights(cfg)
    used = set()

    def tensor(n, shape):
        used.add(n)
        assert tuple(w[n].shape) == shape, n
        return w[n]
    m = nabalix.build(cfg, tensor, torch.float32, 64)
    assert used == set(w) and (m.vocab_size, m.width, m.eps, m.streams) == (cfg["vocab"], cfg["width"], cfg["norm"]["eps"], cfg["streams"])
    n_links = sum(2 if s["mlp"] else 1 for s in cfg["layers"]) + 1
    assert len(m.coefs) == n_links and all(c.numel() == 2 * m.streams + 1 + m.streams ** 2 for c in m.coefs)
    for i, (spec, layer) in enumerate(zip(cfg["layers"], m.layers)):
        assert layer.mixer.kind == spec["type"] and (layer.ffn is None) == (spec["mlp"] is None)
        att, rec = layer.mixer.branches
        left = spec["mixer"]["left"]
        assert (att.window, att.scale, att.softcap) == (left["mask"]["size"], left["scale"], left["softcap"])
        # joint projection: every piece sits where its offset says, keys and values as in the cache's row
        p = f"l{i}.mix."
        v_off = att.k_off + m.new_caches(1)[i].parts[0].v_off
        for off, n in ((att.q_off, "left.q"), (att.k_off, "left.k"), (v_off, "left.v"), (att.g_off, "left.g"), (rec.q_off, "right.q"),
                       (rec.f_off, "right.f"), (rec.v_off, "right.v")):
            assert off % 8 == 0 and torch.equal(layer.mixer.w_in[off:off + w[p + n].shape[0], :m.width], w[p + n]), n
        # the penalty of every distance inside the window
        assert att.penalty.shape == (left["heads"], min(left["mask"]["size"], 64))
        want = np.stack([O.distance_penalty(a, b, np.arange(att.penalty.shape[1])) for a, b in
                         zip(w[p + "left.r1"].double().numpy(), w[p + "left.r2"].double().numpy())])
        assert np.abs(att.penalty.numpy() - want).max() < 1e-6


def test_link_coefficients():
    """What a link reads, through the update of the one before, equals reading the updated streams."""
    from nativebit_b200.layered import Link
    r = np.random.default_rng(5)
    for S in (1, 2, 5):
        a, b = (Link(None, read=torch.from_numpy(r.standard_normal(S)), share=torch.from_numpy(r.standard_normal(S)),
                     mix=torch.from_numpy(r.standard_normal((S, S)))) for _ in range(2))
        x, y = r.standard_normal((S, 7)), r.standard_normal(7)
        c = b.behind(a).double().numpy()
        new = a.mix.numpy().T @ x + a.share.numpy()[:, None] * y
        assert np.allclose(c[:S] @ x + c[S] * y, b.read.numpy() @ new, atol=1e-5)
        assert np.allclose(c[S + 1:2 * S + 1], a.share) and np.allclose(c[2 * S + 1:].reshape(S, S), a.mix)
        first = a.behind(None).double().numpy()
        assert np.allclose(first[:S], a.read) and first[S] == 0


def test_bad_configurations_are_refused():
    from nativebit_b200 import nabalix
    w = nc.weights(nc.CASES["mixed"])

    def build(change):
        cfg = copy.deepcopy(nc.CASES["mixed"])
        change(cfg)
        with pytest.raises((ValueError, KeyError)):
            nabalix.build(cfg, lambda n, s: w[n], torch.float32, 64)
    build(lambda c: c["layers"][0].update(type="something"))
    build(lambda c: c["layers"][0]["mlp"].update(kind="sparse"))
    build(lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=4))             # six heads
    build(lambda c: c["layers"][0]["mixer"]["left"].update(heads=8))
    build(lambda c: c["layers"][0]["mixer"]["right"].update(dim=13))
    build(lambda c: c["layers"][0]["mixer"]["left"].pop("softcap"))


def test_registry():
    from nativebit_b200 import registry
    fam = registry.family({"architecture": "Nabalix"})
    assert fam.library == "layered" and set(fam.dtypes) == {"bfloat16", "float32"}


# ---------------------------------------------------------------- C ABI
def test_argument_checks_need_no_gpu():
    from nativebit_b200 import _lib
    from nativebit_b200.build import build_library
    build_library(which="layered")
    l = _lib.layered_lib()
    fake, ref = 4096, ctypes.byref
    s = dict(x=fake, x_out=8192, y0=fake, w0=fake, y1=None, w1=None, coef=fake, norm_w=fake, eps=1e-6, streams=2, C=8, y_norm=0, norm=0)

    def stream(**kw):
        return l.nb_stream_norm(ref(_lib.StreamArgs(**{**s, **kw})), fake, 0, 8, 1, None)
    assert stream(w0=None) == 1 and stream(y0=None, y1=fake, w1=fake) == 1 and stream(norm=-1) == 1 and stream(streams=9) == 3 and stream(C=9) == 1
    m = dict(w=fake, y=fake, N=8, K=8, ldw=8)

    def matvec(m_kw, **kw):
        return l.nb_matvec_streams(ref(_lib.MatvecArgs(**{**m, **m_kw})), ref(_lib.StreamArgs(**{**s, **kw})), None)
    assert matvec({}, x_out=fake) == 1 and matvec({}, x_out=None) == 1 and matvec({"K": 4}) == 1 and matvec({"act": 3}) == 1
    assert matvec({"N": 7, "act": 2}) == 3 and matvec({"ldw": 12}) == 2
    a = _lib.MatvecArgs(**{**m, "x": fake})
    assert l.nb_matvec_pair(ref(a), ref(_lib.MatvecArgs(**m)), None) == 1                            # no row
    assert l.nb_matvec_pair(ref(a), ref(_lib.MatvecArgs(**{**m, "x": fake, "norm_w": fake})), None) == 1
    g = dict(p=fake, out=fake, state=fake, a2_b=fake, norm_w=fake, lower=fake, eps=1e-6, kind=1, dtype=0, B=1, T=1, H=2, dim=8, vdim=6, ldp=64,
             q_off=0, k_off=16, v_off=32, g_off=-1, lds=8, ldo=16)
    assert l.nb_gla_decode(ref(_lib.GlaArgs(**{**g, "lower": None})), None) == 1
    assert l.nb_gla_decode(ref(_lib.GlaArgs(**{**g, "kind": 2})), None) == 1
    assert l.nb_gla_decode(ref(_lib.GlaArgs(**{**g, "k_off": 56})), None) == 3
    assert l.nb_gla_decode(ref(_lib.GlaArgs(**{**g, "g_off": 60})), None) == 3
    assert l.nb_cache_append(fake, 24, 8, 16, fake, 24, 0, 1, 4, 8, 5, None) == 3                    # past the context
    assert l.nb_cache_append(fake, 24, 4, 16, fake, 24, 0, 1, 4, 8, 0, None) == 2
    t = dict(q=fake, cache=fake, out=fake, penalty=fake, talk=fake, scale=1.0, softcap=1.0, dtype=0, B=1, T=4, H=4, G=2, dim=8, vdim=6, ctx=64,
             ldc=32, v_off=16, ldq=32, ldg=32, ldo=24, pos0=10, window=5, n_pen=5)

    def talk(ws=4096, size=1 << 20, **kw):
        return l.nb_talk_attention(ref(_lib.TalkAttentionArgs(**{**t, **kw})), ws, size, None)
    assert talk(G=3) == 3 and talk(n_pen=4) == 3 and talk(pos0=61) == 3 and talk(ldc=24) == 3 and talk(talk=None) == 1
    assert talk(ws=None) == 7 and talk(size=16) == 7 and talk(ws=4100) == 2
    assert l.nb_talk_attention_workspace_bytes(1, 64, 4, 10, 5, 1) == 4 * 64 * 128 * 4               # 68 positions of reach, in tiles of 64
    d = dict(p=fake, cache=fake, penalty=fake, talk=fake, pos=fake, out=fake, scale=1.0, softcap=1.0, cache_dtype=0, B=1, H=4, G=2, dim=8, vdim=6,
             ctx=64, ldc=32, v_off=16, ldp=96, q_off=0, k_off=32, g_off=64, ldo=24, window=5, n_pen=5)

    def decode(**kw):
        return l.nb_talk_decode(ref(_lib.TalkDecodeArgs(**{**d, **kw})), None)
    assert decode(n_pen=3) == 3 and decode(g_off=80) == 3 and decode(k_off=72) == 3 and decode(v_off=12) == 3 and decode(ldc=28) == 2
    assert decode(pos=None) == 1
