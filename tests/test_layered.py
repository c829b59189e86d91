"""Layered decoders on the CPU: the oracle's own mechanisms against independent expressions, the rotary tables, reading
of configurations and checkpoints, the registry, and the kernels' argument checks (nothing is launched)."""
import ctypes
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import layered_cases as lc
from oracle import hybrid_oracle as O

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.fixture(scope="session")
def layered_lib():
    from nativebit_b200.build import build_library
    return build_library(which="layered")


# ---------------------------------------------------------------- oracle
def test_oracle_attention_against_masked_softmax():
    r = np.random.default_rng(0)
    q, k, v = r.standard_normal((30, 2, 6)), r.standard_normal((30, 2, 6)), r.standard_normal((30, 2, 5))
    for window in (1, 4, 29, 30, 100):
        out = O.windowed_attention(q, k, v, 0.7, window)
        i = np.arange(30)
        seen = (i[None, :] <= i[:, None]) & (i[:, None] - i[None, :] < window)
        s = np.where(seen[None], np.einsum("ihd,jhd->hij", q, k) * 0.7, -np.inf)
        p = torch.softmax(torch.from_numpy(s), -1).numpy()
        assert np.allclose(out, np.einsum("hij,jhd->ihd", p, v))


def test_oracle_window_edge_shows():
    """A key that dominates the scores is seen from exactly window - 1 tokens on and no further."""
    q = np.ones((12, 1, 4))
    k, v = np.zeros((12, 1, 4)), np.zeros((12, 1, 3))
    k[2], v[2] = 10.0, 1.0
    out = O.windowed_attention(q, k, v, 1.0, 5)[:, 0, 0]
    assert (out[2:7] > 0.9).all() and (out[7:] == 0).all() and (out[:2] == 0).all()


def test_oracle_recurrence_carries_its_state():
    r = np.random.default_rng(1)
    q, k, a = r.standard_normal((20, 2, 4)), r.standard_normal((20, 2, 4)), r.uniform(0.2, 1.0, (20, 2, 4))
    v = r.standard_normal((20, 2, 3))
    whole, end = O.gla_recurrence(q, k, v, a)
    first, s = O.gla_recurrence(q[:7], k[:7], v[:7], a[:7])
    second, s = O.gla_recurrence(q[7:], k[7:], v[7:], a[7:], s)
    assert np.allclose(np.concatenate([first, second]), whole) and np.allclose(s, end)
    # the closed form: o_t = sum_{s <= t} (q_t * prod_{s < r <= t} a_r) . k_s v_s
    t = 13
    o = sum(((q[t, 1] * np.prod(a[s + 1:t + 1, 1], 0)) @ k[s, 1]) * v[s, 1] for s in range(t + 1))
    assert np.allclose(o, whole[t, 1])


def test_oracle_norms():
    x = np.random.default_rng(2).standard_normal((3, 7)) + 2.0
    ref = torch.nn.functional.layer_norm(torch.from_numpy(x), (7,), torch.full((7,), 2.0, dtype=torch.float64), None, 1e-3).numpy()
    assert np.allclose(O.layer_norm(x, 2.0, 1e-3), ref)
    assert np.allclose(O.rms_norm(x, 1.0, 1e-3) * np.sqrt((x * x).mean(-1, keepdims=True) + 1e-3), x)


# ---------------------------------------------------------------- rotary tables
@pytest.mark.parametrize("dims,base,yarn", [(12, 300.0, None), (16, 1e4, (4.0, 512, 32.0, 1.0)), (64, 5e5, (8.0, 4096, 16.0, 2.0)),
                                            (4, 50.0, (2.0, 8, 1.0, 1.0)), (8, 1e4, (10.0, 100, 64.0, 0.01)), (2, 100.0, (3.0, 40, 4.0, 1.0))])
def test_rotation_tables(dims, base, yarn):
    from nativebit_b200.layered import Rotation, Yarn
    sc = None if yarn is None else dict(zip(("factor", "original", "fast", "slow"), yarn))
    cos, sin = Rotation(dims, base, None if yarn is None else Yarn(*yarn)).tables(40, "cpu")
    f, m = O.rope_frequencies(dims, base, sc)
    a = np.outer(np.arange(40), f)
    assert cos.shape == (40, dims) and torch.equal(cos[:, ::2], cos[:, 1::2])
    assert np.abs(cos[:, ::2].numpy() - np.cos(a) * m).max() < 1e-6
    assert np.abs(sin[:, ::2].numpy() - np.sin(a) * m).max() < 1e-6
    x = np.random.default_rng(3).standard_normal((40, dims + 3))
    y = O.rotate(x, np.arange(40), {"dims": dims, "base": base, "scaling": sc})
    assert np.array_equal(y[:, dims:], x[:, dims:]) and np.allclose(y[0, :dims], x[0, :dims] * m)
    n = lambda z: (z[:, :dims] ** 2).sum(-1)                                                # noqa: E731
    assert np.allclose(n(y), n(x) * m * m)


# ---------------------------------------------------------------- configurations, weights, registry
def test_checkpoint_round_trip(tmp_path):
    from nativebit_b200.weights import Checkpoint, write_safetensors
    t = {"a": torch.randn(3, 5).bfloat16(), "b": torch.arange(4, dtype=torch.int32), "c": torch.randn(2)}
    path = str(tmp_path / "x.safetensors")
    write_safetensors(path, t)
    c = Checkpoint(path, "cpu")
    for k, v in t.items():
        assert c.get(k).dtype == v.dtype and torch.equal(c.get(k), v)
    assert c.unread() == [] and "a" in c and "z" not in c
    with pytest.raises(KeyError):
        c.get("z")
    with pytest.raises(ValueError):
        c.get("a", (3, 6))
    (tmp_path / "bad").write_bytes(b"\xff" * 12)
    with pytest.raises(ValueError):
        Checkpoint(str(tmp_path / "bad"), "cpu")


@pytest.mark.parametrize("name", sorted(lc.CASES))
def test_layers_are_read_from_the_configuration(name):
    from nativebit_b200 import nerulorn
    cfg = lc.CASES[name]
    w = lc.weights(cfg)
    used = set()

    def tensor(n, shape):
        used.add(n)
        assert len(shape) == w[n].dim() and all(s in (None, g) for s, g in zip(shape, w[n].shape)), n
        return w[n]
    m = nerulorn.build(cfg, tensor, torch.float32, 64)
    assert used == set(w) and m.vocab_size == cfg["vocab"] and m.width == cfg["width"] and m.eps == cfg["norm"]["eps"]
    caches = m.new_caches(2)
    for i, (spec, layer) in enumerate(zip(cfg["layers"], m.layers)):
        assert layer.mixer.kind == spec["type"] and (layer.ffn is None) == (spec["mlp"] is None)
        src = spec["mixer"].get("kv_from")
        if src is not None:
            assert caches[i] is caches[src]
        if spec["type"] == "latent_attention":
            assert layer.mixer.window == spec["mixer"]["mask"]["size"] and layer.mixer.scale == spec["mixer"]["scale"]
    # packed rows: every piece sits where its offset says
    g = m.layers[[s["type"] for s in cfg["layers"]].index("gla")].mixer
    i = [s["type"] for s in cfg["layers"]].index("gla")
    for off, n in ((g.q_off, "q"), (g.k_off, "k"), (g.v_off, "v"), (g.g_off, "g"), (g.a_off, "a1")):
        x = w[f"l{i}.mix.{n}"]
        assert off % 8 == 0 and torch.equal(g.w_in[off:off + x.shape[0], :x.shape[1]], x)


def test_bad_configurations_are_refused():
    from nativebit_b200 import nerulorn
    w = lc.weights(lc.CASES["mixed"])

    def build(cfg):
        return nerulorn.build(cfg, lambda n, s: w[n], torch.float32, 64)
    cfg = lc.config(lc.CASES["mixed"]["layers"])
    cfg["layers"][3]["mixer"]["kv_from"] = 0                       # a recurrent layer has no key/value cache
    with pytest.raises(ValueError):
        build(cfg)
    cfg = lc.config(lc.CASES["mixed"]["layers"])
    cfg["layers"][3]["mixer"]["rot"]["base"] = 301.0               # the shared key part was rotated otherwise
    with pytest.raises(ValueError):
        build(cfg)
    cfg = lc.config(lc.CASES["mixed"]["layers"])
    cfg["layers"][1]["mixer"]["heads"] = 4
    with pytest.raises(ValueError):
        build(cfg)
    cfg = lc.config(lc.CASES["mixed"]["layers"])
    cfg["layers"][0]["type"] = "something"
    with pytest.raises(ValueError):
        build(cfg)


def test_registry():
    from nativebit_b200 import registry
    assert registry.family({"architecture": "Nerulorn"}).library == "layered"
    assert registry.family({"architecture": "PackedGPT"}).library == "packed"
    with pytest.raises(ValueError):
        registry.family({"architecture": "Other"})


def test_packed_models_have_no_32_bit_mode(tmp_path):
    """The trace runner refuses a dtype the family does not run in, before it touches a device."""
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "PackedGPT"}))
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path),
                        "--max-tokens", "8"], stdin=subprocess.DEVNULL, capture_output=True, text=True)
    assert r.returncode == 3, r.stderr


def test_command_line_lists_models():
    r = subprocess.run([sys.executable, "-m", "nativebit_b200", "models"], cwd=ROOT, capture_output=True, text=True)
    assert r.returncode == 0 and "Nerulorn" in r.stdout and "PackedGPT" in r.stdout


# ---------------------------------------------------------------- C ABI
def test_layered_library_exports_every_declared_symbol(layered_lib):
    from nativebit_b200 import _lib
    names = _lib.declared_symbols("layered")
    handle = ctypes.CDLL(layered_lib)
    assert set(names) == set(_lib._LAYERED_SIGNATURES)
    for n in names:
        assert hasattr(handle, n), n


def test_layered_argument_checks_need_no_gpu(layered_lib):
    from nativebit_b200 import _lib
    l = _lib.layered_lib()
    fake, odd = 4096, 4100
    assert l.nb_embed_scaled(None, fake, 1, 8, 8, 1.0, 1, fake, None) == 1
    assert l.nb_residual_norm(fake, fake, None, fake, 1, 1e-6, fake, 0, 8, 1, 8, None) == 1          # y without its weight
    assert l.nb_residual_norm(fake, None, None, fake, 2, 1e-6, fake, 0, 8, 1, 8, None) == 1          # unknown norm
    assert l.nb_residual_norm(fake, None, None, fake, 1, 1e-6, fake, 0, 20000, 1, 20000, None) == 3  # row too long
    assert l.nb_linear_bf16(fake, 12, fake, 16, None, 0, 0.0, 0.0, 4, 8, 12, fake, 2, 8, None, None) == 2      # row stride no multiple of 8
    assert l.nb_linear_bf16(fake, 16, fake, 16, None, 1, 0.0, 0.0, 4, 7, 12, fake, 2, 8, None, None) == 3      # pairs need an even N
    assert l.nb_linear_bf16(odd, 16, fake, 16, None, 0, 0.0, 0.0, 4, 8, 12, fake, 2, 8, None, None) == 2
    assert l.nb_linear_f32(fake, 8, fake, 8, None, 0, 0.0, 0.0, 4, 8, 12, fake, 8, None) == 1                  # stride below K
    a = _lib.MatvecArgs(fake, None, fake, fake, fake, fake, fake, fake, 1e-6, 0.0, 0.0, 8, 8, 8, 0, 1)
    assert l.nb_matvec_bf16(ctypes.byref(a), None) == 1                                              # x_out aliases x
    a = _lib.MatvecArgs(fake, None, fake, fake, None, None, None, None, 0.0, 0.0, 0.0, 8, 9, 12, 0, 0)
    assert l.nb_matvec_bf16(ctypes.byref(a), None) == 2
    g = dict(p=fake, out=fake, state=fake, a2=fake, a2_b=fake, norm_w=fake, tau=4.0, eps=1e-6, dtype=0, B=1, T=1, H=2, dim=8, vdim=6, ldp=64,
             q_off=0, k_off=16, v_off=32, g_off=44, a_off=56, a_rank=4, lda2=8, lds=8, ldo=16)
    assert l.nb_gla_decode(ctypes.byref(_lib.GlaArgs(**{**g, "a_off": 62})), None) == 3              # past the row
    assert l.nb_gla_decode(ctypes.byref(_lib.GlaArgs(**{**g, "tau": 0.0})), None) == 1
    assert l.nb_gla_decode(ctypes.byref(_lib.GlaArgs(**{**g, "dtype": 2})), None) == 1
    assert l.nb_gla_prefill(ctypes.byref(_lib.GlaArgs(**g)), None, 0, None) == 7
    assert l.nb_gla_workspace_bytes(1, 65, 2, 8, 6) > l.nb_gla_workspace_bytes(1, 64, 2, 8, 6) > 0
    t = dict(q=fake, kv=fake, cache=fake, gate=None, out=fake, cos2=fake, sin2=fake, scale=1.0, dtype=0, B=1, T=4, H=2, dim=8, rot=4, vdim=8,
             rank=16, ctx=64, ldc=24, ldq=24, ldkv=32, v_off=16, kv_rows=4, kv_pos0=10, ldg=2, ldo=16, pos0=10, window=3)
    assert l.nb_latent_attention(ctypes.byref(_lib.LatentAttentionArgs(**t)), None) == 3             # keys before kv_pos0 are visible
    assert l.nb_latent_attention(ctypes.byref(_lib.LatentAttentionArgs(**{**t, "kv_pos0": 8, "kv_rows": 5})), None) == 3
    assert l.nb_latent_attention(ctypes.byref(_lib.LatentAttentionArgs(**{**t, "vdim": 300})), None) == 3
    assert l.nb_latent_attention(ctypes.byref(_lib.LatentAttentionArgs(**{**t, "rot": 3})), None) == 1
    assert l.nb_argmax(None, 1, 8, fake, None, None) == 1
