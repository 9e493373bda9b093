"""The float64 statement of the decoder with gated-delta-rule layers and masked attention (oracle/hybrid_ref.py), mechanism
by mechanism against direct formulas, and the host side of the library's registry entry.  No GPU."""
import ctypes as C
import json

import numpy as np
import pytest

from oracle import hybrid_ref as hr


def rng(seed=0):
    return np.random.default_rng(seed)


def test_masks_name_the_visible_keys():
    pos = np.arange(9)
    w, c = hr.window_mask(pos, 3), hr.chunk_mask(pos, 4)
    for i in range(9):
        assert list(np.flatnonzero(w[i])) == list(range(max(0, i - 2), i + 1))
        assert list(np.flatnonzero(c[i])) == list(range(i // 4 * 4, i + 1))
    assert np.array_equal(hr.window_mask(pos, 1), np.eye(9, dtype=bool)) and np.array_equal(hr.chunk_mask(pos, 1), np.eye(9, dtype=bool))
    # chunks are counted from the sequence's start wherever the rows begin
    assert np.array_equal(hr.chunk_mask(pos + 5, 4), hr.chunk_mask(np.arange(14), 4)[5:, 5:])


def test_softmax_with_one_more_term():
    s = np.array([[1.0, 2.0, 50.0]])
    vis = np.array([[True, True, False]])
    e = np.exp([1.0, 2.0])
    assert np.allclose(hr.softmax_plus_one(s, vis)[0], [e[0] / (1 + e.sum()), e[1] / (1 + e.sum()), 0])
    assert np.allclose(hr.softmax_plus_one(s - 700, vis), 0) and np.allclose(hr.softmax_plus_one(s + 700, vis).sum(), 1)


def test_frequencies_are_kept_slowed_and_mixed():
    rot = {"base": 300.0, "dims": 20, "scaling": {"factor": 5.0, "low": 2.0, "high": 9.0, "original": 300}}
    f, plain = hr.frequencies(rot), hr.frequencies({"base": 300.0, "dims": 20})
    kinds = set()
    for i in range(10):
        p = 300.0 ** (-2 * i / 20)
        assert np.isclose(plain[i], p)
        wave = 2 * np.pi / p
        if wave < 300 / 9:
            want, kind = p, "kept"
        elif wave > 300 / 2:
            want, kind = p / 5, "slowed"
        else:
            s = (300 / wave - 2) / (9 - 2)
            want, kind = (1 - s) * p / 5 + s * p, "mixed"
        kinds.add(kind)
        assert np.isclose(f[i], want)
    assert kinds == {"kept", "slowed", "mixed"}


def test_rotation_turns_adjacent_pairs_of_the_first_dimensions():
    rot = {"base": 37.0, "dims": 6}
    v = rng().standard_normal((4, 2, 9))
    pos = np.array([0, 1, 5, 1000])
    got = hr.rotate_pairs(v, pos, rot)
    for t, p in enumerate(pos):
        for i in range(3):
            a = p * 37.0 ** (-2 * i / 6)
            x, y = v[t, :, 2 * i], v[t, :, 2 * i + 1]
            assert np.allclose(got[t, :, 2 * i], x * np.cos(a) - y * np.sin(a)) and np.allclose(got[t, :, 2 * i + 1], y * np.cos(a) + x * np.sin(a))
    assert np.array_equal(got[..., 6:], v[..., 6:])
    assert np.allclose(hr.rms(got, 1e-6), hr.rms(v, 1e-6))              # turning keeps the length


def test_attention_reads_the_group_of_its_head():
    q, k, v = rng(1).standard_normal((5, 6, 4)), rng(2).standard_normal((5, 2, 4)), rng(3).standard_normal((5, 2, 3))
    vis = hr.window_mask(np.arange(5), 2)
    got = hr.attend(q, k, v, vis, 0.7).reshape(5, 6, 3)
    for h in range(6):
        for i in range(5):
            js = [j for j in (i - 1, i) if j >= 0]
            e = np.array([np.exp(0.7 * q[i, h] @ k[j, h // 3]) for j in js])
            assert np.allclose(got[i, h], sum(x * v[j, h // 3] for x, j in zip(e, js)) / (1 + e.sum()))


@pytest.mark.parametrize("taps", [1, 2, 4])
def test_convolution_is_causal_with_the_last_tap_on_the_token(taps):
    x, w = rng(4).standard_normal((6, 3)), rng(5).standard_normal((3, taps))
    got = hr.causal_conv(x, w)
    for t in range(6):
        z = sum(x[t - j] * w[:, taps - 1 - j] for j in range(taps) if t - j >= 0)
        assert np.allclose(got[t], z / (1 + np.exp(-z)))


def test_delta_rule_writes_what_is_missing_and_reads_after_it():
    d, e = 5, 3
    k = hr.unit(rng(6).standard_normal((4, d)))
    v = rng(7).standard_normal((4, e))
    # a full step without decay stores the value under its key exactly (up to the unit vector's eps)
    o, S = hr.delta_steps(k, k, v, np.ones(4), np.ones(4))
    assert np.allclose(o, v, atol=1e-5)
    # decay first, then the error against the decayed memory, then the read of the new one
    S0 = rng(8).standard_normal((d, e))
    q = rng(9).standard_normal(d)
    o, S = hr.delta_steps(q[None], k[:1], v[:1], np.array([0.3]), np.array([0.6]), S0)
    want = 0.3 * S0 + 0.6 * np.outer(k[0], v[0] - 0.3 * S0.T @ k[0])
    assert np.allclose(S, want) and np.allclose(o[0], want.T @ q)
    # carried from call to call
    g, b = rng(10).uniform(0, 1, 4), rng(11).uniform(0, 1, 4)
    whole, S1 = hr.delta_steps(k, k, v, g, b)
    first, Sa = hr.delta_steps(k[:1], k[:1], v[:1], g[:1], b[:1])
    rest, S2 = hr.delta_steps(k[1:], k[1:], v[1:], g[1:], b[1:], Sa)
    assert np.allclose(np.concatenate([first, rest]), whole) and np.allclose(S1, S2)


def test_delta_rule_in_blocks_is_the_same_recurrence():
    """The form the library computes: products with the state ahead of the block, and a triangle inside it."""
    n, d, e = 16, 6, 4
    k, q, v = hr.unit(rng(12).standard_normal((n, d))), rng(13).standard_normal((n, d)), rng(14).standard_normal((n, e))
    g, b = np.where(rng(15).uniform(0, 1, n) < 0.2, 1e-30, rng(16).uniform(0.5, 1, n)), rng(17).uniform(0, 1, n)
    S0 = rng(18).standard_normal((d, e))
    want, S = hr.delta_steps(q, k, v, g, b, S0)
    R = np.array([[np.prod(g[i + 1:t + 1]) for t in range(n)] for i in range(n)])
    G = np.cumprod(g)
    u, o = np.zeros((n, e)), np.zeros((n, e))
    for t in range(n):
        u[t] = b[t] * (v[t] - G[t] * S0.T @ k[t] - sum(R[i, t] * (k[i] @ k[t]) * u[i] for i in range(t)))
        o[t] = G[t] * S0.T @ q[t] + sum(R[i, t] * (k[i] @ q[t]) * u[i] for i in range(t + 1))
    assert np.allclose(o, want) and np.allclose(S, G[-1] * S0 + sum(R[i, n - 1] * np.outer(k[i], u[i]) for i in range(n)))


def small_config():
    delta = {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 5, "conv": 3}
    window = {"heads": 3, "kv_heads": 1, "dim": 7, "vdim": 4, "scale": 0.4, "mask": {"size": 5}}
    chunk = {"heads": 2, "kv_heads": 2, "dim": 8, "vdim": 8, "scale": 0.3, "mask": {"size": 4},
             "rot": {"base": 100.0, "dims": 6, "scaling": {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 64}}}
    mlp = {"kind": "dense", "ff": 12}
    return {"architecture": "Vofusun", "width": 20, "vocab": 11, "norm": {"eps": 1e-5}, "embedding": {"scale": 3.0},
            "loop": {"start": 1, "stop": 3, "times": 3},
            "layers": [{"type": "attention", "mixer": window, "mlp": mlp}, {"type": "delta", "mixer": delta, "mlp": None},
                       {"type": "attention_2", "mixer": chunk, "mlp": mlp}, {"type": "delta", "mixer": delta, "mlp": mlp}]}


def small_weights(cfg, seed=3):
    r = rng(seed)
    return {n: r.standard_normal(s) * 0.3 for n, s in hr.tensor_shapes(cfg).items()}


def test_order_of_passes():
    cfg = small_config()
    assert hr.passes(cfg) == [(0, False), (1, False), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    del cfg["loop"]
    assert hr.passes(cfg) == [(i, False) for i in range(4)]


def test_causality_and_passes():
    cfg = small_config()
    w = small_weights(cfg)
    ids = np.arange(9) % cfg["vocab"]
    out = []
    a = hr.forward(cfg, w, ids, out)
    assert len(out) == 8
    assert np.allclose(hr.forward(cfg, w, ids[:5]), a[:5])
    # one pass of the span is the model without a loop; a second one starts from x plus the embeddings
    once = dict(cfg, loop={"start": 1, "stop": 3, "times": 1})
    plain = {k: v for k, v in cfg.items() if k != "loop"}
    assert np.array_equal(hr.forward(once, w, ids), hr.forward(plain, w, ids))
    assert not np.allclose(hr.forward(once, w, ids), a)
    x = out[2] + w["embed"][ids] * 3.0
    f = lambda p: (lambda n: w[p + n])
    y = x + hr.delta_mixer(x / hr.rms(x, 1e-5) * w["l1.norm1"], cfg["layers"][1]["mixer"], f("l1.mix."), 1e-5, np.arange(9))
    assert np.allclose(out[3], y)


def create(b200p, cfg, shapes):
    """b200p_model_create on the host: the pointers are only stored."""
    L = b200p.lib()
    names = list(shapes)
    dims = [d for n in names for d in shapes[n]]
    k = len(names)
    st = C.c_int(0)
    h = L.b200p_model_create(json.dumps(cfg).encode(), k, (C.c_char_p * k)(*[n.encode() for n in names]), (C.c_void_p * k)(*[4096] * k),
                             (C.c_int * k)(*[b200p.BF16] * k), (C.c_int * k)(*[len(shapes[n]) for n in names]),
                             (C.c_longlong * len(dims))(*dims), C.byref(st))
    return h, st.value


def test_registry_reads_the_configuration(b200p):
    for change in (lambda c: None, lambda c: c.pop("loop"), lambda c: c["layers"][2]["mixer"]["rot"].pop("scaling"), lambda c: c.pop("embedding"),
                   lambda c: c["layers"][2]["mixer"]["rot"].update(dims=0)):
        cfg = small_config()
        change(cfg)
        h, st = create(b200p, cfg, hr.tensor_shapes(cfg))
        assert h and st == 0
        mc, name = b200p.ModelConfig(), C.create_string_buffer(32)
        assert b200p.lib().b200p_model_describe(h, name, 32, C.byref(mc)) == 0
        assert name.value == b"Vofusun" and (mc.n_layers, mc.hidden, mc.vocab_size) == (4, 20, 11)
        b200p.lib().b200p_model_free(h)


def test_registry_refuses_what_it_cannot_run(b200p):
    shapes = hr.tensor_shapes(small_config())

    def status(change=lambda c: None, drop=None, reshape=None):
        c = small_config()
        change(c)
        s = {n: v for n, v in shapes.items() if n != drop}
        if reshape:
            s[reshape] = (1,) + tuple(s[reshape])[1:]
        h, st = create(b200p, c, s)
        assert not h
        return st

    mixer = lambda i: (lambda c: c["layers"][i]["mixer"])
    assert status(lambda c: c["layers"][0].update(type="latent_attention")) == -3
    assert status(lambda c: c["layers"][0]["mlp"].update(kind="sparse")) == -3
    assert status(lambda c: mixer(1)(c).pop("conv")) == -11
    assert status(lambda c: mixer(0)(c).pop("mask")) == -11
    assert status(lambda c: mixer(0)(c)["mask"].update(size=0)) == -11
    assert status(lambda c: mixer(2)(c).pop("rot")) == -11
    assert status(lambda c: mixer(2)(c)["rot"]["scaling"].pop("original")) == -11
    assert status(lambda c: mixer(2)(c)["rot"].update(dims=7)) == -11
    assert status(lambda c: mixer(0)(c).update(kv_heads=2)) == -6
    assert status(lambda c: mixer(2)(c).update(vdim=4)) == -6
    assert status(lambda c: c["loop"].update(stop=5)) == -11
    assert status(lambda c: c["loop"].update(times=0)) == -11
    assert status(drop="l1.mix.k.conv") == -11
    assert status(drop="l2.mix.g") == -11
    assert status(reshape="l3.mix.a") == -6
