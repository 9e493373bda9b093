"""The float64 statement of the latent-attention decoder (oracle/latent_ref.py), mechanism by mechanism against direct
formulas, and the host side of the library's model registry.  No GPU."""
import ctypes as C
import json
import os

import numpy as np
import pytest

from oracle import latent_ref as lr


def test_rms_norm_has_eps_inside_the_root():
    x = np.array([[3.0, -4.0, 0.0, 0.0]])
    w = np.array([1.0, 2.0, 3.0, 4.0])
    got = lr.rms_norm(x, w, 0.75)
    assert np.allclose(got, x * w / np.sqrt(25.0 / 4 + 0.75))
    assert np.all(lr.rms_norm(np.zeros((1, 4)), w, 1e-6) == 0)


def test_gelu_is_the_tanh_form():
    z = np.linspace(-6, 6, 25)
    want = [0.5 * v * (1 + np.tanh(np.sqrt(2 / np.pi) * (v + 0.044715 * v * v * v))) for v in z]
    assert np.allclose(lr.gelu_tanh(z), want)


@pytest.mark.parametrize("rotate,pair", [(lr.rotate_interleaved, lambda i, n: (2 * i, 2 * i + 1)),
                                         (lr.rotate_halves, lambda i, n: (i, i + n // 2))])
def test_rotations(rotate, pair):
    n, base = 6, 37.0
    v = np.random.default_rng(0).standard_normal((4, 2, n))
    pos = np.array([0, 1, 5, 1000])
    got = rotate(v, lr.rotation_angles(pos, n, base))
    for t, p in enumerate(pos):
        for i in range(n // 2):
            a = p * base ** (-2 * i / n)
            u, w = pair(i, n)
            assert np.allclose(got[t, :, u], v[t, :, u] * np.cos(a) - v[t, :, w] * np.sin(a))
            assert np.allclose(got[t, :, w], v[t, :, w] * np.cos(a) + v[t, :, u] * np.sin(a))
    assert np.array_equal(got[0], v[0])                       # position 0 does not turn
    # scores depend on the distance only
    q, k = v[0, 0], v[1, 1]
    at = lambda x, p: rotate(x[None], lr.rotation_angles([p], n, base))[0]
    assert np.isclose(at(q, 9) @ at(k, 4), at(q, 105) @ at(k, 100))


def test_softmax_and_sink():
    s = np.array([[1.0, 2.0, 50.0]])
    vis = np.array([[True, True, False]])
    e = np.exp([1.0, 2.0])
    assert np.allclose(lr.softmax_rows(s, vis)[0], [e[0] / e.sum(), e[1] / e.sum(), 0])
    d = e.sum() + np.exp(1.5)
    assert np.allclose(lr.softmax_rows(s, vis, 1.5)[0], [e[0] / d, e[1] / d, 0])
    assert np.allclose(lr.softmax_rows(s, vis, 900.0), 0)     # and no overflow


def test_causality_and_shared_layers():
    cfg = small_config()
    w = {n: np.random.default_rng(3).standard_normal(s) * 0.2 for n, s in lr.tensor_shapes(cfg).items()}
    ids = np.arange(9) % cfg["vocab"]
    a = lr.forward(cfg, w, ids)
    assert np.allclose(lr.forward(cfg, w, ids[:5]), a[:5])
    copied = json.loads(json.dumps(cfg))
    del copied["layers"][1]["weights_of"]
    w2 = dict(w, **{n.replace("l0.", "l1.", 1): v for n, v in w.items() if n.startswith("l0.")})
    assert np.allclose(lr.forward(copied, w2, ids), a)


def small_config():
    mx = {"heads": 3, "dim": 8, "rot_dim": 4, "vdim": 6, "kv_rank": 10, "q_rank": 7, "scale": 0.3, "rot": {"base": 100.0, "dims": 4}}
    layer = {"type": "latent_attention_2", "mixer": mx, "mlp": {"kind": "dense", "ff": 12}}
    return {"architecture": "Maposun", "width": 20, "vocab": 11, "norm": {"eps": 1e-5},
            "layers": [layer, dict(layer, weights_of=0), {"type": "latent_attention", "mixer": mx, "mlp": None}]}


def create(b200p, cfg, shapes):
    """b200p_model_create on the host: the pointers are only stored."""
    L = b200p.lib()
    names = list(shapes)
    dims = [d for n in names for d in shapes[n]]
    k = len(names)
    st = C.c_int(0)
    h = L.b200p_model_create(cfg if isinstance(cfg, bytes) else json.dumps(cfg).encode(), k, (C.c_char_p * k)(*[n.encode() for n in names]),
                             (C.c_void_p * k)(*[4096] * k), (C.c_int * k)(*[b200p.BF16] * k), (C.c_int * k)(*[len(shapes[n]) for n in names]),
                             (C.c_longlong * len(dims))(*dims), C.byref(st))
    return h, st.value


def test_registry_reads_the_configuration(b200p):
    cfg = small_config()
    h, st = create(b200p, cfg, lr.tensor_shapes(cfg))
    assert h and st == 0
    mc, name = b200p.ModelConfig(), C.create_string_buffer(32)
    assert b200p.lib().b200p_model_describe(h, name, 32, C.byref(mc)) == 0
    assert name.value == b"Maposun" and (mc.n_layers, mc.hidden, mc.vocab_size) == (3, 20, 11)
    b200p.lib().b200p_model_free(h)


def test_registry_refuses_what_it_cannot_run(b200p):
    cfg = small_config()
    shapes = lr.tensor_shapes(cfg)

    def status(change, drop=None, reshape=None):
        c = json.loads(json.dumps(cfg))
        change(c)
        s = {n: v for n, v in shapes.items() if n != drop}
        if reshape:
            s[reshape] = (1,) + tuple(s[reshape])[1:]
        h, st = create(b200p, c, s)
        assert not h
        return st

    nothing = lambda c: None
    assert status(lambda c: c.update(architecture="Nobody")) == -3
    assert status(lambda c: c["layers"][0].update(type="attention")) == -3
    assert status(lambda c: c["layers"][0]["mlp"].update(kind="sparse")) == -3
    assert status(lambda c: c["layers"][0]["mixer"].pop("kv_rank")) == -11
    assert status(lambda c: c["layers"][1].update(weights_of=1)) == -11
    assert status(lambda c: c["layers"][1]["mixer"].update(heads=4)) == -6
    assert status(nothing, drop="l0.mix.sink") == -11
    assert status(nothing, reshape="l2.mix.uk") == -6
    assert create(b200p, b'{"architecture": "Maposun", ', shapes)[1] == -11
    assert b200p.lib().b200p_strerror(-3).decode().startswith("unknown")


def test_model_files_round_trip(tmp_path):
    cfg = small_config()
    rng = np.random.default_rng(1)
    w = {n: rng.standard_normal(s).astype(np.float32) for n, s in lr.tensor_shapes(cfg).items()}
    lr.write_model(str(tmp_path), cfg, w)
    assert json.load(open(os.path.join(tmp_path, "config.json"))) == cfg
    back = lr.read_safetensors(os.path.join(tmp_path, "model.safetensors"))
    assert set(back) == set(w)
    for n in w:
        assert np.all(np.abs(back[n] - w[n]) <= np.abs(w[n]) / 256)
