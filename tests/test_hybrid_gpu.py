"""The decoder with gated-delta-rule layers and masked attention (architecture "Vofusun") through the runtime's session
against its float64 statement (oracle/hybrid_ref.py): whole prompts, portions, single tokens, in fp32 and in bf16, on
shapes that take every kernel.

Where random weights would hide a fault, the weights are made so that it shows: one key that takes nearly all of a row just
inside or just outside a window or a chunk, memories that last for hundreds of tokens or are wiped by a single one.
Errors are the root mean square over the vocabulary of the difference (mean taken off), relative to the logits' standard
deviation: the bar is 1e-4 in fp32 and 0.06 in bf16."""
import json
import os
import subprocess

import numpy as np
import pytest

from oracle import hybrid_ref as hr
from oracle import latent_ref as lr

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BAR = {"f32": 1e-4, "bf16": 0.06}
SCALING = {"factor": 6.0, "low": 1.5, "high": 5.0, "original": 200}


def delta(heads, kv, dim, vdim, taps, ff=None):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": taps}, "mlp": ff and {"kind": "dense", "ff": ff}}


def window(heads, kv, dim, vdim, size, ff=None, scale=None):
    return {"type": "attention", "mlp": ff and {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale or 1.5 / np.sqrt(dim), "mask": {"size": size}}}


def chunk(heads, kv, dim, size, turning, ff=None, scale=None, base=500.0, scaling=SCALING):
    return {"type": "attention_2", "mlp": ff and {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": scale or 1.5 / np.sqrt(dim), "mask": {"size": size},
                      "rot": {"base": base, "dims": turning, "scaling": scaling}}}


def config(width, vocab, layers, loop=None, eps=1e-5, scale=4.0):
    out = {"architecture": "Vofusun", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}
    if loop:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


CONFIGS = {
    # nothing a multiple of 16, an MLP missing, shared query/key heads, a loop in the middle
    "odd": config(200, 333, [delta(6, 2, 24, 40, 3, 168), chunk(6, 3, 40, 24, 20, 100), window(5, 1, 24, 56, 17), delta(3, 3, 40, 22, 5, 72),
                             window(4, 4, 16, 8, 33, 40)], (1, 4, 3), 1e-3, 2.5),
    "ones": config(48, 50, [delta(1, 1, 1, 1, 1, 16), window(1, 1, 1, 1, 1, 16), chunk(1, 1, 2, 1, 2, 16)], (0, 3, 2)),
    # more query heads per key head than one 16-row tile; windows beyond the sequence
    "many_heads": config(96, 130, [window(20, 1, 16, 48, 1000, 64), chunk(40, 2, 32, 70, 32), delta(20, 4, 32, 16, 2, 64)]),
    # the head sizes of large models
    "real_heads": config(288, 200, [delta(4, 2, 128, 128, 4, 352), chunk(8, 2, 128, 160, 64, 352), window(4, 1, 128, 128, 130, 352)], (0, 2, 2)),
    # query/key and value heads of different box counts, S with several 64-column slices
    "unequal": config(128, 96, [window(4, 2, 48, 112, 50, 96), window(4, 2, 96, 64, 129, 96), delta(2, 1, 96, 200, 4, 96), delta(2, 2, 64, 80, 7)]),
    # an MLP too wide for the streaming kernels with eight rows and more
    "wide_mlp": config(64, 70, [window(2, 1, 16, 16, 9, 12304), delta(2, 2, 16, 16, 4, 12304)]),
    # outside the tensor-core and register kernels' domain
    "too_wide": config(128, 96, [delta(2, 1, 160, 300, 4, 96), window(2, 1, 144, 160, 40, 96), chunk(2, 2, 152, 30, 100), delta(2, 2, 16, 272, 4)]),
    "no_scaling": config(80, 60, [chunk(2, 1, 24, 50, 24, 64, scaling=None), delta(2, 2, 32, 64, 4), chunk(2, 1, 24, 50, 0, 64, scaling=None)]),
}
EVERY = sorted(CONFIGS)
_cache = {}


def bf16(a):
    a = np.asarray(a)
    return (lr.bf16_bits(a).astype(np.uint32) << 16).view(np.float32).reshape(a.shape)


def weights(name, cfg=None):
    if name not in _cache:
        cfg = cfg or CONFIGS[name]
        rng = np.random.default_rng(sum(name.encode()))
        w = {}
        for n, s in hr.tensor_shapes(cfg).items():
            if n.endswith("A_log"):
                a = rng.uniform(-4, 1, s)
            elif n.endswith("dt_bias"):
                a = rng.uniform(-3, 1, s)
            elif n.endswith(".conv"):
                a = rng.standard_normal(s) * 0.7
            elif n == "embed":
                a = rng.standard_normal(s) / np.sqrt(s[1]) * 2
            elif "norm" in n:
                a = rng.uniform(0.5, 1.5, s)
            else:
                a = rng.standard_normal(s) / np.sqrt(s[1])
            w[n] = bf16(a)
        _cache[name] = w
    return _cache[name]


def tokens(cfg, n, seed=0):
    return np.random.default_rng(1000 + seed).integers(0, cfg["vocab"], n)


_ref = {}


def reference(name, ids, cfg=None):
    """Causal: a prefix of a longer sequence's logits does."""
    ids = tuple(int(i) for i in ids)
    for (n, other), out in _ref.items():
        if n == name and other[:len(ids)] == ids:
            return out[:len(ids)]
    _ref[name, ids] = hr.forward(cfg or CONFIGS[name], weights(name, cfg), ids)
    return _ref[name, ids]


@pytest.fixture
def opened(b200p, torch_cuda):
    """name -> session; closed at the end of the test."""
    torch = torch_cuda
    live = []

    def make(name, dtype="f32", max_seq=512, batch=1, cfg=None):
        t = {n: torch.from_numpy(np.ascontiguousarray(a)).cuda().bfloat16() for n, a in weights(name, cfg).items()}
        s = b200p.Session.from_model(b200p.Model.from_tensors(cfg or CONFIGS[name], t), max_seq, batch, b200p.F32 if dtype == "f32" else b200p.BF16)
        live.append(s)
        return s

    yield make
    for s in live:
        s.close()
    assert b200p.device_status() == 0


@pytest.fixture
def knob(b200p):
    used = []

    def turn(key, value):
        used.append(key)
        b200p.set_tuning(key, value)

    yield turn
    for key in used:
        b200p.set_tuning(key, -1)


def errors(got, want):
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / want.std()


def check(got, want, dtype, what=""):
    e = errors(got, want)
    if what == "signs":                                         # a few rows may be anything
        e = np.sort(e)[:max(1, int(0.97 * len(e)))]
    assert np.isfinite(e).all() and e.max() < BAR[dtype], (what, int(e.argmax()), float(e.max()))


def run(session, ids, portions):
    """Logits of every token, the sequence fed in the given portions (the last one repeats)."""
    session.reset()
    out, at, k = [], 0, 0
    while at < len(ids):
        n = min(portions[min(k, len(portions) - 1)], len(ids) - at)
        out.append(session.extend([ids[at:at + n]], range(n))[0])
        at += n
        k += 1
    assert session.kv_len == len(ids)
    return np.concatenate(out)


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", EVERY)
def test_whole_prompt(opened, name, dtype):
    s = opened(name, dtype)
    ids = tokens(CONFIGS[name], 170)
    reference(name, ids)
    for n in (170, 1, 2, 3, 15, 16, 17, 33, 150):              # blocks of 16 tokens, tiles of 128 keys
        check(run(s, ids[:n], [n]), reference(name, ids[:n]), dtype, "signs" if name == "ones" and dtype == "bf16" else n)


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", EVERY)
def test_portions_and_single_tokens(opened, name, dtype):
    s = opened(name, dtype)
    ids = tokens(CONFIGS[name], 170)
    want = reference(name, ids)
    for portions in ([1], [2], [3], [60, 3, 2, 17, 1, 1, 33, 2, 16], [129, 5, 20], [1, 2, 1, 40], [150, 1]):
        # heads of one column: a unit vector is a sign, and rounding turns one that is close to zero
        check(run(s, ids, portions), want, dtype, "signs" if name == "ones" and dtype == "bf16" else portions)


@pytest.mark.parametrize("name", ["odd", "real_heads", "unequal"])
def test_fp32_does_not_depend_on_the_cut(opened, name):
    s = opened(name, "f32")
    ids = tokens(CONFIGS[name], 90, 2)
    whole = run(s, ids, [90])
    for portions in ([1], [7], [16], [45, 2]):
        assert errors(run(s, ids, portions), whole).max() < 3e-5


# ---- edges of windows and chunks -------------------------------------------------------------------------------------
# Token 1 asks, token 0 answers, the others do neither: one attention layer whose only large score (about 13) is between the
# two, in a direction that does not turn; all other scores of token 1 are 0.
def pointed(kind, size):
    dim = 32
    layer = window(2, 1, dim, dim, size, scale=0.8) if kind == "window" else chunk(2, 1, dim, size, 8, scale=0.4)
    cfg = config(64, 40, [layer], scale=1.0)
    name = "%s%d" % (kind, size)
    if name not in _cache:
        rng = np.random.default_rng(7)
        w = {n: np.zeros(s) for n, s in hr.tensor_shapes(cfg).items()}
        w["embed"][2:, 8:] = rng.standard_normal((38, 56)) * 0.5
        w["embed"][0, 0] = w["embed"][1, 1] = 2.0                  # 8 after the norm
        w["l0.norm1"][:] = w["final.norm"][:] = 1.0
        w["l0.mix.k"][31, 0] = w["l0.mix.q"][31, 1] = w["l0.mix.q"][dim + 31, 1] = 0.5
        if kind == "window":
            w["l0.mix.v"][:, 0] = rng.standard_normal(dim)
            w["l0.mix.v"][:, 8:] = rng.standard_normal((dim, 56)) * 0.1
        else:
            w["l0.mix.k"][:24, 8:] = rng.standard_normal((24, 56)) * 0.1
            w["l0.mix.g"][:] = rng.standard_normal(w["l0.mix.g"].shape) * 0.2
        w["l0.mix.o"][:] = rng.standard_normal(w["l0.mix.o"].shape)
        _cache[name] = {n: bf16(a) for n, a in w.items()}
    return name, cfg


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("kind,size", [("window", 1), ("window", 2), ("window", 17), ("window", 64), ("window", 100), ("window", 127), ("window", 128), ("window", 129), ("window", 300),
                                       ("chunk", 2), ("chunk", 19), ("chunk", 48), ("chunk", 128), ("chunk", 130), ("chunk", 256)])
def test_edges(opened, kind, size, dtype):
    name, cfg = pointed(kind, size)
    w = weights(name, cfg)
    s = opened(name, dtype, max_seq=700, cfg=cfg)
    rng = np.random.default_rng(size)
    seen = {}
    base = 290 if kind == "window" else (600 // size - 1) * size        # the answer's place or the chunk's first position
    for inside in (True, False):
        if kind == "window":
            at, ask = base, base + size - (1 if inside else 0)
        else:
            at, ask = (base, base + size - 1) if inside else (base - 1, base)
        if at == ask:                                                       # a window of one: the token sees only itself
            continue
        ids = rng.integers(2, 40, ask + 3)
        ids[at], ids[ask] = 0, 1
        want = hr.forward(cfg, w, ids)
        blank = ids.copy()
        blank[at] = 2
        seen[inside] = errors(hr.forward(cfg, w, blank)[ask:ask + 1], want[ask:ask + 1])[0]
        for portions in ([len(ids)], [ask, 1], [max(ask - 40, 1), 39, 2, 1], [at + 1, 1] if inside and size < 200 else [max(at, 1), 3, 1]):
            got = run(s, ids, portions)
            check(got[ask:], want[ask:], dtype, (inside, portions))
            check(got, want, dtype, (inside, portions))
    if len(seen) == 2:
        assert seen[True] > 0.3 and seen[False] < 1e-9                      # the oracle's row depends on the key inside, and not on the one outside


def test_decoding_passes_windows_chunks_and_key_tiles(opened):
    """Long decoding: windows and chunks of every layer pass over decoded tokens many times."""
    name = "odd"
    s = opened(name, "bf16", max_seq=420)
    ids = tokens(CONFIGS[name], 400, 3)
    check(run(s, ids, [5, 1]), reference(name, ids), "bf16")
    name = "real_heads"
    s = opened(name, "bf16", max_seq=420)
    ids = tokens(CONFIGS[name], 400, 3)
    check(run(s, ids, [120, 1]), reference(name, ids), "bf16")


@pytest.mark.parametrize("splits", [1, 2, 3, 8])
def test_key_splits_of_the_step(opened, knob, splits):
    knob("decode_splits", splits)
    for name, n in (("many_heads", 300), ("real_heads", 300), ("unequal", 170)):
        s = opened(name, "bf16", max_seq=400)
        ids = tokens(CONFIGS[name], n)
        check(run(s, ids, [n - 40, 1])[n - 40:], reference(name, ids)[n - 40:], "bf16", name)
        check(run(s, ids[:20], [1]), reference(name, ids[:20]), "bf16", name)


@pytest.mark.parametrize("dtype,splits", [("f32", 0), ("bf16", 0), ("bf16", 1), ("bf16", 2)])
def test_masks_of_many_key_tiles(opened, knob, dtype, splits):
    """Windows and chunks of about a thousand keys: every ring of key tiles goes round more than once, in prompts and in
    decoding."""
    cfg = config(96, 90, [window(4, 2, 64, 48, 1000), window(2, 1, 128, 112, 900), chunk(2, 1, 32, 1040, 32, scale=0.3), delta(2, 2, 32, 32, 4)])
    name = "long"
    ids = tokens(cfg, 1150, 16)
    want = reference(name, ids, cfg)
    if splits:
        knob("decode_splits", splits)
    s = opened(name, dtype, max_seq=1150, cfg=cfg)
    for portions in ([1150], [1030, 1], [600, 300, 130, 2]):
        check(run(s, ids, portions), want, dtype, portions)


# ---- memories ----------------------------------------------------------------------------------------------------------
def memory_model(name, a_log, dt_bias, taps=4):
    cfg = config(96, 120, [delta(4, 2, 40, 72, taps), delta(2, 2, 64, 32, taps)])
    if name in _cache:
        return cfg
    w = weights(name, cfg)
    for n in w:
        if n.endswith("A_log"):
            w[n][:] = bf16(np.resize(a_log, w[n].shape).astype(np.float32))
        elif n.endswith("dt_bias"):
            w[n][:] = bf16(np.resize(dt_bias, w[n].shape).astype(np.float32))
        elif n.endswith(".b") and "lasting" in name:
            w[n][:] = bf16(w[n] * 0.2)
    return cfg


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_lasting_memory(opened, dtype):
    """Decays of almost one: what was written hundreds of tokens ago still moves the logits."""
    name = "lasting"
    cfg = memory_model(name, [-9.0, -7.0], [-2.0])
    ids = tokens(cfg, 420, 4)
    ids[60:] = ids[60 + np.arange(360) % 4]                     # then nothing but four tokens over and over: few keys are overwritten
    want = reference(name, ids, cfg)
    other = ids.copy()
    other[:60] = tokens(cfg, 60, 5)
    assert errors(hr.forward(cfg, weights(name, cfg), other)[-20:], want[-20:]).mean() > 0.05
    s = opened(name, dtype, max_seq=420, cfg=cfg)
    for portions in ([420], [64, 2, 5, 100, 1, 1, 17], [390, 1]):
        check(run(s, ids, portions), want, dtype, portions)


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_decays_from_none_to_total(opened, dtype):
    """Heads whose decay is anything from 1 to exp(-hundreds), some within one block of sixteen tokens."""
    name = "wiped"
    cfg = memory_model(name, [-30.0, 5.0, 2.5, -1.0], [0.0, -4.0, 3.0])
    ids = tokens(cfg, 150, 6)
    want = reference(name, ids, cfg)
    s = opened(name, dtype, max_seq=200, cfg=cfg)
    for portions in ([150], [1], [16, 3, 40, 1, 1, 15]):
        check(run(s, ids, portions), want, dtype, portions)


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6, 9])
def test_convolution_history(opened, taps):
    """Portions shorter and longer than the history, one token at a time, and both mixed."""
    name = "taps%d" % taps
    cfg = memory_model(name, [0.0], [0.0], taps)
    ids = tokens(cfg, 60, 7)
    want = reference(name, ids, cfg)
    s = opened(name, "f32", max_seq=60, cfg=cfg)
    for portions in ([60], [1], [2], [3], [5], [20, 1, 2, 1, 1, 3, 16, 1]):
        check(run(s, ids, portions), want, "f32", portions)


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_far_tokens_reach_through_several_windows(opened, dtype):
    """Layers in a row carry a token further than one window; the first tokens of the sequence included."""
    cfg = config(96, 120, [window(2, 1, 40, 24, 90, scale=0.35), window(2, 2, 24, 40, 70, scale=0.35), chunk(2, 1, 40, 128, 16, scale=0.3)], (0, 3, 3))
    name = "relay"
    ids = tokens(cfg, 420, 8)
    want = reference(name, ids, cfg)
    other = ids.copy()
    other[:40] = tokens(cfg, 40, 9)
    moved = errors(hr.forward(cfg, weights(name, cfg), other), want)
    assert moved[150:250].max() > 0.01                          # further than any one mask
    s = opened(name, dtype, max_seq=420, cfg=cfg)
    for portions in ([420], [200, 100, 30, 2], [380, 1]):
        check(run(s, ids, portions), want, dtype, portions)


def test_one_pass_is_no_loop(opened):
    cfg = CONFIGS["odd"]
    a, b = dict(cfg, loop={"start": 1, "stop": 4, "times": 1}), {k: v for k, v in cfg.items() if k != "loop"}
    _cache["odd_once"] = _cache["odd_plain"] = weights("odd")
    ids = tokens(cfg, 60, 10)
    for dtype in ("f32", "bf16"):
        assert np.array_equal(run(opened("odd_once", dtype, cfg=a), ids, [40, 3, 1]), run(opened("odd_plain", dtype, cfg=b), ids, [40, 3, 1]))


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", ["odd", "too_wide"])
def test_cache_and_state_used_again(opened, name, dtype):
    """A shorter sequence after a longer one, and the first one again: nothing is left over."""
    s = opened(name, dtype, max_seq=300)
    first, second = tokens(CONFIGS[name], 190, 11), tokens(CONFIGS[name], 70, 12)
    a = run(s, first, [100, 17, 1])
    for portions in ([30, 2, 1], [1], [2, 5]):
        check(run(s, second, portions), reference(name, second), dtype, portions)
    assert np.array_equal(run(s, first, [100, 17, 1]), a)


@pytest.mark.parametrize("name,dtype,batch", [("odd", "bf16", 3), ("odd", "f32", 2), ("wide_mlp", "bf16", 8), ("many_heads", "bf16", 5), ("many_heads", "bf16", 20),
                                              ("real_heads", "bf16", 12), ("too_wide", "bf16", 2)])
def test_batch_against_each_alone(opened, name, dtype, batch):
    s = opened(name, dtype, max_seq=128, batch=batch)
    ids = np.stack([tokens(CONFIGS[name], 90, 20 + b) for b in range(batch)])
    got, at = [], 0
    for n in (40, 3, 1, 1, 2, 30, 1, 12):
        got.append(s.extend(ids[:, at:at + n], range(n)))
        at += n
    got = np.concatenate(got, axis=1)
    for b in range(batch):
        check(got[b], reference(name, ids[b]), dtype, b)


def test_wanted_places(opened):
    name = "real_heads"
    s = opened(name, "bf16")
    ids = tokens(CONFIGS[name], 80, 13)
    everything = s.extend([ids], range(80))[0]
    for want in ([79], [0], [3, 3, 70, 12], [], list(range(40))):
        s.reset()
        got = s.extend([ids], want)
        assert got.shape == (1, len(want), CONFIGS[name]["vocab"])
        if want:
            assert errors(got[0], everything[want]).max() < 2e-3


@pytest.mark.parametrize("key", ["grouped_plain", "delta_plain"])
@pytest.mark.parametrize("name", ["odd", "many_heads", "real_heads", "unequal"])
def test_plain_and_fast_kernels_agree(opened, knob, name, key):
    ids = tokens(CONFIGS[name], 150)
    for dtype in ("bf16",) if key == "grouped_plain" else ("f32", "bf16"):
        s = opened(name, dtype)
        fast = run(s, ids, [100, 20, 2, 1])
        knob(key, 1)
        plain = run(s, ids, [100, 20, 2, 1])
        knob(key, -1)
        check(fast, plain.astype(np.float64), dtype)


@pytest.mark.parametrize("columns", [1, 2, 4])
@pytest.mark.parametrize("name", ["odd", "real_heads", "unequal", "no_scaling"])
def test_forms_of_the_block_walk(opened, knob, name, columns):
    """The delta rule's blocks with and without tensor cores, whatever the columns are dealt to."""
    ids = tokens(CONFIGS[name], 150)
    knob("delta_columns", columns)
    for dtype, tensor in (("bf16", 1), ("bf16", 0), ("f32", 1)):
        knob("delta_tensor", tensor)
        s = opened(name, dtype)
        check(run(s, ids, [100, 20, 2, 1]), reference(name, ids), dtype, (tensor, columns))


@pytest.mark.parametrize("name,dtype,batch", [("odd", "bf16", 2), ("odd", "f32", 1), ("real_heads", "bf16", 1), ("too_wide", "bf16", 1)])
def test_greedy_generation(opened, name, dtype, batch):
    """generate() (the greedy loop, replayed as a graph where the step can be captured): the tokens of the host-driven loop
    on the same session, and of the oracle wherever its best logit is clear of the second."""
    cfg = CONFIGS[name]
    T, new = 37, 24
    s = opened(name, dtype, max_seq=T + new, batch=batch)
    ids = np.stack([tokens(cfg, T, 30 + b) for b in range(batch)])
    toks, _ = s.generate(ids, new)
    captured = dtype == "bf16" and name != "too_wide"
    assert s.graph_replays == (new - 2 if captured else 0) and s.kv_len == T + new - 1
    lg = s.prefill_logits(ids)
    for k in range(new):
        assert np.array_equal(np.argmax(bf16(lg) if dtype == "bf16" else lg, -1), toks[:, k]), k
        if k + 1 < new:
            lg = s.step_logits(toks[:, k])
    for b in range(batch):
        seq = np.concatenate([ids[b], toks[b]])
        ref = hr.forward(cfg, weights(name), seq[:-1])[T - 1:]
        top = np.sort(ref, -1)
        clear = top[:, -1] - top[:, -2] > (0.5 if dtype == "bf16" else 1e-3) * ref.std()
        assert np.array_equal(np.argmax(ref, -1)[clear], toks[b][clear])
    again, _ = s.generate(ids, new)
    assert np.array_equal(again, toks)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_programs(tmp_path, torch_cuda, dtype):
    name, cfg = "odd", CONFIGS["odd"]
    lr.write_model(str(tmp_path / "m"), cfg, weights(name))
    out = tmp_path / "out"
    out.mkdir()
    a, b = tokens(cfg, 50, 14), tokens(cfg, 9, 15)
    steps = [("a", a[:30], [0, 29], []), ("a", a[30:32], [], []), ("a", a[32:], [0, 5, 17], ["a"]), ("b", b[:1], [0], []), ("b", b[1:], [7], ["b"])]
    lines = [json.dumps({"step": k, "entries": [{"id": i, "tokens": [int(x) for x in t], "want": w}], "end": e}) for k, (i, t, w, e) in enumerate(steps)]
    model = ["--model", str(tmp_path / "m"), "--dtype", dtype]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), *model, "--out", str(out), "--max-tokens", "64"], input="\n".join(lines) + "\n",
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert r.stdout.split("\n")[:-1] == ["done %d" % k for k in range(len(steps))]
    ra, rb = reference(name, a), reference(name, b)
    for k, rows in ((0, ra[[0, 29]]), (2, ra[[32, 37, 49]]), (3, rb[[0]]), (4, rb[[8]])):
        check(np.fromfile(str(out / ("%d.f32" % k)), "<f4").reshape(rows.shape), rows, {"float32": "f32", "bfloat16": "bf16"}[dtype], k)
    assert not (out / "1.f32").exists()
    r = subprocess.run([os.path.join(ROOT, "bin", "generate"), *model, "--max-new", "3", "--prompt", " ".join(map(str, a))], capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    new = [int(x) for x in r.stdout.split()]
    assert len(new) == 3
    ref = ra[-1]
    if np.sort(ref)[-1] - np.sort(ref)[-2] > 0.5 * ref.std() or dtype == "float32":
        assert new[0] == int(np.argmax(ref))
