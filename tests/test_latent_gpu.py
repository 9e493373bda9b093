"""The decoder with latent attention (architecture "Maposun") through the runtime's session against its float64 statement
(oracle/latent_ref.py): whole prompts, portions, single tokens, in fp32 and in bf16, on shapes that take every kernel.

Weights are random; the attention scale is set so that softmax is far from uniform (a row's largest weight is often above
one half), so a key too many or too few, a wrong rotation or a missing sink moves the logits by far more than rounding.
Errors are the root mean square over the vocabulary of the difference (mean taken off), relative to the logits'
standard deviation: the bar is 1e-4 in fp32 and 0.06 in bf16."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import latent_ref as lr

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BAR = {"f32": 1e-4, "bf16": 0.06}


def mixer(heads, dim, rot, vdim, kv, q, base=10000.0, scale=None, turning=None):
    return {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": kv, "q_rank": q,
            "rot": {"base": base, "dims": rot if turning is None else turning}, "scale": scale or 1.5 / np.sqrt(dim + rot)}


def config(width, vocab, layers, eps=1e-5):
    """layers: (type suffix, mixer, ff or None[, weights_of])."""
    out = []
    for kind, mx, ff, *of in layers:
        e = {"type": "latent_attention" + kind, "mixer": mx, "mlp": {"kind": "dense", "ff": ff} if ff else None}
        if of:
            e["weights_of"] = of[0]
        out.append(e)
    return {"architecture": "Maposun", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": out}


ODD = mixer(5, 24, 12, 40, 72, 56, 500.0)
ODD2 = mixer(3, 40, 6, 22, 100, 36)
ONE = mixer(1, 16, 2, 16, 16, 16, 3.0)
MANY = mixer(20, 16, 16, 16, 48, 32)
REAL = mixer(16, 128, 64, 128, 512, 112)
CONFIGS = {
    # nothing a multiple of 16, layers without MLP, shared layers, both mixers with different sizes
    "odd": config(200, 333, [("", ODD, 168), ("_2", ODD2, None), ("", ODD, 168, 0), ("_2", ODD2, None, 1), ("_2", ODD, 100)], 1e-3),
    "one_head": config(64, 50, [("_2", ONE, 32), ("", ONE, 48)]),
    # more query rows than one 16-row tile for a single token
    "many_heads": config(96, 130, [("_2", MANY, 64), ("", MANY, None), ("", MANY, 64)]),
    # the head sizes of the large models: the widest prefill and decode kernels
    "real_heads": config(288, 200, [("_2", REAL, 352), ("", REAL, 352)]),
    # key and value heads of different box counts
    # an MLP too wide for the streaming kernels with eight rows and more
    "wide_mlp": config(64, 70, [("", mixer(2, 16, 8, 16, 32, 32), 12304)]),
    "wide_keys": config(128, 96, [("", mixer(4, 96, 32, 48, 160, 64), 96), ("_2", mixer(4, 48, 64, 112, 272, 80), 96)]),
    # rotated parts of which only the first dimensions turn, an odd number among them
    "partly_rotated": config(80, 60, [("", mixer(3, 32, 20, 32, 48, 40, 50.0, turning=8), 64), ("_2", mixer(2, 16, 13, 16, 32, 32, 50.0, turning=10), 64)]),
    # outside the tensor-core kernels' domain
    "too_wide": config(128, 96, [("", mixer(2, 144, 80, 160, 600, 64), 96), ("_2", mixer(2, 24, 16, 32, 528, 48), 96)]),
}
EVERY = sorted(CONFIGS)
_cache = {}


def weights(name, cfg=None):
    key = name
    if key not in _cache:
        cfg = cfg or CONFIGS[name]
        rng = np.random.default_rng(sum(name.encode()))
        w = {}
        for n, s in lr.tensor_shapes(cfg).items():
            if n.endswith("sink"):
                a = rng.uniform(-3, 5, s)
            elif n == "embed":
                a = rng.standard_normal(s)
            elif "norm" in n:
                a = rng.uniform(0.5, 1.5, s)
            else:
                a = rng.standard_normal(s) / np.sqrt(s[1])
            w[n] = (lr.bf16_bits(a).astype(np.uint32) << 16).view(np.float32).reshape(s)
        _cache[key] = w
    return _cache[key]


def tokens(cfg, n, seed=0):
    return np.random.default_rng(1000 + seed).integers(0, cfg["vocab"], n)


_ref = {}


def reference(name, ids, cfg=None):
    key = (name, tuple(int(i) for i in ids))
    if key not in _ref:
        _ref[key] = lr.forward(cfg or CONFIGS[name], weights(name, cfg), ids)
    return _ref[key]


@pytest.fixture
def opened(b200p, torch_cuda):
    """name -> session; closed at the end of the test."""
    torch = torch_cuda
    live = []

    def make(name, dtype="f32", max_seq=512, batch=1, cfg=None):
        c = cfg or CONFIGS[name]
        t = {n: torch.from_numpy(np.ascontiguousarray(a)).cuda().bfloat16() for n, a in weights(name, cfg).items()}
        s = b200p.Session.from_model(b200p.Model.from_tensors(c, t), max_seq, batch, b200p.F32 if dtype == "f32" else b200p.BF16)
        live.append(s)
        return s

    yield make
    for s in live:
        s.close()
    assert b200p.device_status() == 0


def errors(got, want):
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / want.std()


def check(got, want, dtype, what=""):
    e = errors(got, want)
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
    cfg = CONFIGS[name]
    s = opened(name, dtype)
    for n in (1, 2, 16, 17, 150):                              # the last is over a 128-key tile; 1..16 run on the streaming kernels
        ids = tokens(cfg, n)
        check(run(s, ids, [n]), reference(name, ids), dtype, n)


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", EVERY)
def test_portions_and_single_tokens(opened, name, dtype):
    cfg = CONFIGS[name]
    s = opened(name, dtype)
    ids = tokens(cfg, 170, 1)
    want = reference(name, ids)
    for portions in ([1], [2], [60, 3, 2, 17, 1, 1, 33, 2, 16], [129, 5, 20], [150, 1]):
        check(run(s, ids, portions), want, dtype, portions)


@pytest.mark.parametrize("name", ["odd", "real_heads"])
def test_fp32_does_not_depend_on_the_cut(opened, name):
    s = opened(name, "f32")
    ids = tokens(CONFIGS[name], 90, 2)
    whole = run(s, ids, [90])
    for portions in ([1], [7], [45, 2]):
        assert errors(run(s, ids, portions), whole).max() < 2e-5


def test_key_tiles_edges_in_decoding(opened):
    """Decoding across the 64-key tiles and the splits of the cache, and prompts that end on their edges."""
    name = "many_heads"
    s = opened(name, "bf16", max_seq=700)
    ids = tokens(CONFIGS[name], 400, 3)
    want = reference(name, ids)
    for n in (62, 63, 64, 65, 127, 128, 129, 191, 256, 395):
        check(run(s, ids[:n + 4], [n, 1]), want[:n + 4], "bf16", n)
    check(run(s, ids, [5, 1]), want, "bf16", "long decoding")


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("sharp", [1.0, 6.0])
def test_far_keys(opened, dtype, sharp):
    """One layer, sharp scores: most rows have one key that takes nearly everything, hundreds of tokens back for many.
    The oracle's own weights say so, and the logits follow."""
    mx = mixer(2, 40, 24, 24, 64, 48, 1e4, sharp * 1.5 / np.sqrt(64))
    cfg = config(96, 120, [("", mx, None)])
    name = "far%g" % sharp
    ids = tokens(cfg, 600, 4)
    want = reference(name, ids, cfg)
    cut = lr.forward(cfg, weights(name, cfg), ids[200:])       # without the first 200 tokens (positions move along: scores do not)
    if sharp > 1:
        assert np.mean(errors(cut[-50:], want[-50:])) > 0.2    # they matter
    s = opened(name, dtype, max_seq=600, cfg=cfg)
    for portions in ([600], [300, 100, 30, 2], [560, 1]):
        check(run(s, ids, portions), want, dtype, portions)


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_sinks(opened, dtype):
    """Sinks from nothing to everything: a layer whose sinks are left out, scaled or counted per key differs grossly."""
    cfg = config(96, 120, [("_2", mixer(6, 40, 24, 24, 64, 48), None)])
    name = "sinks"
    w = weights(name, cfg)
    ids = tokens(cfg, 140, 5)
    s = None
    for sink in (np.full(6, -30.0), np.array([-2.0, 0, 1, 2, 3, 4]), np.full(6, 8.0), np.full(6, 60.0)):
        w["l0.mix.sink"] = (lr.bf16_bits(sink).astype(np.uint32) << 16).view(np.float32)
        want = lr.forward(cfg, w, ids)
        s = opened(name, dtype, cfg=cfg)
        for portions in ([140], [20, 1], [40, 17, 2]):
            check(run(s, ids, portions), want, dtype, (float(sink[0]), portions))


def test_shared_layers_have_their_own_cache(opened):
    """The same as the layers written out twice, bit for bit."""
    cfg = CONFIGS["odd"]
    w = weights("odd")
    full = json.loads(json.dumps(cfg))
    copy = dict(w)
    for i, L in enumerate(full["layers"]):
        j = L.pop("weights_of", None)
        if j is not None:
            copy.update({n.replace("l%d." % j, "l%d." % i, 1): a for n, a in w.items() if n.startswith("l%d." % j)})
    _cache["odd_full"] = {n: copy[n] for n in lr.tensor_shapes(full)}
    ids = tokens(cfg, 60, 6)
    for dtype in ("f32", "bf16"):
        a, b = opened("odd", dtype), opened("odd_full", dtype, cfg=full)
        assert np.array_equal(run(a, ids, [40, 3, 1]), run(b, ids, [40, 3, 1]))


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_cache_used_again(opened, dtype):
    """A shorter sequence after a longer one, and the first one again: nothing is left over."""
    name = "odd"
    s = opened(name, dtype, max_seq=300)
    first, second = tokens(CONFIGS[name], 290, 7), tokens(CONFIGS[name], 70, 8)
    a = run(s, first, [200, 17, 1])
    check(run(s, second, [30, 2, 1]), reference(name, second), dtype)
    assert np.array_equal(run(s, first, [200, 17, 1]), a)


@pytest.mark.parametrize("name,dtype,batch", [("odd", "bf16", 3), ("odd", "f32", 2), ("wide_mlp", "bf16", 8), ("many_heads", "bf16", 5), ("many_heads", "bf16", 20),
                                              ("real_heads", "bf16", 12)])
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


@pytest.mark.parametrize("name", ["odd", "real_heads"])
def test_wanted_places(opened, name):
    s = opened(name, "bf16")
    ids = tokens(CONFIGS[name], 80, 9)
    everything = s.extend([ids], range(80))[0]
    for want in ([79], [0], [3, 3, 70, 12], [], list(range(40))):
        s.reset()
        got = s.extend([ids], want)
        assert got.shape == (1, len(want), CONFIGS[name]["vocab"])
        if want:
            assert errors(got[0], everything[want]).max() < 2e-3


@pytest.mark.parametrize("name", ["odd", "many_heads", "real_heads", "wide_keys"])
def test_plain_and_tensor_core_kernels_agree(b200p, opened, name):
    s = opened(name, "bf16")
    ids = tokens(CONFIGS[name], 150, 10)
    fast = run(s, ids, [100, 20, 2, 1])
    b200p.set_tuning("latent_plain", 1)
    try:
        plain = run(s, ids, [100, 20, 2, 1])
    finally:
        b200p.set_tuning("latent_plain", -1)
    check(fast, plain.astype(np.float64), "bf16")


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
        lg_b = (lr.bf16_bits(lg).astype(np.uint32) << 16).view(np.float32).reshape(lg.shape) if dtype == "bf16" else lg
        assert np.array_equal(np.argmax(lg_b, -1), toks[:, k]), k
        if k + 1 < new:
            lg = s.step_logits(toks[:, k])
    for b in range(batch):
        seq = np.concatenate([ids[b], toks[b]])
        ref = lr.forward(cfg, weights(name), seq[:-1])[T - 1:]
        top = np.sort(ref, -1)
        clear = top[:, -1] - top[:, -2] > (0.5 if dtype == "bf16" else 1e-3) * ref.std()
        assert np.array_equal(np.argmax(ref, -1)[clear], toks[b][clear])
    again, _ = s.generate(ids, new)
    assert np.array_equal(again, toks)


def test_argument_errors_leave_the_session_usable(b200p, opened):
    s = opened("odd", "bf16", max_seq=64)
    ids = tokens(CONFIGS["odd"], 60, 11)
    with pytest.raises(b200p.B200PError) as e:
        s.extend([np.full(3, 333)], [0])                       # no such token
    assert e.value.status == -10
    s.extend([ids], [])
    with pytest.raises(b200p.B200PError) as e:
        s.extend([ids[:5]], [0])                               # 65 tokens in a cache of 64
    assert e.value.status == -4
    with pytest.raises(b200p.B200PError) as e:
        s.extend([ids[:2]], [2])
    assert e.value.status == -10
    assert s.kv_len == 60
    check(s.extend([ids[:4]], range(4))[0], reference("odd", np.concatenate([ids, ids[:4]]))[60:], "bf16")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_program(tmp_path, torch_cuda, dtype):
    name, cfg = "odd", CONFIGS["odd"]
    lr.write_model(str(tmp_path / "m"), cfg, weights(name))
    out = tmp_path / "out"
    out.mkdir()
    a, b = tokens(cfg, 50, 12), tokens(cfg, 9, 13)
    steps = [("a", a[:30], [0, 29], []), ("a", a[30:32], [], []), ("a", a[32:], [0, 5, 17], ["a"]), ("b", b[:1], [0], []), ("b", b[1:], [7], ["b"])]
    lines = [json.dumps({"step": k, "entries": [{"id": i, "tokens": [int(x) for x in t], "want": w}], "end": e}) for k, (i, t, w, e) in enumerate(steps)]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(out),
                        "--max-tokens", "64"], input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert r.stdout.split("\n")[:-1] == ["done %d" % k for k in range(len(steps))]
    ra, rb = reference(name, a), reference(name, b)
    for k, rows in ((0, ra[[0, 29]]), (2, ra[[32, 37, 49]]), (3, rb[[0]]), (4, rb[[8]])):
        got = np.fromfile(str(out / ("%d.f32" % k)), "<f4").reshape(rows.shape)
        check(got, rows, {"float32": "f32", "bfloat16": "bf16"}[dtype], k)
    assert not (out / "1.f32").exists()


def test_trace_and_generate_programs_on_the_llama_format(tmp_path, torch_cuda):
    model = os.path.join(ROOT, "tests", "golden", "tiny_llama")
    run_ = lambda prog, *args, **kw: subprocess.run([os.path.join(ROOT, "bin", prog), "--model", model, *args], capture_output=True, text=True,
                                                    timeout=300, **kw)
    assert run_("trace_run", "--dtype", "float32", "--out", str(tmp_path), input="").returncode == 3
    prompt = [int(x) for x in open(os.path.join(model, "prompt_ids.txt")).read().split()]
    want = [int(x) for x in open(os.path.join(model, "ref_tokens.txt")).read().split()][len(prompt):]     # prompt + continuation
    r = run_("generate", "--max-new", "4", "--prompt", " ".join(map(str, prompt)))
    assert r.returncode == 0, r.stderr
    got = [int(x) for x in r.stdout.split()]
    assert got == want[:4]
    # a portion on top of a cache: the Llama decoder goes token by token
    line = lambda k, t, w: json.dumps({"step": k, "entries": [{"id": "x", "tokens": t, "want": w}], "end": []})
    r = run_("trace_run", "--out", str(tmp_path), input=line(0, prompt[:-2], []) + "\n" + line(1, prompt[-2:], [1]) + "\n")
    assert r.returncode == 0, r.stderr
    assert int(np.argmax(np.fromfile(str(tmp_path / "1.f32"), "<f4"))) == want[0]
