"""Plain float64 statement of the decoder that mixes gated-delta-rule layers with windowed and chunked attention
(architecture "Vofusun"), one function per mechanism.  Slow on purpose: whole sequences, token by token where the
mechanism is a recurrence, no cache and no blocked forms.  For tests and CPU timings only; shares no code with the library.

    x       residual stream, [tokens, width]
    config  the parsed config.json; weights: dict name -> array as stored in model.safetensors
"""
import numpy as np


def rms(x, eps):
    """Root mean square over the last axis, eps inside the root."""
    return np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def silu(z):
    return z / (1.0 + np.exp(-z))


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def softplus(z):
    return np.logaddexp(0.0, z)


def unit(x):
    """x by its length over the last axis."""
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


# ---- attention ------------------------------------------------------------------------------------------
def frequencies(rot):
    """[dims / 2] angles per position; long wavelengths are slowed down by `factor`, with a ramp in between."""
    dims = rot["dims"]
    f = np.power(float(rot["base"]), -2.0 * np.arange(dims // 2) / dims)
    sc = rot.get("scaling")
    if not sc:
        return f
    turns = sc["original"] * f / (2.0 * np.pi)                 # full turns within the original context
    mix = np.clip((turns - sc["low"]) / (sc["high"] - sc["low"]), 0.0, 1.0)
    return (1.0 - mix) * f / sc["factor"] + mix * f


def rotate_pairs(v, positions, rot):
    """Pairs (2i, 2i + 1) of the first rot.dims columns of v [tokens, heads, dim]."""
    n = rot["dims"]
    a = np.asarray(positions, np.float64)[:, None, None] * frequencies(rot)[None, None, :]
    out = v.copy()
    x, y = v[..., 0:n:2], v[..., 1:n:2]
    out[..., 0:n:2] = x * np.cos(a) - y * np.sin(a)
    out[..., 1:n:2] = y * np.cos(a) + x * np.sin(a)
    return out


def window_mask(positions, size):
    """[query, key]: the token itself and the size - 1 before it."""
    d = positions[:, None] - positions[None, :]
    return (d >= 0) & (d < size)


def chunk_mask(positions, size):
    """[query, key]: earlier tokens of the same chunk, and the token itself."""
    return (positions[:, None] >= positions[None, :]) & (positions[:, None] // size == positions[None, :] // size)


def softmax_plus_one(scores, visible):
    """exp(s_j) / (1 + sum exp(s)) over the visible keys."""
    s = np.where(visible, scores, -np.inf)
    m = np.maximum(s.max(axis=-1, keepdims=True), 0.0)
    e = np.exp(s - m)
    return e / (np.exp(-m) + e.sum(axis=-1, keepdims=True))


def attend(q, k, v, visible, scale):
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H * e]; query head h reads key/value head h // (H / G)."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = np.empty((T, H, v.shape[2]))
    for h in range(H):
        out[:, h] = softmax_plus_one(q[:, h] @ k[:, h // per].T * scale, visible) @ v[:, h // per]
    return out.reshape(T, -1)


def window_attention(h, mixer, W, eps, positions):
    """No positions in the scores, a sliding window, separate values."""
    T, H, G = len(h), mixer["heads"], mixer["kv_heads"]
    q = (h @ W("q").T).reshape(T, H, mixer["dim"])
    k = (h @ W("k").T).reshape(T, G, mixer["dim"])
    v = (h @ W("v").T).reshape(T, G, mixer["vdim"])
    return attend(q, k, v, window_mask(positions, mixer["mask"]["size"]), mixer["scale"]) @ W("o").T


def chunk_attention(h, mixer, W, eps, positions):
    """Rotary positions, then q and k by their root mean square; values are the keys before both; chunks; gated output."""
    T, H, G, d = len(h), mixer["heads"], mixer["kv_heads"], mixer["dim"]
    q = (h @ W("q").T).reshape(T, H, d)
    v = (h @ W("k").T).reshape(T, G, d)
    q, k = rotate_pairs(q, positions, mixer["rot"]), rotate_pairs(v, positions, mixer["rot"])
    q, k = q / rms(q, eps), k / rms(k, eps)
    o = attend(q, k, v, chunk_mask(positions, mixer["mask"]["size"]), mixer["scale"])
    return (o * sigmoid(h @ W("g").T)) @ W("o").T


# ---- gated delta rule -----------------------------------------------------------------------------------
def causal_conv(x, w):
    """x [T, channels], w [channels, taps], the last tap is the current token's; silu of the sum."""
    T, taps = len(x), w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, x.shape[1])), x])
    return silu(sum(padded[j:j + T] * w[:, j] for j in range(taps)))


def delta_steps(q, k, v, g, beta, state=None):
    """One head: q, k [T, d], v [T, e], g, beta [T] -> (o [T, e], state [d, e])."""
    S = np.zeros((q.shape[1], v.shape[1])) if state is None else state.copy()
    out = np.empty_like(v)
    for t in range(len(q)):
        S = g[t] * S
        S = S + np.outer(k[t], beta[t] * (v[t] - S.T @ k[t]))
        out[t] = S.T @ q[t]
    return out, S


def delta_mixer(h, mixer, W, eps, positions):
    T, H, G, d, e = len(h), mixer["heads"], mixer["kv_heads"], mixer["dim"], mixer["vdim"]
    q = unit(causal_conv(h @ W("q").T, W("q.conv")).reshape(T, G, d)) * d ** -0.5
    k = unit(causal_conv(h @ W("k").T, W("k.conv")).reshape(T, G, d))
    v = causal_conv(h @ W("v").T, W("v.conv")).reshape(T, H, e)
    beta = sigmoid(h @ W("b").T)
    g = np.exp(-np.exp(W("A_log")) * softplus(h @ W("a").T + W("dt_bias")))
    o = np.empty((T, H, e))
    for hd in range(H):
        o[:, hd], _ = delta_steps(q[:, hd // (H // G)], k[:, hd // (H // G)], v[:, hd], g[:, hd], beta[:, hd])
    o = o / rms(o, eps) * W("norm") * silu(h @ W("g").T).reshape(T, H, e)
    return o.reshape(T, H * e) @ W("o").T


# ---- the model ------------------------------------------------------------------------------------------
MIXERS = {"attention": window_attention, "attention_2": chunk_attention, "delta": delta_mixer}


def feed_forward(h, W):
    return (silu(h @ W("gate").T) * (h @ W("up").T)) @ W("down").T


def passes(config):
    """(layer index, whether the embeddings are added ahead of it) in the order the layers run."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    out = [(i, False) for i in range(a)]
    for t in range(loop["times"]):
        out += [(i, t > 0 and i == a) for i in range(a, b)]
    return out + [(i, False) for i in range(b, n)]


def forward(config, weights, tokens, layers_out=None):
    """Logits [tokens, vocab] of one sequence; layers_out, a list, receives x after every layer run."""
    eps = config["norm"]["eps"]
    f64 = lambda n: np.asarray(weights[n], np.float64)
    x0 = f64("embed")[np.asarray(tokens)] * config["embedding"]["scale"]
    x = x0
    pos = np.arange(len(tokens))
    for i, again in passes(config):
        layer, p = config["layers"][i], "l%d." % i
        if again:
            x = x + x0
        x = x + MIXERS[layer["type"]](x / rms(x, eps) * f64(p + "norm1"), layer["mixer"], lambda n: f64(p + "mix." + n), eps, pos)
        if layer.get("mlp") is not None:
            x = x + feed_forward(x / rms(x, eps) * f64(p + "norm2"), lambda n: f64(p + "mlp." + n))
        if layers_out is not None:
            layers_out.append(x.copy())
    return x / rms(x, eps) * f64("final.norm") @ f64("embed").T


def tensor_shapes(config):
    """name -> shape of every tensor a config asks for."""
    D = config["width"]
    out = {"embed": (config["vocab"], D)}
    for i, L in enumerate(config["layers"]):
        m, p = L["mixer"], "l%d." % i
        H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        mp = p + "mix."
        out[p + "norm1"] = (D,)
        if L["type"] == "delta":
            n = m["conv"]
            out.update({mp + "q": (G * d, D), mp + "q.conv": (G * d, n), mp + "k": (G * d, D), mp + "k.conv": (G * d, n),
                        mp + "v": (H * e, D), mp + "v.conv": (H * e, n), mp + "b": (H, D), mp + "a": (H, D), mp + "A_log": (H,),
                        mp + "dt_bias": (H,), mp + "norm": (e,), mp + "g": (H * e, D)})
        else:
            out.update({mp + "q": (H * d, D), mp + "k": (G * d, D)})
            out[mp + ("g" if L["type"] == "attention_2" else "v")] = (H * e if L["type"] == "attention_2" else G * e, D)
        out[mp + "o"] = (D, H * e)
        if L.get("mlp") is not None:
            ff = L["mlp"]["ff"]
            out.update({p + "norm2": (D,), p + "mlp.gate": (ff, D), p + "mlp.up": (ff, D), p + "mlp.down": (D, ff)})
    out["final.norm"] = (D,)
    return out
