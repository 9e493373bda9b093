"""Plain float64 statement of the decoder with latent attention and output norms (architecture "Maposun"), one
function per mechanism.  Slow on purpose: whole sequences, one head at a time, no cache and no absorbed products.
For tests and CPU timings only; shares no code with the library.

    x       residual stream, [tokens, width]
    config  the parsed config.json; weights: dict name -> array as stored in model.safetensors
"""
import numpy as np


def rms_norm(x, w, eps):
    """Over the last axis: x by the root of (mean square + eps), times w."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def rotation_angles(positions, dims, base):
    """[positions, dims / 2]: p * base^(-2i / dims)."""
    i = np.arange(dims // 2)
    return np.asarray(positions, np.float64)[:, None] * np.power(float(base), -2.0 * i / dims)[None, :]


def rotate_interleaved(v, angles):
    """Pairs (2i, 2i + 1) of the last axis of v [tokens, ..., dims]."""
    a = angles.reshape((angles.shape[0],) + (1,) * (v.ndim - 2) + (angles.shape[1],))
    out = np.empty_like(v)
    x, y = v[..., 0::2], v[..., 1::2]
    out[..., 0::2] = x * np.cos(a) - y * np.sin(a)
    out[..., 1::2] = y * np.cos(a) + x * np.sin(a)
    return out


def rotate_halves(v, angles):
    """Pairs (i, i + dims / 2) of the last axis of v [tokens, ..., dims]."""
    a = angles.reshape((angles.shape[0],) + (1,) * (v.ndim - 2) + (angles.shape[1],))
    h = v.shape[-1] // 2
    x, y = v[..., :h], v[..., h:]
    return np.concatenate([x * np.cos(a) - y * np.sin(a), y * np.cos(a) + x * np.sin(a)], axis=-1)


def softmax_rows(scores, visible, sink=None):
    """Softmax of scores [q, k] over the visible keys; a sink is one more term of the denominator."""
    s = np.where(visible, scores, -np.inf)
    m = s.max(axis=-1, keepdims=True)
    if sink is not None:
        m = np.maximum(m, sink)
    e = np.exp(s - m)
    d = e.sum(axis=-1, keepdims=True)
    if sink is not None:
        d = d + np.exp(sink - m)
    return e / d


# what each mixer type of this architecture means
MIXERS = {"latent_attention": dict(rotate=rotate_interleaved, sink=False),
          "latent_attention_2": dict(rotate=rotate_halves, sink=True)}


def latent_attention(h, positions, mixer, kind, weights, prefix, eps):
    """Causal latent attention of h [tokens, width]; prefix is '<layer>.mix.'."""
    W = lambda n: np.asarray(weights[prefix + n], np.float64)
    how = MIXERS[kind]
    H, dim, rot, vdim, rank = mixer["heads"], mixer["dim"], mixer["rot_dim"], mixer["vdim"], mixer["kv_rank"]
    T = h.shape[0]
    turning = mixer["rot"]["dims"]
    ang = rotation_angles(positions, turning, mixer["rot"]["base"])
    rotate = lambda v: np.concatenate([how["rotate"](v[..., :turning], ang), v[..., turning:]], axis=-1)
    q = (rms_norm(h @ W("dq").T, W("dq.norm"), eps) @ W("uq").T).reshape(T, H, dim + rot)
    q_plain, q_rot = q[..., :dim], rotate(q[..., dim:])
    down = h @ W("dkv").T
    latent = rms_norm(down[:, :rank], W("dkv.norm"), eps)
    k_rot = rotate(down[:, rank:])                       # one for all heads
    k_plain = (latent @ W("uk").T).reshape(T, H, dim)
    v = (latent @ W("uv").T).reshape(T, H, vdim)
    visible = np.asarray(positions)[None, :] <= np.asarray(positions)[:, None]
    out = np.empty((T, H, vdim))
    for hd in range(H):
        s = (q_plain[:, hd] @ k_plain[:, hd].T + q_rot[:, hd] @ k_rot.T) * mixer["scale"]
        p = softmax_rows(s, visible, float(W("sink")[hd]) if how["sink"] else None)
        out[:, hd] = p @ v[:, hd]
    return (out.reshape(T, H * vdim) * sigmoid(h @ W("g").T)) @ W("o").T


def feed_forward(h, weights, prefix):
    W = lambda n: np.asarray(weights[prefix + n], np.float64)
    return (gelu_tanh(h @ W("gate").T) * (h @ W("up").T)) @ W("down").T


def forward(config, weights, tokens, layers_out=None):
    """Logits [tokens, vocab] of one sequence; layers_out, a list, receives x after every layer."""
    eps = config["norm"]["eps"]
    f64 = lambda n: np.asarray(weights[n], np.float64)
    x = f64("embed")[np.asarray(tokens)]
    pos = np.arange(len(tokens))
    for i, layer in enumerate(config["layers"]):
        p = "l%d." % layer.get("weights_of", i)
        x = x + rms_norm(latent_attention(x, pos, layer["mixer"], layer["type"], weights, p + "mix.", eps), f64(p + "norm1"), eps)
        if layer.get("mlp") is not None:
            x = x + rms_norm(feed_forward(x, weights, p + "mlp."), f64(p + "norm2"), eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return rms_norm(x, f64("final.norm"), eps) @ f64("head").T


def read_safetensors(path):
    """name -> array; bfloat16 tensors come back as float32."""
    import json
    raw = open(path, "rb").read()
    n = int.from_bytes(raw[:8], "little")
    out = {}
    for name, t in json.loads(raw[8:8 + n]).items():
        if name == "__metadata__":
            continue
        a, b = t["data_offsets"]
        buf = raw[8 + n + a:8 + n + b]
        if t["dtype"] == "BF16":
            arr = (np.frombuffer(buf, np.uint16).astype(np.uint32) << 16).view(np.float32)
        else:
            arr = np.frombuffer(buf, {"F32": np.float32, "I32": np.int32}[t["dtype"]])
        out[name] = arr.reshape(t["shape"])
    return out


def bf16_bits(a):
    """Round-to-nearest-even bfloat16 bits of a float array."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return ((u + 0x7fff + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def write_model(path, config, weights):
    """config.json and model.safetensors (bfloat16) under the folder `path`."""
    import json
    import os
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(config, f)
    head, blobs, at = {}, [], 0
    for name, a in weights.items():
        b = bf16_bits(a).tobytes()
        head[name] = {"dtype": "BF16", "shape": list(np.shape(a)), "data_offsets": [at, at + len(b)]}
        blobs.append(b)
        at += len(b)
    text = json.dumps(head).encode()
    with open(os.path.join(path, "model.safetensors"), "wb") as f:
        f.write(len(text).to_bytes(8, "little") + text + b"".join(blobs))


def tensor_shapes(config):
    """name -> shape of every tensor a config asks for."""
    D, V = config["width"], config["vocab"]
    out = {"embed": (V, D)}
    for i, L in enumerate(config["layers"]):
        if L.get("weights_of") is not None:
            continue
        m, p = L["mixer"], "l%d." % i
        H = m["heads"]
        out[p + "norm1"] = (D,)
        if L.get("mlp") is not None:
            out[p + "norm2"] = (D,)
        out.update({p + "mix.dq": (m["q_rank"], D), p + "mix.dq.norm": (m["q_rank"],),
                    p + "mix.uq": (H * (m["dim"] + m["rot_dim"]), m["q_rank"]),
                    p + "mix.dkv": (m["kv_rank"] + m["rot_dim"], D), p + "mix.dkv.norm": (m["kv_rank"],),
                    p + "mix.uk": (H * m["dim"], m["kv_rank"]), p + "mix.uv": (H * m["vdim"], m["kv_rank"])})
        if MIXERS[L["type"]]["sink"]:
            out[p + "mix.sink"] = (H,)
        out.update({p + "mix.g": (H * m["vdim"], D), p + "mix.o": (D, H * m["vdim"])})
        if L.get("mlp") is not None:
            ff = L["mlp"]["ff"]
            out.update({p + "mlp.gate": (ff, D), p + "mlp.up": (ff, D), p + "mlp.down": (D, ff)})
    out["final.norm"] = (D,)
    out["head"] = (V, D)
    return out
