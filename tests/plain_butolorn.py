"""Plain, slow restatement of the Butolorn layers, one function per mechanism, in numpy.

Test infrastructure: it shares no code with the library.  Every function takes whole
sequences (rows are tokens) and computes in the floating-point type of its inputs, float64
unless a test asks for less.  A model is a configuration dictionary (the contents of a
config.json) and a dictionary of named [out, in] arrays.
"""
import math

import numpy as np


def unit_rms(x, eps):
    """Last axis divided by sqrt(mean of squares + eps)."""
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + x.dtype.type(eps))


def rms_norm(x, weight, eps):
    return unit_rms(x, eps) * weight


def sigmoid(z):
    return 1 / (1 + np.exp(-z))


def log_sigmoid(z):
    return np.minimum(z, 0) - np.log1p(np.exp(-np.abs(z)))


def gelu_tanh(z):
    return 0.5 * z * (1 + np.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def squared_relu(z):
    return np.maximum(z, 0) ** 2


def angles(positions, rot, dtype):
    """cos and sin [tokens, 1, dims / 2] of position * base^(-2i/dims)."""
    freq = np.array([rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)])
    a = np.asarray(positions, dtype=np.float64)[:, None, None] * freq
    return np.cos(a).astype(dtype), np.sin(a).astype(dtype)


def rotate_halves(x, positions, rot):
    """x [tokens, heads, dim]: of the first `dims` elements, i and i + dims/2 are a pair."""
    n = rot["dims"] // 2
    cos, sin = angles(positions, rot, x.dtype)
    out = x.copy()
    u, v = x[..., :n], x[..., n:2 * n]
    out[..., :n] = u * cos - v * sin
    out[..., n:2 * n] = v * cos + u * sin
    return out


def rotate_interleaved(x, positions, rot):
    """x [tokens, heads, dim]: of the first `dims` elements, 2i and 2i + 1 are a pair."""
    n = 2 * (rot["dims"] // 2)
    cos, sin = angles(positions, rot, x.dtype)
    out = x.copy()
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    out[..., 0:n:2] = u * cos - v * sin
    out[..., 1:n:2] = v * cos + u * sin
    return out


def softmax_plain(s):
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def softmax_sink(s):
    """One more score of 0 in the denominator, without a value."""
    m = np.maximum(s.max(axis=-1, keepdims=True), 0)
    e = np.exp(s - m)
    return e / (np.exp(-m) + e.sum(axis=-1, keepdims=True))


def causal(n):
    """[query, key]: what token i sees."""
    return np.arange(n)[None, :] <= np.arange(n)[:, None]


def attend(q, k, v, scale, softmax):
    """Causal attention, q [tokens, H, dim] against k, v [tokens, G, ...]; query head h reads
    key head h // (H / G).  Returns [tokens, H * vdim]."""
    n, H, _ = q.shape
    G = k.shape[1]
    seen = causal(n)
    out = np.empty((n, H, v.shape[2]), dtype=q.dtype)
    for h in range(H):
        s = q[:, h] @ k[:, h // (H // G)].T * q.dtype.type(scale)
        out[:, h] = softmax(np.where(seen, s, -np.inf)) @ v[:, h // (H // G)]
    return out.reshape(n, -1)


def heads_of(x, n):
    return x.reshape(len(x), n, -1)


def attention(h, c, t, p):
    """Biased projections, split-half rotation, ordinary softmax."""
    pos = np.arange(len(h))
    q, k, v = (h @ t[p + name].T + t[p + name + ".b"] for name in "qkv")
    q = rotate_halves(heads_of(q, c["heads"]), pos, c["rot"])
    k = rotate_halves(heads_of(k, c["kv_heads"]), pos, c["rot"])
    return attend(q, k, heads_of(v, c["kv_heads"]), c["scale"], softmax_plain) @ t[p + "o"].T


def whole_norm(x, weight, eps):
    """Query / key norm over all rows of the projection at once."""
    return rms_norm(x, weight, eps)


def output_gate(o, z):
    return o * sigmoid(z)


def sink_attention(h, c, t, p, eps):
    """Query and key normed over the whole projection, interleaved rotation, a softmax with a sink
    of score 0, an output gate."""
    pos = np.arange(len(h))
    q = whole_norm(h @ t[p + "q"].T, t[p + "q.norm"], eps)
    k = whole_norm(h @ t[p + "k"].T, t[p + "k.norm"], eps)
    q = rotate_interleaved(heads_of(q, c["heads"]), pos, c["rot"])
    k = rotate_interleaved(heads_of(k, c["kv_heads"]), pos, c["rot"])
    o = attend(q, k, heads_of(h @ t[p + "v"].T, c["kv_heads"]), c["scale"], softmax_sink)
    return output_gate(o, h @ t[p + "g"].T) @ t[p + "o"].T


def memory_gates(h, c, t, p):
    """Log input and log forget gates [tokens, heads], soft-capped."""
    cap = h.dtype.type(c["gate_cap"])
    i = cap * np.tanh((h @ t[p + "i"].T + t[p + "i.b"]) / cap)
    f = log_sigmoid(cap * np.tanh((h @ t[p + "f"].T + t[p + "f.b"]) / cap))
    return i, f


def memory_scan(q, k, v, i, f):
    """The stabilised matrix memory, token by token: q, k [tokens, heads, dim], v [tokens, heads,
    vdim], i, f [tokens, heads] -> [tokens, heads, vdim].  Everything starts at zero, the running
    maximum too."""
    n, H, dim = q.shape
    S, z = np.zeros((H, dim, v.shape[2]), dtype=q.dtype), np.zeros((H, dim), dtype=q.dtype)
    m = np.zeros(H, dtype=q.dtype)
    out = np.empty((n, H, v.shape[2]), dtype=q.dtype)
    for t in range(n):
        new = np.maximum(f[t] + m, i[t])
        keep, add = np.exp(f[t] + m - new), np.exp(i[t] - new)
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        z = keep[:, None] * z + add[:, None] * k[t]
        m = new
        num = np.einsum("hdv,hd->hv", S, q[t])
        den = np.maximum(np.abs((z * q[t]).sum(axis=1)), np.exp(-m)) + q.dtype.type(1e-6)
        out[t] = num / den[:, None]
    return out


def matrix_memory(h, c, t, p, eps):
    q = heads_of(h @ t[p + "q"].T, c["heads"]) * h.dtype.type(c["dim"] ** -0.5)
    k, v = heads_of(h @ t[p + "k"].T, c["heads"]), heads_of(h @ t[p + "v"].T, c["heads"])
    o = unit_rms(memory_scan(q, k, v, *memory_gates(h, c, t, p)), eps).reshape(len(h), -1)
    return output_gate(o * t[p + "norm"], h @ t[p + "g"].T) @ t[p + "o"].T


def side_by_side(h, c, t, p, eps):
    left = sink_attention(h, c["left"], t, p + "left.", eps)
    right = matrix_memory(h, c["right"], t, p + "right.", eps)
    return h.dtype.type(c["left_scale"]) * left + h.dtype.type(c["right_scale"]) * right


def feed_forward(h, t, p):
    return squared_relu(h @ t[p + "up"].T) @ t[p + "down"].T


def token_side(x, e, t, p, eps):
    """What a layer's slice e of the per-token table adds to the stream."""
    y = (gelu_tanh(x @ t[p + "side.gate"].T) * e) @ t[p + "side.proj"].T
    return rms_norm(y, t[p + "side.norm"], eps)


def layer_order(config):
    """[(layer, the embedding output is added before it)] of one forward pass."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    order = [(i, False) for i in range(loop["start"])]
    for turn in range(loop["times"]):
        order += [(i, turn > 0 and i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return order + [(i, False) for i in range(loop["stop"], n)]


def forward(config, tensors, tokens, dtype=np.float64, residuals=None):
    """Logits [tokens, vocab] of one sequence; residuals (a list) receives the stream after every
    layer run."""
    t = {k: np.asarray(v).astype(dtype) for k, v in tensors.items()}
    eps, tokens = config["norm"]["eps"], np.asarray(tokens)
    first = t["embed"][tokens] * dtype(config["embedding"]["scale"])
    x = first
    for i, again in layer_order(config):
        c, p = config["layers"][i], f"l{i}."
        if again:
            x = x + first
        h = rms_norm(x, t[p + "norm1"], eps)
        if c["type"] == "attention":
            y = attention(h, c["mixer"], t, p + "mix.")
        else:
            assert c["type"] == "parallel"
            y = side_by_side(h, c["mixer"], t, p + "mix.", eps)
        x = x + rms_norm(y, t[p + "norm1b"], eps)
        if c["mlp"] is not None:
            y = feed_forward(rms_norm(x, t[p + "norm2"], eps), t, p + "mlp.")
            x = x + rms_norm(y, t[p + "norm2b"], eps)
        if config.get("token_side"):
            dim = config["token_side"]["dim"]
            x = x + token_side(x, t["side.embed"][tokens][:, i * dim:(i + 1) * dim], t, p, eps)
        if residuals is not None:
            residuals.append(x)
    return rms_norm(x, t["final.norm"], eps) @ t["embed"].T


def tensor_shapes(config):
    """Names and shapes of all tensors of a configuration."""
    W = config["width"]
    out = {"embed": (config["vocab"], W)}
    side = config["token_side"]["dim"] if config.get("token_side") else 0
    if side:
        out["side.embed"] = (config["vocab"], len(config["layers"]) * side)
    for i, layer in enumerate(config["layers"]):
        m, f, p = layer["mixer"], layer["mlp"], f"l{i}."
        names = ["norm1", "norm1b"] + (["norm2", "norm2b"] if f else [])
        out.update({p + name: (W,) for name in names})
        a, q = (m, p + "mix.") if layer["type"] == "attention" else (m["left"], p + "mix.left.")
        nq, nk, nv, no = a["heads"] * a["dim"], a["kv_heads"] * a["dim"], a["kv_heads"] * a["vdim"], a["heads"] * a["vdim"]
        out[q + "q"], out[q + "k"], out[q + "v"], out[q + "o"] = (nq, W), (nk, W), (nv, W), (W, no)
        if layer["type"] == "attention":
            out[q + "q.b"], out[q + "k.b"], out[q + "v.b"] = (nq,), (nk,), (nv,)
        else:
            out[q + "q.norm"], out[q + "k.norm"], out[q + "g"] = (nq,), (nk,), (no, W)
            r, q = m["right"], p + "mix.right."
            nq, nv = r["heads"] * r["dim"], r["heads"] * r["vdim"]
            out[q + "q"], out[q + "k"], out[q + "v"], out[q + "g"] = (nq, W), (nq, W), (nv, W), (nv, W)
            out[q + "o"], out[q + "norm"] = (W, nv), (nv,)
            for g in "if":
                out[q + g], out[q + g + ".b"] = (r["heads"], W), (r["heads"],)
        if f:
            out[p + "mlp.up"], out[p + "mlp.down"] = (f["ff"], W), (W, f["ff"])
        if side:
            out[p + "side.gate"], out[p + "side.proj"], out[p + "side.norm"] = (side, W), (W, side), (W,)
    out["final.norm"] = (W,)
    return out
