"""Plain, slow restatement of the Talazen layers, one function per mechanism, in numpy.

Test infrastructure: it shares no code with the library.  Every function takes whole
sequences (rows are tokens) and computes in the floating-point type of its inputs, float64
unless a test asks for less.  A model is a configuration dictionary (the contents of a
config.json) and a dictionary of named [out, in] arrays.
"""
import math

import numpy as np


def rms_norm(x, weight, eps):
    """Every row divided by sqrt(mean of squares + eps), times the weight."""
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + x.dtype.type(eps)) * weight


def rotate_pairs(x, positions, base):
    """Rotary positions, interleaved layout: elements (2i, 2i+1) of the last axis form a pair
    turned by position * base^(-2i/n).  x is [tokens, ..., n]."""
    n = x.shape[-1]
    freq = np.array([base ** (-2.0 * i / n) for i in range(n // 2)])
    angle = np.asarray(positions, dtype=np.float64)[:, None] * freq[None, :]
    shape = (len(positions),) + (1,) * (x.ndim - 2) + (n // 2,)
    cos, sin = np.cos(angle).reshape(shape).astype(x.dtype), np.sin(angle).reshape(shape).astype(x.dtype)
    out = np.empty_like(x)
    u, v = x[..., 0::2], x[..., 1::2]
    out[..., 0::2] = u * cos - v * sin
    out[..., 1::2] = v * cos + u * sin
    return out


def window_mask(n, window):
    """[query, key]: token i sees itself and the window - 1 tokens before it (None: all before)."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    seen = j <= i
    if window is not None:
        seen &= (i - j) < window
    return seen


def softmax_rows(s, seen):
    s = np.where(seen, s, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def latent_keys(h, mixer, tensors, prefix, eps):
    """What a layer with a down-projection of its own caches: the normed latent [tokens, rank]
    and the rotated key part [tokens, rot_dim] that all heads share."""
    rank = mixer["kv_rank"]
    down = h @ tensors[prefix + "dkv"].T
    latent = rms_norm(down[:, :rank], tensors[prefix + "dkv.norm"], eps)
    return latent, rotate_pairs(down[:, rank:], np.arange(len(h)), mixer["rot"]["base"])


def latent_attention(h, latent, key_rot, mixer, tensors, prefix):
    """Attention over expanded keys and values, head by head."""
    heads, dim, rot, vdim = mixer["heads"], mixer["dim"], mixer["rot_dim"], mixer["vdim"]
    n = len(h)
    q = (h @ tensors[prefix + "q"].T).reshape(n, heads, dim + rot)
    q_rot = rotate_pairs(q[:, :, dim:], np.arange(n), mixer["rot"]["base"])
    keys = (latent @ tensors[prefix + "uk"].T).reshape(n, heads, dim)
    values = (latent @ tensors[prefix + "uv"].T).reshape(n, heads, vdim)
    mask = mixer.get("mask")
    seen = window_mask(n, mask["size"] if mask else None)
    out = np.empty((n, heads, vdim), dtype=h.dtype)
    for k in range(heads):
        s = (q[:, k, :dim] @ keys[:, k].T + q_rot[:, k] @ key_rot.T) * h.dtype.type(mixer["scale"])
        out[:, k] = softmax_rows(s, seen) @ values[:, k]
    return out.reshape(n, heads * vdim) @ tensors[prefix + "o"].T


def gated_unit(h, gate, up, down, limit):
    """down(g * sigmoid(1.702 g) * (u + 1)), g bounded above, u on both sides."""
    g = np.minimum(h @ gate.T, limit)
    u = np.clip(h @ up.T, -limit, limit)
    return (g / (1 + np.exp(-1.702 * g)) * (u + 1)) @ down.T


def route(h, router, top):
    """Chosen experts [tokens, top] and the softmax over their logits only."""
    z = h @ router.T
    chosen = np.argsort(-z, axis=-1, kind="stable")[:, :top]
    zc = np.take_along_axis(z, chosen, axis=-1)
    e = np.exp(zc - zc.max(axis=-1, keepdims=True))
    return chosen, e / e.sum(axis=-1, keepdims=True)


def route_margin(h, router, top):
    """How far the last chosen expert's logit lies above the first one left out, per token, relative
    to the spread of the logits: a small margin may fall either way under rounding."""
    z = np.sort(h @ router.T, axis=-1)[:, ::-1]
    if top == z.shape[1]:
        return np.full(len(h), np.inf)
    return (z[:, top - 1] - z[:, top]) / z.std()


def mixture(h, mlp, tensors, prefix):
    limit = mlp["expert"]["limit"]
    chosen, weight = route(h, tensors[prefix + "router"], mlp["router"]["top"])
    out = np.zeros_like(h)
    for t in range(len(h)):
        for e, w in zip(chosen[t], weight[t]):
            p = f"{prefix}e{e}."
            out[t] += w * gated_unit(h[t:t + 1], tensors[p + "gate"], tensors[p + "up"], tensors[p + "down"], limit)[0]
    return out


def feed_forward(h, mlp, tensors, prefix):
    if mlp["kind"] == "dense":
        return gated_unit(h, tensors[prefix + "gate"], tensors[prefix + "up"], tensors[prefix + "down"], mlp["limit"])
    return mixture(h, mlp, tensors, prefix)


def forward(config, tensors, tokens, dtype=np.float64, residuals=None, margins=None):
    """Logits [tokens, vocab] of one sequence; residuals (a list) receives the stream after
    every layer, margins (a list) route_margin of every mixture."""
    t = {k: np.asarray(v).astype(dtype) for k, v in tensors.items()}
    eps = config["norm"]["eps"]
    x = t["embed"][np.asarray(tokens)]
    caches = {}
    for i, layer in enumerate(config["layers"]):
        assert layer["type"] == "latent_attention"
        p, mixer = f"l{i}.", layer["mixer"]
        h = rms_norm(x, t[p + "norm1"], eps)
        source = mixer.get("kv_from")
        if source is None:
            caches[i] = latent_keys(h, mixer, t, p + "mix.", eps)
            source = i
        y = latent_attention(h, *caches[source], mixer, t, p + "mix.")
        if margins is not None and layer["mlp"] is not None and layer["mlp"]["kind"] != "dense":
            margins.append(route_margin(h, t[p + "mlp.router"], layer["mlp"]["router"]["top"]))
        if layer["mlp"] is not None:
            y = y + feed_forward(h, layer["mlp"], t, p + "mlp.")
        x = x + y
        if residuals is not None:
            residuals.append(x)
    return rms_norm(x, t["final.norm"], eps) @ t["embed"].T


def tensor_shapes(config):
    """Names and shapes of all tensors of a configuration."""
    W, out = config["width"], {"embed": (config["vocab"], config["width"])}
    for i, layer in enumerate(config["layers"]):
        m, f, p = layer["mixer"], layer["mlp"], f"l{i}."
        out[p + "norm1"] = (W,)
        out[p + "mix.q"] = (m["heads"] * (m["dim"] + m["rot_dim"]), W)
        if m.get("kv_from") is None:
            out[p + "mix.dkv"] = (m["kv_rank"] + m["rot_dim"], W)
            out[p + "mix.dkv.norm"] = (m["kv_rank"],)
        out[p + "mix.uk"] = (m["heads"] * m["dim"], m["kv_rank"])
        out[p + "mix.uv"] = (m["heads"] * m["vdim"], m["kv_rank"])
        out[p + "mix.o"] = (W, m["heads"] * m["vdim"])
        if f is None:
            continue
        units = [("mlp.", f["ff"])] if f["kind"] == "dense" else \
            [(f"mlp.e{e}.", f["expert"]["ff"]) for e in range(f["router"]["experts"])]
        if f["kind"] != "dense":
            out[p + "mlp.router"] = (f["router"]["experts"], W)
        for q, ff in units:
            out[p + q + "gate"], out[p + q + "up"], out[p + q + "down"] = (ff, W), (ff, W), (W, ff)
    out["final.norm"] = (W,)
    return out
