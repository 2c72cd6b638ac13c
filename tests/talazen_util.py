"""Small random Talazen models for the tests: configurations, weights, comparison."""
import json

import numpy as np

import plain_talazen as plain


def attention(heads=3, dim=24, rot=16, vdim=20, rank=40, window=None, base=1000.0, sharp=2.0, kv_from=None):
    """sharp multiplies the usual 1/sqrt(size) scale, so that single keys stand out."""
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank,
         "rot": {"base": base, "dims": rot}, "scale": sharp / (dim + rot) ** 0.5}
    if window is not None:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def gated(ff=56, limit=1.5):
    return {"kind": "dense", "ff": ff, "limit": limit}


def experts(n=5, top=2, ff=24, limit=1.5):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": n, "top": top}}


def config(layers, width=72, vocab=136, eps=1e-5):
    """layers: [(mixer, feed-forward or None)]"""
    return {"architecture": "Talazen", "width": width, "vocab": vocab, "norm": {"eps": eps},
            "layers": [{"type": "latent_attention", "mixer": m, "mlp": f} for m, f in layers]}


def to_bf16(a):
    """float32 -> bfloat16 patterns, nearest even."""
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def from_bf16(p):
    return (p.astype(np.uint32) << 16).view(np.float32)


def weights(cfg, seed):
    """{name: bf16 patterns}; mixed magnitudes so that gates reach their limits and experts differ."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in plain.tensor_shapes(cfg).items():
        if len(shape) == 1:
            a = 1.0 + 0.3 * rng.standard_normal(shape)
        else:
            a = rng.standard_normal(shape) / shape[1] ** 0.5
            if name == "embed":
                a = rng.standard_normal(shape)
            elif name.endswith((".gate", ".up")):
                a *= 2.0
            elif name.endswith(".router"):
                a *= 3.0
        out[name] = to_bf16(a.astype(np.float32))
    return out


def values(w):
    return {k: from_bf16(v) for k, v in w.items()}


def want_logits(cfg, w, tokens):
    return plain.forward(cfg, values(w), tokens)


def clear_of_close_calls(cfg, w, tokens, margin=0.03):
    """Per token: no router had to make a close call, which bfloat16 rounding may turn, for it or for
    any token before it (what a token sees)."""
    margins = []
    plain.forward(cfg, values(w), tokens, margins=margins)
    worst = np.min(margins, axis=0) if margins else np.full(len(tokens), np.inf)
    return np.minimum.accumulate(worst) > margin


def error(got, want):
    """Largest row error: rms over the vocabulary of the difference (mean taken off), relative to
    the rms of the wanted logits."""
    got, want = np.atleast_2d(got).astype(np.float64), np.atleast_2d(want)
    d = got - want
    d -= d.mean(axis=1, keepdims=True)
    return float(np.sqrt((d * d).mean(axis=1)).max() / want.std())


TOLERANCE = {"float32": 2e-5, "bfloat16": 5e-2}


def session(cfg, w, dtype, max_len=256):
    from buddy_mlir_b200 import talazen
    from buddy_mlir_b200.session import ModelSession
    s = ModelSession(talazen.parse(cfg, dtype, max_len))
    s.load_named(w)
    return s


def batch(s, max_seqs=8, page=4, pages=512, context=512):
    from buddy_mlir_b200.session import BatchSession
    return BatchSession(s, max_seqs, page, pages, context)


def write_folder(folder, cfg, w):
    """config.json and model.safetensors."""
    with open(f"{folder}/config.json", "w") as f:
        json.dump(cfg, f)
    header, blobs, at = {}, [], 0
    for name, a in w.items():
        header[name] = {"dtype": "BF16", "shape": list(a.shape), "data_offsets": [at, at + a.nbytes]}
        blobs.append(a.tobytes())
        at += a.nbytes
    head = json.dumps(header).encode()
    with open(f"{folder}/model.safetensors", "wb") as f:
        f.write(len(head).to_bytes(8, "little") + head + b"".join(blobs))


def mixed_model(seed=5):
    """Every branch at once: dense, expert and absent feed-forwards, windows of different size, a
    layer without a window, shared caches under other windows and head shapes."""
    cfg = config([
        (attention(window=11), gated()),
        (attention(heads=5, dim=16, rot=8, vdim=12, rank=24, window=19, base=500.0), experts()),
        (attention(heads=2, dim=40, rot=8, vdim=36, rank=24, window=7, base=500.0, kv_from=1), None),
        (attention(heads=4, dim=8, rot=16, vdim=8, rank=40, window=29, kv_from=0), experts(n=7, top=3, ff=40)),
    ])
    return cfg, weights(cfg, seed)
