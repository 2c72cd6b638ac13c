"""Small random Butolorn models for the tests: configurations, weights, sessions."""
import numpy as np

import plain_butolorn as plain
from talazen_util import batch, error, to_bf16, values, write_folder  # noqa: F401

TOLERANCE = {"float32": 3e-5, "bfloat16": 4e-2}


def heads(heads=4, kv=2, dim=20, vdim=12, rot=16, base=1000.0, sharp=2.0):
    """sharp multiplies the usual 1/sqrt(size) scale, so that single keys stand out."""
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot},
            "scale": sharp / dim ** 0.5}


def attention(ff=56, **kw):
    return {"type": "attention", "mixer": heads(**kw), "mlp": feed(ff)}


def memory(heads=3, dim=10, vdim=14, cap=4.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def parallel(left=None, right=None, left_scale=1.3, right_scale=0.7, ff=56):
    return {"type": "parallel", "mixer": {"left": left or heads(), "right": right or memory(), "left_scale": left_scale,
                                          "right_scale": right_scale}, "mlp": feed(ff)}


def feed(ff):
    return None if ff is None else {"kind": "dense", "ff": ff}


def config(layers, width=72, vocab=136, eps=1e-5, scale=2.5, loop=None, side=12):
    """loop: (start, stop, times); side: size of the per-token layer input."""
    return {"architecture": "Butolorn", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "layers": layers, "loop": dict(zip(("start", "stop", "times"), loop)) if loop else None,
            "token_side": {"dim": side} if side else None}


def weights(cfg, seed):
    """{name: bf16 patterns}.  Forget gates that hold for hundreds of tokens and ones that do not,
    input gates on both sides of zero (the running maximum starts there)."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in plain.tensor_shapes(cfg).items():
        if name.endswith(".f.b"):
            a = rng.uniform(1.0, 6.0, shape)
        elif name.endswith(".i.b"):
            a = rng.uniform(-4.0, 2.0, shape)
        elif name.endswith(".b"):
            a = 0.7 * rng.standard_normal(shape)
        elif len(shape) == 1:
            a = 1.0 + 0.3 * rng.standard_normal(shape)
        else:
            a = rng.standard_normal(shape) / shape[1] ** 0.5
            if name in ("embed", "side.embed"):
                a = rng.standard_normal(shape)
            elif name.endswith((".i", ".f")):
                a *= 1.5
            elif name.endswith(".right.v"):
                a *= 0.004                   # a memory's output is normed: only where it is small does its scale count
        out[name] = to_bf16(a.astype(np.float32))
    return out


def want_logits(cfg, w, tokens):
    return plain.forward(cfg, values(w), tokens)


def session(cfg, w, dtype, max_len=256):
    from buddy_mlir_b200 import butolorn
    from buddy_mlir_b200.session import ModelSession
    s = ModelSession(butolorn.parse(cfg, dtype, max_len))
    s.load_named(w)
    return s


def mixed_model(seed=5):
    """Every branch at once: both kinds of layers in and around a loop, a layer without a
    feed-forward, head counts and sizes that differ everywhere."""
    cfg = config([
        parallel(heads(heads=6, kv=3, dim=10, rot=8, sharp=0.5), memory(heads=2, dim=18, vdim=34, cap=9.0), 2.5),
        attention(heads=6, kv=3, dim=24, vdim=18, rot=24, base=300.0, sharp=1.0, ff=None),
        parallel(heads(heads=5, kv=1, dim=14, vdim=22, rot=4), memory(heads=5, dim=7, vdim=9, cap=2.0), 0.9, 1.1, ff=None),
        attention(heads=4, kv=1, dim=12, vdim=8, rot=6, ff=40),
        parallel(ff=33),
    ], loop=(1, 3, 3))
    return cfg, weights(cfg, seed)
