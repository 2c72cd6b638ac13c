"""Butolorn without a GPU: configuration, weight files, the chunked form of the matrix memory, and
how sharp the GPU tests are: a mistake planted in the restatement moves its logits far beyond the
tolerance those tests allow."""
import math

import numpy as np
import pytest

import butolorn_util as bt
import plain_butolorn as plain
from buddy_mlir_b200 import _lib, butolorn, registry
from buddy_mlir_b200.config import MemoryMixer, SideBySide


def test_configuration_carries_every_size_and_constant():
    cfg = bt.config([bt.attention(heads=6, kv=2, dim=22, vdim=10, rot=6, base=77.0, ff=None),
                     bt.parallel(bt.heads(heads=3, kv=1, dim=8, vdim=4, rot=8, base=5.0), bt.memory(heads=7, dim=9, vdim=11, cap=3.5), 0.25, 4.0,
                                 ff=19)], width=64, vocab=99, eps=1e-3, scale=1.75, loop=(0, 2, 4), side=5)
    c = butolorn.parse(cfg, "float32", 77)
    assert (c.hidden, c.vocab, c.eps, c.n_layers, c.max_len, c.dtype) == (64, 99, 1e-3, 2, 77, "float32")
    assert (c.embed_scale, c.loop, c.side_dim) == (1.75, (0, 2, 4), 5)
    a, b = (layer.to_c() for layer in c.layers)
    assert (a.mixer, a.block, a.heads, a.kv_heads, a.dim, a.vdim, a.rot_dim, a.rot_base) == \
        (_lib.MIX_HEADS, _lib.BLOCK_SANDWICH, 6, 2, 22, 10, 6, 77.0)
    assert (a.rot_halves, a.qkv_bias, a.qk_norm, a.out_gate, a.sink, a.window, a.mix_scale) == (1, 1, 0, 0, -math.inf, 0, 1.0)
    assert a.ff_kind == _lib.FF_NONE and a.scale == pytest.approx(2.0 / 22 ** 0.5)
    assert (b.mixer, b.heads, b.kv_heads, b.dim, b.vdim, b.rot_dim, b.rot_base) == (_lib.MIX_HEADS_MEMORY, 3, 1, 8, 4, 8, 5.0)
    assert (b.rot_halves, b.qkv_bias, b.qk_norm, b.out_gate, b.sink, b.mix_scale) == (0, 0, 1, 1, 0.0, 0.25)
    assert (b.mem_heads, b.mem_dim, b.mem_vdim, b.mem_cap, b.mem_mix_scale) == (7, 9, 11, 3.5, 4.0)
    assert b.mem_q_scale == pytest.approx(1 / 3) and b.mem_floor == pytest.approx(1e-6)
    assert (b.ff_kind, b.ff, b.ff_act) == (_lib.FF_PLAIN, 19, _lib.ACT_RELU2)


def test_absent_loop_and_side_input():
    cfg = bt.config([bt.attention()], loop=None, side=0)
    del cfg["loop"], cfg["token_side"]
    c = butolorn.parse(cfg)
    assert c.loop == (0, 0, 1) and c.side_dim == 0


def test_a_memory_layer_of_its_own_is_described():
    """The mechanisms stand beside one another: another design may use one without the other."""
    from buddy_mlir_b200.config import LayerSpec
    m = butolorn.parse(bt.config([bt.parallel()])).layers[0].mixer
    assert isinstance(m, SideBySide) and isinstance(m.right, MemoryMixer)
    c = LayerSpec(m.right, None).to_c()
    assert c.mixer == _lib.MIX_MEMORY and c.mem_heads == m.right.heads and c.heads == 0


@pytest.mark.parametrize("change", [{"type": "recurrent"}, {"mlp": {"kind": "other"}}])
def test_unknown_layers_are_refused(change):
    cfg = bt.config([bt.attention()])
    cfg["layers"][0].update(change)
    with pytest.raises(ValueError):
        butolorn.parse(cfg)


def test_registry_reads_a_folder(tmp_path):
    cfg, w = bt.mixed_model()
    bt.write_folder(str(tmp_path), cfg, w)
    assert registry.model_config(str(tmp_path), "float32", 9) == butolorn.parse(cfg, "float32", 9)


def test_causality_of_the_restatement():
    cfg, w = bt.mixed_model()
    toks = np.random.default_rng(1).integers(0, cfg["vocab"], 40)
    whole = bt.want_logits(cfg, w, toks)
    assert np.allclose(bt.want_logits(cfg, w, toks[:17]), whole[:17], rtol=0, atol=1e-10)


def chunked_scan(q, k, v, i, f, size):
    """The recurrence unrolled over chunks: with F the running sum of f in a chunk, a = i - F and
    M_t = max(m, a_0 .. a_t), num_t = exp(m - M_t) S^T q_t + sum_s exp(a_s - M_t) (q_t k_s) v_s."""
    n, H, dim = q.shape
    S, z, m = np.zeros((H, dim, v.shape[2])), np.zeros((H, dim)), np.zeros(H)
    out = np.empty((n, H, v.shape[2]))
    for c in range(0, n, size):
        e = min(n, c + size)
        F = np.cumsum(f[c:e], axis=0)
        a = i[c:e] - F
        M = np.maximum(m, np.maximum.accumulate(a, axis=0))
        for h in range(H):
            D = np.tril(np.exp(a[None, :, h] - M[:, None, h]))
            P = (q[c:e, h] @ k[c:e, h].T) * D
            carry = np.exp(m[h] - M[:, h])[:, None]
            num = carry * (q[c:e, h] @ S[h]) + P @ v[c:e, h]
            nq = carry[:, 0] * (q[c:e, h] @ z[h]) + P.sum(axis=1)
            out[c:e, h] = num / (np.maximum(np.abs(nq), np.exp(-(F[:, h] + M[:, h]))) + 1e-6)[:, None]
            w = np.exp(a[:, h] - M[-1, h])
            S[h] = np.exp(m[h] - M[-1, h]) * S[h] + (k[c:e, h] * w[:, None]).T @ v[c:e, h]
            z[h] = np.exp(m[h] - M[-1, h]) * z[h] + w @ k[c:e, h]
        m = F[-1] + M[-1]
    return out


@pytest.mark.parametrize("size", [1, 7, 64, 200])
def test_chunks_of_the_matrix_memory_equal_the_recurrence(size):
    rng = np.random.default_rng(2)
    q, k, v = (rng.standard_normal((150, 3, d)) for d in (6, 6, 9))
    i, f = 4 * rng.standard_normal((150, 3)), -np.exp(2 * rng.standard_normal((150, 3)) - 3)
    want = plain.memory_scan(q, k, v, i, f)
    assert np.allclose(chunked_scan(q, k, v, i, f, size), want, rtol=1e-8, atol=1e-10)


# ---- planted mistakes ------------------------------------------------------------------------------
def swapped_heads(q, k, v, scale, softmax):
    """Query head h reads key head h mod G."""
    H, G = q.shape[1], k.shape[1]
    order = [h % G for h in range(H)]
    return plain_attend(q, k[:, order], v[:, order], scale, softmax)


def floor_one(q, k, v, i, f):
    """max(|n q|, 1) in place of max(|n q|, exp(-m))."""
    n, H, dim = q.shape
    S, z, m = np.zeros((H, dim, v.shape[2])), np.zeros((H, dim)), np.zeros(H)
    out = np.empty((n, H, v.shape[2]))
    for t in range(n):
        new = np.maximum(f[t] + m, i[t])
        keep, add = np.exp(f[t] + m - new), np.exp(i[t] - new)
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        z, m = keep[:, None] * z + add[:, None] * k[t], new
        out[t] = np.einsum("hdv,hd->hv", S, q[t]) / np.maximum(np.abs((z * q[t]).sum(axis=1)), 1.0)[:, None]
    return out


def lost_state(q, k, v, i, f):
    """The state is dropped at token 32."""
    return np.concatenate([plain_scan(q[a:b], k[a:b], v[a:b], i[a:b], f[a:b]) for a, b in ((0, 32), (32, len(q)))])


def uncapped(h, c, t, p):
    return h @ t[p + "i"].T + t[p + "i.b"], plain.log_sigmoid(h @ t[p + "f"].T + t[p + "f.b"])


def whole_norm_by_head(x, weight, eps):
    n = 2 if x.shape[1] % 2 == 0 else 1
    return plain.unit_rms(x.reshape(len(x), n, -1), eps).reshape(x.shape) * weight


def forgetful_loop(config):
    return [(i, False) for i, _ in plain_order(config)]


def eager_loop(config):
    loop = config["loop"]
    seen, out = False, []
    for i, again in plain_order(config):
        first = i == loop["start"] and not seen
        seen = seen or first
        out.append((i, again or first))
    return out


plain_attend, plain_scan, plain_order = plain.attend, plain.memory_scan, plain.layer_order
MISTAKES = {"no sink": ("softmax_sink", plain.softmax_plain), "a sink everywhere": ("softmax_plain", plain.softmax_sink),
            "halves rotated in pairs": ("rotate_halves", plain.rotate_interleaved),
            "pairs rotated in halves": ("rotate_interleaved", plain.rotate_halves),
            "key heads taken in turn": ("attend", swapped_heads),
            "norm head by head": ("whole_norm", whole_norm_by_head), "no query and key norm": ("whole_norm", lambda x, w, eps: x),
            "no output gate": ("output_gate", lambda o, z: o),
            "a token does not see itself": ("causal", lambda n: np.tril(np.ones((n, n), bool), -1) | (np.arange(n) == 0)[:, None] & np.eye(n, dtype=bool)),
            "floor of one": ("memory_scan", floor_one),
            "state dropped": ("memory_scan", lost_state), "gates without a cap": ("memory_gates", uncapped),
            "plain forget gate": ("log_sigmoid", lambda z: np.minimum(z, 0)),
            "relu not squared": ("squared_relu", lambda z: np.maximum(z, 0)),
            "sigmoid in place of gelu": ("gelu_tanh", plain.sigmoid),
            "side input not normed": ("token_side", lambda x, e, t, p, eps: (plain.gelu_tanh(x @ t[p + "side.gate"].T) * e) @ t[p + "side.proj"].T),
            "no embedding before a pass": ("layer_order", forgetful_loop), "embedding before the first pass": ("layer_order", eager_loop)}


@pytest.mark.parametrize("name", MISTAKES)
def test_planted_mistakes_show(name, monkeypatch):
    cfg, w = bt.mixed_model()
    toks = np.random.default_rng(7).integers(0, cfg["vocab"], 60)
    good = bt.want_logits(cfg, w, toks)
    monkeypatch.setattr(plain, *MISTAKES[name])
    assert bt.error(bt.want_logits(cfg, w, toks), good) > 2 * bt.TOLERANCE["bfloat16"]


@pytest.mark.parametrize("change", [("embedding", "scale"), ("norm", "eps")])
def test_model_constants_show(change):
    cfg, w = bt.mixed_model()
    toks = np.random.default_rng(7).integers(0, cfg["vocab"], 60)
    good = bt.want_logits(cfg, w, toks)
    cfg[change[0]][change[1]] *= 2 if change[1] == "scale" else 1e4
    assert bt.error(bt.want_logits(cfg, w, toks), good) > 2 * bt.TOLERANCE["bfloat16"]
