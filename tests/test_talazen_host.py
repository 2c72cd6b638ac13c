"""Talazen without a GPU: configuration, weight files, and how sharp the GPU tests are: a mistake
planted in the restatement moves its logits far beyond the tolerance those tests allow."""
import numpy as np
import pytest

import plain_talazen as plain
import talazen_util as tz
from buddy_mlir_b200 import _lib, registry, safetensors_file, talazen


def test_configuration_carries_every_size_and_constant():
    cfg = tz.config([(tz.attention(window=11), tz.gated(ff=10, limit=2.5)),
                     (tz.attention(kv_from=0, window=3), tz.experts(n=6, top=4, ff=9, limit=0.5)),
                     (tz.attention(kv_from=0), None)], width=64, vocab=99, eps=1e-3)
    c = talazen.parse(cfg, "float32", 77)
    assert (c.hidden, c.vocab, c.eps, c.n_layers, c.max_len, c.dtype) == (64, 99, 1e-3, 3, 77, "float32")
    a, b, d = (layer.to_c() for layer in c.layers)
    assert (a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank, a.window, a.kv_from) == (3, 24, 16, 20, 40, 11, -1)
    assert (a.ff_kind, a.ff, a.limit) == (_lib.FF_GATED, 10, 2.5)
    assert a.gate_slope == pytest.approx(1.702) and a.up_offset == 1.0
    assert (b.ff_kind, b.ff, b.experts, b.top, b.kv_from, b.window) == (_lib.FF_EXPERTS, 9, 6, 4, 0, 3)
    assert (d.ff_kind, d.window) == (_lib.FF_NONE, 0)
    assert a.scale == pytest.approx(2.0 / 40 ** 0.5) and a.rot_base == 1000.0


@pytest.mark.parametrize("change", [{"type": "recurrent"}, {"mlp": {"kind": "other"}}])
def test_unknown_layers_are_refused(change):
    cfg = tz.config([(tz.attention(), None)])
    cfg["layers"][0].update(change)
    with pytest.raises(ValueError):
        talazen.parse(cfg)


def test_registry_reads_a_folder(tmp_path):
    cfg, w = tz.mixed_model()
    tz.write_folder(str(tmp_path), cfg, w)
    c = registry.model_config(str(tmp_path), "float32", 9)
    assert c == talazen.parse(cfg, "float32", 9)
    t = safetensors_file.read(str(tmp_path / "model.safetensors"))
    assert set(t) == set(w) and all(d == "BF16" and np.array_equal(a, w[k]) for k, (d, a) in t.items())
    (tmp_path / "config.json").write_text('{"architecture": "Nothing"}')
    with pytest.raises(ValueError, match="unknown architecture"):
        registry.model_config(str(tmp_path))


def test_a_truncated_weight_file_is_refused(tmp_path):
    cfg, w = tz.mixed_model()
    tz.write_folder(str(tmp_path), cfg, w)
    p = tmp_path / "model.safetensors"
    p.write_bytes(p.read_bytes()[:-10])
    with pytest.raises(ValueError, match="does not fit"):
        safetensors_file.read(str(p))


def test_causality_of_the_restatement():
    cfg, w = tz.mixed_model()
    toks = np.random.default_rng(1).integers(0, cfg["vocab"], 40)
    whole = tz.want_logits(cfg, w, toks)
    assert np.allclose(tz.want_logits(cfg, w, toks[:17]), whole[:17], rtol=0, atol=1e-12)


def off_by_one(delta):
    def mask(n, window):
        i, j = np.arange(n)[:, None], np.arange(n)[None, :]
        return (j <= i) & ((i - j) < (window + delta if window is not None else n))
    return mask


def no_offset(h, gate, up, down, limit):
    g = np.minimum(h @ gate.T, limit)
    return (g / (1 + np.exp(-1.702 * g)) * np.clip(h @ up.T, -limit, limit)) @ down.T


def unbounded(h, gate, up, down, limit):
    g = h @ gate.T
    return (g / (1 + np.exp(-1.702 * g)) * (h @ up.T + 1)) @ down.T


def silu_gate(h, gate, up, down, limit):
    g = np.minimum(h @ gate.T, limit)
    return (g / (1 + np.exp(-g)) * (np.clip(h @ up.T, -limit, limit) + 1)) @ down.T


def halves(x, positions, base):
    n = x.shape[-1]
    perm = np.concatenate([np.arange(0, n, 2), np.arange(1, n, 2)])
    out = np.empty_like(x)
    out[..., :] = plain_rotate(x[..., np.argsort(perm)], positions, base)[..., perm]
    return out


def softmax_over_all(h, router, top):
    z = h @ router.T
    chosen = np.argsort(-z, axis=-1, kind="stable")[:, :top]
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    return chosen, np.take_along_axis(e / e.sum(axis=-1, keepdims=True), chosen, axis=-1)


plain_rotate = plain.rotate_pairs
MISTAKES = {"window one longer": ("window_mask", off_by_one(1)), "window one shorter": ("window_mask", off_by_one(-1)),
            "no offset on the up branch": ("gated_unit", no_offset), "no limit": ("gated_unit", unbounded),
            "another gate slope": ("gated_unit", silu_gate), "split halves rotated": ("rotate_pairs", halves),
            "positions stretched": ("rotate_pairs", lambda x, p, b: plain_rotate(x, np.asarray(p) * 1.05, b)),
            "router softmax over all": ("route", softmax_over_all),
            "latent not normed": ("latent_keys", None)}


@pytest.mark.parametrize("name", MISTAKES)
def test_planted_mistakes_show(name, monkeypatch):
    cfg, w = tz.mixed_model()
    toks = np.random.default_rng(7).integers(0, cfg["vocab"], 60)
    good = tz.want_logits(cfg, w, toks)
    attr, fn = MISTAKES[name]
    if name == "latent not normed":
        def fn(h, mixer, tensors, prefix, eps):
            down = h @ tensors[prefix + "dkv"].T
            return down[:, :mixer["kv_rank"]], plain_rotate(down[:, mixer["kv_rank"]:], np.arange(len(h)), mixer["rot"]["base"])
    monkeypatch.setattr(plain, attr, fn)
    assert tz.error(tz.want_logits(cfg, w, toks), good) > 2 * tz.TOLERANCE["bfloat16"]
