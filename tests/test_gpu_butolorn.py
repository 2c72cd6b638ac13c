"""Butolorn on the GPU against the plain restatement (plain_butolorn.py): each mechanism alone,
prompts against token-by-token decoding, portions, mixed batches, pages and slots used again, far
keys and old state, generation."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import butolorn_util as bt
from buddy_mlir_b200 import _lib, butolorn
from buddy_mlir_b200.session import ModelSession, run_generation

pytestmark = pytest.mark.gpu
DTYPES = ("float32", "bfloat16")


def tokens(cfg, n, seed=0):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n)


def step_logits(b, seq, toks, sizes):
    """All logits of a sequence fed in portions of the given sizes."""
    out, at = [], 0
    for n in sizes:
        part = toks[at:at + n]
        lo, _ = b.step([(seq, part)], [list(range(len(part)))])
        out.append(lo)
        at += len(part)
    assert at == len(toks)
    return np.concatenate(out)


def cut(n, size):
    return [size] * (n // size) + ([n % size] if n % size else [])


def check_model(cfg, w, dtype, n=150, singles=40):
    """A whole prompt, token-by-token decoding, and a batch in portions."""
    tol = bt.TOLERANCE[dtype]
    toks = tokens(cfg, n)
    want = bt.want_logits(cfg, w, toks)
    s = bt.session(cfg, w, dtype)
    assert bt.error(s.prefill_rows(toks, 0), want) < tol
    s.reset_position()
    for i, t in enumerate(toks[:singles]):
        s.decode(int(t))
        assert bt.error(s.logits_data(), want[i]) < tol, i
    b = bt.batch(s)
    sizes = [70, 1, 2, 17, 1, 16, 9, 8, 5]
    assert bt.error(step_logits(b, b.add(), toks, sizes + [n - sum(sizes)]), want) < tol
    b.close()
    s.close()


# ---- mechanisms alone -------------------------------------------------------------------------
HEADS = [
    dict(),
    dict(heads=6, kv=6, dim=2, vdim=1, rot=2),
    dict(heads=3, kv=3, dim=33, vdim=7, rot=10),                 # nothing aligned
    dict(heads=34, kv=2, dim=8, vdim=8, rot=8),                  # more query heads per key head than a tile has rows
    dict(heads=12, kv=2, dim=64, vdim=72, rot=32, sharp=1.0),
    dict(heads=4, kv=4, dim=96, vdim=40, rot=64, base=50.0, sharp=1.0),
    dict(heads=2, kv=1, dim=128, vdim=136, rot=128, sharp=1.0),  # two groups of value columns
    dict(heads=2, kv=2, dim=200, vdim=16, rot=4, sharp=1.0),
    dict(heads=3, kv=1, dim=264, vdim=48, rot=30, sharp=1.0),    # wider than the tensor-core kernels take
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kw", HEADS)
def test_attention_alone(kw, dtype):
    cfg = bt.config([bt.attention(ff=None, **kw)], side=0)
    check_model(cfg, bt.weights(cfg, 1), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kw", HEADS)
def test_sink_attention_alone(kw, dtype):
    cfg = bt.config([bt.parallel(bt.heads(**kw), ff=None)], side=0)
    w = bt.weights(cfg, 2)
    w["l0.mix.right.o"][:] = 0               # the memory contributes nothing
    check_model(cfg, w, dtype)


MEMORY = [
    dict(),
    dict(heads=1, dim=1, vdim=1),
    dict(heads=2, dim=7, vdim=33, cap=0.5),
    dict(heads=2, dim=32, vdim=32, cap=20.0),
    dict(heads=1, dim=64, vdim=65),
    dict(heads=2, dim=65, vdim=96),
    dict(heads=1, dim=128, vdim=40),
    dict(heads=1, dim=160, vdim=72),
    dict(heads=1, dim=256, vdim=31),
    dict(heads=1, dim=300, vdim=20),                             # wider than the chunked kernel takes
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kw", MEMORY)
def test_matrix_memory_alone(kw, dtype):
    cfg = bt.config([bt.parallel(bt.heads(heads=1, kv=1, dim=2, vdim=2, rot=2), bt.memory(**kw), ff=None)], side=0)
    w = bt.weights(cfg, 3)
    w["l0.mix.left.o"][:] = 0                # the attention contributes nothing
    check_model(cfg, w, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("bias", [-9.0, 0.0, 9.0])
def test_matrix_memory_with_extreme_input_gates(bias, dtype):
    """Input gates far below the start of the running maximum, and far above it."""
    cfg = bt.config([bt.parallel(bt.heads(heads=1, kv=1, dim=2, vdim=2, rot=2), bt.memory(dim=24, vdim=24, cap=15.0), ff=None)], side=0)
    w = bt.weights(cfg, 4)
    w["l0.mix.left.o"][:] = 0
    w["l0.mix.right.i.b"] = bt.to_bf16(np.full(3, bias, np.float32))
    check_model(cfg, w, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("ff", [1, 7, 333])
def test_feed_forward_alone(ff, dtype):
    cfg = bt.config([bt.attention(heads=1, kv=1, dim=2, vdim=2, rot=2, ff=ff)], width=100, side=0)
    w = bt.weights(cfg, 5)
    w["l0.mix.o"][:] = 0
    check_model(cfg, w, dtype, n=130, singles=3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("side", [1, 5, 64])
def test_side_input_alone(side, dtype):
    layer = dict(heads=1, kv=1, dim=2, vdim=2, rot=2, ff=None)
    cfg = bt.config([bt.attention(**layer), bt.attention(**layer), bt.attention(**layer)], side=side)
    w = bt.weights(cfg, 6)
    for i in range(3):
        w[f"l{i}.mix.o"][:] = 0
    check_model(cfg, w, dtype, n=130, singles=3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("loop", [None, (0, 1, 2), (0, 3, 2), (2, 3, 4), (1, 2, 1), (1, 1, 3)])
def test_loops(loop, dtype):
    cfg = bt.config([bt.parallel(), bt.attention(ff=24), bt.parallel(ff=None)], loop=loop, side=4)
    check_model(cfg, bt.weights(cfg, 7), dtype, n=130, singles=12)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("vocab,width,side", [(131, 75, 9), (2, 1, 1), (4099, 8, 3)])
def test_odd_sizes_everywhere(vocab, width, side, dtype):
    cfg = bt.config([bt.parallel(bt.heads(heads=3, kv=3, dim=7, vdim=5, rot=2), bt.memory(heads=1, dim=3, vdim=5), 1.0, 1.0, ff=13),
                     bt.attention(heads=3, kv=1, dim=9, vdim=1, rot=0, ff=1)], width=width, vocab=vocab, loop=(1, 2, 2), side=side)
    w = bt.weights(cfg, 8)
    if width < 10:                           # few elements: a norm is little more than signs, and rounding may turn one
        for k in w:
            if k.endswith(("norm1b", "norm2b", "side.norm")):
                w[k] = bt.to_bf16(np.full(width, 0.1, np.float32))
    check_model(cfg, w, dtype, n=130, singles=20)


@pytest.mark.parametrize("dtype", DTYPES)
def test_wide_projections(dtype):
    """Large enough for every form of the contractions: 256-column tiles, a split k range, activations
    staged in several pieces."""
    cfg = bt.config([bt.parallel(bt.heads(heads=8, kv=2, dim=128, vdim=128, rot=64, sharp=1.0), bt.memory(heads=4, dim=128, vdim=256), ff=4100),
                     bt.attention(heads=16, kv=4, dim=64, vdim=64, rot=64, sharp=1.0, ff=520)], width=1032, vocab=1000, side=40)
    w = bt.weights(cfg, 9)
    toks = tokens(cfg, 538, 1)
    want = bt.want_logits(cfg, w, toks)
    tol = bt.TOLERANCE[dtype]
    s = bt.session(cfg, w, dtype, max_len=640)
    assert bt.error(s.prefill_rows(toks, 0), want) < tol
    s.reset_position()
    s.prefill_rows(toks[:500], 0)
    assert bt.error(s.prefill_rows(toks[500:530], 500), want[500:530]) < tol
    for i in range(530, 538):
        s.decode(int(toks[i]))
        assert bt.error(s.logits_data(), want[i]) < tol
    s.close()


# ---- the whole model under schedules -----------------------------------------------------------
@pytest.fixture(scope="module", params=DTYPES)
def mixed(request):
    cfg, w = bt.mixed_model()
    s = bt.session(cfg, w, request.param)
    toks = tokens(cfg, 200, 7)
    yield cfg, w, s, toks, bt.want_logits(cfg, w, toks), bt.TOLERANCE[request.param]
    s.close()


@pytest.mark.parametrize("page", [1, 4, 16, 100])
@pytest.mark.parametrize("size", [2, 3, 8, 9, 16, 17, 50, 63, 64, 65, 127, 128, 129, 200])
def test_portions(mixed, size, page):
    cfg, w, s, toks, want, tol = mixed
    n = 60 if size < 8 else len(toks)
    b = bt.batch(s, page=page, pages=300)
    assert bt.error(step_logits(b, b.add(), toks[:n], cut(n, size)), want[:n]) < tol
    b.close()


def test_uneven_portions_and_single_tokens(mixed):
    cfg, w, s, toks, want, tol = mixed
    b = bt.batch(s)
    sizes = [1, 2, 40, 1, 1, 17, 3, 2, 30, 1, 60, 2]
    sizes += [1] * (len(toks) - sum(sizes))
    assert bt.error(step_logits(b, b.add(), toks, sizes), want) < tol
    b.close()


def test_prompt_equals_token_by_token(mixed):
    cfg, w, s, toks, want, tol = mixed
    s.reset_position()
    rows = s.prefill_rows(toks[:90], 0)
    s.reset_position()
    one = []
    for t in toks[:90]:
        s.decode(int(t))
        one.append(s.logits_data().copy())
    assert bt.error(np.array(one), want[:90]) < tol
    assert bt.error(rows, np.array(one, dtype=np.float64)) < tol


def test_long_decoding(mixed):
    cfg, w, s, toks, want, tol = mixed
    s.reset_position()
    s.prefill_rows(toks[:3], 0)
    for i, t in enumerate(toks[3:], 3):
        s.decode(int(t))
        assert bt.error(s.logits_data(), want[i]) < tol, i


def test_a_prompt_longer_than_one_pass(mixed):
    """Thousands of rows go through the layers in several passes; the result is that of portions."""
    cfg, w, s, _, _, tol = mixed
    toks = tokens(cfg, 4500, 13)
    b = bt.batch(s, page=64, pages=160, context=5000)
    places = [0, 511, 512, 2999, 4095, 4096, 4097, 4499]
    whole, _ = b.step([(b.add(), toks)], [places])
    q = b.add()
    parts, at = [], 0
    for n in (1500, 7, 2500, 493):
        got, _ = b.step([(q, toks[at:at + n])], [[p - at for p in places if at <= p < at + n]], want_logits=True)
        parts.append(got)
        at += n
    assert bt.error(whole, np.concatenate(parts).astype(np.float64)) < tol
    b.close()


def test_first_tokens(mixed):
    cfg, w, s, toks, want, tol = mixed
    for n in (1, 2, 3, 8, 9, 10, 16, 17, 18):
        s.reset_position()
        assert bt.error(s.prefill_rows(toks[:n], 0), want[:n]) < tol


def test_unequal_batch_against_each_alone(mixed):
    cfg, w, s, toks, _, tol = mixed
    rng = np.random.default_rng(11)
    seqs = [rng.integers(0, cfg["vocab"], n) for n in (75, 1, 33, 120, 18, 2)]
    wants = [bt.want_logits(cfg, w, t) for t in seqs]
    b = bt.batch(s, page=8)
    ids = [b.add() for _ in seqs]
    at = [0] * len(seqs)
    while any(a < len(t) for a, t in zip(at, seqs)):
        # prompts and single tokens together, a random subset in a random order
        live = [i for i in rng.permutation(len(seqs)) if at[i] < len(seqs[i]) and rng.random() < 0.8]
        entries, want_places, expect = [], [], []
        for i in live:
            n = min(int(rng.choice([1, 1, 2, 5, 20, 40])), len(seqs[i]) - at[i])
            entries.append((ids[i], seqs[i][at[i]:at[i] + n]))
            want_places.append(sorted(set(rng.integers(0, n, 2).tolist())))
            expect += [wants[i][at[i] + p] for p in want_places[-1]]
            at[i] += n
        if entries:
            got, nxt = b.step(entries, want_places)
            assert bt.error(got, np.array(expect)) < tol
            assert np.array_equal(nxt, got.argmax(axis=1))
    b.close()


def test_many_sequences_in_one_step(mixed):
    cfg, w, s, _, _, tol = mixed
    rng = np.random.default_rng(17)
    seqs = [rng.integers(0, cfg["vocab"], 5 + i % 4) for i in range(70)]
    b = bt.batch(s, max_seqs=70, page=4)
    ids = [b.add() for _ in seqs]
    b.step([(q, t[:-3]) for q, t in zip(ids, seqs)])
    got = [b.step([(q, t[k:k + 1] if k < -1 else t[-1:]) for q, t in zip(ids, seqs)])[0] for k in (-3, -2, -1)]
    for i, t in enumerate(seqs):
        assert bt.error(np.array([g[i] for g in got]), bt.want_logits(cfg, w, t)[-3:]) < tol
    b.close()


def test_freed_pages_and_slots_are_used_again(mixed):
    """A slot's state and a page's rows of a finished sequence leave no trace in the next."""
    cfg, w, s, toks, want, tol = mixed
    b = bt.batch(s, max_seqs=2, page=4, pages=40, context=160)
    rng = np.random.default_rng(3)
    for k in range(6):
        other = b.add()
        b.step([(other, rng.integers(0, cfg["vocab"], 13 + 5 * k))])
        q = b.add()
        n = 70 + k
        first = (1, 2, 30, 64, 8, 17)[k]
        got = step_logits(b, q, toks[:n], [first, n - 6 - first, 2, 1, 1, 2])
        assert bt.error(got, want[:n]) < tol
        b.remove(other)
        b.remove(q)
        assert b.free_pages() == 40
    b.close()


def test_a_step_that_does_not_fit_changes_nothing():
    cfg = bt.config([bt.parallel()])
    w = bt.weights(cfg, 8)
    s = bt.session(cfg, w, "float32")
    toks = tokens(cfg, 20)
    want = bt.want_logits(cfg, w, toks)
    b = bt.batch(s, max_seqs=2, page=4, pages=5, context=20)
    q, r = b.add(), b.add()
    b.step([(q, toks[:8])])
    with pytest.raises(_lib.B200Error):
        b.step([(r, toks[:4]), (q, toks[:12])])
    assert b.free_pages() == 3 and b.length(q) == 8 and b.length(r) == 0
    got, _ = b.step([(q, toks[8:])], [list(range(12))])
    assert bt.error(got, want[8:]) < bt.TOLERANCE["float32"]
    b.close()
    s.close()


def test_a_session_with_state_runs_from_where_it_is():
    """A recurrent state cannot go back: only to the start, or on from the last token."""
    cfg = bt.config([bt.parallel()])
    w = bt.weights(cfg, 8)
    s = bt.session(cfg, w, "float32")
    toks = tokens(cfg, 30)
    want = bt.want_logits(cfg, w, toks)
    s.prefill_rows(toks[:20], 0)
    with pytest.raises(_lib.B200Error, match="recurrent state"):
        s.prefill_rows(toks[10:12], 10)
    assert bt.error(s.prefill_rows(toks[20:], 20), want[20:]) < bt.TOLERANCE["float32"]
    s.reset_position()
    s.decode(int(toks[0]))
    assert bt.error(s.logits_data(), want[0]) < bt.TOLERANCE["float32"]
    s.close()
    att = bt.config([bt.attention()])        # no state: any earlier position will do
    s = bt.session(att, bt.weights(att, 8), "float32")
    s.prefill_rows(toks[:20], 0)
    s.prefill_rows(toks[10:12], 10)
    s.close()


# ---- far keys and old state ---------------------------------------------------------------------
def far_places(query):
    return (0, 1, 15, 16, 63, 64, 127, 128, query - 64, query - 1)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["attention", "parallel"])
def test_a_far_key_among_hundreds(kind, dtype):
    """Token 1 asks for token 0 and for nothing else: one head's query answers feature 1 on the key
    element that carries feature 0, at a pair that hardly turns."""
    m = dict(heads=2, kv=1, dim=24, vdim=20, rot=8, base=1e4, sharp=1.0)
    layer = bt.attention(ff=None, **m) if kind == "attention" else bt.parallel(bt.heads(**m), ff=None)
    cfg = bt.config([layer], width=80, side=0, scale=1.0)
    w = bt.values(bt.weights(cfg, 6))
    e, p = w["embed"], "l0.mix." if kind == "attention" else "l0.mix.left."
    if kind == "parallel":
        w["l0.mix.right.o"][:] = 0
    e[:, :2] = 0
    e[0, 0] = e[1, 1] = 6.0
    at = 20                                  # an element that is not rotated
    for name in ("q", "k"):
        w[p + name][:, :2] = 0
        w[p + name][at, :] = 0
    w[p + "q"][at, 1] = 40.0
    w[p + "k"][at, 0] = 8.0
    w = {k: bt.to_bf16(v) for k, v in w.items()}
    s = bt.session(cfg, w, dtype, max_len=512)
    rng = np.random.default_rng(12)
    for query in (511, 300):
        for place in far_places(query):
            toks = rng.integers(2, cfg["vocab"], query + 1)
            toks[place], toks[query] = 0, 1
            want = bt.want_logits(cfg, w, toks)[-1]
            other = toks.copy()
            other[place] = 2
            assert bt.error(bt.want_logits(cfg, w, other)[-1], want) > 5 * bt.TOLERANCE[dtype]
            s.reset_position()
            assert bt.error(s.prefill_rows(toks, 0)[-1], want) < bt.TOLERANCE[dtype]
            b = bt.batch(s, page=16, context=512)
            q = b.add()
            got = step_logits(b, q, toks, [query - 20, 19, 1, 1])
            assert bt.error(got[-1], want) < bt.TOLERANCE[dtype]
            b.close()
    s.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_an_old_memory_after_hundreds_of_tokens(dtype):
    """Token 0 opens the input gate wide and the forget gate holds: what it wrote is read by every
    later token, at and around the edges of the chunks the state is carried over.  A query that is
    nearly orthogonal to that one key divides by next to nothing: the restatement itself, in 32-bit,
    is 3.5e-5 away from its 64-bit result here."""
    tol = max(bt.TOLERANCE[dtype], 1e-4)
    cfg = bt.config([bt.parallel(bt.heads(heads=1, kv=1, dim=2, vdim=2, rot=2), bt.memory(heads=2, dim=16, vdim=24, cap=12.0), ff=None)],
                    width=80, side=0, scale=1.0)
    w = bt.values(bt.weights(cfg, 16))
    e, p = w["embed"], "l0.mix.right."
    w["l0.mix.left.o"][:] = 0
    e[:, 0] = 0
    e[0, 0] = 8.0
    w[p + "i"][:] = 0
    w[p + "i"][:, 0] = 4.0
    w[p + "i.b"][:] = -2.0
    w[p + "f"][:] = 0
    w[p + "f.b"][:] = 9.0
    w = {k: bt.to_bf16(v) for k, v in w.items()}
    s = bt.session(cfg, w, dtype, max_len=512)
    rng = np.random.default_rng(12)
    for place in (0, 1, 62, 63, 64, 65, 127, 128):
        toks = rng.integers(2, cfg["vocab"], 400)
        toks[place] = 0
        want = bt.want_logits(cfg, w, toks)
        other = toks.copy()
        other[place] = 2
        assert bt.error(bt.want_logits(cfg, w, other)[-1], want[-1]) > 5 * tol
        s.reset_position()
        assert bt.error(s.prefill_rows(toks, 0), want) < tol
        b = bt.batch(s, page=16, context=512)
        got = step_logits(b, b.add(), toks, [64, 1, 65, 2, 63, 100, 17] + [1] * 88)
        assert bt.error(got, want) < tol
        b.close()
    s.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_every_earlier_token_is_seen_and_no_later_one(dtype):
    cfg = bt.config([bt.attention(ff=None, sharp=0.5)], side=0)
    w = bt.weights(cfg, 4)
    s = bt.session(cfg, w, dtype)
    base = tokens(cfg, 140, 9)
    for sizes in ([140], [100] + [1] * 40, cut(140, 9)):
        b = bt.batch(s, page=8)
        q = b.add()
        ref = step_logits(b, q, base, sizes)
        b.remove(q)
        for j in (0, 55, 110):
            other = base.copy()
            other[j] = (other[j] + 1) % cfg["vocab"]
            q = b.add()
            got = step_logits(b, q, other, sizes)
            b.remove(q)
            changed = np.abs(got - ref).max(axis=1) > 0
            assert not changed[:j].any() and changed[j:].mean() > 0.95
        b.close()
    s.close()


# ---- generation -----------------------------------------------------------------------------------
def plain_greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(bt.want_logits(cfg, w, toks)[-1])))
    return toks[len(prompt):]


def test_greedy_generation_and_device_loop():
    cfg, w = bt.mixed_model(21)
    s = bt.session(cfg, w, "float32")
    prompt = [int(t) for t in tokens(cfg, 24, 1)]
    want = plain_greedy(cfg, w, prompt, 24)
    ids, _ = run_generation(s, prompt, len(prompt) + 23)
    assert ids == want
    s.prefill(prompt)
    first = int(np.argmax(s.logits_data()))
    assert [first] + s.generate(first, 23).tolist() == want
    assert s.decode_greedy(want[-1]) == plain_greedy(cfg, w, prompt + want, 1)[0]
    s.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["attention", "parallel"])
def test_full_cache_drops_positions_and_turns_keys_back(kind, dtype):
    """One layer: its cached rows depend on nothing but token and position, so after the overflow
    the session must continue like a fresh sequence of the tokens that were kept."""
    cfg = bt.config([bt.attention() if kind == "attention" else bt.parallel()])
    w = bt.weights(cfg, 31)
    if kind == "parallel":
        w["l0.mix.right.o"][:] = 0           # a recurrent state has no positions to drop
    s = bt.session(cfg, w, dtype, max_len=48)
    toks = tokens(cfg, 48, 3)
    s.prefill_rows(toks, 0)
    assert s.handle_kv_cache_overflow(10)
    kept = np.concatenate([toks[:10], toks[29:]])
    assert s.position() == len(kept)
    for t in (5, 6, 7):
        kept = np.append(kept, t)
        s.decode(t)
        assert bt.error(s.logits_data(), bt.want_logits(cfg, w, kept)[-1]) < bt.TOLERANCE[dtype]
    ids, _ = run_generation(s, [int(t) for t in toks[:40]], 40 + 30)   # runs past the cache's end
    assert len(ids) == 31
    s.close()


def test_batched_greedy_generation():
    cfg, w = bt.mixed_model(22)
    s = bt.session(cfg, w, "float32")
    b = bt.batch(s, max_seqs=12, page=4)
    prompts = [[int(t) for t in tokens(cfg, n, 30 + n)] for n in (5, 1, 40, 17, 9, 3, 21, 2, 11, 6)]
    ids = [b.add() for _ in prompts]
    _, nxt = b.step(list(zip(ids, prompts)), want_logits=False)
    out = [[int(t)] for t in nxt]
    for _ in range(7):
        _, nxt = b.decode(ids, [o[-1] for o in out], want_logits=False)
        for o, t in zip(out, nxt):
            o.append(int(t))
    for p, o in zip(prompts, out):
        assert o == plain_greedy(cfg, w, p, 8)
    b.close()
    s.close()


def test_command_line_generates_and_replays(tmp_path):
    cfg, w = bt.mixed_model(23)
    model = tmp_path / "model"
    model.mkdir()
    bt.write_folder(str(model), cfg, w)
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    prompt = [int(t) for t in tokens(cfg, 9, 2)]
    out = subprocess.run([sys.executable, "-m", "buddy_mlir_b200", "generate", "--model", str(model), "--dtype", "float32",
                          "--tokens", ",".join(map(str, prompt)), "--max-new", "8", "--max-len", "64"],
                         cwd=root, capture_output=True, text=True, timeout=300)
    assert out.returncode == 0, out.stderr
    assert [int(t) for t in out.stdout.split()] == plain_greedy(cfg, w, prompt, 8)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": prompt, "want": [8, 0]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [3], "want": []}, {"id": "b", "tokens": [1, 2], "want": [1]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": [4, 5], "want": [0]}], "end": ["a"]}]
    run = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(model), "--dtype", "float32",
                          "--out", str(tmp_path), "--max-tokens", "32"], cwd=str(tmp_path), capture_output=True, text=True,
                         input="".join(json.dumps(x) + "\n" for x in steps), timeout=300)
    assert run.returncode == 0, run.stderr
    assert [l for l in run.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    a, b = bt.want_logits(cfg, w, prompt + [3, 4, 5]), bt.want_logits(cfg, w, [1, 2])
    for name, rows in (("0", [a[8], a[0]]), ("1", [b[1]]), ("2", [a[10]])):
        got = np.fromfile(tmp_path / f"{name}.f32", dtype="<f4").reshape(len(rows), -1)
        assert bt.error(got, np.array(rows)) < bt.TOLERANCE["float32"]


def test_wrong_tensors_and_layers_are_refused():
    cfg = bt.config([bt.attention(ff=None), bt.parallel()])
    w = bt.weights(cfg, 1)
    s = ModelSession(butolorn.parse(cfg, "float32", 16))
    with pytest.raises(_lib.B200Error, match="no tensor"):
        s.load_named({"l1.mix.q": w["l0.mix.q"]})
    with pytest.raises(_lib.B200Error, match="got"):
        s.load_named({"l0.mix.q.b": w["l0.mix.q.b"][:-1]})
    with pytest.raises(_lib.B200Error, match="missing"):
        s.load_named({k: v for k, v in w.items() if k != "l1.mix.right.f.b"})
    s.close()
    for bad in (bt.attention(heads=5, kv=2), bt.attention(dim=8, rot=10), bt.parallel(right=bt.memory(dim=600)),
                bt.parallel(right=bt.memory(cap=0.0))):
        with pytest.raises(_lib.B200Error, match="sizes"):
            ModelSession(butolorn.parse(bt.config([bad]), "float32", 16))
    with pytest.raises(_lib.B200Error, match="loop"):
        ModelSession(butolorn.parse(bt.config([bt.attention()], loop=(0, 2, 1)), "float32", 16))


def test_norms_of_an_absent_feed_forward_may_come_along():
    cfg = bt.config([bt.attention(ff=None)])
    w = bt.weights(cfg, 1)
    w["l0.norm2"] = w["l0.norm2b"] = w["l0.norm1"]
    toks = tokens(cfg, 12)
    s = bt.session(cfg, w, "float32")
    assert bt.error(s.prefill_rows(toks, 0), bt.want_logits(cfg, w, toks)) < bt.TOLERANCE["float32"]
    s.close()
