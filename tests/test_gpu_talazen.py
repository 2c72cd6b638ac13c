"""Talazen on the GPU against the plain restatement (plain_talazen.py): each mechanism alone,
prompts against token-by-token decoding, portions, mixed batches, page reuse, window edges,
generation."""
import os
import subprocess
import sys

import numpy as np
import pytest

import plain_talazen as plain
import talazen_util as tz
from buddy_mlir_b200 import _lib
from buddy_mlir_b200.session import run_generation

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


# ---- mechanisms alone -------------------------------------------------------------------------
ATTENTION = [
    dict(),                                                                    # no window
    dict(window=1),                                                            # only itself
    dict(window=9),
    dict(heads=1, dim=32, rot=8, vdim=16, rank=16, window=5),
    dict(heads=17, dim=8, rot=4, vdim=4, rank=12, window=33),                  # more heads than one CTA takes
    dict(heads=2, dim=5, rot=6, vdim=7, rank=9, window=12),                    # nothing aligned
    dict(heads=2, dim=120, rot=72, vdim=128, rank=264, window=40, sharp=1.0),
    dict(heads=2, dim=200, rot=56, vdim=136, rank=520, window=30, sharp=1.0),  # two groups of value columns
    dict(heads=2, dim=260, rot=2, vdim=16, rank=24, window=8, sharp=1.0),      # wider than the expanded form takes
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kw", ATTENTION)
def test_attention_alone(kw, dtype):
    cfg = tz.config([(tz.attention(**kw), None)])
    w = tz.weights(cfg, 1)
    toks = tokens(cfg, 150)
    want = tz.want_logits(cfg, w, toks)
    s = tz.session(cfg, w, dtype)
    assert tz.error(s.prefill_rows(toks, 0), want) < tz.TOLERANCE[dtype]
    s.reset_position()
    for i, t in enumerate(toks[:45]):
        s.decode(int(t))
        assert tz.error(s.logits_data(), want[i]) < tz.TOLERANCE[dtype], i
    s.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("ff", [tz.gated(), tz.gated(ff=1, limit=0.5), tz.gated(ff=333, limit=7.0),
                                tz.experts(), tz.experts(n=1, top=1), tz.experts(n=4, top=4, ff=1), tz.experts(n=40, top=1, ff=33),
                                tz.experts(n=9, top=6, ff=130, limit=0.7)])
def test_feed_forward_alone(ff, dtype):
    cfg = tz.config([(tz.attention(heads=1, dim=2, rot=2, vdim=2, rank=2), ff)], width=100)
    w = tz.weights(cfg, 2)
    w["l0.mix.o"][:] = 0                     # the attention contributes nothing
    toks = tokens(cfg, 70)
    want = tz.want_logits(cfg, w, toks)
    s = tz.session(cfg, w, dtype)
    assert tz.error(s.prefill_rows(toks, 0), want) < tz.TOLERANCE[dtype]
    s.reset_position()
    assert tz.error(s.prefill_rows(toks[:5], 0), want[:5]) < tz.TOLERANCE[dtype]
    s.reset_position()
    s.decode(int(toks[0]))
    assert tz.error(s.logits_data(), want[0]) < tz.TOLERANCE[dtype]
    s.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_shared_cache_has_its_own_heads_and_window(dtype):
    m = dict(rank=32, rot=8, base=300.0)
    cfg = tz.config([(tz.attention(window=4, **m), None), (tz.attention(window=6, **m), None),
                     (tz.attention(heads=2, dim=50, vdim=10, window=25, kv_from=0, sharp=3.0, **m), None),
                     (tz.attention(heads=7, dim=6, vdim=30, window=2, kv_from=1, **m), None),
                     (tz.attention(kv_from=0, sharp=3.0, **m), None)])
    w = tz.weights(cfg, 3)
    toks = tokens(cfg, 90)
    want = tz.want_logits(cfg, w, toks)
    s = tz.session(cfg, w, dtype)
    assert tz.error(s.prefill_rows(toks, 0), want) < tz.TOLERANCE[dtype]
    b = tz.batch(s)
    got = step_logits(b, b.add(), toks, [60] + [1] * 30)
    assert tz.error(got, want) < tz.TOLERANCE[dtype]
    b.close()
    s.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_odd_sizes_everywhere(dtype):
    cfg = tz.config([(tz.attention(heads=3, dim=7, rot=2, vdim=5, rank=11, window=13), tz.gated(ff=13)),
                     (tz.attention(heads=1, dim=9, rot=6, vdim=3, rank=21, window=4), tz.experts(n=3, top=1, ff=7)),
                     (tz.attention(heads=5, dim=3, rot=2, vdim=1, rank=11, kv_from=0, window=50), tz.experts(n=3, top=3, ff=9))],
                    width=75, vocab=131)
    w = tz.weights(cfg, 14)
    toks = tokens(cfg, 80, 1)
    want = tz.want_logits(cfg, w, toks)
    s = tz.session(cfg, w, dtype)
    assert tz.error(s.prefill_rows(toks, 0), want) < tz.TOLERANCE[dtype]
    b = tz.batch(s)
    assert tz.error(step_logits(b, b.add(), toks, [40, 1, 1, 10, 3, 25]), want) < tz.TOLERANCE[dtype]
    b.close()
    s.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_wide_projections(dtype):
    """Large enough for every form of the contractions: 256-column tiles, a split k range, activations
    staged in several pieces, grouped tiles of many experts."""
    cfg = tz.config([(tz.attention(heads=6, dim=64, rot=32, vdim=64, rank=128, window=90, sharp=1.0), tz.gated(ff=4100)),
                     (tz.attention(heads=6, dim=64, rot=32, vdim=64, rank=128, window=300, sharp=1.0), tz.experts(n=40, top=2, ff=520))],
                    width=1032, vocab=1000)
    w = tz.weights(cfg, 15)
    toks = tokens(cfg, 600, 1)
    margins = []
    want = plain.forward(cfg, tz.values(w), toks, margins=margins)
    clear = margins[0] > 0.03                # a close call of the router may fall either way in bfloat16
    assert clear.mean() > 0.8
    s = tz.session(cfg, w, dtype, max_len=640)
    got = s.prefill_rows(toks, 0)
    assert tz.error(got[clear], want[clear]) < tz.TOLERANCE[dtype]
    s.reset_position()
    s.prefill_rows(toks[:500], 0)
    part = s.prefill_rows(toks[500:530], 500)
    assert tz.error(part[clear[500:530]], want[500:530][clear[500:530]]) < tz.TOLERANCE[dtype]
    for i in range(530, 538):
        s.decode(int(toks[i]))
        if clear[i]:
            assert tz.error(s.logits_data(), want[i]) < tz.TOLERANCE[dtype]
    s.close()


# ---- the whole model under schedules -----------------------------------------------------------
@pytest.fixture(scope="module", params=DTYPES)
def mixed(request):
    cfg, w = tz.mixed_model()
    s = tz.session(cfg, w, request.param)
    toks = tokens(cfg, 200, 7)
    yield cfg, w, s, toks, tz.want_logits(cfg, w, toks), tz.TOLERANCE[request.param]
    s.close()


@pytest.mark.parametrize("page", [1, 4, 16, 100])
@pytest.mark.parametrize("size", [2, 3, 8, 9, 16, 17, 50, 200])
def test_portions(mixed, size, page):
    cfg, w, s, toks, want, tol = mixed
    n = 60 if size < 8 else len(toks)
    b = tz.batch(s, page=page, pages=300)
    assert tz.error(step_logits(b, b.add(), toks[:n], cut(n, size)), want[:n]) < tol
    b.close()


def test_uneven_portions_and_single_tokens(mixed):
    cfg, w, s, toks, want, tol = mixed
    b = tz.batch(s)
    sizes = [1, 2, 40, 1, 1, 17, 3, 2, 30, 1, 60, 2]
    sizes += [1] * (len(toks) - sum(sizes))
    assert tz.error(step_logits(b, b.add(), toks, sizes), want) < tol
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
    assert tz.error(np.array(one), want[:90]) < tol
    assert tz.error(rows, np.array(one, dtype=np.float64)) < tol


def test_long_decoding(mixed):
    cfg, w, s, toks, want, tol = mixed
    s.reset_position()
    s.prefill_rows(toks[:3], 0)
    for i, t in enumerate(toks[3:], 3):
        s.decode(int(t))
        assert tz.error(s.logits_data(), want[i]) < tol, i


def test_a_prompt_longer_than_one_pass(mixed):
    """Thousands of rows go through the layers in several passes; the result is that of portions."""
    cfg, w, s, _, _, tol = mixed
    toks = tokens(cfg, 4500, 13)
    b = tz.batch(s, page=64, pages=160, context=5000)
    places = [0, 511, 512, 2999, 4095, 4096, 4097, 4499]
    whole, _ = b.step([(b.add(), toks)], [places])
    q = b.add()
    parts, at = [], 0
    for n in (1500, 7, 2500, 493):
        got, _ = b.step([(q, toks[at:at + n])], [[p - at for p in places if at <= p < at + n]], want_logits=True)
        parts.append(got)
        at += n
    assert tz.error(whole, np.concatenate(parts).astype(np.float64)) < tol
    b.close()


def test_first_tokens(mixed):
    cfg, w, s, toks, want, tol = mixed
    for n in (1, 2, 3, 10, 11, 12):
        s.reset_position()
        assert tz.error(s.prefill_rows(toks[:n], 0), want[:n]) < tol


def test_unequal_batch_against_each_alone(mixed):
    cfg, w, s, toks, _, tol = mixed
    rng = np.random.default_rng(11)
    seqs = [rng.integers(0, cfg["vocab"], n) for n in (75, 1, 33, 120, 18, 2)]
    wants = [tz.want_logits(cfg, w, t) for t in seqs]
    b = tz.batch(s, page=8)
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
            assert tz.error(got, np.array(expect)) < tol
            assert np.array_equal(nxt, got.argmax(axis=1))
    b.close()


def test_many_sequences_in_one_step(mixed):
    cfg, w, s, _, _, tol = mixed
    rng = np.random.default_rng(17)
    seqs = [rng.integers(0, cfg["vocab"], 5 + i % 4) for i in range(70)]
    b = tz.batch(s, max_seqs=70, page=4)
    ids = [b.add() for _ in seqs]
    b.step([(q, t[:-3]) for q, t in zip(ids, seqs)])
    got = [b.step([(q, t[k:k + 1] if k < -1 else t[-1:]) for q, t in zip(ids, seqs)])[0] for k in (-3, -2, -1)]
    compared = 0
    for i, t in enumerate(seqs):
        if tol < 1e-3 or tz.clear_of_close_calls(cfg, w, t)[-1]:
            compared += 1
            assert tz.error(np.array([g[i] for g in got]), tz.want_logits(cfg, w, t)[-3:]) < tol
    assert compared > 20
    b.close()


def test_freed_pages_and_slots_are_used_again(mixed):
    cfg, w, s, toks, want, tol = mixed
    b = tz.batch(s, max_seqs=2, page=4, pages=40, context=160)
    rng = np.random.default_rng(3)
    for k in range(6):
        other = b.add()
        b.step([(other, rng.integers(0, cfg["vocab"], 13 + 5 * k))])
        q = b.add()
        n = 70 + k
        got = step_logits(b, q, toks[:n], [n - 6, 2, 1, 1, 2])
        assert tz.error(got, want[:n]) < tol
        b.remove(other)
        b.remove(q)
        assert b.free_pages() == 40
    b.close()


def test_pages_behind_every_window_return_to_the_pool():
    cfg = tz.config([(tz.attention(window=9), tz.gated()), (tz.attention(window=14, kv_from=0), None)])
    w = tz.weights(cfg, 8)
    toks = tokens(cfg, 120, 5)
    want = tz.want_logits(cfg, w, toks)
    s = tz.session(cfg, w, "float32")
    b = tz.batch(s, max_seqs=3, page=4, pages=12, context=400)   # far fewer pages than the sequence is long
    q = b.add()
    got = step_logits(b, q, toks, [30] + [1] * 50 + [5] * 8)
    assert tz.error(got, want) < tz.TOLERANCE["float32"]
    assert b.free_pages() >= 12 - 5
    b.remove(q)
    assert b.free_pages() == 12
    b.close()
    s.close()


def test_a_step_that_does_not_fit_changes_nothing():
    cfg = tz.config([(tz.attention(), None)])
    w = tz.weights(cfg, 8)
    s = tz.session(cfg, w, "float32")
    toks = tokens(cfg, 20)
    want = tz.want_logits(cfg, w, toks)
    b = tz.batch(s, max_seqs=2, page=4, pages=5, context=20)
    q, r = b.add(), b.add()
    b.step([(q, toks[:8])])
    with pytest.raises(_lib.B200Error):
        b.step([(r, toks[:4]), (q, toks[:12])])
    assert b.free_pages() == 3 and b.length(q) == 8 and b.length(r) == 0
    got, _ = b.step([(q, toks[8:])], [list(range(12))])
    assert tz.error(got, want[8:]) < tz.TOLERANCE["float32"]
    b.close()
    s.close()


# ---- window edges: a token just inside changes the logits, one just outside leaves every bit ------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [1, 2, 8, 9, 64, 65])
def test_window_edge_in_prompt_portions_and_decoding(window, dtype):
    cfg = tz.config([(tz.attention(window=window, sharp=1.0), None)])
    w = tz.weights(cfg, 4)
    s = tz.session(cfg, w, dtype)
    n = 140
    base = tokens(cfg, n, 9)
    for sizes in ([n], [100] + [1] * 40, cut(n, 9), cut(n, 3)):
        if sizes[0] == 3 and window not in (8, 9):
            continue
        b = tz.batch(s, page=8)
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
            assert not changed[:j].any()
            assert changed[j:min(n, j + window)].all()
            assert not changed[j + window:].any()
        b.close()
    s.close()


def planted_key(cfg, at, query):
    """Tokens where the query's token is matched by one key token at position `at` and by nothing
    else: q and k are made to agree on one direction that only those two tokens carry."""
    rng = np.random.default_rng(12)
    toks = rng.integers(2, cfg["vocab"], query + 1)
    toks[at], toks[query] = 0, 1
    return toks


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_far_key_among_hundreds(dtype):
    cfg = tz.config([(tz.attention(heads=2, dim=24, rot=8, vdim=20, rank=40, sharp=1.0), None)], width=80)
    w = tz.values(tz.weights(cfg, 6))
    # token 0 carries feature 0, token 1 feature 1; the latent keeps feature 0, head 0's key is that
    # latent element and its query answers feature 1 on the same element with a large factor
    e = w["embed"]
    e[:, :2] = 0
    e[0, 0] = e[1, 1] = 6.0
    w["l0.mix.q"][:, :2] = 0
    w["l0.mix.q"][0, 1] = 40.0
    w["l0.mix.dkv"][:, :2] = 0
    w["l0.mix.dkv"][0, :] = 0
    w["l0.mix.dkv"][0, 0] = 3.0
    w["l0.mix.uk"][0, :] = 0
    w["l0.mix.uk"][0, 0] = 3.0
    w = {k: tz.to_bf16(v) for k, v in w.items()}
    s = tz.session(cfg, w, dtype, max_len=512)
    for at, query in ((0, 400), (3, 260), (255, 511), (256, 300)):
        toks = planted_key(cfg, at, query)
        want = tz.want_logits(cfg, w, toks)
        plain_toks = toks.copy()
        plain_toks[at] = 2
        assert tz.error(tz.want_logits(cfg, w, plain_toks)[-1], want[-1]) > 5 * tz.TOLERANCE[dtype]
        s.reset_position()
        assert tz.error(s.prefill_rows(toks, 0)[-1], want[-1]) < tz.TOLERANCE[dtype]
        b = tz.batch(s, page=16, context=512)
        got = step_logits(b, b.add(), toks, [query - 20, 19, 1, 1])
        assert tz.error(got[-1], want[-1]) < tz.TOLERANCE[dtype]
        b.close()
    s.close()


# ---- generation -----------------------------------------------------------------------------------
def plain_greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(tz.want_logits(cfg, w, toks)[-1])))
    return toks[len(prompt):]


def test_greedy_generation_and_device_loop():
    cfg, w = tz.mixed_model(21)
    s = tz.session(cfg, w, "float32")
    prompt = [int(t) for t in tokens(cfg, 24, 1)]
    want = plain_greedy(cfg, w, prompt, 40)
    ids, _ = run_generation(s, prompt, len(prompt) + 39)
    assert ids == want
    s.prefill(prompt)
    first = int(np.argmax(s.logits_data()))
    assert [first] + s.generate(first, 39).tolist() == want
    assert s.decode_greedy(want[-1]) == plain_greedy(cfg, w, prompt + want, 1)[0]
    s.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_full_cache_drops_positions_and_turns_keys_back(dtype):
    """One layer: its cached rows depend on nothing but token and position, so after the overflow
    the session must continue like a fresh sequence of the tokens that were kept."""
    cfg = tz.config([(tz.attention(window=30), tz.gated())])
    w = tz.weights(cfg, 31)
    s = tz.session(cfg, w, dtype, max_len=48)
    toks = tokens(cfg, 48, 3)
    s.prefill_rows(toks, 0)
    assert not tz.session(cfg, w, dtype, max_len=60).handle_kv_cache_overflow(4)
    assert s.handle_kv_cache_overflow(10)
    kept = np.concatenate([toks[:10], toks[29:]])
    assert s.position() == len(kept)
    for t in (5, 6, 7):
        kept = np.append(kept, t)
        s.decode(t)
        assert tz.error(s.logits_data(), tz.want_logits(cfg, w, kept)[-1]) < tz.TOLERANCE[dtype]
    ids, _ = run_generation(s, [int(t) for t in toks[:40]], 40 + 30)   # runs past the cache's end
    assert len(ids) == 31
    s.close()


def test_batched_greedy_generation():
    cfg, w = tz.mixed_model(22)
    s = tz.session(cfg, w, "float32")
    b = tz.batch(s, max_seqs=12, page=4)
    prompts = [[int(t) for t in tokens(cfg, n, 30 + n)] for n in (5, 1, 40, 17, 9, 3, 21, 2, 11, 6)]
    ids = [b.add() for _ in prompts]
    _, nxt = b.step(list(zip(ids, prompts)), want_logits=False)
    out = [[int(t)] for t in nxt]
    for _ in range(11):
        _, nxt = b.decode(ids, [o[-1] for o in out], want_logits=False)
        for o, t in zip(out, nxt):
            o.append(int(t))
    for p, o in zip(prompts, out):
        assert o == plain_greedy(cfg, w, p, 12)
    b.close()
    s.close()


def test_command_line_generates_and_replays(tmp_path):
    import json
    cfg, w = tz.mixed_model(23)
    model = tmp_path / "model"
    model.mkdir()
    tz.write_folder(str(model), cfg, w)
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
    a, b = tz.want_logits(cfg, w, prompt + [3, 4, 5]), tz.want_logits(cfg, w, [1, 2])
    for name, rows in (("0", [a[8], a[0]]), ("1", [b[1]]), ("2", [a[10]])):
        got = np.fromfile(tmp_path / f"{name}.f32", dtype="<f4").reshape(len(rows), -1)
        assert tz.error(got, np.array(rows)) < tz.TOLERANCE["float32"]


def test_wrong_tensors_and_layers_are_refused():
    cfg = tz.config([(tz.attention(), None), (tz.attention(kv_from=0), None)])
    w = tz.weights(cfg, 1)
    from buddy_mlir_b200 import talazen
    from buddy_mlir_b200.session import ModelSession
    s = ModelSession(talazen.parse(cfg, "float32", 16))
    with pytest.raises(_lib.B200Error, match="no tensor"):
        s.load_named({"l1.mix.dkv": w["l0.mix.dkv"]})
    with pytest.raises(_lib.B200Error, match="got"):
        s.load_named({"embed": w["embed"][:-1]})
    with pytest.raises(_lib.B200Error, match="missing"):
        s.load_named({"embed": w["embed"]})
    s.close()
    bad = tz.config([(tz.attention(), None), (tz.attention(kv_from=0, rank=48), None)])
    with pytest.raises(_lib.B200Error, match="differ"):
        ModelSession(talazen.parse(bad, "float32", 16))
    bad = tz.config([(tz.attention(), tz.experts(n=2, top=3))])
    with pytest.raises(_lib.B200Error, match="experts"):
        ModelSession(talazen.parse(bad, "float32", 16))
