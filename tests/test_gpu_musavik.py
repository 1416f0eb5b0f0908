"""Musavik on the GPU against the plain restatement (oracle/musavik.py): each mechanism alone, prompts, decoding through the
caches and states, portions of prompts, mixed batches, reuse of pages and lanes, window and kept-key edges, far keys, sampling
and greedy generation, in f32 and bf16 and with each implementation of the mixers."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import musavik_cases as K
from oracle import musavik as G

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {"float32": 2e-5, "bfloat16": 3e-2}
OPTIONS = ("gqa_attention", "linear_attention", "short_conv")
IMPLS = {"auto": ("auto", "auto", "auto"), "plain": ("plain", "plain", "plain"), "small": ("paged", "recurrent", "auto")}


@pytest.fixture(scope="module")
def rb():
    from rew_b200 import _lib, api
    _lib.init()
    return api


@pytest.fixture(params=["float32", "bfloat16"])
def dtype(request):
    return request.param


@pytest.fixture(params=list(IMPLS))
def impl(request, rb):
    for o, v in zip(OPTIONS, IMPLS[request.param]):
        rb.set_option(o, v)
    yield request.param
    for o in OPTIONS:
        rb.set_option(o, "auto")


def build(rb, cfg, t, dtype, max_seq=2048):
    from rew_b200 import models, musavik
    c = musavik.config_from_json(cfg, dtype=models.DTYPES[dtype], max_seq=max_seq)
    return rb.CausalLM(c).load(c.canonical_tensors(t))


def row_errors(got, want):
    """rms of every row's difference over the rms of all wanted values."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    assert got.shape == want.shape and np.isfinite(got).all()
    return np.sqrt(((got - want) ** 2).mean(-1)) / max(np.sqrt((want ** 2).mean()), 1e-30)


def err(got, want):
    return float(np.sqrt((row_errors(got, want) ** 2).mean()))


def close(got, want, dtype):
    """All rows together within the tolerance, and no row far above it (16-bit rounding can move a sharp softmax at one
    position)."""
    e = row_errors(got, want)
    assert np.sqrt((e ** 2).mean()) <= TOL[dtype] and e.max() <= 2.5 * TOL[dtype], (np.sqrt((e ** 2).mean()), e.max())


def feed_all(sess, lane, ids, cuts):
    """Logits of every position of one request, fed in portions of the given sizes (the last repeats)."""
    out, at, i = [], 0, 0
    while at < len(ids):
        n = min(cuts[min(i, len(cuts) - 1)], len(ids) - at)
        lg, _ = sess.feed([(lane, ids[at:at + n])], want=range(n))
        out.append(lg)
        at, i = at + n, i + 1
    return np.concatenate(out)


def silence(t, *suffixes):
    return {k: np.zeros_like(v) if k.endswith(suffixes) else v for k, v in t.items()}


# ---------------------------------------------------------------- each mechanism alone

@pytest.mark.parametrize("what", ["all", "attention", "delta", "lru", "dense", "norms", "embedding"])
def test_residual_after_every_layer_run(rb, dtype, what):
    cfg = K.small()
    t = K.weights(cfg, seed=2, score_gain=2.0)
    outs = {"attention": "left.o", "delta": "right.o", "lru": "mix.o"}
    if what in outs:
        t = silence(t, ".down", ".down.b", *[o for k, o in outs.items() if k != what])
    elif what == "dense":
        t = silence(t, *outs.values())
    elif what == "embedding":
        t = silence(t, ".down", ".down.b", *outs.values())
    elif what == "norms":     # an eps that matters in every norm
        cfg["norm"]["eps"] = 0.3
    ids = K.tokens(cfg, 90, seed=2)
    want = []
    logits = G.forward(cfg, t, ids, want)
    rb.set_option("record_layers", "1")
    try:
        sess = build(rb, cfg, t, dtype).paged_session(2, 128, 5)
        got, _ = sess.feed([(1, ids)], want=range(len(ids)))
        layers = sess.layers(len(ids))
    finally:
        rb.set_option("record_layers", "0")
    close(got, logits, dtype)
    assert len(layers) == len(want) == 9
    for i, w in enumerate(want):
        close(layers[i], w, dtype)


P, R = K.parallel, K.rglru
SIZES = [
    ([P(heads=1, kv_heads=1, dim=8, vdim=8, rot=2, base=10.0, size=1, keep=1, right=(1, 1, 8, 8, 1)), R(width=8, blocks=1, conv=1)], 40, 33, 150),
    ([P(heads=8, kv_heads=8, dim=16, vdim=16, rot=16, size=200, keep=64, right=(4, 4, 32, 32, 2)), R(width=128, blocks=4, conv=2)], 96, 64, 200),
    ([P(heads=8, kv_heads=2, dim=128, vdim=128, rot=128, base=1e6, size=96, keep=65, right=(4, 4, 128, 128, 4)), R(width=512, blocks=2, conv=4)], 128, 96, 300),
    ([P(heads=33, kv_heads=1, dim=24, vdim=8, rot=12, size=65, keep=3, right=(6, 2, 24, 8, 3)), R(width=136, blocks=17, conv=3)], 136, 72, 150),    # a group above 16; 33 heads
    ([P(heads=6, kv_heads=3, dim=13, vdim=19, rot=10, size=50, keep=21, right=(2, 2, 13, 19, 7)), R(width=63, blocks=7, conv=5)], 61, 101, 120),    # nothing divides by 8
    ([P(heads=4, kv_heads=2, dim=192, vdim=72, rot=64, size=3, keep=100, right=(2, 1, 72, 136, 5)), R(width=88, blocks=2, conv=9)], 88, 50, 150),   # long convolutions, states above the chunk kernel
    ([P(heads=2, kv_heads=2, dim=256, vdim=256, rot=252, size=64, keep=7, right=(1, 1, 256, 256, 2)), R(width=40, blocks=1, conv=8)], 64, 40, 100),
    ([P(heads=40, kv_heads=2, dim=64, vdim=64, rot=64, scale=0.3, size=128, keep=128, right=(5, 5, 64, 64, 6)), R(width=320, blocks=10, conv=6)], 112, 70, 330),
    ([P(heads=3, kv_heads=1, dim=300, vdim=40, rot=44, size=129, keep=0, right=(3, 3, 40, 300, 3)), R(width=60, blocks=5, conv=3)], 80, 48, 130),
    ([P(heads=10, kv_heads=2, dim=72, vdim=136, rot=6, size=70, keep=60, right=(2, 2, 120, 104, 12)), R(width=216, blocks=3, conv=12)], 72, 56, 280),
    ([P(heads=16, kv_heads=16, dim=32, vdim=48, rot=32, size=256, keep=2, right=(3, 1, 48, 48, 4)), R(width=96, blocks=12, conv=4)], 64, 40, 300),
]


@pytest.mark.parametrize("i", range(len(SIZES)))
def test_other_sizes(rb, dtype, i):
    layers, width, vocab, n = SIZES[i]
    cfg = K.config([dict(layers[i % 2], mlp=K.dense(13)), dict(layers[1 - i % 2], mlp=K.dense(30 + i))], vocab=vocab, width=width, bigram=(1 + 6 * i, 3 + i, 100003),
                   scale=[1.0, 3.0, 0.2][i % 3], loop=[None, dict(start=0, stop=1, times=1), dict(start=0, stop=2, times=2), dict(start=1, stop=2, times=3)][i % 4])
    t = K.weights(cfg, seed=i, score_gain=1.5)
    ids = K.tokens(cfg, n, seed=i)
    want = G.forward(cfg, t, ids)
    sess = build(rb, cfg, t, dtype).paged_session(1, 448, 8)
    close(feed_all(sess, 0, ids, [n]), want, dtype)
    sess.release(0)
    close(feed_all(sess, 0, ids, [80, 1, 1, 3, 2, 33, 1]), want, dtype)


@pytest.mark.parametrize("seed", range(4))
def test_values_are_normed_keys_rotated_and_heads_mixed(rb, dtype, seed):
    """Values of very unequal sizes, biases that outweigh the projections, heads that take all their weights from one another."""
    cfg = K.config([P(heads=4, kv_heads=2, size=40, keep=9)])
    t = {k: v.copy() for k, v in K.weights(cfg, seed=seed, score_gain=2.0).items()}
    t["l0.mix.right.o"][:] = 0.0
    y = "l0.mix.left."
    t[y + "v"] *= np.float32(100.0 if seed % 2 else 0.01)
    t[y + "v.b"] *= np.float32(100.0 if seed % 2 else 0.01)
    for n in "qk":
        t[y + n + ".b"] *= 4.0
    t[y + "talk"] = np.roll(np.eye(4, dtype=np.float32), seed, axis=1) * np.float32(1.5)
    ids = K.tokens(cfg, 130, seed=seed)
    want = G.forward(cfg, t, ids)
    sess = build(rb, cfg, t, dtype).paged_session(1, 192, 4)
    for cuts in ([130], [1], [20, 2, 64]):
        close(feed_all(sess, 0, ids, cuts), want, dtype)
        sess.release(0)


# ---------------------------------------------------------------- cuts, batches, pages

@pytest.mark.parametrize("cuts", [[300], [2], [1], [7, 2, 31], [3], [64], [33, 31], [63, 2, 65], [130, 1, 129, 1], [100, 160], [32], [40, 2, 90]])
def test_portions_agree_with_the_whole_prompt(rb, dtype, cuts, impl):
    cfg = K.small()
    t = K.weights(cfg, seed=3, score_gain=1.5)
    ids = K.tokens(cfg, 260, seed=3)
    sess = build(rb, cfg, t, dtype).paged_session(2, 320, 6)
    close(feed_all(sess, 1, ids, cuts), G.forward(cfg, t, ids), dtype)


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 9])
def test_convolutions_reach_back_over_every_cut(rb, dtype, taps):
    """Only the oldest tap weighs anything: every convolved value is that of taps - 1 tokens ago, whatever step that was in."""
    cfg = K.config([K.parallel(right=(3, 3, 16, 24, taps)), K.rglru(conv=taps + 1), K.rglru(width=60, blocks=4, conv=taps)])
    t = {k: v.copy() for k, v in K.weights(cfg, seed=taps, score_gain=1.5).items()}
    for k in t:
        if k.endswith(".conv"):
            t[k][:, 1:] = 0.0
            t[k][:, 0] = 1.0
    ids = K.tokens(cfg, 75, seed=taps)
    want = G.forward(cfg, t, ids)
    sess = build(rb, cfg, t, dtype).paged_session(2, 128, 4)
    for i, cuts in enumerate(([75], [1], [2], [3], [taps], [64, 1, 2], [2, 1, 5, 1, 1, 8])):
        close(feed_all(sess, i % 2, ids, cuts), want, dtype)
        sess.release(i % 2)


@pytest.mark.parametrize("forget", [-9.0, 4.0])
def test_states_that_last_and_states_that_fade(rb, dtype, forget, impl):
    """Decays near one (the first tokens still count at the end) and near zero (exponents far from zero inside a chunk)."""
    cfg = K.config([K.parallel(right=(4, 2, 32, 40, 3), size=8, keep=0), K.rglru()])
    t = {k: v.copy() for k, v in K.weights(cfg, seed=21, forget=forget).items()}
    t["l0.mix.left.o"][:] = 0.0
    if forget > 0:
        t["l0.mix.right.A_log"] += 4.0
    ids = K.tokens(cfg, 400, seed=21)
    want = G.forward(cfg, t, ids)
    if forget < 0:
        other = ids.copy()
        other[:3] = (other[:3] + 5) % cfg["vocab"]
        assert err(G.forward(cfg, t, other)[-1:], want[-1:]) > 1e-3
    sess = build(rb, cfg, t, dtype).paged_session(1, 448, 8)
    for cuts in ([400], [37, 1, 2, 64, 31], [390, 1]):
        close(feed_all(sess, 0, ids, cuts), want, dtype)
        sess.release(0)


def test_mixed_batches_against_each_request_alone(rb, dtype):
    """Portions of some requests beside single tokens of others, requests left out of a step, lanes and pages used again."""
    cfg = K.small()
    t = K.weights(cfg, seed=5, score_gain=1.5)
    rng = np.random.default_rng(5)
    reqs = [K.tokens(cfg, n, seed=50 + n) for n in (150, 3, 90, 64, 33, 200, 65, 1, 2)]
    want = [G.forward(cfg, t, r) for r in reqs]
    sess = build(rb, cfg, t, dtype).paged_session(3, 256, 9)
    got, at = [[] for _ in reqs], [0] * len(reqs)
    queue, live = list(range(len(reqs))), {}
    while queue or live:
        for lane in range(3):
            if lane not in live and queue and sess.free_blocks() >= (len(reqs[queue[0]]) + 63) // 64:
                live[lane] = queue.pop(0)
        fits, need = [], 0
        for lane, r in live.items():
            if len(live) > 1 and rng.random() < 0.2:
                continue
            n = min(len(reqs[r]) - at[r], int(rng.choice([1, 1, 2, 5, 31, 32, 40, 70, 128])))
            grow = (at[r] + n + 63) // 64 - (at[r] + 63) // 64      # a lane that cannot grow waits
            if need + grow <= sess.free_blocks():
                need += grow
                fits.append((lane, r, n))
        if not fits:
            continue
        rows = sum(n for _, _, n in fits)
        lg, _ = sess.feed([(lane, reqs[r][at[r]:at[r] + n]) for lane, r, n in fits], want=range(rows))
        row = 0
        for lane, r, n in fits:
            got[r].append(lg[row:row + n])
            at[r] += n
            row += n
            if at[r] == len(reqs[r]):
                sess.release(lane)
                del live[lane]
    for r in range(len(reqs)):
        close(np.concatenate(got[r]), want[r], dtype)


def test_freed_pages_and_states_hold_nothing_over(rb):
    """A request on pages and a lane that others used gives the same bits as on a fresh session."""
    cfg = K.small()
    t = K.weights(cfg, seed=6, score_gain=2.0)
    model = build(rb, cfg, t, "bfloat16")
    ids = K.tokens(cfg, 120, seed=6)
    first = feed_all(model.paged_session(1, 128, 3), 0, ids, [1, 50, 1, 68])
    sess = model.paged_session(3, 128, 6)
    for i in range(4):
        feed_all(sess, i % 3, K.tokens(cfg, 60 + i, seed=40 + i), [61])
        if i >= 1:
            sess.release((i - 1) % 3)
    sess.step(2)
    sess.release(0)
    assert np.array_equal(feed_all(sess, 2 if sess.lane_length(2) < 0 else 0, ids, [1, 50, 1, 68]), first)


def test_the_last_token_belongs_to_its_lane(rb, dtype):
    """Bigram rows across steps that interleave lanes, and after a lane was given to another request."""
    cfg = K.config([K.rglru(None, width=16, blocks=1, conv=1)], bigram=(1009, 29, 13))
    t = {k: v.copy() for k, v in K.weights(cfg, seed=16).items()}
    t["bigram"] *= 4.0
    t["l0.mix.o"][:] = 0.0
    sess = build(rb, cfg, t, dtype).paged_session(3, 64, 4)
    a, b, c = (K.tokens(cfg, 20, seed=s) for s in (1, 2, 3))
    want = {n: G.forward(cfg, t, r) for n, r in (("a", a), ("b", b), ("c", c))}
    lg, _ = sess.feed([(0, a[:5]), (2, b[:1])], want=range(6))
    close(lg, np.concatenate([want["a"][:5], want["b"][:1]]), dtype)
    lg, _ = sess.feed([(2, b[1:2]), (0, a[5:7])], want=range(3))
    close(lg, np.concatenate([want["b"][1:2], want["a"][5:7]]), dtype)
    sess.release(0)
    lg, _ = sess.feed([(0, c[:2]), (2, b[2:20])], want=range(20))
    close(lg, np.concatenate([want["c"][:2], want["b"][2:]]), dtype)
    close(sess.feed([(0, c[2:])], want=range(18))[0], want["c"][2:], dtype)


def test_errors_change_nothing(rb):
    from rew_b200._lib import RewB200Error
    from rew_b200 import musavik
    cfg = K.small()
    sess = build(rb, cfg, K.weights(cfg), "float32").paged_session(2, 128, 3)
    for bad in ([(0, [1] * 129)], [(0, [])], [(0, [1]), (0, [2])], [(2, [1])], [(0, [cfg["vocab"]])], [(0, [1] * 128), (1, [1])]):
        with pytest.raises(RewB200Error):
            sess.feed(bad)
    assert sess.free_blocks() == 2 and sess.lane_length(0) == -1
    for side, change in (("left", dict(kv_heads=3)), ("left", dict(rot=dict(base=10.0, dims=26))), ("left", dict(rot=dict(base=10.0, dims=5))),
                         ("left", dict(mask=dict(size=0, keep_first=3))), ("right", dict(kv_heads=2)), ("right", dict(conv=0))):
        bad = K.small()
        bad["layers"][1]["mixer"][side].update(change)
        with pytest.raises(RewB200Error):
            rb.CausalLM(musavik.config_from_json(bad))
    with pytest.raises(RewB200Error):
        rb.CausalLM(musavik.config_from_json(K.small(loop=dict(start=4, stop=7, times=2))))


# ---------------------------------------------------------------- keys at every distance

@pytest.mark.parametrize("window", [1, 2, 50, 63, 64, 65, 128, 129, 200])
def test_keys_just_inside_and_outside_the_window(rb, dtype, window, impl):
    cfg, t, filler, key, query = K.marked(K.parallel(None, heads=4, kv_heads=2, dim=24, vdim=16, rot=8, size=window, keep=2))
    sess = build(rb, cfg, t, dtype).paged_session(2, 512, 10)
    for q_pos in (window + 3, 63 + window, 64 + window, 191, 320):
        seqs = {}
        for dist in (window - 1, window):           # the oldest key that is seen, and the first that is not
            if q_pos - dist < 2:
                continue
            ids = np.full(q_pos + 1, filler, np.int32)
            ids[q_pos - dist] = key
            ids[q_pos] = query
            seqs[dist] = ids
        want = {k: G.forward(cfg, t, v)[-1:] for k, v in seqs.items()}
        if len(want) == 2 and window > 1:
            assert err(want[window - 1], want[window]) > 5 * TOL["bfloat16"]     # a shifted edge would show
        for dist, ids in seqs.items():
            for cuts in ([q_pos + 1], [q_pos, 1], [max(1, q_pos - 2), 3], [max(1, q_pos - dist), 2, 70]):
                close(feed_all(sess, 0, ids, cuts)[-1:], want[dist], dtype)
                sess.release(0)


@pytest.mark.parametrize("keep", [0, 1, 20, 63, 64, 65, 130])
def test_first_keys_are_kept(rb, dtype, keep, impl):
    """The last kept key and the next one, from queries far behind them and from queries whose window touches them."""
    size = 40
    cfg, t, filler, key, query = K.marked(K.parallel(None, heads=6, kv_heads=2, dim=24, vdim=16, rot=8, size=size, keep=keep))
    sess = build(rb, cfg, t, dtype).paged_session(1, 512, 9)
    for q_pos in (keep + size - 1, keep + size, keep + size + 1, keep + 64, 300):
        seqs = {}
        for where in (keep - 1, keep):
            if where < 0:
                continue
            ids = np.full(q_pos + 1, filler, np.int32)
            ids[where] = key
            ids[q_pos] = query
            seqs[where] = ids
        want = {k: G.forward(cfg, t, v)[-1:] for k, v in seqs.items()}
        if len(want) == 2 and q_pos >= keep + size:
            assert err(want[keep - 1], want[keep]) > 5 * TOL["bfloat16"]
        for where, ids in seqs.items():
            for cuts in ([q_pos + 1], [q_pos, 1], [max(1, q_pos - 2), 3], [where + 1, 2, 70]):
                close(feed_all(sess, 0, ids, cuts)[-1:], want[where], dtype)
                sess.release(0)


def test_far_keys_and_page_borders(rb, dtype, impl):
    """A marked key at the first token and around every page border of a long context, found by prompts and by decoding."""
    cfg, t, filler, key, query = K.marked(K.parallel(None, heads=4, kv_heads=2, dim=24, vdim=24, rot=8, size=660, keep=3))
    sess = build(rb, cfg, t, dtype).paged_session(1, 1024, 17)
    base = np.full(700, filler, np.int32)
    base[-1] = query
    none = G.forward(cfg, t, base)[-1:]
    for where in (0, 1, 2, 40, 62, 63, 64, 65, 127, 128, 383, 384, 640, 697, 698):
        ids = base.copy()
        ids[where] = key
        want = G.forward(cfg, t, ids)[-1:]
        assert err(want, none) > 5 * TOL["bfloat16"]
        for cuts in ([700], [699, 1], [350, 300, 50]):
            got, at = None, 0
            for n in cuts:
                got, _ = sess.feed([(0, ids[at:at + n])], want=[n - 1])
                at += n
            close(got, want, dtype)
            sess.release(0)


@pytest.mark.parametrize("dim,vdim,heads,kv,size,keep", [(64, 64, 8, 2, 300, 90), (128, 128, 4, 1, 129, 0), (128, 128, 16, 4, 500, 64), (96, 120, 6, 6, 257, 130),
                                                        (64, 128, 3, 1, 1000, 1)])
def test_long_prompts(rb, dtype, dim, vdim, heads, kv, size, keep):
    """Windows across many tiles of queries and keys, with kept keys inside and outside the window's first tile."""
    cfg = K.config([P(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, rot=dim // 2, size=size, keep=keep, right=(2, 2, 32, 32, 3))])
    t = K.weights(cfg, seed=dim + size, score_gain=2.0)
    ids = K.tokens(cfg, 900, seed=size)
    want = G.forward(cfg, t, ids)
    sess = build(rb, cfg, t, dtype).paged_session(2, 960, 31)
    close(feed_all(sess, 0, ids, [900]), want, dtype)
    close(feed_all(sess, 1, ids, [200, 3, 500, 1, 196]), want, dtype)
    # two portions in one step, one of them inside a page
    sess.release(0)
    sess.release(1)
    sess.feed([(0, ids[:333]), (1, ids[:90])])
    lg, _ = sess.feed([(1, ids[90:400]), (0, ids[333:900])], want=range(877))
    close(lg, np.concatenate([want[90:400], want[333:900]]), dtype)


def test_rotation_at_far_positions(rb, dtype):
    """Fast and slow features a long way into the sequence, rotated whole and in part."""
    cfg = K.config([K.parallel(None, heads=2, kv_heads=1, dim=32, rot=32, base=10.0, size=300), K.parallel(None, heads=2, kv_heads=2, dim=24, rot=12, base=1e7, size=2000)])
    t = K.weights(cfg, seed=13, score_gain=1.5)
    ids = K.tokens(cfg, 1200, seed=13)
    want = G.forward(cfg, t, ids)[-130:]
    sess = build(rb, cfg, t, dtype).paged_session(1, 1216, 20)
    sess.feed([(0, ids[:1070])])
    got = [sess.feed([(0, ids[1070:1120])], want=range(50))[0]] + [sess.feed([(0, ids[i:i + 1])], want=[0])[0] for i in range(1120, 1130)] \
        + [sess.feed([(0, ids[1130:])], want=range(70))[0]]
    close(np.concatenate(got), want, dtype)


def test_long_decoding(rb, dtype):
    cfg = K.config([K.parallel(K.dense(), size=80, keep=10), K.rglru(K.dense())], loop=dict(start=0, stop=1, times=2))
    t = K.weights(cfg, seed=8, score_gain=1.5)
    ids = K.tokens(cfg, 300, seed=8)
    sess = build(rb, cfg, t, dtype).paged_session(1, 320, 6)
    close(feed_all(sess, 0, ids, [20, 1]), G.forward(cfg, t, ids), dtype)


# ---------------------------------------------------------------- the mechanisms in other designs

def other_design(block, seed, first, beside, dtype):
    """A layered model of one kind of block whose first layer has mixer `first`, with `beside` next to it."""
    from rew_b200 import models
    from rew_b200.layered import LayeredConfig, LayerSpec
    from rew_b200.weights import bf16_round
    kinds = {
        "attention": dict(mixer="attention", heads=4, kv_heads=2, dim=24, vdim=16, scale=0.2, window=33, keep_first=4, out_gate=True, qk_norm=False,
                          rope_base=60.0, rope_dims=8, rope_pairs=True, v_norm=True),
        "delta": dict(mixer="delta", heads=4, kv_heads=2, dim=24, vdim=16, conv_taps=3),
        "lru": dict(mixer="lru", heads=4, dim=16, vdim=16, conv_taps=4),
        "gla": dict(mixer="gla", heads=2, dim=24, vdim=16, decay_rank=5, tau=4.0),
    }
    second = LayerSpec(ff="none", mix_scale=0.5, **kinds[beside]) if beside else None
    layers = [LayerSpec(ff="dense", ffn=40, ff_act="gelu_tanh" if block != "output_norm" else "gated_silu", beside=second,
                        beside_names=("a.", "b.") if second else ("", ""), **kinds[first]),
              LayerSpec(ff="none", **kinds["attention"])]
    cfg = LayeredConfig(vocab=72, d_model=64, layers=layers, eps=1e-5, norm_zero_centred=False, block=block, own_head=True, max_seq=320, dtype=models.DTYPES[dtype])
    rng = np.random.default_rng(seed)
    t = {}
    for n, shape in cfg.tensor_specs():
        x = rng.normal(0, 1.2 if n == "embed" or n.endswith("conv") else shape[-1] ** -0.5 if n.endswith((".ra", ".ri")) else shape[0] ** -0.5 if len(shape) == 2 else 0.3, size=shape)
        if "norm" in n:
            x = 1 + 0.5 * x
        if n.endswith((".lam", ".A_log")):
            x = x - 2.0
        t[n] = bf16_round(x.astype(np.float32))
    return cfg, t


def other_mixer(spec, w, h):
    """One mixer of an other design, out of the oracles' functions; w(name) -> tensor with Linear weights [out, in]."""
    from oracle import girulorn as GG
    T, H, D, V = len(h), spec.heads, spec.dim, spec.vdim
    if spec.mixer == "delta":
        return G.delta_rule(h, dict(heads=H, kv_heads=spec.kv_heads, dim=D, vdim=V), w, 1e-5)
    if spec.mixer == "lru":
        return G.rglru(h, dict(width=H * D, blocks=H), w)
    if spec.mixer == "gla":
        return GG.gla(h, dict(heads=H, dim=D, vdim=V, tau=spec.tau), w, 1e-5)
    N = spec.kv_heads
    q, k = (G.rotated_pairs((h @ w(n).T).reshape(T, x, D), range(T), spec.rope_base, spec.rope_dims) for n, x in (("q", H), ("k", N)))
    v = G.rms_norm((h @ w("v").T).reshape(T, N, V), 1.0, 1e-5)
    gate, vis = G.sigmoid(h @ w("g").T), G.visible(T, spec.window, spec.keep_first)
    out = np.stack([G.softmax(q[:, a] @ k[:, a // (H // N)].T * spec.scale, vis) @ v[:, a // (H // N)] * gate[:, a:a + 1] for a in range(H)], 1)
    return out.reshape(T, H * V) @ w("o").T


@pytest.mark.parametrize("block,first,beside", [("parallel", "attention", None), ("parallel", "delta", None), ("parallel_one_norm", "lru", None),
                                                ("output_norm", "attention", "lru"), ("parallel_one_norm", "gla", "delta"), ("sandwich", "delta", "lru"),
                                                ("parallel", "lru", "delta")])
def test_mechanisms_in_other_blocks(rb, dtype, block, first, beside):
    """A window and kept keys without mixed heads, recurrences alone and beside other mixers, in every kind of block."""
    cfg, t = other_design(block, 3, first, beside, dtype)
    ids = np.random.default_rng(4).integers(0, 72, size=300).astype(np.int32)
    f = {k: v.astype(np.float64) for k, v in t.items()}
    norm = lambda x, n: G.rms_norm(x, f[n], 1e-5)
    x = f["embed"][ids]
    for i, spec in enumerate(cfg.layers):
        p = "l%d." % i

        def mix(h):
            y = 0.0
            for m, sub, scale in ((spec, spec.beside_names[0], 1.0), (spec.beside, spec.beside_names[1], 0.5)):
                if m is None:
                    continue
                raw = lambda n: f[p + "mix." + sub + n]
                def w(n):
                    a = raw(n)
                    if n in ("ra", "ri"):
                        return a.reshape(m.heads, m.dim, m.dim)
                    if n in ("ra.b", "ri.b"):
                        return a.reshape(m.heads, m.dim)
                    return a.T if a.ndim == 2 and not n.endswith("conv") else a
                y = y + scale * other_mixer(m, w, h)
            return y

        def ff(h):
            if spec.ff_act == "gelu_tanh":
                return G.gelu_tanh(h @ f[p + "mlp.up"]) @ f[p + "mlp.down"]
            return (G.silu(h @ f[p + "mlp.gate"]) * (h @ f[p + "mlp.up"])) @ f[p + "mlp.down"]

        has = spec.ff != "none"
        if block == "parallel":
            x = x + mix(norm(x, p + "norm1")) + (ff(norm(x, p + "norm2")) if has else 0.0)
        elif block == "parallel_one_norm":
            h = norm(x, p + "norm1")
            x = x + mix(h) + (ff(h) if has else 0.0)
        elif block == "output_norm":
            x = x + norm(mix(x), p + "norm1")
            x = x + norm(ff(x), p + "norm2") if has else x
        else:
            x = x + norm(mix(norm(x, p + "norm1")), p + "norm1b")
            x = x + norm(ff(norm(x, p + "norm2")), p + "norm2b") if has else x
    want = norm(x, "final.norm") @ f["head"]
    sess = rb.CausalLM(cfg).load([t[n] for n, _ in cfg.tensor_specs()]).paged_session(1, 320, 6)
    for cuts in ([300], [150, 1, 2, 70, 1], [3, 297]):
        close(feed_all(sess, 0, ids, cuts), want, dtype)
        sess.release(0)


# ---------------------------------------------------------------- generation

def test_greedy_generation_follows_the_oracle(rb):
    """Session.generate, the paged lanes with a captured decode step, and steps that mix prompts with decoding."""
    cfg = K.small()
    t = K.weights(cfg, seed=9, score_gain=1.5)
    model = build(rb, cfg, t, "float32")
    prompts = [K.tokens(cfg, n, seed=60 + n) for n in (5, 1, 70, 33)]
    want = []
    for p in prompts:
        ids, margin = G.generate_greedy(cfg, t, p, 12)
        assert margin > 1e-4
        want.append(ids)
    s = model.session(2, 64)
    same = np.stack([prompts[0], prompts[0][::-1]])
    got = s.generate(same, 12)
    assert got[0].tolist() == want[0] and got[1].tolist() == G.generate_greedy(cfg, t, prompts[0][::-1], 12)[0]
    assert s.generate(same[:1].repeat(2, 0), 12)[1].tolist() == want[0]        # a second call starts over
    ps = model.paged_session(3, 128, 7)
    out = {}
    queue, live = list(range(4)), {}
    while queue or live:
        for lane in range(3):
            if lane not in live and queue:
                r = queue.pop(0)
                live[lane] = r
                out[r] = [ps.admit(lane, prompts[r])]
        got = ps.step(3)
        for lane, r in list(live.items()):
            out[r] += got[lane].tolist()
            if len(out[r]) >= 12:
                ps.release(lane)
                del live[lane]
    assert [out[r][:12] for r in range(4)] == want
    # feed: prompt portions beside decoded tokens, then the captured step takes over from the fed state
    ps = model.paged_session(4, 128, 9)
    out = {0: [], 2: []}
    _, n = ps.feed([(0, prompts[0]), (2, prompts[2][:40])], sample=[True, False])
    out[0].append(int(n[0]))
    _, n = ps.feed([(2, prompts[2][40:]), (0, [out[0][-1]])], sample=True)
    out[2].append(int(n[0]))
    out[0].append(int(n[1]))
    got = ps.step(10)
    assert np.all(got[1] == -1) and np.all(got[3] == -1)
    assert (out[0] + got[0].tolist())[:12] == want[0] and (out[2] + got[2].tolist())[:11] == want[2][:11]
    # ... and hands back to it: the state the captured step left serves the next portion
    lane, full = 2, np.concatenate([prompts[2], out[2], got[2]])
    lg, _ = ps.feed([(lane, [int(full[-1]), 7, 8])], want=range(3))
    close(lg, G.forward(cfg, t, np.concatenate([full, [7, 8]]))[-3:], "float32")


def test_bf16_decode_step_matches_the_fed_step(rb):
    """The captured decode step against rewb200_lanes_feed of the same tokens: same kernels up to the launch shapes."""
    cfg = K.small()
    t = K.weights(cfg, seed=11, score_gain=1.5)
    model = build(rb, cfg, t, "bfloat16")
    p = K.tokens(cfg, 90, seed=11)
    a = model.session(1, 256)
    a.forward(p)
    ids, logits = a.decode(40, want_logits=True)
    full = np.concatenate([p, [a.generate(p, 1)[0, 0]], ids[0][:-1]])
    close(logits, G.forward(cfg, t, full)[-1:], "bfloat16")
    ps = model.paged_session(2, 256, 6)
    lg = feed_all(ps, 1, full, [90, 1])
    assert err(lg[-1:], logits) < 1e-2


def test_wide_batches_of_decoding_lanes(rb):
    """More lanes than a small step has rows, each at its own length."""
    cfg = K.config([K.parallel(K.dense(), heads=4, kv_heads=4, dim=64, vdim=64, rot=64, size=30, keep=3), K.rglru(K.dense())])
    t = K.weights(cfg, seed=13)
    model = build(rb, cfg, t, "bfloat16", max_seq=128)
    lanes = 70
    reqs = [K.tokens(cfg, 20 + i, seed=200 + i) for i in range(lanes)]
    ps = model.paged_session(lanes, 128, 2 * lanes + 1)
    ps.feed([(i, r[:-2]) for i, r in enumerate(reqs)])
    ps.feed([(i, r[-2:-1]) for i, r in enumerate(reqs)])
    lg, _ = ps.feed([(i, r[-1:]) for i, r in enumerate(reqs)], want=range(lanes))
    for i in (0, 1, 31, 63, 64, 69):
        close(lg[i:i + 1], G.forward(cfg, t, reqs[i])[-1:], "bfloat16")


@pytest.mark.parametrize("taps,rot", [(3, 16), (4, 8), (1, 24)])
def test_hundreds_of_sequences_in_one_step(rb, dtype, taps, rot):
    """Short portions, each starting inside a tile of rows, from the state of the step ahead; then captured decode steps."""
    cfg = K.config([K.parallel(K.dense(), rot=rot, size=12, keep=2, right=(2, 1, 16, 24, taps)), K.rglru(K.dense(), conv=taps + 1)], loop=dict(start=0, stop=2, times=1))
    t = K.weights(cfg, seed=14)
    s = build(rb, cfg, t, dtype, max_seq=64).session(516, 64)
    ids = np.stack([K.tokens(cfg, 19, seed=i) for i in range(516)])
    some = (0, 1, 2, 3, 255, 511, 512, 515)
    for lo, hi in ((0, 6), (6, 8), (8, 9), (9, 19)):
        first, logits = s.forward(ids[:, lo:hi], want_logits=True)
        close(logits[list(some)], np.stack([G.forward(cfg, t, ids[i, :hi])[-1] for i in some]), dtype)
    got, logits = s.decode(5, want_logits=True)
    for i in some:
        full = np.concatenate([ids[i], [first[i]], got[i][:-1]])
        close(logits[i:i + 1], G.forward(cfg, t, full)[-1:], dtype)


def test_forward_all_and_chunked_session_forward(rb, dtype):
    cfg = K.small()
    t = K.weights(cfg, seed=12)
    ids = np.stack([K.tokens(cfg, 80, seed=12), K.tokens(cfg, 80, seed=13)])
    want = np.stack([G.forward(cfg, t, r) for r in ids])
    s = build(rb, cfg, t, dtype).session(2, 128)
    close(s.forward_all(ids).reshape(160, -1), want.reshape(160, -1), dtype)
    s.reset()
    for lo, hi in ((0, 30), (30, 31), (31, 80)):
        _, lg = s.forward(ids[:, lo:hi], want_logits=True)
        close(lg, want[:, hi - 1], dtype)


def test_sampling_is_the_engines_own(rb):
    """Sampled ids of a lane: the same whether the prompt is admitted or fed in portions, and whoever shares the batch."""
    cfg = K.small()
    model = build(rb, cfg, K.weights(cfg, seed=14), "float32")
    p, other = K.tokens(cfg, 45, seed=14), K.tokens(cfg, 20, seed=15)
    kw = dict(temperature=0.9, top_k=20, repetition_penalty=1.2)
    a = model.paged_session(2, 128, 5)
    a.set_sampling(**kw)
    ref = [a.admit(0, p, seed=77)] + a.step(10)[0].tolist()
    b = model.paged_session(3, 128, 7)
    b.set_sampling(**kw)
    b.feed([(1, p[:17])], seeds=[77])
    _, n = b.feed([(0, other), (1, p[17:])], sample=[False, True], seeds=[5, 77])
    out = [int(n[1])]
    _, n = b.feed([(1, [out[-1]])], sample=True)
    out.append(int(n[0]))
    out += b.step(9)[1].tolist()
    assert out == ref and len(set(ref)) > 2


# ---------------------------------------------------------------- the folder on disk and the trace runner

@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    from rew_b200 import safetensors as st
    path = tmp_path_factory.mktemp("model")
    cfg = K.small()
    t = K.weights(cfg, seed=20, score_gain=1.5)
    st.write_safetensors(str(path / "model.safetensors"), t, dtype="BF16")
    (path / "config.json").write_text(json.dumps(cfg))
    return path, cfg, t


def test_registry_loads_a_folder(rb, folder, dtype):
    from rew_b200 import models
    path, cfg, t = folder
    ids = K.tokens(cfg, 40, seed=21)
    s = models.load_model(str(path), dtype=dtype, max_seq=64).session(1, 64)
    _, lg = s.forward(ids, want_logits=True)
    close(lg, G.forward(cfg, t, ids)[-1:], dtype)


def test_command_line_generates(rb, folder):
    path, cfg, t = folder
    p = K.tokens(cfg, 9, seed=22)
    want, margin = G.generate_greedy(cfg, t, p, 5)
    assert margin > 1e-4
    r = subprocess.run([sys.executable, "-m", "rew_b200", "generate", "--model", str(path), "--dtype", "float32", "--ids",
                        ",".join(map(str, p)), "--max-new", "5"], capture_output=True, text=True, cwd=ROOT)
    assert r.returncode == 0, r.stderr
    assert [int(v) for v in r.stdout.split()] == want


def test_trace_runner_end_to_end(rb, folder, dtype, tmp_path):
    """Requests that come and go on a pool of three pages, one step left out, wanted places out of order."""
    path, cfg, t = folder
    a, b, c = (K.tokens(cfg, n, seed=30 + n) for n in (100, 60, 70))
    full = {"a": G.forward(cfg, t, a), "b": G.forward(cfg, t, b), "c": G.forward(cfg, t, c)}
    steps = [
        ([("a", a[:50], [49, 0]), ("b", b[:2], [])], []),
        ([("b", b[2:60], [57])], ["b"]),
        ([("a", a[50:51], [0])], []),
        ([("a", a[51:100], [3, 48])], ["a"]),
        ([("c", c[:64], [63]), ("b2", b[:3], [1])], []),
        ([("b2", b[3:60], [56]), ("c", c[64:], [0, 5])], ["b2", "c"]),
    ]
    lines, want, at = [], {}, {}
    for n, (entries, end) in enumerate(steps):
        rows = []
        for rid, toks, w in entries:
            rows += [full[rid[0]][at.get(rid, 0) + k] for k in w]
            at[rid] = at.get(rid, 0) + len(toks)
        want[n] = rows
        lines.append(json.dumps({"step": n, "entries": [{"id": r, "tokens": [int(v) for v in k], "want": w} for r, k, w in entries], "end": end}))
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(path), "--dtype", dtype, "--out", str(tmp_path),
                        "--max-tokens", "192"], input="\n".join(lines) + "\n", capture_output=True, text=True)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done %d" % n for n in range(len(steps))]
    for n, rows in want.items():
        f = tmp_path / ("%d.f32" % n)
        assert f.exists() == bool(rows)
        if rows:
            close(np.fromfile(str(f), "<f4").reshape(len(rows), -1), np.array(rows), dtype)


def test_serving_loop_matches_generation_alone(rb, folder):
    """The command line's scheduler: more prompts than lanes, chunked prompts beside decoding lanes, stop ids."""
    from rew_b200 import models
    from rew_b200.__main__ import serve
    path, cfg, t = folder
    model = models.load_model(str(path), dtype="float32", max_seq=256)
    prompts = [K.tokens(cfg, n, seed=70 + n).tolist() for n in (50, 4, 33, 90, 1)]
    want = []
    for p in prompts:
        ids, margin = G.generate_greedy(cfg, t, p, 9)
        assert margin > 1e-4
        want.append(ids)
    assert serve(model, prompts, 9, lanes=2, chunk=16, decode_steps=4) == want
    stop = want[0][3]
    cut = [w[:w.index(stop) + 1] if stop in w else w for w in want]
    assert serve(model, prompts, 9, stop_ids=[stop], lanes=3, chunk=40) == cut
