"""Kugirax on the GPU against the plain restatement (oracle/kugirax.py): each mechanism alone, prompts, decoding through the
paged caches and the convolution state, portions of prompts, mixed batches, reuse of pages and lanes, window edges, far keys,
sinks, capped logits, sampling and greedy generation, in f32 and bf16 and with each implementation of the mixers."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import kugirax_cases as K
from oracle import kugirax as G

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {"float32": 2e-5, "bfloat16": 3e-2}
IMPLS = {"auto": ("auto", "auto"), "plain": ("plain", "plain"), "small": ("paged", "absorbed")}


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
    a, l = IMPLS[request.param]
    rb.set_option("gqa_attention", a)
    rb.set_option("latent_attention", l)
    yield request.param
    rb.set_option("gqa_attention", "auto")
    rb.set_option("latent_attention", "auto")


def build(rb, cfg, t, dtype, max_seq=2048):
    from rew_b200 import kugirax, models
    c = kugirax.config_from_json(cfg, dtype=models.DTYPES[dtype], max_seq=max_seq)
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

@pytest.mark.parametrize("what", ["all", "attention", "latent", "dense", "experts", "shared", "norms"])
def test_residual_after_every_layer(rb, dtype, what):
    cfg = K.small()
    t = K.weights(cfg, seed=2, score_gain=2.0)
    outs = {kind: ["l%d.mix.o" % i for i, l in enumerate(cfg["layers"]) if l["type"] == kind] for kind in ("attention", "latent_attention")}
    if what == "attention":
        t = silence(t, ".down", *outs["latent_attention"])
    elif what == "latent":
        t = silence(t, ".down", *outs["attention"])
    elif what == "dense":
        t = silence(t, "mix.o", "shared.down", *["e%d.down" % e for e in range(8)])
    elif what == "experts":
        t = silence(t, "mix.o", "mlp.down", "shared.down")
    elif what == "shared":
        t = silence(t, "mix.o", "mlp.down", *["e%d.down" % e for e in range(8)])
    elif what == "norms":     # an eps that matters in every norm, those of the latents included
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
    for i, w in enumerate(want):
        close(layers[i], w, dtype)


A, L = K.attention, K.latent
SIZES = [
    ([A(heads=1, kv_heads=1, dim=8, conv=1, rot=2, base=10.0), L(heads=1, dim=8, vdim=8, q_rank=8, kv_rank=8, window=1)], 40, 33, 150),
    ([A(heads=8, kv_heads=8, dim=16, conv=2, rot=16), L(heads=8, dim=16, vdim=16, q_rank=16, kv_rank=16, window=200)], 96, 64, 200),
    ([A(heads=8, kv_heads=2, dim=128, conv=4, rot=128, base=1e6), L(heads=4, dim=128, vdim=128, q_rank=64, kv_rank=128, window=96)], 128, 96, 300),
    ([A(heads=33, kv_heads=1, dim=24, conv=3, rot=12), L(heads=33, dim=24, vdim=8, q_rank=40, kv_rank=72, window=65)], 136, 72, 150),    # a group above 16; 33 heads
    ([A(heads=6, kv_heads=3, dim=13, conv=7, rot=10), L(heads=2, dim=13, vdim=19, q_rank=21, kv_rank=27, window=50)], 61, 101, 120),   # nothing divides by 8
    ([A(heads=4, kv_heads=2, dim=192, conv=5, rot=64), L(heads=2, dim=200, vdim=72, q_rank=88, kv_rank=160, window=3)], 88, 50, 150),  # value heads above 128
    ([A(heads=2, kv_heads=2, dim=256, conv=2, rot=252), L(heads=1, dim=256, vdim=256, q_rank=24, kv_rank=520, window=64)], 64, 40, 100),
    ([A(heads=40, kv_heads=2, dim=64, conv=6, rot=64, scale=0.3), L(heads=40, dim=64, vdim=64, q_rank=32, kv_rank=64, window=128)], 112, 70, 330),
    ([A(heads=3, kv_heads=1, dim=300, conv=3, rot=44), L(heads=3, dim=120, vdim=40, q_rank=9, kv_rank=88, window=129)], 80, 48, 130),
    ([A(heads=2, kv_heads=1, dim=72, conv=12, rot=6), L(heads=2, dim=72, vdim=136, q_rank=72, kv_rank=104, window=70)], 72, 56, 280),
]


@pytest.mark.parametrize("i", range(len(SIZES)))
def test_other_sizes(rb, dtype, i):
    layers, width, vocab, n = SIZES[i]
    m = layers[1]["mixer"]
    reader = L(heads=m["heads"] + 1, dim=24, vdim=m["vdim"] + 8, q_rank=m["q_rank"] + 4, kv_rank=m["kv_rank"], window=m["mask"]["size"] + 9, kv_from=1)
    cfg = K.config([dict(layers[0], mlp=K.moe(7, 1, 13, 21, scale=1.0)), dict(layers[1], mlp=K.moe(9, 9, 16, 0, scale=3.0)), dict(reader, mlp=K.dense(30))],
                   vocab=vocab, width=width, cap=[None, 3.0, 50.0][i % 3])
    t = K.weights(cfg, seed=i, score_gain=1.5)
    ids = K.tokens(cfg, n, seed=i)
    want = G.forward(cfg, t, ids)
    sess = build(rb, cfg, t, dtype).paged_session(1, 448, 8)
    close(feed_all(sess, 0, ids, [n]), want, dtype)
    sess.release(0)
    close(feed_all(sess, 0, ids, [80, 1, 1, 3, 2, 33, 1]), want, dtype)


# ---------------------------------------------------------------- cuts, batches, pages

@pytest.mark.parametrize("cuts", [[300], [2], [1], [7, 2, 31], [3], [64], [33, 31], [63, 2, 65], [130, 1, 129, 1], [100, 160]])
def test_portions_agree_with_the_whole_prompt(rb, dtype, cuts, impl):
    cfg = K.small()
    t = K.weights(cfg, seed=3, score_gain=1.5)
    ids = K.tokens(cfg, 260, seed=3)
    sess = build(rb, cfg, t, dtype).paged_session(2, 320, 6)
    close(feed_all(sess, 1, ids, cuts), G.forward(cfg, t, ids), dtype)


@pytest.mark.parametrize("taps", [2, 3, 4, 5, 9])
def test_convolution_reaches_back_over_every_cut(rb, dtype, taps):
    """Only the oldest tap weighs anything: every query and key is that of taps - 1 tokens ago, whatever step that was in."""
    cfg = K.config([K.attention(None, conv=taps), K.attention(None, heads=2, kv_heads=1, dim=20, rot=20, conv=taps + 1)], cap=None)
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


def test_long_prompt_with_many_routed_pairs(rb, dtype):
    """More (token, expert) pairs than the small-step sort takes, beside a decoding lane."""
    cfg = K.config([K.latent(K.moe(6, 4, 16), window=90), K.attention(K.moe(6, 3, 16))])
    t = K.weights(cfg, seed=17)
    a, b = K.tokens(cfg, 700, seed=17), K.tokens(cfg, 30, seed=18)
    wa, wb = G.forward(cfg, t, a), G.forward(cfg, t, b)
    sess = build(rb, cfg, t, dtype).paged_session(2, 704, 13)
    close(sess.feed([(1, b[:29])], want=range(29))[0], wb[:29], dtype)
    lg, _ = sess.feed([(0, a[:640]), (1, b[29:])], want=range(641))
    close(lg, np.concatenate([wa[:640], wb[29:]]), dtype)
    close(sess.feed([(0, a[640:])], want=range(60))[0], wa[640:], dtype)


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


def test_errors_change_nothing(rb):
    from rew_b200._lib import RewB200Error
    from rew_b200 import kugirax
    cfg = K.small()
    sess = build(rb, cfg, K.weights(cfg), "float32").paged_session(2, 128, 3)
    for bad in ([(0, [1] * 129)], [(0, [])], [(0, [1]), (0, [2])], [(2, [1])], [(0, [cfg["vocab"]])], [(0, [1] * 128), (1, [1])]):
        with pytest.raises(RewB200Error):
            sess.feed(bad)
    assert sess.free_blocks() == 2 and sess.lane_length(0) == -1
    for layer, change in ((1, dict(kv_heads=3)), (1, dict(rot=dict(base=10.0, dims=26))), (1, dict(rot=dict(base=10.0, dims=5))), (1, dict(vdim=16)),
                          (3, dict(kv_from=1)), (3, dict(kv_from=4)), (6, dict(kv_from=3)), (6, dict(kv_rank=32))):
        bad = K.small()
        bad["layers"][layer]["mixer"].update(change)
        with pytest.raises(RewB200Error):
            rb.CausalLM(kugirax.config_from_json(bad))


# ---------------------------------------------------------------- keys at every distance

@pytest.mark.parametrize("window", [1, 2, 50, 63, 64, 65, 128, 129, 200])
def test_keys_just_inside_and_outside_the_window(rb, dtype, window, impl):
    cfg, t, filler, key, query = K.marked(K.latent(None, heads=2, dim=24, vdim=16, q_rank=32, kv_rank=40, window=window))
    sess = build(rb, cfg, t, dtype).paged_session(2, 512, 10)
    for q_pos in (window + 3, 63 + window, 64 + window, 191, 320):
        seqs = {}
        for dist in (window - 1, window):           # the oldest key that is seen, and the first that is not
            if q_pos - dist < 0:
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


@pytest.mark.parametrize("kind", ["attention", "latent"])
def test_far_keys_and_page_borders(rb, dtype, impl, kind):
    """A marked key at the first token and around every page border of a long context, found by prompts and by decoding."""
    layer = K.attention(None, heads=4, kv_heads=2, dim=24, rot=8) if kind == "attention" else K.latent(None, heads=2, dim=24, vdim=16, q_rank=32, window=700)
    cfg, t, filler, key, query = K.marked(layer)
    sess = build(rb, cfg, t, dtype).paged_session(1, 1024, 17)
    base = np.full(700, filler, np.int32)
    base[-1] = query
    none = G.forward(cfg, t, base)[-1:]
    for where in (0, 1, 62, 63, 64, 65, 127, 128, 383, 384, 640, 697, 698):
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


@pytest.mark.parametrize("sink", [-30.0, 0.0, 3.0, 30.0])
def test_learned_sinks_take_their_share(rb, dtype, impl, sink):
    cfg = K.config([K.latent(None, window=50), K.latent(None, heads=4, kv_from=0)])
    t = K.weights(cfg, seed=9, score_gain=1.5)
    t["l0.mix.sink"][:] = t["l1.mix.sink"][:] = sink
    t["l0.mix.sink"][1] = -sink
    ids = K.tokens(cfg, 150, seed=9)
    want = G.forward(cfg, t, ids)
    sess = build(rb, cfg, t, dtype).paged_session(1, 192, 4)
    for cuts in ([150], [1, 2, 64, 1]):
        close(feed_all(sess, 0, ids, cuts), want, dtype)
        sess.release(0)


@pytest.mark.parametrize("gain", [0.0, 1.0, 3.0])
def test_the_one_in_the_denominator(rb, dtype, impl, gain):
    """Scores from all equal (the one is a further key without a value) to far below and above zero, first tokens first."""
    cfg = K.config([K.attention(None, heads=2, kv_heads=1, conv=2), K.attention(None, heads=3, kv_heads=3, conv=1)])
    t = K.weights(cfg, seed=12, score_gain=gain)
    ids = K.tokens(cfg, 100, seed=12)
    want = G.forward(cfg, t, ids)
    plain = {"sink_softmax": G.sink_softmax}
    G.sink_softmax = lambda s, vis, sink: plain["sink_softmax"](s, vis, -np.inf)
    try:
        assert err(G.forward(cfg, t, ids)[:3], want[:3]) > 0.05        # without it the first tokens differ
    finally:
        G.sink_softmax = plain["sink_softmax"]
    sess = build(rb, cfg, t, dtype).paged_session(1, 128, 3)
    for cuts in ([100], [1], [2]):
        close(feed_all(sess, 0, ids, cuts), want, dtype)
        sess.release(0)


def test_rotation_at_far_positions(rb, dtype):
    """Fast and slow features a long way into the sequence, rotated whole and in part."""
    cfg = K.config([K.attention(None, heads=2, kv_heads=1, dim=32, rot=32, base=10.0), K.attention(None, heads=2, kv_heads=2, dim=24, rot=12, base=1e7)])
    t = K.weights(cfg, seed=13, score_gain=1.5)
    ids = K.tokens(cfg, 1200, seed=13)
    want = G.forward(cfg, t, ids)[-130:]
    sess = build(rb, cfg, t, dtype).paged_session(1, 1216, 20)
    sess.feed([(0, ids[:1070])])
    got = [sess.feed([(0, ids[1070:1120])], want=range(50))[0]] + [sess.feed([(0, ids[i:i + 1])], want=[0])[0] for i in range(1120, 1130)] \
        + [sess.feed([(0, ids[1130:])], want=range(70))[0]]
    close(np.concatenate(got), want, dtype)


def mixed_attention(T, spec, t, p, h, kv):
    """Attention with every option of the layered one: convolution, norms, temperature, rotation, values of their own, a
    learned sink and a gate per head, keys and values of another layer (kv)"""
    from oracle import girulorn as GG
    H, N, D, V = spec.heads, spec.kv_heads, spec.dim, spec.vdim
    w = lambda n: t[p + "mix." + n].astype(np.float64)
    turn = lambda x: G.rotated_halves(x, np.arange(T), spec.rope_base, spec.rope_dims)
    q = GG.rms_norm(G.short_conv(h @ w("q"), w("q.conv")).reshape(T, H, D), w("q.norm"), 1e-5)
    q = turn(q * GG.query_temperature(range(T), dict(coef=spec.temp_coef, every=spec.temp_every))[:, None, None])
    if kv is None:
        kv = (turn(GG.rms_norm(G.short_conv(h @ w("k"), w("k.conv")).reshape(T, N, D), w("k.norm"), 1e-5)), (h @ w("v")).reshape(T, N, V))
    gate = G.sigmoid(h @ w("g"))
    out = np.stack([G.sink_softmax(q[:, a] @ kv[0][:, a // (H // N)].T * spec.scale, G.visible(T), w("sink")[a]) @ kv[1][:, a // (H // N)] * gate[:, a:a + 1]
                    for a in range(H)], 1)
    return out.reshape(T, H * V) @ w("o"), kv


@pytest.mark.parametrize("dim,vdim,taps,rope", [(24, 40, 3, 16), (16, 16, 4, 12), (40, 24, 6, 40), (136, 64, 2, 64)])
def test_convolution_norms_temperature_rotation_and_values_together(rb, dtype, dim, vdim, taps, rope):
    from rew_b200 import models
    from rew_b200.layered import LayeredConfig, LayerSpec
    from rew_b200.weights import bf16_round
    base = dict(mixer="attention", heads=4, kv_heads=2, dim=dim, vdim=vdim, scale=dim ** -0.5, conv_taps=taps, rope_base=90.0, rope_dims=rope, qk_norm=True,
                sink=True, out_gate=True, temp_every=7, temp_coef=0.3, ff="none")
    cfg = LayeredConfig(vocab=72, d_model=64, layers=[LayerSpec(**base), LayerSpec(kv_from=0, **base)], eps=1e-5, norm_zero_centred=False,
                        block="parallel_one_norm", own_head=True, max_seq=640, dtype=models.DTYPES[dtype])
    rng = np.random.default_rng(dim)
    t = {n: bf16_round(rng.normal(1.0 if n.endswith("norm") or n.endswith("norm1") else 0.0, 0.2 if "norm" in n else 1.2 if n.endswith("conv") or n == "embed"
                                  else shape[0] ** -0.5, size=shape).astype(np.float32)) for n, shape in cfg.tensor_specs()}
    ids = rng.integers(0, 72, size=600).astype(np.int32)
    f = {k: v.astype(np.float64) for k, v in t.items()}
    x, kv = f["embed"][ids], None
    for i, spec in enumerate(cfg.layers):
        y, kv = mixed_attention(600, spec, t, "l%d." % i, G.rms_norm(x, f["l%d.norm1" % i], 1e-5), kv)
        x = x + y
    want = G.rms_norm(x, f["final.norm"], 1e-5) @ f["head"]
    sess = rb.CausalLM(cfg).load([t[n] for n, _ in cfg.tensor_specs()]).paged_session(1, 640, 11)
    for cuts in ([600], [520, 1, 2, 70, 1], [3, 597]):
        close(feed_all(sess, 0, ids, cuts), want, dtype)
        sess.release(0)


def test_long_decoding(rb, dtype):
    cfg = K.config([K.attention(K.moe()), K.latent(K.moe(), window=80), K.latent(None, window=120, kv_from=1)])
    t = K.weights(cfg, seed=8, score_gain=1.5)
    ids = K.tokens(cfg, 300, seed=8)
    sess = build(rb, cfg, t, dtype).paged_session(1, 320, 6)
    close(feed_all(sess, 0, ids, [20, 1]), G.forward(cfg, t, ids), dtype)


@pytest.mark.parametrize("vocab", [150, 160])
def test_capped_logits(rb, dtype, vocab):
    """Logits far beyond the cap, whole rows and with a padded vocabulary."""
    cfg = K.config([K.attention(None)], vocab=vocab, cap=1.5)
    t = K.weights(cfg, seed=15)
    ids = K.tokens(cfg, 40, seed=15)
    want = G.forward(cfg, t, ids)
    assert np.abs(want).max() > 1.4 and np.abs(want).max() <= 1.5
    s = build(rb, cfg, t, dtype).session(1, 64)
    _, lg = s.forward(ids, want_logits=True)
    close(lg, want[-1:], dtype)
    close(s.forward_all(ids).reshape(40, -1), want, dtype)


# ---------------------------------------------------------------- generation

def test_greedy_generation_follows_the_oracle(rb):
    """Session.generate, the paged lanes with a captured decode step, and steps that mix prompts with decoding."""
    cfg = K.small(cap=12.0)
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
    cfg = K.small(cap=25.0)
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
    cfg = K.config([K.latent(K.moe()), K.attention(K.moe(), heads=4, kv_heads=4, dim=64, rot=64)])
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


@pytest.mark.parametrize("conv,rot", [(3, 16), (4, 20), (7, 24), (1, 8)])
def test_hundreds_of_sequences_in_one_step(rb, dtype, conv, rot):
    """Short portions, each starting inside a tile of rows, from the state of the step ahead; then captured decode steps."""
    cfg = K.config([K.attention(K.dense(), conv=conv, rot=rot), K.latent(K.dense())], cap=25.0)
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
    cfg = K.small(cap=12.0)
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
