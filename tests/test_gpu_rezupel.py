"""Rezupel on the GPU against the plain restatement (oracle/rezupel.py): each mechanism alone, prompts, decoding through
the paged latent cache, portions of prompts, mixed batches, reuse of pages and lanes, window edges, sampling and greedy
generation, in f32 and bf16 and with each implementation of the attention."""
import json
import os
import subprocess

import numpy as np
import pytest

import rezupel_cases as K
from oracle import rezupel as R

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {"float32": 2e-5, "bfloat16": 3e-2}


@pytest.fixture(scope="module")
def rb():
    from rew_b200 import _lib, api
    _lib.init()
    return api


@pytest.fixture(params=["float32", "bfloat16"])
def dtype(request):
    return request.param


def build(rb, cfg, t, dtype, max_seq=2048):
    from rew_b200 import models, rezupel
    c = rezupel.config_from_json(cfg, dtype=models.DTYPES[dtype], max_seq=max_seq)
    return rb.CausalLM(c).load(rezupel.canonical_tensors(c, t))


def err(got, want):
    """Worst row: rms of the difference over the rms of all wanted values."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    assert got.shape == want.shape and np.isfinite(got).all()
    return float(np.sqrt(((got - want) ** 2).mean(-1)).max() / max(np.sqrt((want ** 2).mean()), 1e-30))


def close(got, want, dtype, slack=1.0):
    e = err(got, want)
    assert e <= TOL[dtype] * slack, e


def feed_all(sess, lane, ids, cuts):
    """Logits of every position of one request, fed in portions of the given sizes (the last repeats)."""
    out, at, i = [], 0, 0
    while at < len(ids):
        n = min(cuts[min(i, len(cuts) - 1)], len(ids) - at)
        lg, _ = sess.feed([(lane, ids[at:at + n])], want=range(n))
        out.append(lg)
        at, i = at + n, i + 1
    return np.concatenate(out)


# ---------------------------------------------------------------- each mechanism alone

def silence(t, *suffixes):
    return {k: np.zeros_like(v) if k.endswith(suffixes) else v for k, v in t.items()}


@pytest.mark.parametrize("what", ["all", "attention", "dense", "experts", "loop", "norms"])
def test_residual_after_every_layer_run(rb, dtype, what):
    cfg = K.small()
    t = K.weights(cfg, seed=2, score_gain=2.0)
    if what == "attention":
        t = silence(t, ".down")
    elif what in ("dense", "experts"):
        t = silence(t, "mix.o")
        if what == "experts":
            t = silence(t, "mlp.gate")
    elif what == "loop":
        t = silence(t, "mix.o", ".down")
    elif what == "norms":     # an eps that matters in every norm, the latents' included
        cfg["norm"]["eps"] = 0.3
    ids = K.tokens(cfg, 50, seed=2)
    want = []
    logits = R.forward(cfg, t, ids, want)
    rb.set_option("record_layers", "1")
    try:
        sess = build(rb, cfg, t, dtype).paged_session(2, 64, 4)
        got, _ = sess.feed([(1, ids)], want=range(len(ids)))
        layers = sess.layers(len(ids))
    finally:
        rb.set_option("record_layers", "0")
    close(got, logits, dtype)
    for i, w in enumerate(want):
        close(layers[i], w, dtype)


def test_gate_and_scale_are_applied(rb, dtype):
    """A gate driven hard to one side removes a head; a larger score scale sharpens the softmax."""
    for scale in (0.05, 1.0):
        cfg = K.config([K.layer(None, heads=2, scale=scale)])
        t = K.weights(cfg, seed=5)
        t["l0.mix.g"] = t["l0.mix.g"] * 8
        ids = K.tokens(cfg, 30, seed=5)
        close(feed_all(build(rb, cfg, t, dtype).paged_session(1, 64, 2), 0, ids, [30]), R.forward(cfg, t, ids), dtype)


SIZES = [
    dict(heads=1, dim=8, rot_dim=2, vdim=8, q_rank=8, kv_rank=8, window=1),
    dict(heads=7, dim=16, rot_dim=8, vdim=48, q_rank=24, kv_rank=16, window=2),
    dict(heads=4, dim=64, rot_dim=64, vdim=32, q_rank=72, kv_rank=192, window=200),
    dict(heads=16, dim=128, rot_dim=64, vdim=128, q_rank=96, kv_rank=512, window=70, base=10000.0),
    dict(heads=33, dim=24, rot_dim=16, vdim=24, q_rank=40, kv_rank=64, window=64),
    dict(heads=5, dim=13, rot_dim=6, vdim=11, q_rank=19, kv_rank=27, window=30, rope_dims=4),     # nothing divides by 8
    dict(heads=2, dim=192, rot_dim=32, vdim=160, q_rank=64, kv_rank=256, window=129),
    dict(heads=8, dim=32, rot_dim=16, vdim=64, q_rank=64, kv_rank=640, window=100),
    dict(heads=3, dim=192, rot_dim=64, vdim=128, q_rank=48, kv_rank=72, window=150),     # four score boxes: one query tile a CTA
    dict(heads=2, dim=136, rot_dim=24, vdim=40, q_rank=32, kv_rank=56, window=300),      # ... two, with one value stage
    dict(heads=4, dim=128, rot_dim=64, vdim=128, q_rank=80, kv_rank=256, window=130),
]


@pytest.mark.parametrize("i", range(len(SIZES)))
def test_other_sizes(rb, dtype, i):
    width, vocab = [(40, 33), (96, 64), (256, 130), (320, 200), (136, 72), (61, 101), (128, 90), (200, 88), (112, 70), (96, 50),
                    (192, 96)][i]
    cfg = K.config([K.layer(K.dense(37), **SIZES[i]), K.layer(K.moe(6, 1, 13), **SIZES[i])], vocab=vocab, width=width, loop=(0, 2, 2))
    t = K.weights(cfg, seed=i, score_gain=2.0)
    n = 150 if i < 8 else 400
    ids = K.tokens(cfg, n, seed=i)
    want = R.forward(cfg, t, ids)
    sess = build(rb, cfg, t, dtype).paged_session(1, 448, 8)
    close(feed_all(sess, 0, ids, [n]), want, dtype)
    sess.release(0)
    close(feed_all(sess, 0, ids, [100, 1, 1, 3, 2, 80, 1]), want, dtype)


# ---------------------------------------------------------------- cuts, batches, pages

@pytest.mark.parametrize("impl", ["auto", "plain", "absorbed"])
@pytest.mark.parametrize("cuts", [[300], [2], [1], [7, 2, 31], [64], [63, 2, 65], [130, 1, 129, 1], [100, 160]])
def test_portions_agree_with_the_whole_prompt(rb, dtype, cuts, impl):
    cfg = K.small()
    t = K.weights(cfg, seed=3, score_gain=2.5)
    ids = K.tokens(cfg, 260, seed=3)
    rb.set_option("latent_attention", impl)
    try:
        sess = build(rb, cfg, t, dtype).paged_session(2, 320, 6)
        close(feed_all(sess, 1, ids, cuts), R.forward(cfg, t, ids), dtype)
    finally:
        rb.set_option("latent_attention", "auto")


def test_mixed_batches_against_each_request_alone(rb, dtype):
    """Four live requests in portions of 1 .. 140 tokens on a pool that is too small for all of them at once; lanes and
    pages go from request to request."""
    cfg = K.small()
    t = K.weights(cfg, seed=4, score_gain=2.0)
    rng = np.random.default_rng(0)
    reqs = [K.tokens(cfg, int(n), seed=10 + i) for i, n in enumerate([170, 3, 90, 1, 64, 65, 200, 40, 129])]
    want = [R.forward(cfg, t, r) for r in reqs]
    sess = build(rb, cfg, t, dtype).paged_session(4, 256, 9)
    got = [[] for _ in reqs]
    todo, live = list(range(len(reqs))), {}
    at = [0] * len(reqs)
    steps = 0
    while todo or live:
        held = sum(-(-len(reqs[r]) // 64) for r in live.values())
        for lane in range(4):
            if lane not in live and todo and held + -(-len(reqs[todo[0]]) // 64) <= 8:
                held += -(-len(reqs[todo[0]]) // 64)
                live[lane] = todo.pop(0)
        portions, spans = [], []
        for lane, r in live.items():
            if len(live) > 1 and rng.random() < 0.2:
                continue                                    # left out of this step
            n = int(rng.choice([1, 1, 2, 5, 33, 64, 140]))
            n = min(n, len(reqs[r]) - at[r])
            portions.append((lane, reqs[r][at[r]:at[r] + n]))
            spans.append((r, n))
        if not portions:
            continue
        lg, _ = sess.feed(portions, want=range(sum(n for _, n in spans)))
        o = 0
        for r, n in spans:
            got[r].append(lg[o:o + n])
            o, at[r] = o + n, at[r] + n
        for lane in [l for l, r in live.items() if at[r] == len(reqs[r])]:
            sess.release(lane)
            del live[lane]
        steps += 1
    assert sess.free_blocks() == 8 and steps > 8
    for r in range(len(reqs)):
        close(np.concatenate(got[r]), want[r], dtype)


def test_long_prompt_with_many_routed_pairs(rb, dtype):
    """More (token, expert) pairs than the small-step sort takes, beside a decoding lane."""
    cfg = K.config([K.layer(K.moe(6, 4, 16), window=90)], loop=(0, 1, 2))
    t = K.weights(cfg, seed=17)
    a, b = K.tokens(cfg, 700, seed=17), K.tokens(cfg, 30, seed=18)
    wa, wb = R.forward(cfg, t, a), R.forward(cfg, t, b)
    sess = build(rb, cfg, t, dtype).paged_session(2, 704, 13)
    close(sess.feed([(1, b[:29])], want=range(29))[0], wb[:29], dtype)
    lg, _ = sess.feed([(0, a[:640]), (1, b[29:])], want=range(641))
    close(lg, np.concatenate([wa[:640], wb[29:]]), dtype)
    close(sess.feed([(0, a[640:])], want=range(60))[0], wa[640:], dtype)


def test_freed_pages_hold_nothing_over(rb):
    """A request on pages and a lane that others used gives the same bits as on a fresh session."""
    cfg = K.small()
    t = K.weights(cfg, seed=6, score_gain=2.0)
    model = build(rb, cfg, t, "bfloat16")
    ids = K.tokens(cfg, 120, seed=6)
    first = feed_all(model.paged_session(1, 128, 3), 0, ids, [50, 1, 1, 68])
    sess = model.paged_session(3, 128, 6)
    for i in range(4):
        feed_all(sess, i % 3, K.tokens(cfg, 60 + i, seed=40 + i), [61])
        if i >= 1:
            sess.release((i - 1) % 3)
    sess.release(0)
    assert np.array_equal(feed_all(sess, 2, ids, [50, 1, 1, 68]) if sess.lane_length(2) < 0 else
                          feed_all(sess, 0, ids, [50, 1, 1, 68]), first)


def test_errors_change_nothing(rb):
    from rew_b200._lib import RewB200Error
    cfg = K.small()
    sess = build(rb, cfg, K.weights(cfg), "float32").paged_session(2, 128, 3)
    for bad in ([(0, [1] * 129)], [(0, [])], [(0, [1]), (0, [2])], [(2, [1])], [(0, [cfg["vocab"]])], [(0, [1] * 128), (1, [1])]):
        with pytest.raises(RewB200Error):
            sess.feed(bad)
    with pytest.raises(RewB200Error):
        sess.feed([(0, [1, 2])], want=[2])
    assert sess.free_blocks() == 2 and sess.lane_length(0) == -1


# ---------------------------------------------------------------- window edges

def edge_case(window, seed=0):
    """One layer without a feed-forward whose second vocabulary half carries a mark: the last token's query (a token of
    the third kind) meets marked keys with a score far above all others.  Returns (cfg, tensors, filler, key, query)."""
    cfg = K.config([K.layer(None, heads=2, dim=24, rot_dim=8, vdim=16, q_rank=32, kv_rank=40, window=window, base=50.0)], vocab=96, width=88)
    t = {k: v.copy() for k, v in K.weights(cfg, seed=seed).items()}
    d, m = cfg["width"], cfg["layers"][0]["mixer"]
    filler, key, query = 1, 2, 3
    t["l0.norm1"][:] = 0
    for tok, col in ((key, 0), (query, 1)):
        t["embed"][tok] = 0.0
        t["embed"][tok, col] = 8.0
    t["embed"][filler, :2] = 0.0
    # the mark of the key reaches latent feature 0, the mark of the query query-latent feature 0, and they meet in
    # unrotated feature 0 of both heads
    for n, col in (("dkv", 0), ("dq", 1)):
        t["l0.mix." + n][:, col] = 0.0
        t["l0.mix." + n][0] = 0.0
        t["l0.mix." + n][0, col] = 4.0
    t["l0.mix.uq"][:, 0] = 0.0
    t["l0.mix.uk"][:, 0] = 0.0
    for h in range(m["heads"]):
        t["l0.mix.uq"][h * (m["dim"] + m["rot_dim"]), 0] = 6.0
        t["l0.mix.uk"][h * m["dim"], 0] = 4.0
    return cfg, t, filler, key, query


@pytest.mark.parametrize("impl", ["auto", "plain", "absorbed"])
@pytest.mark.parametrize("window", [1, 2, 50, 63, 64, 65, 128, 129, 200])
def test_keys_just_inside_and_outside_the_window(rb, dtype, window, impl):
    cfg, t, filler, key, query = edge_case(window)
    rb.set_option("latent_attention", impl)
    try:
        sess = build(rb, cfg, t, dtype).paged_session(2, 512, 10)
        for q_pos in (window + 3, 63 + window, 64 + window, 191, 320):
            seqs = {}
            for dist in (window - 1, window):           # the oldest key that is seen, and the first that is not
                ids = np.full(q_pos + 1, filler, np.int32)
                if q_pos - dist < 0:
                    continue
                ids[q_pos - dist] = key
                ids[q_pos] = query
                seqs[dist] = ids
            want = {k: R.forward(cfg, t, v)[-1:] for k, v in seqs.items()}
            if len(want) == 2 and window > 1:
                assert err(want[window - 1], want[window]) > 10 * TOL["bfloat16"]     # a shifted edge would show
            for dist, ids in seqs.items():
                for cuts in ([q_pos + 1], [q_pos, 1], [max(1, q_pos - 2), 3], [max(1, q_pos - dist), 2, 70]):
                    got = feed_all(sess, 0, ids, cuts)[-1:]
                    close(got, want[dist], dtype)
                    sess.release(0)
    finally:
        rb.set_option("latent_attention", "auto")


@pytest.mark.parametrize("impl", ["auto", "plain", "absorbed"])
def test_far_keys_and_page_borders(rb, dtype, impl):
    """A marked key at the first token and around every page border of a long context, found by prompts and by decoding."""
    cfg, t, filler, key, query = edge_case(1000)
    rb.set_option("latent_attention", impl)
    try:
        sess = build(rb, cfg, t, dtype).paged_session(1, 1024, 17)
        base = np.full(700, filler, np.int32)
        base[-1] = query
        none = R.forward(cfg, t, base)[-1:]
        for where in (0, 1, 62, 63, 64, 65, 127, 128, 383, 384, 640, 697, 698):
            ids = base.copy()
            ids[where] = key
            want = R.forward(cfg, t, ids)[-1:]
            assert err(want, none) > 10 * TOL["bfloat16"]
            for cuts in ([700], [699, 1], [350, 300, 50]):
                close(feed_all(sess, 0, ids, cuts)[-1:], want, dtype)
                sess.release(0)
    finally:
        rb.set_option("latent_attention", "auto")


def test_window_passes_over_decoded_tokens(rb, dtype):
    """Long decoding: the window leaves the prompt and wraps over several pages of decoded tokens."""
    cfg = K.config([K.layer(K.dense(40), window=70), K.layer(K.moe(), window=33)], loop=(0, 1, 2))
    t = K.weights(cfg, seed=8, score_gain=3.0)
    ids = K.tokens(cfg, 260, seed=8)
    want = R.forward(cfg, t, ids)
    sess = build(rb, cfg, t, dtype).paged_session(1, 320, 6)
    close(feed_all(sess, 0, ids, [20, 1]), want, dtype)


# ---------------------------------------------------------------- generation

def test_greedy_generation_follows_the_oracle(rb):
    """Session.generate, the paged lanes with a captured decode step, and steps that mix prompts with decoding."""
    cfg = K.small()
    t = K.weights(cfg, seed=9, score_gain=1.5)
    model = build(rb, cfg, t, "float32")
    prompts = [K.tokens(cfg, n, seed=60 + n) for n in (5, 1, 70, 33)]
    want = []
    for p in prompts:
        ids, margin = R.generate_greedy(cfg, t, p, 12)
        assert margin > 1e-4
        want.append(ids)
    # uniform batch through generate()
    s = model.session(2, 64)
    same = np.stack([prompts[0], prompts[0][::-1]])
    got = s.generate(same, 12)
    assert got[0].tolist() == want[0] and got[1].tolist() == R.generate_greedy(cfg, t, prompts[0][::-1], 12)[0]
    assert s.generate(same[:1].repeat(2, 0), 12)[1].tolist() == want[0]        # a second call starts over
    # lanes: admit, then the captured step over all lanes
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
    assert n.tolist()[1] == -1
    out[0].append(int(n[0]))
    _, n = ps.feed([(2, prompts[2][40:]), (0, [out[0][-1]])], sample=True)
    out[2].append(int(n[0]))
    out[0].append(int(n[1]))
    got = ps.step(10)
    assert np.all(got[1] == -1) and np.all(got[3] == -1)
    assert (out[0] + got[0].tolist())[:12] == want[0] and (out[2] + got[2].tolist())[:11] == want[2][:11]


def test_bf16_decode_step_matches_the_fed_step(rb):
    """The captured decode step against rewb200_lanes_feed of the same tokens: same kernels up to the launch shapes."""
    cfg = K.small()
    t = K.weights(cfg, seed=11, score_gain=2.0)
    model = build(rb, cfg, t, "bfloat16")
    p = K.tokens(cfg, 90, seed=11)
    a = model.session(1, 256)
    a.forward(p)
    ids, logits = a.decode(40, want_logits=True)
    full = np.concatenate([p, [a.generate(p, 1)[0, 0]], ids[0][:-1]])
    close(logits, R.forward(cfg, t, full)[-1:], "bfloat16")
    ps = model.paged_session(2, 256, 6)
    lg = feed_all(ps, 1, full, [90, 1])
    assert err(lg[-1:], logits) < 1e-2


@pytest.mark.parametrize("rope_dims,heads", [(12, 3), (6, 5), (0, 4)])
def test_hundreds_of_sequences_in_one_step(rb, dtype, rope_dims, heads):
    """Large steps of short portions: rotated pairs whole and in part, gates of any number of heads."""
    cfg = K.config([K.layer(K.dense(), heads=heads, rope_dims=rope_dims), K.layer(None, heads=2, window=9)])
    t = K.weights(cfg, seed=21, score_gain=2.0)
    s = build(rb, cfg, t, dtype, max_seq=64).session(260, 64)
    ids = np.stack([K.tokens(cfg, 11, seed=i) for i in range(260)])
    some = [0, 1, 7, 128, 255, 259]
    for lo, hi in ((0, 5), (5, 11)):
        _, logits = s.forward(ids[:, lo:hi], want_logits=True)
        close(logits[some], np.stack([R.forward(cfg, t, ids[i, :hi])[-1] for i in some]), dtype)


def test_forward_all_and_chunked_session_forward(rb, dtype):
    cfg = K.small()
    t = K.weights(cfg, seed=12)
    ids = np.stack([K.tokens(cfg, 80, seed=12), K.tokens(cfg, 80, seed=13)])
    want = np.stack([R.forward(cfg, t, r) for r in ids])
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


def test_feed_serves_grouped_query_models_too(rb, orc):
    from rew_b200 import weights as W
    cfg = W.tiny_llama(norm_kind=0, mask_kind=1)
    t = W.init_weights(cfg, seed=1)
    p = np.random.default_rng(3).integers(0, cfg.vocab, size=(1, 30)).astype(np.int32)
    want_ids, _ = orc.generate_greedy(cfg, t, p, 8)
    want = orc.model_forward(cfg, t, p, 0, True)[0]
    s = rb.CausalLM(cfg).load(t).paged_session(3, 64, 4)
    lg, n = s.feed([(2, p[0, :11]), (0, p[0, :5])], want=[3, 10, 12], sample=[False, False])
    close(lg, want[[3, 10, 1]], "float32")
    lg, n = s.feed([(2, p[0, 11:])], want=[18], sample=True)
    close(lg, want[29:], "float32")
    assert [int(n[0])] + s.step(7)[2].tolist() == want_ids[0].tolist()


# ---------------------------------------------------------------- the folder on disk and the trace runner

@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    from rew_b200 import safetensors as st
    path = tmp_path_factory.mktemp("model")
    cfg = K.small()
    t = K.weights(cfg, seed=20, score_gain=2.0)
    st.write_safetensors(str(path / "model.safetensors"), t, dtype="BF16")
    (path / "config.json").write_text(json.dumps(cfg))
    return path, cfg, t


def test_registry_loads_a_folder(rb, folder, dtype):
    from rew_b200 import models
    path, cfg, t = folder
    ids = K.tokens(cfg, 40, seed=21)
    s = models.load_model(str(path), dtype=dtype, max_seq=64).session(1, 64)
    _, lg = s.forward(ids, want_logits=True)
    close(lg, R.forward(cfg, t, ids)[-1:], dtype)


def test_command_line_generates(rb, folder):
    import sys
    path, cfg, t = folder
    p = K.tokens(cfg, 9, seed=22)
    want, margin = R.generate_greedy(cfg, t, p, 5)
    assert margin > 1e-4
    r = subprocess.run([sys.executable, "-m", "rew_b200", "generate", "--model", str(path), "--dtype", "float32", "--ids",
                        ",".join(map(str, p)), "--max-new", "5"], capture_output=True, text=True, cwd=ROOT)
    assert r.returncode == 0, r.stderr
    assert [int(v) for v in r.stdout.split()] == want


def test_trace_runner_end_to_end(rb, folder, dtype, tmp_path):
    """Requests that come and go on a pool of three pages, one step left out, wanted places out of order."""
    path, cfg, t = folder
    a, b, c = (K.tokens(cfg, n, seed=30 + n) for n in (100, 60, 70))
    full = {"a": R.forward(cfg, t, a), "b": R.forward(cfg, t, b), "c": R.forward(cfg, t, c)}
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
        ids, margin = R.generate_greedy(cfg, t, p, 9)
        assert margin > 1e-4
        want.append(ids)
    assert serve(model, prompts, 9, lanes=2, chunk=16, decode_steps=4) == want
    stop = want[0][3]
    cut = [w[:w.index(stop) + 1] if stop in w else w for w in want]
    assert serve(model, prompts, 9, stop_ids=[stop], lanes=3, chunk=40) == cut
