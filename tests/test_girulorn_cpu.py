"""Girulorn on the host: config reader, tensor mapping, registry, and properties of the plain restatement the GPU tests
compare with (oracle/girulorn.py)."""
import json
import math

import numpy as np
import pytest

import girulorn_cases as K
from oracle import girulorn as G
from rew_b200 import _lib, girulorn, models, safetensors as st


def test_config_reader_takes_every_size_from_the_file():
    cfg = K.small()
    t = K.weights(cfg)
    c = girulorn.config_from_json(K.public(cfg), K.shapes(t), max_seq=77, dtype=_lib.BF16)
    assert (c.vocab, c.d_model, c.eps, c.max_seq, c.dtype, c.block, c.own_head) == (152, 104, 1e-5, 77, _lib.BF16, "output_norm", True)
    assert [l.mixer for l in c.layers] == ["gla", "attention", "attention", "gla", "attention"]
    assert [l.ff for l in c.layers] == ["experts", "experts", "none", "none", "experts"]
    assert [(l.experts, l.top_k, l.ffn, l.shared_ffn) for l in c.layers if l.ff == "experts"] == [(5, 3, 24, 40), (7, 2, 40, 0), (5, 3, 24, 40)]
    assert [l.kv_from for l in c.layers] == [-1, -1, -1, -1, 1]
    assert [l.bias_rows for l in c.layers] == [0, 12, 7, 0, 16] and [l.bias_max for l in c.layers] == [0, 50, 50, 0, 90]
    assert [(l.temp_every, l.temp_coef) for l in c.layers] == [(0, 0.0), (16, 0.4), (0, 0.0), (0, 0.0), (16, 0.4)]
    assert [(l.tau, l.decay_rank) for l in c.layers if l.mixer == "gla"] == [(8.0, 6), (2.0, 3)]
    assert (c.layers[2].heads, c.layers[2].kv_heads, c.layers[2].dim, c.layers[2].vdim) == (6, 1, 32, 40)
    assert c.layers[1].renormalize and c.layers[1].expert_gated and c.layers[1].router_bias and c.layers[1].sink
    bad = K.public(cfg)
    bad["layers"][0]["type"] = "something"
    with pytest.raises(ValueError, match="unknown mixer"):
        girulorn.config_from_json(bad, K.shapes(t))
    bad = K.public(K.small())
    bad["layers"][0]["mlp"]["kind"] = "something"
    with pytest.raises(ValueError, match="unknown feed-forward"):
        girulorn.config_from_json(bad, K.shapes(t))


def test_canonical_tensors_cover_the_file_and_check_shapes():
    cfg = K.small()
    t = K.weights(cfg)
    c = girulorn.config_from_json(K.public(cfg), K.shapes(t))
    out = dict(zip([n for n, _ in c.tensor_specs()], c.canonical_tensors(t)))
    assert set(out) == set(t)
    assert np.array_equal(out["embed"], t["embed"]) and np.array_equal(out["l1.mix.rel"], t["l1.mix.rel"])      # tables stay
    for n in ("head", "l0.mix.a2", "l1.mix.g", "l0.mlp.e3.down", "l4.mlp.shared.up", "l1.mlp.router"):
        assert np.array_equal(out[n], t[n].T)
    assert "l4.mix.k" not in out and "l4.mix.v" not in out and "l4.mix.k.norm" not in out
    short = dict(t)
    del short["l0.mix.norm"]
    with pytest.raises(KeyError, match="l0.mix.norm"):
        c.canonical_tensors(short)
    with pytest.raises(ValueError, match="l1.mix.sink"):
        c.canonical_tensors(dict(t, **{"l1.mix.sink": np.zeros(9, np.float32)}))


def test_registry_picks_the_family_by_config(tmp_path):
    cfg = K.small()
    assert models.family_of(json.loads(json.dumps(K.public(cfg)))) == "girulorn"
    t = K.weights(cfg, seed=3)
    st.write_safetensors(str(tmp_path / "model.safetensors"), t, dtype="BF16")
    back = st.read_safetensors_dir(str(tmp_path))
    assert set(back) == set(t) and all(np.array_equal(back[k], t[k]) for k in t)


def test_step_bytes_counts_state_and_cache():
    cfg = K.config([K.gla(), K.attention()])
    t = K.weights(cfg)
    c = girulorn.config_from_json(K.public(cfg), K.shapes(t), dtype=_lib.BF16)
    g, a = cfg["layers"][0]["mixer"], cfg["layers"][1]["mixer"]
    one, far = c.step_bytes(1, 10), c.step_bytes(1, 11)
    assert far - one == 2 * a["kv_heads"] * (a["dim"] + a["vdim"])
    assert c.step_bytes(2, 10) - one == 10 * (far - one) + 8 * g["heads"] * g["dim"] * g["vdim"]


# ---- the restatement itself

def test_oracle_buckets():
    B, D = 16, 90
    b = [G.distance_bucket(n, B, D) for n in range(200)]
    assert b[:9] == [0, 1, 2, 3, 4, 5, 6, 7, 8] and b[90:] == [15] * 110 and b == sorted(b) and set(b) == set(range(16))
    first = [b.index(k) for k in range(8, 16)]
    want = [math.ceil(8 * (D / 8) ** (k / 8) - 1e-9) for k in range(8)]
    assert first == want
    assert [G.distance_bucket(n, 7, 12) for n in (0, 2, 3, 12, 99)] == [0, 2, 3, 6, 6]
    bias = G.distance_bias(5, np.arange(6.0).reshape(3, 2), 4)
    assert bias.shape == (2, 5, 5) and bias[1, 4].tolist() == [5.0, 5.0, 3.0 if G.distance_bucket(2, 3, 4) == 1 else 5.0,
                                                               3.0 if G.distance_bucket(1, 3, 4) == 1 else 5.0, 1.0]


def test_oracle_temperature_sink_and_router():
    f = G.query_temperature(range(9), dict(coef=0.5, every=4))
    assert np.allclose(f[:3], 1.0) and np.allclose(f[3:7], 1 + 0.5 * np.log(2)) and np.allclose(f[7:], 1 + 0.5 * np.log(3))
    assert np.array_equal(G.query_temperature(range(3), None), np.ones(3))
    s = np.array([[0.3, -1.0], [0.1, 0.2]])
    p = G.sink_softmax(s, np.tril(np.ones((2, 2), bool)), 0.7)
    e = np.exp([0.1, 0.2])
    assert np.allclose(p[1], e / (e.sum() + np.exp(0.7))) and np.allclose(p[0], [np.exp(0.3) / (np.exp(0.3) + np.exp(0.7)), 0.0])
    w, i = G.route(np.array([[1.0]]), np.array([[2.0], [1.0], [0.0]]), np.array([0.0, 0.0, 1.5]), 2)
    assert i.tolist() == [[0, 2]] and np.allclose(w, np.exp([2.0, 1.5]) / np.exp([2.0, 1.5]).sum())


def test_oracle_recurrence_equals_its_sum():
    """o_t = sum over s <= t of v_s times k_s . q_t, each channel weighted by the product of the decays in between."""
    m = dict(heads=1, dim=3, vdim=2, tau=2.0)
    rng = np.random.default_rng(0)
    t = {n: rng.normal(size=s) for n, s in dict(q=(3, 4), k=(3, 4), v=(2, 4), a1=(2, 4), a2=(3, 2), g=(2, 4), o=(4, 2), norm=(2,)).items()}
    t["a2.b"] = rng.normal(size=3)
    h = rng.normal(size=(6, 4))
    states = []
    got = G.gla(h, m, lambda n: t[n], 1e-6, states)
    al = G.sigmoid(h @ t["a1"].T @ t["a2"].T + t["a2.b"]) ** 0.5
    q, k, v = h @ t["q"].T * 3 ** -0.5, h @ t["k"].T, h @ t["v"].T
    o = np.array([sum((q[i] * np.prod(al[j + 1:i + 1], axis=0) * k[j]).sum() * v[j] for j in range(i + 1)) for i in range(6)])
    want = (G.rms_norm(o, t["norm"], 1e-6) * G.silu(h @ t["g"].T)) @ t["o"].T
    assert np.allclose(got, want) and states[0].shape == (1, 3, 2) and np.allclose(states[0][0], np.outer(k[0], v[0]))


def test_oracle_is_causal_and_shares_keys():
    cfg = K.small()
    t = K.weights(cfg, seed=1)
    a = K.tokens(cfg, 12)
    b = a.copy()
    b[5] = (b[5] + 1) % cfg["vocab"]
    d = np.abs(G.forward(cfg, t, a) - G.forward(cfg, t, b)).max(-1)
    assert np.all(d[:5] == 0) and np.all(d[5:] > 1e-6)
    # layer 4 reads layer 1's keys: changing layer 1's key weights alone changes what layer 4 adds
    one, two = [], []
    G.forward(cfg, t, a, one)
    silent = dict(t, **{"l1.mix.o": np.zeros_like(t["l1.mix.o"])})
    other = dict(silent, **{"l1.mix.k": -t["l1.mix.k"]})
    one, two = [], []
    G.forward(cfg, silent, a, one)
    G.forward(cfg, other, a, two)
    assert np.allclose(one[3], two[3]) and np.abs(one[4] - two[4]).max() > 1e-3


def test_routing_of_the_cases_is_far_from_ties():
    """The GPU tests in bf16 rely on it: the last chosen and the first left-out expert are well apart everywhere."""
    for cfg in (K.small(), K.config([K.gla(K.moe(6, 4, 16)), K.attention(K.moe(6, 1, 16))])):
        t = {k: v.astype(np.float64) for k, v in K.weights(cfg).items()}
        gaps, used = [], []
        orig = G.route

        def spy(h, router, bias, top):
            z = np.sort(h @ router.T + bias, -1)[:, ::-1]
            gaps.append((z[:, top - 1] - z[:, top]).min())
            w, ids = orig(h, router, bias, top)
            used.append((len(np.unique(ids)), router.shape[0]))
            return w, ids

        G.route = spy
        try:
            G.forward(cfg, t, K.tokens(cfg, 80))
        finally:
            G.route = orig
        assert min(gaps) > 0.05, min(gaps)
        assert all(u >= min(n, 4) for u, n in used), used
