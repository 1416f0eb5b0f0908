"""Musavik on the host: config reader, tensor mapping, registry, and properties of the plain restatement the GPU tests
compare with (oracle/musavik.py)."""
import json

import numpy as np
import pytest

import musavik_cases as K
from oracle import musavik as G
from rew_b200 import _lib, models, musavik, safetensors as st


def test_config_reader_takes_every_size_from_the_file():
    c = musavik.config_from_json(K.small(eps=2e-4, scale=0.3, bigram=(41, 7, 13)), max_seq=77, dtype=_lib.BF16)
    assert (c.vocab, c.d_model, c.eps, c.max_seq, c.dtype, c.block, c.own_head, c.norm_zero_centred) == (150, 104, 2e-4, 77, _lib.BF16, "sandwich", True, True)
    assert c.embed_scale == 0.3 and c.bigram == (41, 7, 13) and c.loop == (1, 4, 2) and c.loop_in
    assert c.layer_runs == [0, 1, 2, 3, 1, 2, 3, 4, 5]
    assert [l.mixer for l in c.layers] == ["lru", "attention", "lru", "attention", "attention", "lru"]
    assert [(l.ff, l.ffn) for l in c.layers] == [("dense", 56), ("dense", 88), ("none", 0), ("none", 0), ("dense", 40), ("dense", 88)]
    assert all(l.ff_act == "gelu_tanh" and l.ff_bias for l in c.layers if l.ff == "dense")
    assert [(l.heads, l.dim, l.vdim, l.conv_taps) for l in c.layers if l.mixer == "lru"] == [(3, 24, 24, 4), (2, 40, 40, 3), (8, 8, 8, 2)]
    left = [l for l in c.layers if l.mixer == "attention"]
    assert [(l.heads, l.kv_heads, l.dim, l.vdim, l.rope_dims, l.window, l.keep_first, l.mix_scale) for l in left] == \
        [(4, 2, 24, 40, 16, 70, 5, 1.2), (6, 1, 32, 16, 32, 9, 0, 1.2), (3, 3, 16, 24, 8, 130, 70, 0.5)]
    assert all(l.head_mix and l.qkv_bias and l.v_norm and l.qk_norm and l.rope_pairs and l.gate_kind == 2 for l in left)
    right = [l.beside for l in left]
    assert [(l.mixer, l.heads, l.kv_heads, l.dim, l.vdim, l.conv_taps, l.mix_scale) for l in right] == \
        [("delta", 3, 3, 16, 24, 4, 0.7), ("delta", 4, 2, 24, 40, 2, 0.7), ("delta", 2, 1, 40, 16, 3, 1.5)]
    plain = musavik.config_from_json(K.small(loop=None))
    assert plain.loop is None and not plain.loop_in and "loop.in" not in dict(plain.tensor_specs())
    for change, why in ((dict(type="something"), "unknown mixer"), (dict(mlp=dict(kind="something")), "unknown feed-forward"),
                        (dict(mixer=dict(width=10, blocks=3, conv=2)), "do not divide")):
        bad = K.small()
        bad["layers"][0].update(change)
        with pytest.raises(ValueError, match=why):
            musavik.config_from_json(bad)


def test_canonical_tensors_cover_the_file_and_check_shapes():
    cfg = K.small()
    t = K.weights(cfg)
    c = musavik.config_from_json(cfg)
    out = dict(zip([n for n, _ in c.tensor_specs()], c.canonical_tensors(t)))
    assert set(out) == set(t)
    for n in ("embed", "bigram", "l0.mix.conv", "l1.mix.left.talk", "l1.mix.right.v.conv", "l1.mix.left.q.b"):      # tables stay
        assert np.array_equal(out[n], t[n])
    for n in ("head", "loop.in", "l1.mix.left.g", "l1.mix.right.b", "l3.mix.right.o", "l0.mlp.down"):
        assert np.array_equal(out[n], t[n].T)
    assert np.array_equal(out["l0.mix.ra"], t["l0.mix.ra"].reshape(72, 24)) and np.array_equal(out["l0.mix.ri.b"], t["l0.mix.ri.b"].reshape(72))
    assert "l2.norm2" not in out and "l0.norm2b" in out
    short = dict(t)
    del short["l3.mix.right.dt_bias"]
    with pytest.raises(KeyError, match="l3.mix.right.dt_bias"):
        c.canonical_tensors(short)
    with pytest.raises(ValueError, match="l1.mix.left.talk"):
        c.canonical_tensors(dict(t, **{"l1.mix.left.talk": np.zeros((4, 5), np.float32)}))


def test_registry_picks_the_family_by_config(tmp_path):
    cfg = K.small()
    assert models.family_of(json.loads(json.dumps(cfg))) == "musavik"
    t = K.weights(cfg, seed=3)
    st.write_safetensors(str(tmp_path / "model.safetensors"), t, dtype="BF16")
    back = st.read_safetensors_dir(str(tmp_path))
    assert set(back) == set(t) and all(np.array_equal(back[k], t[k]) for k in t)


def test_step_bytes_counts_windows_states_and_passes():
    cfg = K.config([K.parallel(size=10, keep=3)])
    c = musavik.config_from_json(cfg, dtype=_lib.BF16)
    m = cfg["layers"][0]["mixer"]
    a, r = m["left"], m["right"]
    per_key = 2 * a["kv_heads"] * (a["dim"] + a["vdim"])
    assert c.step_bytes(1, 7) - c.step_bytes(1, 6) == per_key and c.step_bytes(1, 500) - c.step_bytes(1, 6) == 7 * per_key
    state = r["heads"] * r["dim"] * r["vdim"] + (r["conv"] - 1) * (2 * r["kv_heads"] * r["dim"] + r["heads"] * r["vdim"])
    assert c.step_bytes(2, 6) - c.step_bytes(1, 6) == 6 * per_key + 8 * state
    one, two = (musavik.config_from_json(K.config([K.rglru()], loop=dict(start=0, stop=1, times=n)), dtype=_lib.BF16) for n in (1, 2))
    d, w, n = 104, 72, 24
    assert two.step_bytes(1, 6) - one.step_bytes(1, 6) == 2 * (3 * d * w + 2 * w * n + 4 * w + 2 * d * d) + 8 * 4 * w


# ---- the restatement itself

def test_oracle_embedding_and_loop():
    cfg = K.config([K.rglru()], vocab=9, width=4, scale=0.5, bigram=(7, 3, 5))
    t = K.weights(cfg)
    x = G.embedding(cfg, t, [2, 8, 2])
    assert G.bigram_rows([2, 8, 2], cfg["embedding"]["bigram"]) == [7, (2 * 3 + 8 * 5) % 7, (8 * 3 + 2 * 5) % 7]
    assert np.allclose(x[1], 0.5 * t["embed"][8] + t["bigram"][46 % 7]) and np.allclose(x[0], 0.5 * t["embed"][2] + t["bigram"][7])
    runs = G.layer_runs(dict(layers=[0] * 4, loop=dict(start=1, stop=3, times=2)))
    assert runs == [(0, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    # with W_in = [0 | I] every pass starts from the embeddings: two passes end where one does
    cfg = K.small()
    t = K.weights(cfg, seed=1)
    t["loop.in"] = np.concatenate([np.zeros((104, 104)), np.eye(104)], 1).astype(np.float32)
    one, two = [], []
    ids = K.tokens(cfg, 12)
    G.forward(dict(cfg, loop=dict(start=1, stop=4, times=1)), t, ids, one)
    G.forward(cfg, t, ids, two)
    assert np.allclose(one[-1], two[-1]) and np.allclose(two[1:4], two[4:7])


def test_oracle_rotation_mask_and_mixing():
    rng = np.random.default_rng(0)
    x = rng.normal(size=(9, 2, 10))
    r = G.rotated_pairs(x, range(9), 50.0, 6)
    assert np.array_equal(r[..., 6:], x[..., 6:]) and np.array_equal(r[0], x[0])
    z, zr = x[..., 0:6:2] + 1j * x[..., 1:6:2], r[..., 0:6:2] + 1j * r[..., 1:6:2]
    assert np.allclose(zr, z * np.exp(1j * np.arange(9)[:, None, None] * 50.0 ** (-np.arange(3) / 3.0)))
    assert G.visible(5, 2, 1).astype(int).tolist() == [[1, 0, 0, 0, 0], [1, 1, 0, 0, 0], [1, 1, 1, 0, 0], [1, 0, 1, 1, 0], [1, 0, 0, 1, 1]]
    p = rng.random((2, 3, 3))
    assert np.allclose(G.talk(p, np.array([[1.0, -2.0], [0.5, 0.0]])), [p[0] - 2 * p[1], 0.5 * p[0]])
    y = G.short_conv(rng.normal(size=(6, 3)) * 0 + np.arange(6)[:, None], np.array([[1.0, 0, 0, 10.0]] * 3))
    assert np.allclose(y[:, 0], [0, 10, 20, 30, 41, 52])


def test_oracle_delta_rule_stores_and_overwrites():
    """With step one and no decay, reading a stored key returns its latest value, whatever was stored at other (orthogonal) keys."""
    m = dict(heads=1, kv_heads=1, dim=4, vdim=2, conv=1)
    big = 50.0
    w = {"q": np.eye(4), "k": np.eye(4), "v": np.zeros((2, 4)), "q.conv": np.full((4, 1), big), "k.conv": np.full((4, 1), big),
         "v.conv": np.ones((2, 1)), "b": np.full((1, 4), big), "a": np.zeros((1, 4)), "A_log": np.full(1, -50.0), "dt_bias": np.zeros(1),
         "norm": np.ones(2), "g": np.ones((2, 4)), "o": np.eye(2)}
    states = []
    h = np.eye(4)[[0, 1, 0]]
    w["v"] = np.array([[3.0, 5.0, 0, 0], [1.0, 2.0, 0, 0]])
    G.delta_rule(h, m, lambda n: w[n], 1e-5, states)
    assert np.allclose(states[2][0, 0], G.silu(w["v"][:, 0]), atol=1e-4) and np.allclose(states[2][0, 1], G.silu(w["v"][:, 1]), atol=1e-4)


def test_oracle_recurrent_unit_keeps_and_forgets():
    m = dict(width=2, blocks=1, conv=1)
    w = {"y": np.eye(2), "y.b": np.zeros(2), "x": np.eye(2), "x.b": np.zeros(2), "conv": np.ones((2, 1)), "conv.b": np.zeros(2),
         "ra": np.zeros((1, 2, 2)), "ra.b": np.full((1, 2), 50.0), "ri": np.zeros((1, 2, 2)), "ri.b": np.full((1, 2), 50.0),
         "lam": np.array([-50.0, 50.0]), "o": np.eye(2)}
    states = []
    G.rglru(np.array([[1.0, 1.0], [2.0, 3.0]]), m, lambda n: w[n], states)
    assert np.allclose(states[1], [0.0, 3.0], atol=1e-6)      # a = 1: nothing enters; a = 0: only the current input


def test_oracle_is_causal():
    cfg = K.small()
    t = K.weights(cfg, seed=1)
    a = K.tokens(cfg, 12)
    b = a.copy()
    b[5] = (b[5] + 1) % cfg["vocab"]
    d = np.abs(G.forward(cfg, t, a) - G.forward(cfg, t, b)).max(-1)
    assert np.all(d[:5] == 0) and np.all(d[5:] > 1e-6)
