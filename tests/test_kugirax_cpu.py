"""Kugirax on the host: config reader, tensor mapping, registry, and properties of the plain restatement the GPU tests
compare with (oracle/kugirax.py)."""
import json

import numpy as np
import pytest

import kugirax_cases as K
from oracle import kugirax as G
from rew_b200 import _lib, kugirax, models, safetensors as st


def test_config_reader_takes_every_size_from_the_file():
    c = kugirax.config_from_json(K.small(cap=7.5, eps=2e-4), max_seq=77, dtype=_lib.BF16)
    assert (c.vocab, c.d_model, c.eps, c.max_seq, c.dtype, c.block, c.own_head) == (150, 104, 2e-4, 77, _lib.BF16, "parallel_one_norm", True)
    assert c.logit_softcap == 7.5 and kugirax.config_from_json(K.small(cap=None)).logit_softcap == 0.0
    assert [l.mixer for l in c.layers] == ["latent", "attention", "attention", "latent", "latent", "attention", "latent"]
    assert [l.ff for l in c.layers] == ["experts", "dense", "experts", "dense", "none", "none", "experts"]
    assert [(l.experts, l.top_k, l.ffn, l.router_scale, l.shared_ffn, l.shared_gate) for l in c.layers if l.ff == "experts"] == \
        [(5, 3, 24, 1.7, 40, True), (7, 2, 40, 1.7, 0, False), (5, 3, 24, 0.6, 64, True)]
    assert [l.kv_from for l in c.layers] == [-1, -1, -1, 0, -1, -1, 4]
    assert [l.window for l in c.layers] == [70, 0, 0, 9, 64, 0, 130]
    assert [(l.conv_taps, l.rope_dims, l.rope_base) for l in c.layers if l.mixer == "attention"] == [(4, 16, 700.0), (2, 32, 700.0), (3, 8, 700.0)]
    assert [(l.q_rank, l.kv_rank, l.vdim) for l in c.layers if l.mixer == "latent"] == [(36, 40, 28), (20, 40, 24), (36, 24, 28), (36, 24, 28)]
    assert all(l.sink == ("one" if l.mixer == "attention" else True) and not l.out_gate for l in c.layers)
    for change, why in ((dict(type="something"), "unknown mixer"), (dict(mlp=dict(kind="something")), "unknown feed-forward")):
        bad = K.small()
        bad["layers"][0].update(change)
        with pytest.raises(ValueError, match=why):
            kugirax.config_from_json(bad)


def test_canonical_tensors_cover_the_file_and_check_shapes():
    cfg = K.small()
    t = K.weights(cfg)
    c = kugirax.config_from_json(cfg)
    out = dict(zip([n for n, _ in c.tensor_specs()], c.canonical_tensors(t)))
    assert set(out) == set(t)
    assert np.array_equal(out["embed"], t["embed"]) and np.array_equal(out["l1.mix.q.conv"], t["l1.mix.q.conv"])      # tables stay
    for n in ("head", "l0.mix.uk", "l1.mix.k", "l0.mlp.e3.down", "l6.mlp.shared.sg", "l2.mlp.router"):
        assert np.array_equal(out[n], t[n].T)
    assert "l3.mix.dkv" not in out and "l3.mix.uk" in out and "l1.mix.v" not in out and "l1.norm2" not in out
    short = dict(t)
    del short["l5.mix.k.conv"]
    with pytest.raises(KeyError, match="l5.mix.k.conv"):
        c.canonical_tensors(short)
    with pytest.raises(ValueError, match="l0.mix.sink"):
        c.canonical_tensors(dict(t, **{"l0.mix.sink": np.zeros(9, np.float32)}))


def test_registry_picks_the_family_by_config(tmp_path):
    cfg = K.small()
    assert models.family_of(json.loads(json.dumps(cfg))) == "kugirax"
    t = K.weights(cfg, seed=3)
    st.write_safetensors(str(tmp_path / "model.safetensors"), t, dtype="BF16")
    back = st.read_safetensors_dir(str(tmp_path))
    assert set(back) == set(t) and all(np.array_equal(back[k], t[k]) for k in t)


def test_step_bytes_counts_caches_windows_and_convolution_state():
    cfg = K.config([K.attention(conv=5), K.latent(window=8)])
    c = kugirax.config_from_json(cfg, dtype=_lib.BF16)
    a, l = cfg["layers"][0]["mixer"], cfg["layers"][1]["mixer"]
    one, two, far = c.step_bytes(1, 6), c.step_bytes(1, 7), c.step_bytes(1, 100)
    per_key, per_latent = 4 * a["kv_heads"] * a["dim"], 2 * l["kv_rank"]
    assert two - one == per_key + per_latent and far - two == 93 * per_key + per_latent
    assert c.step_bytes(2, 6) - one == 6 * (per_key + per_latent) + 8 * 4 * (a["heads"] + a["kv_heads"]) * a["dim"]


# ---- the restatement itself

def test_oracle_convolution_and_rotation():
    rng = np.random.default_rng(0)
    u, w = rng.normal(size=(6, 3)), rng.normal(size=(3, 4))
    y = G.short_conv(u, w)
    for t in range(6):
        want = sum(w[:, j] * u[t - 3 + j] for j in range(4) if t - 3 + j >= 0)
        assert np.allclose(y[t], want)
    x = rng.normal(size=(9, 2, 10))
    r = G.rotated_halves(x, range(9), 50.0, 6)
    assert np.array_equal(r[..., 6:], x[..., 6:]) and np.array_equal(r[0], x[0])
    z, zr = x[..., :3] + 1j * x[..., 3:6], r[..., :3] + 1j * r[..., 3:6]
    assert np.allclose(zr, z * np.exp(1j * np.arange(9)[:, None, None] * 50.0 ** (-np.arange(3) / 3.0)))


def test_oracle_sink_window_router_and_cap():
    s = np.array([[0.3, -1.0], [0.1, 0.2]])
    e = np.exp([0.1, 0.2])
    p = G.sink_softmax(s, G.visible(2), 0.0)
    assert np.allclose(p[1], e / (1 + e.sum())) and np.allclose(p[0], [np.exp(0.3) / (1 + np.exp(0.3)), 0.0])
    assert np.allclose(G.sink_softmax(s, G.visible(2), 800.0), 0.0)
    assert G.visible(4, 2).astype(int).tolist() == [[1, 0, 0, 0], [1, 1, 0, 0], [0, 1, 1, 0], [0, 0, 1, 1]]
    w, i = G.route(np.array([[1.0]]), np.array([[2.0], [1.0], [0.0]]), 2, 3.0)
    assert i.tolist() == [[0, 1]] and np.allclose(w, 3 * np.exp([2.0, 1.0]) / np.exp([2.0, 1.0]).sum())
    assert np.allclose(G.soft_cap(np.array([1e-3, 400.0, -400.0]), 5.0), [1e-3, 5.0, -5.0]) and G.soft_cap(3.0, None) == 3.0


def test_oracle_is_causal_and_shares_latents():
    cfg = K.small()
    t = K.weights(cfg, seed=1)
    a = K.tokens(cfg, 12)
    b = a.copy()
    b[5] = (b[5] + 1) % cfg["vocab"]
    d = np.abs(G.forward(cfg, t, a) - G.forward(cfg, t, b)).max(-1)
    assert np.all(d[:5] == 0) and np.all(d[5:] > 1e-6)
    # layer 3 reads layer 0's latents: changing their projection alone changes what layer 3 adds
    silent = dict(t, **{"l0.mix.o": np.zeros_like(t["l0.mix.o"])})
    other = dict(silent, **{"l0.mix.dkv": -t["l0.mix.dkv"]})
    one, two = [], []
    G.forward(cfg, silent, a, one)
    G.forward(cfg, other, a, two)
    assert np.allclose(one[2], two[2]) and np.abs(one[3] - two[3]).max() > 1e-3


def test_routing_of_the_cases_is_far_from_ties():
    """The GPU tests in bf16 rely on it: the last chosen and the first left-out expert are well apart everywhere."""
    for cfg in (K.small(), K.config([K.attention(K.moe(6, 4, 16)), K.latent(K.moe(6, 1, 16))])):
        t = K.weights(cfg)
        gaps, used = [], []
        orig = G.route

        def spy(h, router, top, scale):
            z = np.sort(h @ router.T, -1)[:, ::-1]
            gaps.append((z[:, top - 1] - z[:, top]).min())
            w, ids = orig(h, router, top, scale)
            used.append((len(np.unique(ids)), router.shape[0]))
            return w, ids

        G.route = spy
        try:
            G.forward(cfg, t, K.tokens(cfg, 80))
        finally:
            G.route = orig
        assert min(gaps) > 0.05, gaps
        assert all(u >= min(n, 4) for u, n in used), used
