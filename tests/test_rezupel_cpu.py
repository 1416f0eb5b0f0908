"""Rezupel on the host: config reader, tensor mapping, registry, trace replay bookkeeping, and properties of the plain
restatement the GPU tests compare with (oracle/rezupel.py)."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import rezupel_cases as K
from oracle import rezupel as R
from rew_b200 import _lib, models, rezupel, safetensors as st, weights as W

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def test_config_reader_takes_every_size_from_the_file():
    cfg = K.small()
    c = rezupel.config_from_json(cfg, max_seq=77, dtype=_lib.BF16)
    assert (c.vocab, c.d_model, c.eps, c.loop, c.max_seq, c.dtype) == (152, 104, 1e-5, (1, 3, 3), 77, _lib.BF16)
    assert [l.ff for l in c.layers] == ["dense", "experts", "none", "experts", "dense"]
    assert [l.window for l in c.layers] == [37, 37, 9, 37, 64]
    assert [l.heads for l in c.layers] == [3, 3, 2, 3, 5]
    assert (c.layers[3].experts, c.layers[3].top_k, c.layers[3].ffn) == (7, 2, 40)
    assert c.layers[2].rope_base == 300.0 and c.layers[0].rope_dims == 12
    assert not c.layers[1].renormalize and not c.layers[1].expert_gated
    assert c.layer_runs == [0, 1, 2, 1, 2, 1, 2, 3, 4]
    assert rezupel.config_from_json(dict(cfg, loop=None)).loop is None
    cfg["layers"][0]["type"] = "something"
    with pytest.raises(ValueError, match="unknown mixer"):
        rezupel.config_from_json(cfg)


def test_canonical_tensors_transpose_linears_and_check_shapes():
    cfg = K.small()
    c, t = rezupel.config_from_json(cfg), K.weights(cfg)
    out = dict(zip([n for n, _ in c.tensor_specs()], rezupel.canonical_tensors(c, t)))
    assert set(out) == set(t)                                   # every tensor of the file has a place
    assert np.array_equal(out["embed"], t["embed"]) and np.array_equal(out["loop.step"], t["loop.step"])
    assert np.array_equal(out["l1.mix.uk"], t["l1.mix.uk"].T) and np.array_equal(out["l3.mlp.e6.down"], t["l3.mlp.e6.down"].T)
    bad = dict(t)
    bad["l0.mix.g"] = bad["l0.mix.g"][:2]
    with pytest.raises(ValueError, match="l0.mix.g"):
        rezupel.canonical_tensors(c, bad)
    del bad["l0.mix.g"]
    with pytest.raises(KeyError, match="l0.mix.g"):
        rezupel.canonical_tensors(c, bad)


def test_registry_picks_the_family_by_config():
    assert models.family_of(K.small()) == "rezupel"
    assert models.family_of({"architectures": ["LlamaForCausalLM"]}) == "llama"
    with pytest.raises(ValueError, match="no model family"):
        models.family_of({"architecture": "Unheard"})


def test_safetensors_round_trip_of_a_model(tmp_path):
    cfg = K.config([K.layer(K.dense(24), heads=2)], vocab=40, width=32)
    t = K.weights(cfg, seed=3)
    st.write_safetensors(str(tmp_path / "model.safetensors"), t, dtype="BF16")
    back = st.read_safetensors_dir(str(tmp_path))
    assert all(np.array_equal(back[k], t[k]) for k in t) and set(back) == set(t)


def test_struct_layouts_match_the_header(tmp_path):
    """The ctypes mirrors of rewb200_layer and rewb200_stack against gcc's view of the header."""
    src = tmp_path / "l.c"
    fields = [("rewb200_layer", _lib.Layer), ("rewb200_stack", _lib.Stack)]
    lines = ["#include <stddef.h>", "#include <stdio.h>", "#include \"rew_b200.h\"", "int main(void) {"]
    for name, cls in fields:
        lines.append('printf("%s %%zu\\n", sizeof(%s));' % (name, name))
        for f in cls._fields_:
            lines.append('printf("%s.%s %%zu\\n", offsetof(%s, %s));' % (name, f[0], name, f[0]))
    src.write_text("\n".join(lines + ["return 0; }"]))
    exe = str(tmp_path / "l")
    r = subprocess.run(["gcc", "-std=c99", "-I", os.path.join(ROOT, "include"), str(src), "-o", exe], capture_output=True, text=True)
    assert r.returncode == 0, r.stderr
    got = dict(l.split() for l in subprocess.run([exe], capture_output=True, text=True, check=True).stdout.splitlines())
    import ctypes
    for name, cls in fields:
        assert int(got[name]) == ctypes.sizeof(cls)
        for f in cls._fields_:
            assert int(got["%s.%s" % (name, f[0])]) == getattr(cls, f[0]).offset


def test_trace_replay_maps_requests_to_lanes():
    """Lane bookkeeping of the trace runner with a stand-in session: order of the wanted logits, reuse of lanes."""
    from rew_b200 import trace_run

    class FakeSession:
        def __init__(self):
            self.calls, self.released = [], []
            self.model = type("M", (), {"cfg": type("C", (), {"vocab": 3})()})()

        def feed(self, portions, want=()):
            self.calls.append((portions, list(want)))
            flat = [t for _, ids in portions for t in ids]
            return np.array([[flat[w]] * 3 for w in want], np.float32).reshape(-1, 3), None

        def release(self, lane):
            self.released.append(lane)

    class FakeModel:
        def paged_session(self, lanes, max_len, blocks):
            self.args = (lanes, max_len, blocks)
            return FakeSession()

    fm = FakeModel()
    r = trace_run.Replay(fm, 130)
    assert fm.args == (4, 192, 4)
    got = r.step([dict(id="a", tokens=[5, 6, 7], want=[2, 0]), dict(id="b", tokens=[9], want=[0])], [])
    assert got[:, 0].tolist() == [7, 5, 9]
    assert len(r.step([dict(id="b", tokens=[1, 2], want=[])], ["a"])) == 0
    r.step([dict(id=i, tokens=[1], want=[]) for i in "cde"], [])
    assert r.session.released == [0] and len(r.lanes) == 4 and r.lanes["e"] == 0
    with pytest.raises(ValueError, match="live requests"):
        r.step([dict(id="f", tokens=[1], want=[])], [])


def test_trace_runner_without_a_gpu_fails_loudly(tmp_path):
    import torch
    if torch.cuda.is_available():
        pytest.skip("a GPU is present")
    cfg = K.config([K.layer(K.dense(24), heads=2)], vocab=40, width=32)
    st.write_safetensors(str(tmp_path / "model.safetensors"), K.weights(cfg), dtype="BF16")
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "bfloat16", "--out", str(tmp_path),
                        "--max-tokens", "64"], input='{"step": 0, "entries": [{"id": "a", "tokens": [1], "want": [0]}], "end": []}\n',
                       capture_output=True, text=True)
    assert r.returncode != 0 and "no CUDA device" in r.stderr and "done" not in r.stdout


# ---- the restatement itself

def test_oracle_rotation_is_relative_and_leaves_the_rest():
    rng = np.random.default_rng(0)
    a, b = rng.normal(size=(1, 10)), rng.normal(size=(1, 10))
    def dot(p, q):
        return (R.rotate_interleaved(a, [p], 100.0, 6) * R.rotate_interleaved(b, [q], 100.0, 6)).sum()
    assert abs(dot(3, 7) - dot(10, 14)) < 1e-12 and abs(dot(3, 7) - dot(3, 8)) > 1e-3
    assert np.array_equal(R.rotate_interleaved(a, [9], 100.0, 6)[:, 6:], a[:, 6:])
    u = R.rotate_interleaved(np.array([[1.0, 0.0]]), [2], 10.0, 2)
    np.testing.assert_allclose(u, [[np.cos(2.0), np.sin(2.0)]])


def test_oracle_window_and_router():
    v = R.window_visible(6, 3)
    assert v[5].tolist() == [False, False, False, True, True, True] and v[0].tolist() == [True] + [False] * 5
    z = np.array([[2.0, 1.0, 0.0, -1.0]])
    w, i = R.route(np.array([[1.0]]), z.T, 2)
    p = np.exp(z[0]) / np.exp(z[0]).sum()
    assert i.tolist() == [[0, 1]] and np.allclose(w, p[:2]) and w.sum() < 1.0


def test_oracle_loop_adds_embedding_and_steps():
    """With every branch silenced the residual is the embedding once per pass plus the step vectors."""
    cfg = K.small()
    t = {k: v.astype(np.float64) for k, v in K.weights(cfg).items()}
    for k in t:
        if k.endswith(("mix.o", ".down")):
            t[k] = np.zeros_like(t[k])
    ids = K.tokens(cfg, 4)
    col = []
    R.forward(cfg, t, ids, col)
    x0 = t["embed"][ids]
    np.testing.assert_allclose(col[0], x0)
    for run, p in ((1, 0), (2, 0), (3, 1), (6, 2), (8, 2)):
        np.testing.assert_allclose(col[run], (p + 1) * x0 + t["loop.step"][:p + 1].sum(0))


def test_oracle_is_causal_and_windowed():
    cfg = K.config([K.layer(K.dense(24), window=5)])
    t = K.weights(cfg, seed=1)
    a = K.tokens(cfg, 12)
    b = a.copy()
    b[3] = (b[3] + 1) % cfg["vocab"]
    d = np.abs(R.forward(cfg, t, a) - R.forward(cfg, t, b)).max(-1)
    assert np.all(d[:3] == 0) and np.all(d[3:8] > 1e-6) and np.all(d[8:] == 0)


def test_routing_of_the_cases_is_far_from_ties():
    """The GPU tests in bf16 rely on it: the last chosen and the first left-out expert are well apart everywhere."""
    cfg = K.small()
    t = {k: v.astype(np.float64) for k, v in K.weights(cfg).items()}
    gaps = []
    orig = R.route

    def spy(h, router, top):
        z = np.sort(h @ router.T, -1)[:, ::-1]
        gaps.append((z[:, top - 1] - z[:, top]).min())
        return orig(h, router, top)

    R.route = spy
    try:
        R.forward(cfg, t, K.tokens(cfg, 60))
    finally:
        R.route = orig
    assert min(gaps) > 0.05, min(gaps)
