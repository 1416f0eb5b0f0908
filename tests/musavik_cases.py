"""Small Musavik configurations with seeded weights, shared by the tests."""
import numpy as np

from rew_b200.weights import bf16_round


def dense(ff=88):
    return dict(kind="dense", ff=ff)


def parallel(mlp=None, heads=4, kv_heads=2, dim=24, vdim=40, rot=16, base=700.0, size=70, keep=5, scale=None, right=(3, 3, 16, 24, 4), scales=(1.2, 0.7)):
    """right: heads, kv_heads, dim, vdim and taps of the delta rule."""
    left = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, rot=dict(base=base, dims=rot), mask=dict(size=size, keep_first=keep),
                scale=dim ** -0.5 if scale is None else scale)
    return dict(type="parallel", mlp=mlp, mixer=dict(left=left, right=dict(zip(("heads", "kv_heads", "dim", "vdim", "conv"), right)),
                                                     left_scale=scales[0], right_scale=scales[1]))


def rglru(mlp=None, width=72, blocks=3, conv=4):
    return dict(type="rglru", mlp=mlp, mixer=dict(width=width, blocks=blocks, conv=conv))


def config(layers, vocab=150, width=104, eps=1e-5, scale=0.6, bigram=(37, 5, 11), loop=None):
    cfg = dict(architecture="Musavik", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers, loop=loop,
               embedding=dict(scale=scale, bigram=dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))))
    return cfg


def small(**kw):
    """Every branch of the design: both mixers in several sizes, feed-forwards and none, a loop in the middle of the stack."""
    return config([rglru(dense(56)), parallel(dense()), rglru(None, width=80, blocks=2, conv=3),
                   parallel(None, heads=6, kv_heads=1, dim=32, vdim=16, rot=32, size=9, keep=0, right=(4, 2, 24, 40, 2)),
                   parallel(dense(40), heads=3, kv_heads=3, dim=16, vdim=24, rot=8, size=130, keep=70, right=(2, 1, 40, 16, 3), scales=(0.5, 1.5)), rglru(dense(), width=64, blocks=8, conv=2)],
                  **{**dict(loop=dict(start=1, stop=4, times=2)), **kw})


def weights(cfg, seed=0, score_gain=1.0, forget=0.0):
    """{name: float32 array, bf16-representable}, Linear weights [out, in].  score_gain sharpens the attention, forget moves
    the decays of both recurrences (negative: longer memory)."""
    rng = np.random.default_rng(seed)
    d, t = cfg["width"], {}

    def lin(o, i, gain=1.0):
        return rng.normal(0, gain * i ** -0.5, size=(o, i))

    def bias(n):
        return rng.normal(0, 0.3, size=n)

    def near_one(n):
        return 1 + rng.normal(0, 0.2, size=n)

    def near_zero(n):
        return rng.normal(0, 0.2, size=n)

    t["embed"] = rng.normal(0, 1.5, size=(cfg["vocab"], d))
    t["bigram"] = rng.normal(0, 0.7, size=(cfg["embedding"]["bigram"]["buckets"] + 1, d))
    if cfg["loop"]:
        t["loop.in"] = lin(d, 2 * d, 1.4)
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], "l%d." % i
        x = p + "mix."
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if L["mlp"] else ()):
            t[p + n] = near_zero(d)
        if L["type"] == "parallel":
            a, y = m["left"], x + "left."
            H, G, K, V = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            for n, o in (("q", H * K), ("k", G * K), ("v", G * V)):
                t[y + n], t[y + n + ".b"] = lin(o, d), bias(o)
            t[y + "q.norm"], t[y + "k.norm"] = near_one(K) * score_gain, near_one(K)
            t[y + "talk"] = np.eye(H) + rng.normal(0, 0.4, size=(H, H))
            t[y + "g"], t[y + "o"] = lin(H * V, d), lin(d, H * V, 1.5)
            a, y = m["right"], x + "right."
            H, G, K, V = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            for n, o in (("q", G * K), ("k", G * K), ("v", H * V)):
                t[y + n], t[y + n + ".conv"] = lin(o, d), lin(o, a["conv"], 1.4)
            t[y + "b"], t[y + "a"] = lin(H, d), lin(H, d)
            t[y + "A_log"], t[y + "dt_bias"] = rng.normal(-1.0, 0.7, size=H), rng.normal(-1.0 + forget, 0.7, size=H)
            t[y + "norm"], t[y + "g"], t[y + "o"] = near_one(V), lin(H * V, d), lin(d, H * V, 1.5)
        else:
            w, n = m["width"], m["width"] // m["blocks"]
            for b in ("y", "x"):
                t[x + b], t[x + b + ".b"] = lin(w, d), bias(w)
            t[x + "conv"], t[x + "conv.b"] = lin(w, m["conv"], 1.4), bias(w)
            for b in ("ra", "ri"):
                t[x + b], t[x + b + ".b"] = rng.normal(0, 1.5 * n ** -0.5, size=(m["blocks"], n, n)), bias((m["blocks"], n))
            t[x + "lam"] = rng.normal(-2.5 + forget, 1.0, size=w)
            t[x + "o"] = lin(d, w, 1.5)
        if L["mlp"] is None:
            continue
        f, q = L["mlp"]["ff"], p + "mlp."
        t[q + "up"], t[q + "up.b"], t[q + "down"], t[q + "down.b"] = lin(f, d, 1.5), bias(f), lin(d, f), bias(d)
    t["final.norm"] = near_zero(d)
    t["head"] = lin(cfg["vocab"], d, 2.0)
    return {k: bf16_round(np.asarray(v, np.float32)) for k, v in t.items()}


def tokens(cfg, n, seed=0):
    return np.random.default_rng(1000 + seed).integers(0, cfg["vocab"], size=n).astype(np.int32)


def marked(layer, seed=0):
    """One attention layer (its delta rule and feed-forward silent) in which three kinds of tokens matter: a filler, a key and a
    query whose score with the key stands out far above all others.  Returns (cfg, tensors, filler, key, query)."""
    assert layer["type"] == "parallel" and layer["mlp"] is None
    cfg = config([layer], vocab=96, width=88, scale=1.0)
    t = {k: v.copy() for k, v in weights(cfg, seed=seed).items()}
    m, p = layer["mixer"]["left"], "l0.mix.left."
    H, G, K = m["heads"], m["kv_heads"], m["dim"]
    filler, key, query = 1, 2, 3
    t["bigram"][:] = 0.0
    t["l0.norm1"][:] = 0.0
    t["l0.mix.right.o"][:] = 0.0
    for tok, col in ((key, 0), (query, 1)):
        t["embed"][tok] = 0.0
        t["embed"][tok, col] = 8.0
    t["embed"][filler, :2] = 0.0
    # the marks meet in the last feature of every head, which must not be rotated
    assert m["rot"]["dims"] < K
    for n, col, heads in (("k", 0, G), ("q", 1, H)):
        last = np.arange(heads) * K + K - 1
        t[p + n][last] = 0.0
        t[p + n][last, col] = 8.0
        t[p + n + ".b"][last] = 0.0
        t[p + n + ".norm"][K - 1] = 2.5
    return cfg, {k: bf16_round(v) for k, v in t.items()}, filler, key, query
