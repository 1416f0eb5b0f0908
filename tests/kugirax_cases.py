"""Small Kugirax configurations with seeded weights, shared by the tests.

Expert choices must not hang on rounding, or a bf16 run could pick another expert than the float64 restatement: the
first features of the residual (as many as the widest router has experts) are reserved for the router.  Every token's
embedding holds a shuffled ladder of values there, no layer writes to them, the norm weighs them alike, and the router
reads (almost) only them.
"""
import numpy as np

from rew_b200.weights import bf16_round


def dense(ff=88):
    return dict(kind="dense", ff=ff)


def moe(experts=5, top=3, ff=24, shared=40, scale=1.7):
    m = dict(kind="moe", router=dict(experts=experts, top=top, scale=scale), expert=dict(ff=ff))
    if shared:
        m["shared"] = dict(ff=shared)
    return m


def attention(mlp=None, heads=4, kv_heads=2, dim=24, conv=4, rot=16, base=700.0, scale=None):
    return dict(type="attention", mlp=mlp,
                mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, conv=conv, rot=dict(base=base, dims=rot),
                           scale=dim ** -0.5 if scale is None else scale))


def latent(mlp=None, heads=3, dim=20, vdim=28, q_rank=36, kv_rank=40, window=37, scale=None, kv_from=None):
    m = dict(heads=heads, dim=dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, mask=dict(size=window), scale=dim ** -0.5 if scale is None else scale)
    if kv_from is not None:
        m["kv_from"] = kv_from
    return dict(type="latent_attention", mixer=m, mlp=mlp)


def config(layers, vocab=150, width=104, eps=1e-5, cap=5.0):
    cfg = dict(architecture="Kugirax", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers)
    if cap:
        cfg["logit_softcap"] = cap
    return cfg


def small(**kw):
    """Every branch of the design: both mixers, latents of another layer, dense, routed (with and without a shared expert)
    and absent feed-forwards."""
    return config([latent(moe(), window=70), attention(dense()), attention(moe(experts=7, top=2, ff=40, shared=0), heads=6, kv_heads=1, dim=32, rot=32, conv=2),
                   latent(dense(56), heads=5, dim=16, vdim=24, q_rank=20, window=9, kv_from=0), latent(None, heads=2, kv_rank=24, window=64),
                   attention(None, heads=2, kv_heads=2, dim=16, rot=8, conv=3), latent(moe(shared=64, scale=0.6), window=130, kv_from=4, kv_rank=24)], **kw)


def weights(cfg, seed=0, score_gain=1.0):
    """{name: float32 array, bf16-representable}, Linear weights [out, in].  score_gain sharpens the attention."""
    rng = np.random.default_rng(seed)
    d, t = cfg["width"], {}
    E = max([l["mlp"]["router"]["experts"] for l in cfg["layers"] if l["mlp"] and l["mlp"]["kind"] == "moe"] or [0])
    assert E < d // 2

    def lin(o, i, gain=1.0):
        return rng.normal(0, gain * i ** -0.5, size=(o, i))

    def into_residual(i, gain=1.0):
        w = lin(d, i, gain)
        w[:E] = 0.0
        return w

    def norm(n):
        return 1 + rng.normal(0, 0.2, size=n)

    t["embed"] = rng.normal(0, 1.0, size=(cfg["vocab"], d))
    for v in range(cfg["vocab"]):
        t["embed"][v, :E] = rng.permutation(np.linspace(-2.0, 2.0, E)) if E else []
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], "l%d." % i
        x, H, K, V = p + "mix.", m["heads"], m["dim"], m["vdim"]
        t[p + "norm1"] = norm(d)
        t[p + "norm1"][:E] = 1.0
        if L["type"] == "attention":
            G, taps = m["kv_heads"], m["conv"]
            t[x + "q"], t[x + "k"] = lin(H * K, d, score_gain), lin(G * K, d)
            t[x + "q.conv"], t[x + "k.conv"] = lin(H * K, taps, 1.4), lin(G * K, taps, 1.4)
        else:
            t[x + "dq"], t[x + "dq.norm"], t[x + "uq"] = lin(m["q_rank"], d), norm(m["q_rank"]), lin(H * K, m["q_rank"], score_gain)
            if m.get("kv_from") is None:
                t[x + "dkv"], t[x + "dkv.norm"] = lin(m["kv_rank"], d), norm(m["kv_rank"])
            t[x + "uk"], t[x + "uv"] = lin(H * K, m["kv_rank"]), lin(H * V, m["kv_rank"])
            t[x + "sink"] = rng.normal(1.0, 1.0, size=H)
        t[x + "o"] = into_residual(H * V, 1.5)
        if L["mlp"] is None:
            continue
        q = p + "mlp."
        if L["mlp"]["kind"] == "dense":
            f = L["mlp"]["ff"]
            t[q + "gate"], t[q + "up"], t[q + "down"] = lin(f, d, 1.5), lin(f, d, 1.5), into_residual(f)
            continue
        e_n, f = L["mlp"]["router"]["experts"], L["mlp"]["expert"]["ff"]
        r = rng.normal(0, 0.002, size=(e_n, d))
        r[np.arange(e_n), rng.permutation(E)[:e_n]] += 1.5
        t[q + "router"] = r
        for e in ["e%d." % e for e in range(e_n)]:
            t[q + e + "gate"], t[q + e + "up"], t[q + e + "down"] = lin(f, d, 1.5), lin(f, d, 1.5), into_residual(f, 1.5)
        if L["mlp"].get("shared"):
            f = L["mlp"]["shared"]["ff"]
            t[q + "shared.gate"], t[q + "shared.up"], t[q + "shared.down"] = lin(f, d, 1.5), lin(f, d, 1.5), into_residual(f)
            t[q + "shared.sg"] = lin(1, d, 2.0)
    t["final.norm"] = norm(d)
    t["head"] = lin(cfg["vocab"], d, 2.0)
    return {k: bf16_round(np.asarray(v, np.float32)) for k, v in t.items()}


def tokens(cfg, n, seed=0):
    return np.random.default_rng(1000 + seed).integers(0, cfg["vocab"], size=n).astype(np.int32)


def marked(layer, seed=0):
    """One layer without a feed-forward in which three kinds of tokens matter: a filler, a key and a query whose score with
    the key stands out far above all others.  Returns (cfg, tensors, filler, key, query)."""
    cfg = config([layer], vocab=96, width=88)
    t = {k: v.copy() for k, v in weights(cfg, seed=seed).items()}
    m = layer["mixer"]
    H, K = m["heads"], m["dim"]
    filler, key, query = 1, 2, 3
    t["l0.norm1"][:] = 1.0
    for tok, col in ((key, 0), (query, 1)):
        t["embed"][tok] = 0.0
        t["embed"][tok, col] = 8.0
    t["embed"][filler, :2] = 0.0
    if layer["type"] == "attention":
        # the marks meet in the last feature of every head, which must not be rotated, nor smeared by the convolution
        assert m["rot"]["dims"] < K
        for n, col, heads in (("k", 0, m["kv_heads"]), ("q", 1, H)):
            last = np.arange(heads) * K + K - 1
            t["l0.mix." + n][:, col] = 0.0
            t["l0.mix." + n][last] = 0.0
            t["l0.mix." + n][last, col] = 1.5
            t["l0.mix." + n + ".conv"][last] = 0.0
            t["l0.mix." + n + ".conv"][last, -1] = 1.0
        for n in ("q", "k"):                        # the mark is also the key's value: the rest is kept small
            t["l0.mix." + n] *= np.where(np.arange(len(t["l0.mix." + n])) % K == K - 1, 1.0, 0.25).astype(np.float32)[:, None]
    else:
        for n, col in (("dkv", 0), ("dq", 1)):
            t["l0.mix." + n][:, col] = 0.0
            t["l0.mix." + n][0] = 0.0
            t["l0.mix." + n][0, col] = 4.0
        t["l0.mix.uq"][:, 0] = 0.0
        t["l0.mix.uk"][:, 0] = 0.0
        t["l0.mix.uq"][np.arange(H) * K, 0] = 6.0
        t["l0.mix.uk"][np.arange(H) * K, 0] = 4.0
    return cfg, {k: bf16_round(v) for k, v in t.items()}, filler, key, query
