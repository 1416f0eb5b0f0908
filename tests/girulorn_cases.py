"""Small Girulorn configurations with seeded weights, shared by the tests.

Expert choices must not hang on rounding, or a bf16 run could pick another expert than the float64 restatement: the
first features of the residual (as many as the widest router has experts) are reserved for the router.  Every token's
embedding holds a shuffled ladder of values there, the sublayers' norm weights are zero there, and the router reads
(almost) only them.
"""
import numpy as np

from rew_b200.weights import bf16_round


def moe(experts=5, top=3, ff=24, shared=40):
    m = dict(kind="moe", router=dict(experts=experts, top=top), expert=dict(ff=ff))
    if shared:
        m["shared"] = dict(ff=shared)
    return m


def attention(mlp=None, heads=4, kv_heads=2, dim=24, vdim=40, scale=None, bias_max=50, rows=12, temp=(0.4, 16), kv_from=None):
    """rows: rows of the bias table (not part of the config: the tensor's shape says it)."""
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=dim ** -0.5 if scale is None else scale, bias_max=bias_max)
    if temp:
        m["q_temp"] = dict(coef=temp[0], every=temp[1])
    if kv_from is not None:
        m["kv_from"] = kv_from
    return dict(type="attention", mixer=m, mlp=mlp, _rows=rows)


def gla(mlp=None, heads=3, dim=32, vdim=24, tau=8.0, rank=6):
    return dict(type="gla", mixer=dict(heads=heads, dim=dim, vdim=vdim, tau=tau), mlp=mlp, _rank=rank)


def config(layers, vocab=152, width=104, eps=1e-5):
    return dict(architecture="Girulorn", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers)


def public(cfg):
    """The configuration as a file holds it."""
    return dict(cfg, layers=[{k: v for k, v in l.items() if not k.startswith("_")} for l in cfg["layers"]])


def small(**kw):
    """Every branch of the design: both mixers, keys and values of another layer, routed feed-forwards with and without a
    shared expert, and none at all."""
    return config([gla(moe()), attention(moe(experts=7, top=2, ff=40, shared=0)), attention(None, heads=6, kv_heads=1, dim=32, rows=7, temp=None),
                   gla(None, heads=2, dim=16, vdim=48, tau=2.0, rank=3), attention(moe(), heads=4, kv_from=1, rows=16, bias_max=90)], **kw)


def weights(cfg, seed=0, score_gain=1.0, decay=2.0):
    """{name: float32 array, bf16-representable}, Linear weights [out, in].  score_gain sharpens the attention; decay is the
    middle of the decay logits."""
    rng = np.random.default_rng(seed)
    d, t = cfg["width"], {}
    E = max([l["mlp"]["router"]["experts"] for l in cfg["layers"] if l["mlp"]] or [0])
    assert E < d // 2

    def lin(o, i, gain=1.0):
        return rng.normal(0, gain * i ** -0.5, size=(o, i))

    def norm(n):
        return 1 + rng.normal(0, 0.2, size=n)

    def back(n):
        w = norm(n)
        w[:E] = 0.0
        return w

    t["embed"] = rng.normal(0, 1.0, size=(cfg["vocab"], d))
    for v in range(cfg["vocab"]):
        t["embed"][v, :E] = rng.permutation(np.linspace(-2.0, 2.0, E)) if E else []
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], "l%d." % i
        x, H, K, V = p + "mix.", m["heads"], m["dim"], m["vdim"]
        t[p + "norm1"] = back(d)
        if L["type"] == "attention":
            G = m["kv_heads"]
            t[x + "q"] = lin(H * K, d)
            if m.get("kv_from") is None:
                t[x + "k"], t[x + "v"], t[x + "k.norm"] = lin(G * K, d), lin(G * V, d), norm(K)
            t[x + "q.norm"] = norm(K) * score_gain
            t[x + "rel"] = rng.normal(0, 1.5, size=(L["_rows"], H))
            t[x + "sink"] = rng.normal(1.0, 1.0, size=H)
            t[x + "g"] = lin(H, d, 2.0)
        else:
            t[x + "q"], t[x + "k"], t[x + "v"] = lin(H * K, d), lin(H * K, d), lin(H * V, d)
            t[x + "a1"], t[x + "a2"] = lin(L["_rank"], d), lin(H * K, L["_rank"], 2.0)
            t[x + "a2.b"] = rng.normal(decay, 1.0, size=H * K)
            t[x + "g"], t[x + "norm"] = lin(H * V, d), norm(V)
        t[x + "o"] = lin(d, H * V)
        if L["mlp"] is None:
            continue
        q = p + "mlp."
        t[p + "norm2"] = back(d)
        e_n, f = L["mlp"]["router"]["experts"], L["mlp"]["expert"]["ff"]
        r = rng.normal(0, 0.002, size=(e_n, d))
        r[np.arange(e_n), rng.permutation(E)[:e_n]] += 1.5
        t[q + "router"] = r
        # the bias moves the choice: by whole rungs of the ladder, plus a fraction of one of its own for every expert
        rung = 1.5 * 4.0 / max(E - 1, 1)
        t[q + "router.b"] = rung * (rng.integers(-1, 2, size=e_n) + rng.permutation(e_n) / (e_n + 1.0))
        for e in ["e%d." % e for e in range(e_n)]:
            t[q + e + "gate"], t[q + e + "up"], t[q + e + "down"] = lin(f, d, 1.5), lin(f, d, 1.5), lin(d, f, 1.5)
        if L["mlp"].get("shared"):
            f = L["mlp"]["shared"]["ff"]
            t[q + "shared.gate"], t[q + "shared.up"], t[q + "shared.down"] = lin(f, d, 1.5), lin(f, d, 1.5), lin(d, f)
    t["final.norm"] = norm(d)
    t["head"] = lin(cfg["vocab"], d)
    return {k: bf16_round(np.asarray(v, np.float32)) for k, v in t.items()}


def tokens(cfg, n, seed=0):
    return np.random.default_rng(1000 + seed).integers(0, cfg["vocab"], size=n).astype(np.int32)


def shapes(t):
    return {k: v.shape for k, v in t.items()}
