"""Small Rezupel configurations with seeded weights, shared by the tests.

Expert choices must not hang on rounding, or a bf16 run could pick another expert than the float64 restatement: the
first `experts` features of the residual are reserved for the router.  Every token's embedding holds a shuffled ladder
of values there, no layer writes to them, and the router reads (almost) only them.
"""
import numpy as np

from rew_b200.weights import bf16_round


def mixer(heads=3, dim=20, rot_dim=12, vdim=28, q_rank=36, kv_rank=44, window=37, base=5000.0, scale=None, rope_dims=None):
    return dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, mask=dict(size=window),
                rot=dict(base=base, dims=rot_dim if rope_dims is None else rope_dims),
                scale=(dim + rot_dim) ** -0.5 if scale is None else scale)


def dense(ff=88):
    return dict(kind="dense", ff=ff)


def moe(experts=5, top=3, ff=24):
    return dict(kind="moe", router=dict(experts=experts, top=top), expert=dict(ff=ff))


def layer(mlp, **kw):
    return dict(type="latent_attention", mixer=mixer(**kw), mlp=mlp)


def config(layers, vocab=152, width=104, eps=1e-5, loop=None):
    cfg = dict(architecture="Rezupel", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers)
    if loop:
        cfg["loop"] = dict(start=loop[0], stop=loop[1], times=loop[2])
    return cfg


def small(**kw):
    """Every branch of the design: dense, routed and absent feed-forwards, two windows, a loop in the middle."""
    return config([layer(dense()), layer(moe()), layer(None, heads=2, window=9, base=300.0), layer(moe(experts=7, top=2, ff=40)),
                   layer(dense(56), heads=5, vdim=16, window=64)], **dict(dict(loop=(1, 3, 3)), **kw))


def weights(cfg, seed=0, score_gain=1.0):
    """{name: float32 array, bf16-representable}, Linear weights [out, in].  score_gain sharpens the attention."""
    rng = np.random.default_rng(seed)
    d, t = cfg["width"], {}
    E = max([l["mlp"]["router"]["experts"] for l in cfg["layers"] if l["mlp"] and l["mlp"]["kind"] == "moe"] or [0])
    assert E < d // 2

    def lin(o, i, gain=1.0):
        return rng.normal(0, gain * i ** -0.5, size=(o, i))

    def into_residual(i, gain):
        w = lin(d, i, gain)
        w[:E] = 0.0
        return w

    def norm(n):
        return rng.normal(0, 0.2, size=n)

    t["embed"] = rng.normal(0, 1.0, size=(cfg["vocab"], d))
    for v in range(cfg["vocab"]):
        t["embed"][v, :E] = rng.permutation(np.linspace(-2.0, 2.0, E)) if E else []
    if cfg.get("loop"):
        t["loop.step"] = rng.normal(0, 0.5, size=(cfg["loop"]["times"], d))
        t["loop.step"][:, :E] = 0.0
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], "l%d." % i
        x = p + "mix."
        H = m["heads"]
        t[p + "norm1"] = norm(d)
        t[x + "dq"] = lin(m["q_rank"], d)
        t[x + "dq.norm"] = 1 + norm(m["q_rank"])
        t[x + "uq"] = lin(H * (m["dim"] + m["rot_dim"]), m["q_rank"], score_gain)
        t[x + "dkv"] = lin(m["kv_rank"] + m["rot_dim"], d)
        t[x + "dkv.norm"] = 1 + norm(m["kv_rank"])
        t[x + "uk"] = lin(H * m["dim"], m["kv_rank"])
        t[x + "uv"] = lin(H * m["vdim"], m["kv_rank"])
        t[x + "g"] = lin(H, d, 2.0)
        t[x + "o"] = into_residual(H * m["vdim"], 1.5)
        if L["mlp"] is None:
            continue
        q = p + "mlp."
        n2 = norm(d)
        n2[:E] = 0.0
        t[p + "norm2"] = n2
        if L["mlp"]["kind"] == "dense":
            f = L["mlp"]["ff"]
            t[q + "gate"], t[q + "up"], t[q + "down"] = lin(f, d, 1.5), lin(f, d, 1.5), into_residual(f, 1.0)
        else:
            e_n, f = L["mlp"]["router"]["experts"], L["mlp"]["expert"]["ff"]
            r = rng.normal(0, 0.002, size=(e_n, d))
            r[np.arange(e_n), rng.permutation(E)[:e_n]] += 1.5
            t[q + "router"] = r
            for e in range(e_n):
                t[q + "e%d.up" % e], t[q + "e%d.down" % e] = lin(f, d, 1.5), into_residual(f, 1.5)
    t["final.norm"] = norm(d)
    return {k: bf16_round(np.asarray(v, np.float32)) for k, v in t.items()}


def tokens(cfg, n, seed=0):
    return np.random.default_rng(1000 + seed).integers(0, cfg["vocab"], size=n).astype(np.int32)
