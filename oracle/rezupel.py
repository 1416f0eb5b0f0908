"""Plain, slow restatement of the Rezupel decoder in numpy, one function per mechanism.

Test infrastructure only: what the CUDA path is compared with, sharing no code with it.  Everything is computed on
whole sequences without a cache, in the precision of the arrays it is given (float64 by default).

A model is (cfg, t): cfg the parsed config.json, t {tensor name: array}, Linear weights [out, in].
"""
import numpy as np


def rms_norm(x, w, eps):
    """x / rms(x) * w over the last axis, eps inside the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def zero_centred_norm(x, w, eps):
    """RMS norm whose stored weight is the distance from one."""
    return rms_norm(x, 1.0 + w, eps)


def rotate_interleaved(x, pos, base, dims):
    """Rotates the pairs (2i, 2i+1) of the first `dims` features by pos * base^(-2i/dims); x [T, ..., >= dims]."""
    out = x.copy()
    for i in range(dims // 2):
        ang = np.asarray(pos, np.float64) * float(base) ** (-2.0 * i / dims)
        c, s = np.cos(ang), np.sin(ang)
        shape = (len(ang),) + (1,) * (x.ndim - 2)
        c, s = c.reshape(shape), s.reshape(shape)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def window_visible(T, size):
    """[T, T] bool: query i sees key j when 0 <= i - j < size."""
    i = np.arange(T)[:, None]
    j = np.arange(T)[None, :]
    return (i - j >= 0) & (i - j < size)


def masked_softmax(s, visible):
    s = np.where(visible, s, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def relu_squared(z):
    r = np.maximum(z, 0.0)
    return r * r


def latent_attention(h, m, w, eps):
    """h [T, d]; m the mixer entry of the config; w(name) -> tensor of this mixer.  Keys and values are expanded
    per head from the latent, as the definition has it (no absorbed projections)."""
    T = h.shape[0]
    H, dn, dr, dv, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(T)
    cq = rms_norm(h @ w("dq").T, w("dq.norm"), eps)
    q = (cq @ w("uq").T).reshape(T, H, dn + dr)
    ckr = h @ w("dkv").T
    c = rms_norm(ckr[:, :r], w("dkv.norm"), eps)
    kr = rotate_interleaved(ckr[:, r:], pos, m["rot"]["base"], m["rot"]["dims"])
    qn = q[:, :, :dn]
    qr = rotate_interleaved(q[:, :, dn:], pos, m["rot"]["base"], m["rot"]["dims"])
    k = (c @ w("uk").T).reshape(T, H, dn)
    v = (c @ w("uv").T).reshape(T, H, dv)
    vis = window_visible(T, m["mask"]["size"])
    gate = sigmoid(h @ w("g").T)
    out = np.empty((T, H, dv), h.dtype)
    for a in range(H):
        s = (qn[:, a] @ k[:, a].T + qr[:, a] @ kr.T) * m["scale"]
        out[:, a] = masked_softmax(s, vis) @ v[:, a] * gate[:, a:a + 1]
    return out.reshape(T, H * dv) @ w("o").T


def dense_ff(h, w):
    return (silu(h @ w("gate").T) * (h @ w("up").T)) @ w("down").T


def route(h, router, top):
    """(weights [T, top], ids [T, top]): the `top` largest softmax scores, not renormalised."""
    z = h @ router.T
    s = masked_softmax(z, np.ones_like(z, bool))
    ids = np.argsort(-s, axis=-1, kind="stable")[:, :top]
    return np.take_along_axis(s, ids, axis=-1), ids


def moe_ff(h, mlp, w, record=None):
    wt, ids = route(h, w("router"), mlp["router"]["top"])
    if record is not None:
        record.append(ids)
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(ids.shape[1]):
            e = int(ids[t, j])
            out[t] += wt[t, j] * (w("e%d.down" % e) @ relu_squared(w("e%d.up" % e) @ h[t]))
    return out


def layer(x, i, cfg, t, record=None):
    """Parallel block: mixer and feed-forward each read their own norm of the same x."""
    L, eps, p = cfg["layers"][i], cfg["norm"]["eps"], "l%d." % i
    mixed = latent_attention(zero_centred_norm(x, t[p + "norm1"], eps), L["mixer"], lambda n: t[p + "mix." + n], eps)
    y = x + mixed
    if L.get("mlp") is not None:
        h2 = zero_centred_norm(x, t[p + "norm2"], eps)
        w = lambda n: t[p + "mlp." + n]
        y = y + (dense_ff(h2, w) if L["mlp"]["kind"] == "dense" else moe_ff(h2, L["mlp"], w, record))
    return y


def layer_runs(cfg):
    """[(layer, pass or None, starts a pass)] in execution order."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None, False) for i in range(n)]
    a, b, k = loop["start"], loop["stop"], loop["times"]
    runs = [(i, None, False) for i in range(a)]
    for p in range(k):
        runs += [(i, p, i == a) for i in range(a, b)]
    return runs + [(i, None, False) for i in range(b, n)]


def forward(cfg, t, tokens, collect=None, record=None, dtype=np.float64):
    """Logits [T, vocab] of one sequence; collect: list that receives the residual after every layer run;
    record: list that receives every routed layer run's expert ids."""
    t = {k: np.asarray(v, dtype) for k, v in t.items()}
    x0 = t["embed"][np.asarray(tokens)]
    x = x0.copy()
    for i, p, first in layer_runs(cfg):
        if first:
            if p > 0:
                x = x + x0
            x = x + t["loop.step"][p]
        x = layer(x, i, cfg, t, record)
        if collect is not None:
            collect.append(x.copy())
    return zero_centred_norm(x, t["final.norm"], cfg["norm"]["eps"]) @ t["embed"].T


def generate_greedy(cfg, t, prompt, n):
    """n greedy tokens; ids of the whole sequence are recomputed every step.  Returns (ids, smallest margin between
    the two largest logits seen)."""
    seq, out, margin = list(prompt), [], np.inf
    for _ in range(n):
        lg = forward(cfg, t, seq)[-1]
        top = np.sort(lg)[-2:]
        margin = min(margin, top[1] - top[0])
        out.append(int(np.argmax(lg)))
        seq.append(out[-1])
    return out, margin
