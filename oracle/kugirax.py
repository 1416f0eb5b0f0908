"""Plain, slow restatement of the Kugirax decoder in numpy, one function per mechanism.

Test infrastructure only: what the CUDA path is compared with, sharing no code with it.  Everything is computed on
whole sequences without a cache, in the precision of the arrays it is given (float64 by default).

A model is (cfg, t): cfg the parsed config.json, t {tensor name: array}, Linear weights [out, in].
"""
import numpy as np


def rms_norm(x, w, eps):
    """x / rms(x) * w over the last axis, eps inside the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def short_conv(u, w):
    """y[t] = sum_j w[:, j] u[t - taps + 1 + j] per channel, zeros ahead of the sequence; u [T, C], w [C, taps]."""
    taps = w.shape[1]
    y = np.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j                     # this tap reads the value `back` tokens ago
        if back < len(u):
            y[back:] += u[:len(u) - back] * w[:, j]
    return y


def rotated_halves(x, pos, base, dims):
    """Rotates the pairs (i, i + dims/2) of the first `dims` features by pos * base^(-2i/dims); x [T, heads, >= dims]."""
    out = x.copy()
    for i in range(dims // 2):
        ang = np.asarray(pos, np.float64) * float(base) ** (-2.0 * i / dims)
        c, s = np.cos(ang)[:, None], np.sin(ang)[:, None]
        u, v = x[..., i], x[..., i + dims // 2]
        out[..., i] = u * c - v * s
        out[..., i + dims // 2] = v * c + u * s
    return out


def visible(T, size=None):
    """[T, T] bool: query i sees key j when 0 <= i - j (< size)."""
    back = np.arange(T)[:, None] - np.arange(T)[None, :]
    return (back >= 0) & (back < (T if size is None else size))


def sink_softmax(s, vis, sink):
    """Softmax over the last axis whose denominator has exp(sink) besides; s [T, T], sink a number."""
    s = np.where(vis, s, -np.inf)
    m = np.maximum(s.max(axis=-1, keepdims=True), sink)
    e = np.exp(s - m)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(sink - m))


def attention(h, m, w):
    """Grouped-query attention whose values are the keys ahead of their rotation; h [T, d], m the mixer entry of the
    config, w(name) -> tensor of this mixer."""
    T, H, G, K = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    pos = np.arange(T)
    q = short_conv(h @ w("q").T, w("q.conv")).reshape(T, H, K)
    k = short_conv(h @ w("k").T, w("k.conv")).reshape(T, G, K)
    v = k
    q, k = (rotated_halves(x, pos, m["rot"]["base"], m["rot"]["dims"]) for x in (q, k))
    out = np.empty((T, H, K), h.dtype)
    for a in range(H):
        g = a // (H // G)
        out[:, a] = sink_softmax(q[:, a] @ k[:, g].T * m["scale"], visible(T), 0.0) @ v[:, g]
    return out.reshape(T, H * K) @ w("o").T


def latent(h, w, eps):
    """The cached latent [T, kv_rank]."""
    return rms_norm(h @ w("dkv").T, w("dkv.norm"), eps)


def latent_attention(h, c, m, w, eps):
    """h [T, d]; c: the latents, this layer's or another's.  Keys and values are expanded per head."""
    T, H, K, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (rms_norm(h @ w("dq").T, w("dq.norm"), eps) @ w("uq").T).reshape(T, H, K)
    k = (c @ w("uk").T).reshape(T, H, K)
    v = (c @ w("uv").T).reshape(T, H, V)
    vis = visible(T, m["mask"]["size"])
    out = np.empty((T, H, V), h.dtype)
    for a in range(H):
        out[:, a] = sink_softmax(q[:, a] @ k[:, a].T * m["scale"], vis, w("sink")[a]) @ v[:, a]
    return out.reshape(T, H * V) @ w("o").T


def gated_ff(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def route(h, router, top, scale):
    """(weights [T, top], ids [T, top]): the `top` largest softmax scores, made to sum to `scale`."""
    z = h @ router.T
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    s = e / e.sum(axis=-1, keepdims=True)
    ids = np.argsort(-s, axis=-1, kind="stable")[:, :top]
    chosen = np.take_along_axis(s, ids, axis=-1)
    return chosen / (chosen.sum(axis=-1, keepdims=True) + 1e-20) * scale, ids


def moe_ff(h, mlp, w, record=None):
    wt, ids = route(h, w("router"), mlp["router"]["top"], mlp["router"]["scale"])
    if record is not None:
        record.append(ids)
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(ids.shape[1]):
            e = "e%d." % ids[t, j]
            out[t] += wt[t, j] * gated_ff(h[t], w(e + "gate"), w(e + "up"), w(e + "down"))
    if mlp.get("shared"):
        y = gated_ff(h, w("shared.gate"), w("shared.up"), w("shared.down"))
        out += sigmoid(h @ w("shared.sg").reshape(1, -1).T) * y
    return out


def layer(x, i, cfg, t, latents, record=None):
    """Parallel block: mixer and feed-forward read the same norm of x; latents {layer: c} of the layers so far."""
    L, eps, p = cfg["layers"][i], cfg["norm"]["eps"], "l%d." % i
    m, w = L["mixer"], lambda n: t[p + "mix." + n]
    h = rms_norm(x, t[p + "norm1"], eps)
    if L["type"] == "attention":
        y = attention(h, m, w)
    else:
        src = m.get("kv_from")
        latents[i] = latent(h, w, eps) if src is None else latents[src]
        y = latent_attention(h, latents[i], m, w, eps)
    mlp = L.get("mlp")
    if mlp is not None:
        f = lambda n: t[p + "mlp." + n]
        y = y + (gated_ff(h, f("gate"), f("up"), f("down")) if mlp["kind"] == "dense" else moe_ff(h, mlp, f, record))
    return x + y


def soft_cap(z, cap):
    return z if not cap else cap * np.tanh(z / cap)


def forward(cfg, t, tokens, collect=None, record=None, dtype=np.float64):
    """Logits [T, vocab] of one sequence; collect: list that receives the residual after every layer; record: list
    that receives every routed layer's expert ids."""
    t = {k: np.asarray(v, dtype) for k, v in t.items()}
    x, latents = t["embed"][np.asarray(tokens)], {}
    for i in range(len(cfg["layers"])):
        x = layer(x, i, cfg, t, latents, record)
        if collect is not None:
            collect.append(x.copy())
    return soft_cap(rms_norm(x, t["final.norm"], cfg["norm"]["eps"]) @ t["head"].T, cfg.get("logit_softcap"))


def generate_greedy(cfg, t, prompt, n):
    """n greedy tokens; the whole sequence is recomputed every step.  Returns (ids, smallest margin between the two
    largest logits seen)."""
    seq, out, margin = list(prompt), [], np.inf
    for _ in range(n):
        lg = forward(cfg, t, seq)[-1]
        top = np.sort(lg)[-2:]
        margin = min(margin, top[1] - top[0])
        out.append(int(np.argmax(lg)))
        seq.append(out[-1])
    return out, margin
