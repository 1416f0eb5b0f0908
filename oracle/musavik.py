"""Plain, slow restatement of the Musavik decoder in numpy, one function per mechanism.

Test infrastructure only: what the CUDA path is compared with, sharing no code with it.  Everything is computed on
whole sequences without a cache, in the precision of the arrays it is given (float64 by default).

A model is (cfg, t): cfg the parsed config.json, t {tensor name: array}, Linear weights [out, in].
"""
import math

import numpy as np

UNIT_EPS = 1e-6      # of the unit queries and keys of the delta rule
DECAY_GAIN = 8.0     # of the linear recurrent unit


def rms_norm(x, w, eps):
    """x / rms(x) * w over the last axis, eps inside the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(z, 0.0)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def bigram_rows(tokens, big):
    """Rows of the bigram table: a hash of the token and the one before it; the row behind the hashed ones for the first."""
    tokens = [int(v) for v in tokens]
    return [big["buckets"]] + [(a * big["mul_prev"] + b * big["mul_cur"]) % big["buckets"] for a, b in zip(tokens, tokens[1:])]


def embedding(cfg, t, tokens):
    e = cfg["embedding"]
    x = t["embed"][np.asarray(tokens)] * e["scale"]
    return x + t["bigram"][bigram_rows(tokens, e["bigram"])] if e.get("bigram") else x


def short_conv(u, w):
    """Causal convolution over time per channel; u [T, C], w [C, taps], the last column is the current token's."""
    T, taps = u.shape[0], w.shape[1]
    y = np.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j
        y[back:] += w[:, j] * u[:T - back] if back < T else 0.0
    return y


def rotated_pairs(x, pos, base, dims):
    """x [T, heads, dim]: features (2i, 2i + 1) of the first `dims` turned by pos * base^(-2i / dims)."""
    out = x.copy()
    a = np.outer(np.asarray(pos, np.float64), base ** (-np.arange(0, dims, 2) / dims))[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * np.cos(a) - v * np.sin(a)
    out[..., 1:dims:2] = v * np.cos(a) + u * np.sin(a)
    return out


def visible(T, size, keep_first):
    """[T, T]: query i sees key j <= i of its window, and the first keys of the sequence."""
    i, j = np.arange(T)[:, None], np.arange(T)[None]
    return (j <= i) & ((i - j < size) | (j < keep_first))


def softmax(s, vis):
    s = np.where(vis, s, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def talk(p, mix):
    """Weights [H, T, T] of the heads mixed: head h gets sum_g mix[h, g] p[g]."""
    return np.einsum("hg,gij->hij", mix, p)


def attention(h, m, w, eps):
    """h [T, d]; m the entry of the config; w(name) -> tensor of this mixer."""
    T = h.shape[0]
    H, G, K, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm((h @ w("q").T + w("q.b")).reshape(T, H, K), w("q.norm"), eps)
    k = rms_norm((h @ w("k").T + w("k.b")).reshape(T, G, K), w("k.norm"), eps)
    v = rms_norm((h @ w("v").T + w("v.b")).reshape(T, G, V), 1.0, eps)
    r = m["rot"]
    q, k = rotated_pairs(q, range(T), r["base"], r["dims"]), rotated_pairs(k, range(T), r["base"], r["dims"])
    vis = visible(T, m["mask"]["size"], m["mask"]["keep_first"])
    p = np.stack([softmax(q[:, a] @ k[:, a // (H // G)].T * m["scale"], vis) for a in range(H)])
    p = talk(p, w("talk"))
    o = np.stack([p[a] @ v[:, a // (H // G)] for a in range(H)], axis=1).reshape(T, H * V)
    return (o * sigmoid(h @ w("g").T)) @ w("o").T


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + UNIT_EPS)


def delta_rule(h, m, w, eps, states=None):
    """Gated delta rule, token by token; states: list that receives the state after every token."""
    T = h.shape[0]
    H, G, K, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    act = lambda n: silu(short_conv(h @ w(n).T, w(n + ".conv")))
    q = np.repeat(unit(act("q").reshape(T, G, K)), H // G, axis=1) * K ** -0.5
    k = np.repeat(unit(act("k").reshape(T, G, K)), H // G, axis=1)
    v = act("v").reshape(T, H, V)
    beta = sigmoid(h @ w("b").T)
    g = np.exp(-np.exp(w("A_log")) * softplus(h @ w("a").T + w("dt_bias")))
    S, o = np.zeros((H, K, V), h.dtype), np.empty((T, H, V), h.dtype)
    for i in range(T):
        S = g[i][:, None, None] * S
        u = beta[i][:, None] * (v[i] - np.einsum("hkv,hk->hv", S, k[i]))
        S = S + k[i][:, :, None] * u[:, None, :]
        o[i] = np.einsum("hkv,hk->hv", S, q[i])
        if states is not None:
            states.append(S.copy())
    o = rms_norm(o, w("norm"), eps).reshape(T, H * V)
    return (o * silu(h @ w("g").T)) @ w("o").T


def parallel(h, m, w, eps):
    """Attention and the delta rule beside one another, both on h."""
    return m["left_scale"] * attention(h, m["left"], lambda n: w("left." + n), eps) + \
        m["right_scale"] * delta_rule(h, m["right"], lambda n: w("right." + n), eps)


def rglru(h, m, w, states=None):
    """Recurrent block with a real-gated linear recurrent unit; states: list that receives the state after every token."""
    T, n = h.shape[0], m["width"] // m["blocks"]
    y = gelu_tanh(h @ w("y").T + w("y.b"))
    u = short_conv(h @ w("x").T + w("x.b"), w("conv")) + w("conv.b")
    part = u.reshape(T, m["blocks"], n)
    r = sigmoid(np.einsum("boi,tbi->tbo", w("ra"), part) + w("ra.b")).reshape(T, -1)
    i = sigmoid(np.einsum("boi,tbi->tbo", w("ri"), part) + w("ri.b")).reshape(T, -1)
    a = np.exp(-DECAY_GAIN * r * softplus(w("lam")))
    S, out = np.zeros(m["width"], h.dtype), np.empty_like(u)
    for s in range(T):
        S = a[s] * S + np.sqrt(1.0 - a[s] ** 2) * i[s] * u[s]
        out[s] = S
        if states is not None:
            states.append(S.copy())
    return (out * y) @ w("o").T


def dense_ff(h, w):
    return gelu_tanh(h @ w("up").T + w("up.b")) @ w("down").T + w("down.b")


def layer(x, i, cfg, t):
    """Every sublayer reads a norm of the residual and is normed on the way back."""
    L, eps, p = cfg["layers"][i], cfg["norm"]["eps"], "l%d." % i
    w, norm = lambda n: t[p + "mix." + n], lambda z, n: rms_norm(z, 1.0 + t[p + n], eps)
    h = norm(x, "norm1")
    y = parallel(h, L["mixer"], w, eps) if L["type"] == "parallel" else rglru(h, L["mixer"], w)
    x = x + norm(y, "norm1b")
    if L.get("mlp") is not None:
        x = x + norm(dense_ff(norm(x, "norm2"), lambda n: t[p + "mlp." + n]), "norm2b")
    return x


def layer_runs(cfg):
    """(layer, whether a pass of the loop starts ahead of it) of every layer run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return [(i, False) for i in range(a)] + [(i, i == a) for i in range(a, b)] * loop["times"] + [(i, False) for i in range(b, n)]


def forward(cfg, t, tokens, collect=None, dtype=np.float64):
    """Logits [T, vocab] of one sequence; collect: list that receives the residual after every layer run."""
    t = {k: np.asarray(v, dtype) for k, v in t.items()}
    x0 = x = embedding(cfg, t, tokens)
    for i, enters in layer_runs(cfg):
        if enters:
            x = np.concatenate([x, x0], axis=-1) @ t["loop.in"].T
        x = layer(x, i, cfg, t)
        if collect is not None:
            collect.append(x.copy())
    return rms_norm(x, 1.0 + t["final.norm"], cfg["norm"]["eps"]) @ t["head"].T


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
