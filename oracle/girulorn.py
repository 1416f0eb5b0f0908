"""Plain, slow restatement of the Girulorn decoder in numpy, one function per mechanism.

Test infrastructure only: what the CUDA path is compared with, sharing no code with it.  Everything is computed on
whole sequences without a cache, in the precision of the arrays it is given (float64 by default).

A model is (cfg, t): cfg the parsed config.json, t {tensor name: array}, Linear weights [out, in].
"""
import math

import numpy as np


def rms_norm(x, w, eps):
    """x / rms(x) * w over the last axis, eps inside the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def query_temperature(pos, temp):
    """Factor of the queries at each position; temp None or {coef, every}."""
    if not temp:
        return np.ones(len(pos))
    return np.array([1.0 + temp["coef"] * math.log((p + 1) // temp["every"] + 1) for p in pos])


def distance_bucket(n, B, D):
    """Row of the bias table for a key n tokens back: exact below B/2, then logarithmic up to D."""
    h = B // 2
    if n < h:
        return n
    return min(B - 1, h + math.floor(math.log(n / h) / math.log(D / h) * (B - h)))


def distance_bias(T, table, D):
    """[H, T, T]: the bias of query i on key j (0 where j > i)."""
    B, H = table.shape
    row = table[[distance_bucket(n, B, D) for n in range(T)]]          # [T, H] by distance
    out = np.zeros((H, T, T), table.dtype)
    for i in range(T):
        out[:, i, :i + 1] = row[i - np.arange(i + 1)].T
    return out


def sink_softmax(s, visible, sink):
    """Softmax over the last axis whose denominator has exp(sink) besides; s [T, T], sink a number."""
    s = np.where(visible, s, -np.inf)
    m = np.maximum(s.max(axis=-1, keepdims=True), sink)
    e = np.exp(s - m)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(sink - m))


def keys_values(h, m, w, eps):
    """(k [T, G, dim] after the norm, v [T, G, vdim])."""
    T, G = h.shape[0], m["kv_heads"]
    k = rms_norm((h @ w("k").T).reshape(T, G, m["dim"]), w("k.norm"), eps)
    return k, (h @ w("v").T).reshape(T, G, m["vdim"])


def attention(h, m, w, eps, kv):
    """h [T, d]; m the mixer entry of the config; w(name) -> tensor of this mixer; kv: keys and values (its own or
    another layer's)."""
    T = h.shape[0]
    H, G = m["heads"], m["kv_heads"]
    k, v = kv
    q = rms_norm((h @ w("q").T).reshape(T, H, m["dim"]), w("q.norm"), eps)
    q = q * query_temperature(range(T), m.get("q_temp"))[:, None, None]
    bias = distance_bias(T, w("rel"), m["bias_max"])
    vis = np.tril(np.ones((T, T), bool))
    gate = sigmoid(h @ w("g").T)
    out = np.empty((T, H, m["vdim"]), h.dtype)
    for a in range(H):
        g = a // (H // G)
        p = sink_softmax(q[:, a] @ k[:, g].T * m["scale"] + bias[a], vis, w("sink")[a])
        out[:, a] = p @ v[:, g] * gate[:, a:a + 1]
    return out.reshape(T, -1) @ w("o").T


def gla(h, m, w, eps, states=None):
    """Gated linear attention, token by token; states: list that receives the state after every token."""
    T, H, K, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w("q").T).reshape(T, H, K) * K ** -0.5
    k = (h @ w("k").T).reshape(T, H, K)
    v = (h @ w("v").T).reshape(T, H, V)
    z = (h @ w("a1").T @ w("a2").T + w("a2.b")).reshape(T, H, K)
    alpha = sigmoid(z) ** (1.0 / m["tau"])
    S = np.zeros((H, K, V), h.dtype)
    o = np.empty((T, H, V), h.dtype)
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hkv,hk->hv", S, q[t])
        if states is not None:
            states.append(S.copy())
    o = rms_norm(o, w("norm"), eps).reshape(T, H * V)
    return (o * silu(h @ w("g").T)) @ w("o").T


def gated_ff(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def route(h, router, bias, top):
    """(weights [T, top], ids [T, top]): the `top` largest logits and the softmax over them."""
    z = h @ router.T + bias
    ids = np.argsort(-z, axis=-1, kind="stable")[:, :top]
    s = np.take_along_axis(z, ids, axis=-1)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True), ids


def moe_ff(h, mlp, w, record=None):
    wt, ids = route(h, w("router"), w("router.b"), mlp["router"]["top"])
    if record is not None:
        record.append(ids)
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(ids.shape[1]):
            e = "e%d." % ids[t, j]
            out[t] += wt[t, j] * gated_ff(h[t], w(e + "gate"), w(e + "up"), w(e + "down"))
    if mlp.get("shared"):
        out += gated_ff(h, w("shared.gate"), w("shared.up"), w("shared.down"))
    return out


def layer(x, i, cfg, t, kvs, record=None):
    """Both sublayers read the residual itself and are normed on the way back; kvs {layer: keys and values} of the
    attention layers so far."""
    L, eps, p = cfg["layers"][i], cfg["norm"]["eps"], "l%d." % i
    m, w = L["mixer"], lambda n: t[p + "mix." + n]
    if L["type"] == "gla":
        y = gla(x, m, w, eps)
    else:
        src = m.get("kv_from")
        kvs[i] = keys_values(x, m, w, eps) if src is None else kvs[src]
        y = attention(x, m, w, eps, kvs[i])
    x = x + rms_norm(y, t[p + "norm1"], eps)
    if L.get("mlp") is not None:
        x = x + rms_norm(moe_ff(x, L["mlp"], lambda n: t[p + "mlp." + n], record), t[p + "norm2"], eps)
    return x


def forward(cfg, t, tokens, collect=None, record=None, dtype=np.float64):
    """Logits [T, vocab] of one sequence; collect: list that receives the residual after every layer; record: list
    that receives every routed layer's expert ids."""
    t = {k: np.asarray(v, dtype) for k, v in t.items()}
    x, kvs = t["embed"][np.asarray(tokens)], {}
    for i in range(len(cfg["layers"])):
        x = layer(x, i, cfg, t, kvs, record)
        if collect is not None:
            collect.append(x.copy())
    return rms_norm(x, t["final.norm"], cfg["norm"]["eps"]) @ t["head"].T


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
