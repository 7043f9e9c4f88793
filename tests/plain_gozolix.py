"""A plain, slow Gozolix in NumPy float64: whole sequences only, no cache, no batching, no step
function. One function for each mechanism of the design, written from its equations; nothing
here imports the package under test.

Notation: n tokens, W the model's width, H heads, G key/value heads, D a head's key size, Dv its
value size. Linear weights are [out, in] and applied as `x @ w.T`.
"""

from __future__ import annotations

import math

import numpy as np

from plain_model import read_model_folder      # the tests' own safetensors reader

__all__ = ["read_model_folder", "rms_norm", "sigmoid", "silu", "softplus", "bigram_rows", "embed",
           "query_temperature", "head_slopes", "soft_cap", "causal_softmax", "attention",
           "causal_conv", "unit", "decay", "delta_scan", "norm_then_gate", "delta_mixer",
           "dense_mlp", "route", "gated_mlp", "experts", "feed_forward", "layer", "forward",
           "generate"]

UNIT_EPS = 1e-6        # a unit vector is x / sqrt(sum(x^2) + UNIT_EPS)


def rms_norm(x, w, eps):
    """x / sqrt(mean(x^2) + eps) (* w): eps inside the root."""
    y = x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)
    return y if w is None else y * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def bigram_rows(ids, b):
    """The bigram table's row of every token: a number made of the token and the one before it;
    the first token has the last row, number `buckets`."""
    ids = [int(i) for i in ids]
    return [b["buckets"]] + [(ids[i - 1] * b["mul_prev"] + ids[i] * b["mul_cur"]) % b["buckets"]
                             for i in range(1, len(ids))]


def embed(t, ids, embedding):
    """Rows of the table times the scale, plus the bigram's row as it is."""
    x = t["embed"][np.asarray(ids)] * embedding.get("scale", 1.0)
    b = embedding.get("bigram")
    return x if b is None else x + t["bigram"][bigram_rows(ids, b)]


def query_temperature(n, temp):
    """[n] factors of the queries at positions 0 .. n-1: 1 + coef ln(floor((p+1) / every) + 1)."""
    if temp is None:
        return np.ones(n)
    return np.array([1.0 + temp["coef"] * math.log(math.floor((p + 1) / temp["every"]) + 1)
                     for p in range(n)])


def head_slopes(heads):
    """What a key loses a position of distance, head by head: 2^(-8 (h + 1) / heads)."""
    return np.array([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)])


def soft_cap(s, cap):
    return s if cap is None else cap * np.tanh(s / cap)


def causal_softmax(scores):
    """Softmax of each row of [n, n] scores over the columns up to the row's own."""
    n = scores.shape[0]
    s = np.where(np.tri(n, dtype=bool), scores, -np.inf)
    e = np.exp(s - s.max(-1, keepdims=True))
    return e / e.sum(-1, keepdims=True)


def attention(h, t, p, m, kv=None):
    """(output, (keys, values)): grouped-query attention without a rotation. Scores are scaled,
    soft-capped, and lose `slope * distance`. `kv`: another layer's keys and values instead of
    ones made here."""
    n = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ t[p + "q"].T + t[p + "q.b"]).reshape(n, H, D)
    q = q * query_temperature(n, m.get("q_temp"))[:, None, None]
    if kv is None:
        kv = ((h @ t[p + "k"].T + t[p + "k.b"]).reshape(n, G, D),
              (h @ t[p + "v"].T + t[p + "v.b"]).reshape(n, G, Dv))
    k, v = kv
    distance = np.arange(n)[:, None] - np.arange(n)[None, :]
    out = np.zeros((n, H, Dv))
    for a in range(H):
        g = a // (H // G)
        scores = soft_cap(q[:, a] @ k[:, g].T * m["scale"], m.get("softcap"))
        out[:, a] = causal_softmax(scores - head_slopes(H)[a] * distance) @ v[:, g]
    return out.reshape(n, H * Dv) @ t[p + "o"].T, kv


def causal_conv(x, w):
    """silu of a causal convolution a channel: x [n, channels], w [channels, taps] (its last
    column multiplies the token itself), zeros before the start."""
    taps = w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, x.shape[1])), x])
    return silu(sum(padded[j:j + x.shape[0]] * w[:, j] for j in range(taps)))


def unit(x):
    return x / np.sqrt((x * x).sum(-1, keepdims=True) + UNIT_EPS)


def decay(a, a_log, dt_bias):
    """One factor a head, between 0 and 1."""
    return np.exp(-np.exp(a_log) * softplus(a + dt_bias))


def delta_scan(q, k, v, g, beta, state=None):
    """q and k [n, G, D], v [n, H, Dv], g and beta [n, H]: per head S [D, Dv] <- g S; u = beta (v -
    S^T k); S <- S + k u^T; o = S^T q; head h reads q/k head floor(h / (H / G)). Returns o [n, H,
    Dv] and the last state [H, D, Dv]."""
    n, H, Dv = v.shape
    G, D = k.shape[1:]
    S = np.zeros((H, D, Dv)) if state is None else state.copy()
    of = np.arange(H) // (H // G)
    o = np.empty_like(v)
    for i in range(n):
        S = g[i][:, None, None] * S
        u = beta[i][:, None] * (v[i] - np.einsum("hdv,hd->hv", S, k[i, of]))
        S = S + k[i, of][:, :, None] * u[:, None, :]
        o[i] = np.einsum("hdv,hd->hv", S, q[i, of])
    return o, S


def norm_then_gate(o, z, w, eps):
    """Each head's outputs over their own root mean square, times the heads' common weight, times
    silu(z): o [n, H, Dv], z [n, H * Dv]."""
    return rms_norm(o, w, eps).reshape(z.shape) * silu(z)


def delta_mixer(h, t, p, m, eps):
    n = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (causal_conv(h @ t[p + x].T, t[p + x + ".conv"]) for x in "qkv")
    q = unit(q.reshape(n, G, D)) * D ** -0.5
    k = unit(k.reshape(n, G, D))
    beta = sigmoid(h @ t[p + "b"].T)
    g = decay(h @ t[p + "a"].T, t[p + "A_log"], t[p + "dt_bias"])
    o, _ = delta_scan(q, k, v.reshape(n, H, Dv), g, beta)
    return norm_then_gate(o, h @ t[p + "g"].T, t[p + "norm"], eps) @ t[p + "o"].T


def dense_mlp(h, t, p):
    """Wdown (relu(Wup h))^2."""
    return np.maximum(h @ t[p + "up"].T, 0.0) ** 2 @ t[p + "down"].T


def route(h, t, p, router):
    """(chosen [n, top], weights [n, top]): sigmoid scores; the experts form `count` equal groups
    of neighbours whose score is the sum of their two largest, and only the experts of the `keep`
    best groups can be chosen (ties: the lowest index); the chosen scores over their sum + 1e-20,
    times the router's scale."""
    s = sigmoid(h @ t[p + "router"].T)
    n, E = s.shape
    groups = router.get("groups") or {"count": 1, "keep": 1}
    by_group = np.sort(s.reshape(n, groups["count"], -1), axis=-1)
    best = by_group[:, :, -2:].sum(-1)
    kept = np.argsort(-best, axis=-1, kind="stable")[:, :groups["keep"]]
    open_ = np.zeros((n, groups["count"]), dtype=bool)
    np.put_along_axis(open_, kept, True, axis=-1)
    allowed = np.where(np.repeat(open_, E // groups["count"], axis=-1), s, -np.inf)
    chosen = np.argsort(-allowed, axis=-1, kind="stable")[:, :router["top"]]
    w = np.take_along_axis(s, chosen, axis=-1)
    return chosen, w / (w.sum(-1, keepdims=True) + 1e-20) * router.get("scale", 1.0)


def gated_mlp(h, t, q):
    """Wdown (silu(Wgate h) (Wup h))."""
    return (silu(h @ t[q + "gate"].T) * (h @ t[q + "up"].T)) @ t[q + "down"].T


def experts(h, t, p, mlp):
    chosen, weights = route(h, t, p, mlp["router"])
    out = gated_mlp(h, t, p + "shared.") if mlp.get("shared") else np.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        rows, place = np.nonzero(chosen == e)
        if rows.size:
            out[rows] += weights[rows, place][:, None] * gated_mlp(h[rows], t, f"{p}e{e}.")
    return out


def feed_forward(h, t, p, mlp):
    return dense_mlp(h, t, p) if mlp["kind"] == "dense" else experts(h, t, p, mlp)


def layer(x, t, config, i, kept):
    """h = norm1(x); x <- x + mixer(h) + ff(h). `kept`: the keys and values of the attention
    layers so far, by layer."""
    entry = config["layers"][i]
    p, eps, m = f"l{i}.", config["norm"]["eps"], entry["mixer"]
    h = rms_norm(x, t[p + "norm1"], eps)
    if entry["type"] == "delta":
        y = delta_mixer(h, t, p + "mix.", m, eps)
    else:
        y, kept[i] = attention(h, t, p + "mix.", m,
                               None if m.get("kv_from") is None else kept[m["kv_from"]])
    if entry.get("mlp"):
        y = y + feed_forward(h, t, p + "mlp.", entry["mlp"])
    return x + y


def forward(config, tensors, ids, hidden_states=None):
    """float64 logits [n, vocab] of one whole sequence; with `hidden_states` (a list), the
    stream after every layer is appended to it."""
    t = {k: np.asarray(v, dtype=np.float64) for k, v in tensors.items()}
    x, kept = embed(t, ids, config.get("embedding") or {}), {}
    for i in range(len(config["layers"])):
        x = layer(x, t, config, i, kept)
        if hidden_states is not None:
            hidden_states.append(x.copy())
    return rms_norm(x, t["final.norm"], config["norm"]["eps"]) @ t["head"].T


def generate(config, tensors, ids, new_tokens):
    """The `new_tokens` tokens that greedy decoding adds to `ids`."""
    ids = list(ids)
    for _ in range(new_tokens):
        ids.append(int(np.argmax(forward(config, tensors, ids)[-1])))
    return ids[len(ids) - new_tokens:]
