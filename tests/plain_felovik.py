"""A plain, slow Felovik in NumPy float64: whole sequences only, no cache, no batching, no step
function. One function for each mechanism of the design, written from its equations; nothing
here imports the package under test.

Notation: n tokens, W the model's width, H heads, G key/value heads (or groups of B and C), D a
head's key size, Dv its value size, N a recurrent head's state size. Linear weights are
[out, in] and applied as `x @ w.T`.
"""

from __future__ import annotations

import math

import numpy as np

from plain_model import read_model_folder      # the tests' own safetensors reader

__all__ = ["read_model_folder", "rms_norm", "sigmoid", "silu", "softplus", "embed",
           "query_temperature", "causal_softmax", "attention", "causal_conv", "dual_scan",
           "gate_then_norm", "dual_mixer", "parallel", "clamped_mlp", "route", "experts",
           "feed_forward", "layer", "forward", "generate"]

ALPHA = 1.702          # the dense feed-forward's activation: g * sigmoid(ALPHA g)


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


def embed(t, ids, scale):
    """Rows of the table times `scale`, plus the position's learned vector as it is."""
    ids = np.asarray(ids)
    return t["embed"][ids] * scale + t["pos"][:ids.size]


def query_temperature(n, temp):
    """[n] factors of the queries at positions 0 .. n-1: 1 + coef ln(floor((p+1) / every) + 1)."""
    if temp is None:
        return np.ones(n)
    return np.array([1.0 + temp["coef"] * math.log(math.floor((p + 1) / temp["every"]) + 1)
                     for p in range(n)])


def causal_softmax(scores):
    """Softmax of each row of [n, n] scores over the columns up to the row's own."""
    n = scores.shape[0]
    s = np.where(np.tri(n, dtype=bool), scores, -np.inf)
    e = np.exp(s - s.max(-1, keepdims=True))
    return e / e.sum(-1, keepdims=True)


def attention(h, t, p, m, eps):
    """Grouped-query attention without a rotation: q and k of every head over their own root
    mean square, queries times their position's temperature, a causal softmax, the heads'
    outputs times sigmoid(Wg h) element by element, Wo."""
    n = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm((h @ t[p + "q"].T).reshape(n, H, D), None, eps)
    k = rms_norm((h @ t[p + "k"].T).reshape(n, G, D), None, eps)
    v = (h @ t[p + "v"].T).reshape(n, G, Dv)
    q = q * query_temperature(n, m.get("q_temp"))[:, None, None]
    out = np.zeros((n, H, Dv))
    for a in range(H):
        g = a // (H // G)
        out[:, a] = causal_softmax(q[:, a] @ k[:, g].T * m["scale"]) @ v[:, g]
    return (out.reshape(n, H * Dv) * sigmoid(h @ t[p + "g"].T)) @ t[p + "o"].T


def causal_conv(x, w, b):
    """silu of a causal convolution a channel: x [n, channels], w [channels, taps] (its last
    column multiplies the token itself), zeros before the start."""
    taps = w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, x.shape[1])), x])
    out = sum(padded[j:j + x.shape[0]] * w[:, j] for j in range(taps))
    return silu(out + b)


def dual_scan(x, B, C, dt, a_log, d_skip, state=None):
    """x [n, H, Dv], B and C [n, G, N], dt [n, H] (positive), a_log and d_skip [H]: per head S
    [N, Dv] <- exp(-exp(a_log) dt) S + dt B x^T, y = S^T C + D x; head h reads group floor(h /
    (H / G)). Returns y [n, H, Dv] and the last state [H, N, Dv]."""
    n, H, Dv = x.shape
    G, N = B.shape[1:]
    S = np.zeros((H, N, Dv)) if state is None else state.copy()
    group = np.arange(H) // (H // G)
    y = np.empty_like(x)
    for i in range(n):
        fade = np.exp(-np.exp(a_log) * dt[i])
        S = fade[:, None, None] * S + (dt[i][:, None] * B[i, group])[:, :, None] * x[i][:, None, :]
        y[i] = np.einsum("hnv,hn->hv", S, C[i, group]) + d_skip[:, None] * x[i]
    return y, S


def gate_then_norm(y, z, w, parts, eps):
    """y * silu(z), then each of `parts` equal pieces of a row over its own root mean square,
    times w."""
    n, width = y.shape
    g = (y * silu(z)).reshape(n, parts, width // parts)
    return rms_norm(g, None, eps).reshape(n, width) * w


def dual_mixer(h, t, p, m, eps):
    """The state-space mixer: [z | x | B | C | dt] = Win h; x, B and C together through the
    convolution; dt <- softplus(dt + bias); the scan; the gate and the norm in parts; Wo."""
    n = h.shape[0]
    H, Dv, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * Dv
    proj = h @ t[p + "in"].T
    z, xbc, dt = np.split(proj, [inner, 2 * inner + 2 * G * N], axis=1)
    xbc = causal_conv(xbc, t[p + "conv"], t[p + "conv.b"])
    x, B, C = np.split(xbc, [inner, inner + G * N], axis=1)
    dt = softplus(dt + t[p + "dt_bias"])
    y, _ = dual_scan(x.reshape(n, H, Dv), B.reshape(n, G, N), C.reshape(n, G, N), dt,
                     t[p + "A_log"], t[p + "D"])
    y = gate_then_norm(y.reshape(n, inner), z, t[p + "norm"], m["norm_groups"], eps)
    return y @ t[p + "o"].T


def parallel(h, t, p, m, eps):
    """Half the sum of the two mixers' outputs, each normed over the width with its weight."""
    left = attention(h, t, p + "left.", m["left"], eps)
    right = dual_mixer(h, t, p + "right.", m["right"], eps)
    return 0.5 * (rms_norm(left, t[p + "left.out"], eps) + rms_norm(right, t[p + "right.out"], eps))


def clamped_mlp(h, t, p, limit):
    """g = min(Wgate h, limit), u = Wup h within +-limit; Wdown (g sigmoid(ALPHA g) (u + 1))."""
    g = np.minimum(h @ t[p + "gate"].T, limit)
    u = np.clip(h @ t[p + "up"].T, -limit, limit)
    return (g * sigmoid(ALPHA * g) * (u + 1.0)) @ t[p + "down"].T


def route(h, t, p, router):
    """(chosen [n, top], weights [n, top]): softmax scores over all experts; the experts form
    `count` equal groups of neighbours whose score is their largest, and only the experts of the
    `keep` best groups can be chosen (ties: the lowest index); the chosen scores over their
    sum + 1e-20."""
    z = h @ t[p + "router"].T
    e = np.exp(z - z.max(-1, keepdims=True))
    s = e / e.sum(-1, keepdims=True)
    n, E = s.shape
    groups = router.get("groups") or {"count": 1, "keep": 1}
    best = s.reshape(n, groups["count"], -1).max(-1)
    kept = np.argsort(-best, axis=-1, kind="stable")[:, :groups["keep"]]
    open_ = np.zeros((n, groups["count"]), dtype=bool)
    np.put_along_axis(open_, kept, True, axis=-1)
    allowed = np.where(np.repeat(open_, E // groups["count"], axis=-1), s, -np.inf)
    chosen = np.argsort(-allowed, axis=-1, kind="stable")[:, :router["top"]]
    w = np.take_along_axis(s, chosen, axis=-1)
    return chosen, w / (w.sum(-1, keepdims=True) + 1e-20)


def experts(h, t, p, mlp):
    chosen, weights = route(h, t, p, mlp["router"])
    out = np.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        rows, place = np.nonzero(chosen == e)
        if rows.size:
            q = f"{p}e{e}."
            y = (silu(h[rows] @ t[q + "gate"].T) * (h[rows] @ t[q + "up"].T)) @ t[q + "down"].T
            out[rows] += weights[rows, place][:, None] * y
    return out


def feed_forward(h, t, p, mlp):
    if mlp["kind"] == "dense":
        return clamped_mlp(h, t, p, mlp["limit"])
    return experts(h, t, p, mlp)


def layer(x, t, config, i):
    """x <- norm1(alpha x + mixer(x)); x <- norm2(alpha x + ff(x))."""
    entry = config["layers"][i]
    p, eps, alpha = f"l{i}.", config["norm"]["eps"], config["postln_alpha"]
    x = rms_norm(alpha * x + parallel(x, t, p + "mix.", entry["mixer"], eps), t[p + "norm1"], eps)
    if entry.get("mlp"):
        x = rms_norm(alpha * x + feed_forward(x, t, p + "mlp.", entry["mlp"]), t[p + "norm2"], eps)
    return x


def forward(config, tensors, ids, hidden_states=None):
    """float64 logits [n, vocab] of one whole sequence; with `hidden_states` (a list), the
    stream after every layer is appended to it."""
    t = {k: np.asarray(v, dtype=np.float64) for k, v in tensors.items()}
    x = embed(t, ids, config["embedding"]["scale"])
    for i in range(len(config["layers"])):
        x = layer(x, t, config, i)
        if hidden_states is not None:
            hidden_states.append(x.copy())
    return rms_norm(x, t["final.norm"], config["norm"]["eps"]) @ t["head"].T


def generate(config, tensors, ids, new_tokens):
    """The `new_tokens` tokens that greedy decoding adds to `ids`."""
    ids = list(ids)
    for _ in range(new_tokens):
        ids.append(int(np.argmax(forward(config, tensors, ids)[-1])))
    return ids[len(ids) - new_tokens:]
