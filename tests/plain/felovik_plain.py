"""Felovik in plain float64 NumPy, one function per mechanism, written from the architecture's equations and sharing no
code with the engine. Slow on purpose: the recurrence is a visible loop over tokens, the attention a loop over
(head, query).

Notation: T tokens, d model width, a sequence's positions count from 0. ``W`` maps tensor names to float64 arrays
(matrices stored [out, in] and applied as W x); ``p`` is the prefix of a part's tensor names; ``m`` the part's sizes as
config.json gives them. A layer is x <- norm1(alpha x + mixer(x)); x <- norm2(alpha x + ff(x)).
"""
import math

import numpy as np

#: the slope inside the dense feed-forward's gate, g * logistic(SLOPE * g)
SLOPE = 1.702


def logistic(x):
    return 1.0 / (1.0 + np.exp(-np.asarray(x, dtype=np.float64)))


def silu(x):
    return x * logistic(x)


def softplus(x):
    return np.logaddexp(0.0, x)


def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def embed(W, tokens, scale):
    """The token's row times ``scale`` plus the position's row (not scaled)."""
    return W["embed"][np.asarray(tokens)] * scale + W["pos"][np.arange(len(tokens))]


def query_temperature(position, q_temp):
    """What the query at ``position`` is multiplied by: constant over ``every`` positions, growing with their logarithm."""
    if q_temp is None:
        return 1.0
    return 1.0 + q_temp["coef"] * math.log(math.floor((position + 1) / q_temp["every"]) + 1)


def softmax(s):
    e = np.exp(s - np.max(s))
    return e / e.sum()


def attention(h, W, p, m, eps):
    """Causal grouped-query softmax attention: unit-RMS queries and keys, a temperature on the queries, a gate per output
    channel."""
    T = h.shape[0]
    H, G, D, V = m["heads"], m.get("kv_heads", m["heads"]), m["dim"], m["vdim"]
    q = rms_unit((h @ W[p + "q"].T).reshape(T, H, D), eps)
    k = rms_unit((h @ W[p + "k"].T).reshape(T, G, D), eps)
    v = (h @ W[p + "v"].T).reshape(T, G, V)
    out = np.zeros((T, H, V))
    for head in range(H):
        g = head // (H // G)
        for i in range(T):
            qi = q[i, head] * query_temperature(i, m.get("q_temp"))
            w = softmax(k[:i + 1, g] @ qi * m["scale"])
            out[i, head] = w @ v[:i + 1, g]
    return (out.reshape(T, H * V) * logistic(h @ W[p + "g"].T)) @ W[p + "o"].T


def causal_conv(x, w, b):
    """x [T, C], w [C, taps] (last column weighs the current token), b [C]: b + sum_j w[:, j] x_(t - taps + 1 + j), zeros
    before the start."""
    T, taps = x.shape[0], w.shape[1]
    y = np.zeros_like(x) + b
    for t in range(T):
        for j in range(taps):
            src = t - taps + 1 + j
            if src >= 0:
                y[t] += w[:, j] * x[src]
    return y


def ssd_scan(x, B, C, dt, a_log, D):
    """x [T, H, V], B and C [T, G, N], dt [T, H] (positive): per head S <- exp(-exp(a_log) dt) S + dt B x^T, y = S^T C + D x."""
    T, H, V = x.shape
    G, N = B.shape[1], B.shape[2]
    y = np.zeros((T, H, V))
    for head in range(H):
        g = head // (H // G)
        S = np.zeros((N, V))
        for t in range(T):
            S = math.exp(-math.exp(a_log[head]) * dt[t, head]) * S + dt[t, head] * np.outer(B[t, g], x[t, head])
            y[t, head] = S.T @ C[t, g] + D[head] * x[t, head]
    return y


def grouped_gated_norm(y, z, w, groups, eps):
    """rms over each of ``groups`` equal parts of y * silu(z), times w per channel."""
    T, inner = y.shape
    return rms_unit((y * silu(z)).reshape(T, groups, inner // groups), eps).reshape(T, inner) * w


def state_space(h, W, p, m, eps):
    T = h.shape[0]
    H, V, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner, gn = H * V, G * N
    row = h @ W[p + "in"].T
    z, xbc, dt = row[:, :inner], row[:, inner:2 * inner + 2 * gn], row[:, 2 * inner + 2 * gn:]
    xbc = silu(causal_conv(xbc, W[p + "conv"], W[p + "conv.b"]))
    x, B, C = xbc[:, :inner], xbc[:, inner:inner + gn], xbc[:, inner + gn:]
    y = ssd_scan(x.reshape(T, H, V), B.reshape(T, G, N), C.reshape(T, G, N), softplus(dt + W[p + "dt_bias"]), W[p + "A_log"],
                 W[p + "D"])
    return grouped_gated_norm(y.reshape(T, inner), z, W[p + "norm"], m["norm_groups"], eps) @ W[p + "o"].T


def parallel(h, W, p, m, eps):
    """Half the sum of the two mixers' outputs, each normed over the model width first."""
    left = attention(h, W, p + "left.", m["left"], eps)
    right = state_space(h, W, p + "right.", m["right"], eps)
    return 0.5 * (rms_unit(left, eps) * W[p + "left.out"] + rms_unit(right, eps) * W[p + "right.out"])


def dense_ff(h, W, p, mlp):
    g = np.minimum(h @ W[p + "gate"].T, mlp["limit"])
    u = np.clip(h @ W[p + "up"].T, -mlp["limit"], mlp["limit"])
    return (g * logistic(SLOPE * g) * (u + 1.0)) @ W[p + "down"].T


def choose(scores, top, groups, keep):
    """The ``top`` experts with the largest scores among those of the ``keep`` groups whose largest score is largest."""
    per = len(scores) // groups
    best = [max(scores[g * per:(g + 1) * per]) for g in range(groups)]
    kept = sorted(range(groups), key=lambda g: -best[g])[:keep]
    allowed = [e for g in kept for e in range(g * per, (g + 1) * per)]
    return sorted(allowed, key=lambda e: (-scores[e], e))[:top]


def route(h, W, p, router):
    """([T, top] experts, [T, top] weights): softmax over all experts, the chosen scores divided by their sum."""
    groups = router.get("groups") or {"count": 1, "keep": 1}
    order, weight = [], []
    for t in range(h.shape[0]):
        s = softmax(W[p + "router"] @ h[t])
        chosen = choose(list(s), router["top"], groups["count"], groups["keep"])
        order.append(chosen)
        weight.append(s[chosen] / (s[chosen].sum() + 1e-20))
    return np.array(order), np.array(weight)


def expert(h_row, W, p, e):
    q = f"{p}e{e}."
    return W[q + "down"] @ (silu(W[q + "gate"] @ h_row) * (W[q + "up"] @ h_row))


def moe_ff(h, W, p, mlp):
    order, weight = route(h, W, p, mlp["router"])
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(order[t], weight[t]):
            out[t] += w * expert(h[t], W, p, int(e))
    return out


def feed_forward(h, W, p, mlp):
    return dense_ff(h, W, p, mlp) if mlp["kind"] == "dense" else moe_ff(h, W, p, mlp)


def forward(cfg, W, tokens, collect=None):
    """tokens -> logits [T, vocab]. ``collect`` (a list) receives the residual after every layer."""
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = embed(W, tokens, cfg["embedding"]["scale"])
    for i, L in enumerate(cfg["layers"]):
        t = f"l{i}."
        x = rms_unit(alpha * x + parallel(x, W, t + "mix.", L["mixer"], eps), eps) * W[t + "norm1"]
        if L.get("mlp") is not None:
            x = rms_unit(alpha * x + feed_forward(x, W, t + "mlp.", L["mlp"]), eps) * W[t + "norm2"]
        if collect is not None:
            collect.append(x.copy())
    return rms_unit(x, eps) * W["final.norm"] @ W["head"].T
