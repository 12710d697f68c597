"""Lodenex in plain float64 NumPy, one function per mechanism, written from the architecture's equations and sharing no code
with the engine. Slow on purpose: attention is a loop over (head, query), the latent attention forms every head's keys and
values before it scores them.

Notation: T tokens, d model width, a sequence's positions count from 0. ``W`` maps tensor names to float64 arrays (matrices
stored [out, in] and applied as W x); ``p`` is the prefix of a part's tensor names; ``m`` the part's sizes as config.json gives
them. A layer is x <- x + norm1(mixer(x)); x <- x + norm2(ff(x)).
"""
import math

import numpy as np


def logistic(x):
    return 1.0 / (1.0 + np.exp(-np.asarray(x, dtype=np.float64)))


def rms(x, weight, eps):
    """weight * x / sqrt(mean(x^2) + eps) over the last axis."""
    return weight * x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def gelu(x):
    """x times the normal distribution's cumulative function."""
    x = np.asarray(x, dtype=np.float64)
    return 0.5 * x * (1.0 + np.vectorize(math.erf, otypes=[np.float64])(x / math.sqrt(2.0)))


def tanh_cap(x, cap):
    return x if cap is None else cap * np.tanh(x / cap)


def embed(W, tokens, scale):
    return W["embed"][np.asarray(tokens)] * scale


# ------------------------------------------------------------------------------------------------------------- rotation
def base_frequencies(dims, base):
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def frequencies_by_wavelength(dims, base, sc):
    """Short wavelengths keep their frequency, long ones are slowed by the factor, the ones between are blended."""
    out = []
    for f in base_frequencies(dims, base):
        if sc is not None:
            wavelength = 2.0 * math.pi / f
            if wavelength > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif not wavelength < sc["original"] / sc["high"]:
                s = (sc["original"] / wavelength - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out, 1.0


def frequencies_by_turns(dims, base, sc):
    """Pairs are slowed along a ramp over their index, whose ends are the pairs that turn ``fast`` and ``slow`` times within
    the original context; sine and cosine are lengthened."""
    f = base_frequencies(dims, base)
    if sc is None:
        return f, 1.0

    def index_of(turns):
        return dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(index_of(sc["fast"])), 0), min(math.ceil(index_of(sc["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * ramp + fi * (1.0 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, position, freqs, length):
    """x [..., >= 2 len(freqs)]: component i is turned with component i + len(freqs), the rest stays."""
    half = len(freqs)
    y = np.array(x, dtype=np.float64)
    for i, f in enumerate(freqs):
        c, s = length * math.cos(position * f), length * math.sin(position * f)
        u, v = x[..., i], x[..., i + half]
        y[..., i], y[..., i + half] = u * c - v * s, v * c + u * s
    return y


def rotate_all(x, freqs, length):
    return np.stack([rotate(x[t], t, freqs, length) for t in range(len(x))]) if len(x) else x


# ------------------------------------------------------------------------------------------------------------ attention
def chunk_keys(i, size):
    """The keys that the query at position i sees: those of its own chunk, up to itself."""
    return [j for j in range(i + 1) if size is None or j // size == i // size]


def window_keys(i, size):
    return [j for j in range(i + 1) if size is None or i - j < size]


def sink_softmax(scores, sink):
    """exp(s_j) / (sum_j exp(s_j) + exp(sink)); ``sink`` None: an ordinary softmax."""
    top = scores.max() if sink is None else max(scores.max(), sink)
    e = np.exp(scores - top)
    return e / (e.sum() + (0.0 if sink is None else math.exp(sink - top)))


def capped_attention(q, k, v, scale, cap, sink, size):
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H, V]: chunks of ``size`` positions, capped scores, a sink per head."""
    T, H = q.shape[:2]
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for head in range(H):
        g = head // (H // G)
        for i in range(T):
            js = chunk_keys(i, size)
            s = tanh_cap(k[js, g] @ q[i, head] * scale, cap)
            out[i, head] = sink_softmax(s, None if sink is None else sink[head]) @ v[js, g]
    return out


def attention(h, W, p, m, eps):
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms(h @ W[p + "q"].T, W[p + "q.norm"], eps).reshape(T, H, D)        # normed before the heads are told apart
    k = rms(h @ W[p + "k"].T, W[p + "k.norm"], eps).reshape(T, G, D)
    v = (h @ W[p + "v"].T).reshape(T, G, V)
    freqs, length = frequencies_by_wavelength(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
    out = capped_attention(rotate_all(q, freqs, length), rotate_all(k, freqs, length), v, m["scale"], m.get("softcap"), W[p + "sink"],
                           m["mask"]["size"] if m.get("mask") else None)
    gate = logistic(h @ W[p + "g"].T)                                        # one number per head
    return (out * gate[:, :, None]).reshape(T, H * V) @ W[p + "o"].T


def latent_attention(h, W, p, m, eps):
    T = h.shape[0]
    H, D, R, V, c = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (rms(h @ W[p + "dq"].T, W[p + "dq.norm"], eps) @ W[p + "uq"].T).reshape(T, H, D + R)
    down = h @ W[p + "dkv"].T
    latent = rms(down[:, :c], W[p + "dkv.norm"], eps)
    k = (latent @ W[p + "uk"].T).reshape(T, H, D)
    v = (latent @ W[p + "uv"].T).reshape(T, H, V)
    freqs, length = frequencies_by_turns(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
    q_rot, k_rot = rotate_all(q[:, :, D:], freqs, length), rotate_all(down[:, c:], freqs, length)
    out = np.zeros((T, H, V))
    for head in range(H):
        for i in range(T):
            js = window_keys(i, m["mask"]["size"] if m.get("mask") else None)
            s = (k[js, head] @ q[i, head, :D] + k_rot[js] @ q_rot[i, head]) * m["scale"]
            out[i, head] = sink_softmax(s, None) @ v[js, head]
    gate = logistic(h @ W[p + "g"].T)                                        # one number per output channel
    return (out.reshape(T, H * V) * gate) @ W[p + "o"].T


# -------------------------------------------------------------------------------------------------------- feed-forward, model
def dense_ff(h, W, p):
    return gelu(h @ W[p + "up"].T) @ W[p + "down"].T


def forward(cfg, W, tokens, collect=None):
    """tokens -> logits [T, vocab]. ``collect`` (a list) receives the residual after every layer."""
    eps = cfg["norm"]["eps"]
    x = embed(W, tokens, cfg["embedding"]["scale"])
    for i, L in enumerate(cfg["layers"]):
        t = f"l{i}."
        mixer = {"attention": attention, "latent_attention": latent_attention}[L["type"]]
        x = x + rms(mixer(x, W, t + "mix.", L["mixer"], eps), W[t + "norm1"], eps)
        if L.get("mlp") is not None:
            x = x + rms(dense_ff(x, W, t + "mlp."), W[t + "norm2"], eps)
        if collect is not None:
            collect.append(x.copy())
    return tanh_cap(rms(x, W["final.norm"], eps) @ W["head"].T, cfg.get("logit_softcap"))
