"""Plain float64 restatement of the Vogerax decoder: whole sequences, no cache, no batching, one function per
mechanism, NumPy only.  It shares no code with the package and is the oracle of its tests.

Notation: x [T, width] a sequence's hidden rows; W matrices stored [out, in] and applied as x @ W.T;
`cfg` is the dict of a config.json, `w` a dict name -> float64 array.  `rnd` (default: the identity) is applied
to what a 16-bit implementation may round: the input and the output of every matrix product, what the cache holds.
The tests take the deviation it causes as the scale of their bfloat16 tolerance.
"""
from __future__ import annotations

import math

import numpy as np


def same(x):
    return x


def round_bf16(x):
    """Round to the nearest bfloat16 (ties to even), as float64."""
    u = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32).astype(np.uint64)
    u = ((u + 0x7FFF + ((u >> 16) & 1)) >> 16) << 16
    return u.astype(np.uint32).view(np.float32).astype(np.float64).reshape(np.shape(x))


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def relu_squared(z):
    return np.maximum(z, 0.0) ** 2


def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, weight, eps):
    return rms_unit(x, eps) * weight


def group_norm(x, weight, eps, groups):
    """Every one of `groups` equal consecutive parts of a row to unit rms by itself, then the weight over the whole row."""
    parts = x.reshape(x.shape[:-1] + (groups, x.shape[-1] // groups))
    return rms_unit(parts, eps).reshape(x.shape) * weight


def product(x, W, rnd=same):
    """x @ W.T with the rounding points of a 16-bit product: its input and its output."""
    return rnd(rnd(x) @ W.T)


# ---------------------------------------------------------------- rotation
def plain_frequencies(base, dims):
    return np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])


def yarn(base, dims, scaling):
    """(frequencies, factor on cosine and sine): low frequencies divided by `factor`, high ones kept, a linear ramp over
    the pair's index between the pairs that turn `fast` and `slow` times over `original` positions."""
    factor, original = scaling["factor"], scaling["original"]

    def index_of(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(index_of(scaling["fast"])), 0)
    hi = min(math.ceil(index_of(scaling["slow"])), dims - 1)
    freq = plain_frequencies(base, dims)
    for i in range(dims // 2):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        freq[i] = freq[i] / factor * ramp + freq[i] * (1.0 - ramp)
    return freq, 0.1 * math.log(factor) + 1.0


def rotary(v, positions, freq, magnitude=1.0, sign=1.0):
    """Rotate the first 2 len(freq) values of the last axis of v [T, heads, n] in pairs (i, i + len(freq)) by
    sign * position * freq_i; cosine and sine are multiplied by `magnitude`."""
    half = len(freq)
    a = sign * np.asarray(positions, dtype=np.float64)[:, None] * freq[None, :]
    c, s = magnitude * np.cos(a)[:, None, :], magnitude * np.sin(a)[:, None, :]
    out = v.copy()
    u, t = v[..., :half], v[..., half:2 * half]
    out[..., :half] = u * c - t * s
    out[..., half:2 * half] = t * c + u * s
    return out


# ---------------------------------------------------------------- softmax attention
def pooled_blocks(x, size):
    """[blocks, ...]: the mean of every whole block of `size` rows."""
    n = x.shape[0] // size
    return x[:n * size].reshape((n, size) + x.shape[1:]).mean(axis=1)


def visible(T, window, pool):
    """Masks of tokens [T, T] and of blocks [T, T // pool]: token j from i if 0 <= i - j < window; block b, the positions
    b pool .. b pool + pool - 1, if its last position lies before i's window."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    last = np.arange(T // pool)[None, :] * pool + pool - 1
    return (j <= i) & (i - j < window), last <= i - window


def softmax_attention(q, k, v, scale, mask, sink=None):
    """q [T, H, d], k [S, G, d], v [S, G, vd], mask [T, S]; query head h reads key/value head h // (H / G).  `sink` [H]:
    one more term exp(sink_h) in the denominator.  Returns [T, H, vd]."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        s = np.where(mask, (q[:, h] @ k[:, g].T) * scale, -np.inf)
        top = s.max(axis=1, keepdims=True)
        if sink is not None:
            top = np.maximum(top, sink[h])
        p = np.exp(s - top)
        total = p.sum(axis=1, keepdims=True)
        if sink is not None:
            total = total + np.exp(sink[h] - top)
        out[:, h] = (p / total) @ v[:, g]
    return out


def pooled_window_attention(h, w, p, m, rnd=same):
    """The 'attention' mixer: values are the projected keys, rotation with linearly scaled frequencies on q and k, a sliding
    window beside which every block of `pool` tokens that has left it is seen as one mean key and one mean value."""
    T = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    q = product(h, w[p + "q"], rnd).reshape(T, H, d)
    k = product(h, w[p + "k"], rnd).reshape(T, G, d)
    v = k
    rot = m.get("rot")
    if rot and rot["dims"]:
        freq = plain_frequencies(rot["base"], rot["dims"])
        if rot.get("scaling"):
            freq = freq / rot["scaling"]["factor"]
        q, k = rotary(q, range(T), freq), rotary(k, range(T), freq)
    q, k = rnd(q), rnd(k)
    mask = m["mask"]
    tokens, blocks = visible(T, mask["size"], mask["pool"])
    keys = np.concatenate([k, rnd(pooled_blocks(k, mask["pool"]))])
    values = np.concatenate([v, rnd(pooled_blocks(v, mask["pool"]))])
    o = softmax_attention(q, keys, values, m["scale"], np.concatenate([tokens, blocks], axis=1))
    return product(o.reshape(T, H * d), w[p + "o"], rnd)


def rotated_value_attention(h, w, p, m, eps, rnd=same):
    """The left half of the 'parallel' mixer: normed queries and keys, YaRN rotation, values rotated by their own position
    and turned back by the query's after the sum, every earlier key, a learned sink, an elementwise output gate."""
    T = h.shape[0]
    H, G, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = product(h, w[p + "q"], rnd).reshape(T, H, d)
    k = product(h, w[p + "k"], rnd).reshape(T, G, d)
    v = product(h, w[p + "v"], rnd).reshape(T, G, vd)
    q, k = rms_norm(q, w[p + "q.norm"], eps), rms_norm(k, w[p + "k.norm"], eps)
    rot = m["rot"]
    freq, magnitude = plain_frequencies(rot["base"], rot["dims"]), 1.0
    if rot.get("scaling"):
        freq, magnitude = yarn(rot["base"], rot["dims"], rot["scaling"])
    q, k = rotary(q, range(T), freq, magnitude), rotary(k, range(T), freq, magnitude)
    value_freq = plain_frequencies(rot["base"], vd)
    v = rotary(v, range(T), value_freq)
    causal = np.tril(np.ones((T, T), dtype=bool))
    o = softmax_attention(rnd(q), rnd(k), rnd(v), m["scale"], causal, w[p + "sink"])
    o = rotary(rnd(o), range(T), value_freq, sign=-1.0)
    o = o.reshape(T, H * vd) * sigmoid(product(h, w[p + "g"], rnd))
    return product(o, w[p + "o"], rnd)


# ---------------------------------------------------------------- retention
def retention(h, w, p, m, eps, rnd=same):
    """The right half of the 'parallel' mixer: S_t = decay_h S_(t-1) + k_t v_t^T, o_t = S_t^T q_t with rotated q and k."""
    T = h.shape[0]
    H, d, vd = m["heads"], m["dim"], m["vdim"]
    q = product(h, w[p + "q"], rnd).reshape(T, H, d)
    k = product(h, w[p + "k"], rnd).reshape(T, H, d)
    v = product(h, w[p + "v"], rnd).reshape(T, H, vd)
    rot = m.get("rot")
    if rot and rot["dims"]:
        freq = plain_frequencies(rot["base"], rot["dims"])
        q, k = rotary(q, range(T), freq), rotary(k, range(T), freq)
    k = k * d ** -0.5
    out = np.zeros((T, H, vd))
    for a in range(H):
        S = np.zeros((d, vd))
        for t in range(T):
            S = m["decay"][a] * S + np.outer(k[t, a], v[t, a])
            out[t, a] = S.T @ q[t, a]
    o = rms_unit(out, eps).reshape(T, H * vd) * silu(product(h, w[p + "g"], rnd))
    return product(o, w[p + "o"], rnd)


def parallel_mixer(h, w, p, m, eps, rnd=same):
    """Half the sum of the two mixers' outputs, each to unit rms over the width with a weight."""
    left = rotated_value_attention(h, w, p + "left.", m["left"], eps, rnd)
    right = retention(h, w, p + "right.", m["right"], eps, rnd)
    return rnd(0.5 * (rms_norm(left, w[p + "left.out"], eps) + rms_norm(right, w[p + "right.out"], eps)))


# ---------------------------------------------------------------- feed-forwards
def squared_relu_mlp(h, w, p, rnd=same):
    return product(relu_squared(product(h, w[p + "up"], rnd)), w[p + "down"], rnd)


def route(h, w, p, r, rnd=same):
    """For every token the experts with the largest scores (softmax over all of them) and those scores as weights."""
    z = rnd(h) @ w[p + "router"].T
    s = np.exp(z - z.max(axis=1, keepdims=True))
    s /= s.sum(axis=1, keepdims=True)
    ids = np.argsort(-s, axis=1, kind="stable")[:, :r["top"]]
    return ids, np.take_along_axis(s, ids, axis=1)


def mixture(h, w, p, mlp, rnd=same):
    ids, weights = route(h, w, p, mlp["router"], rnd)
    out = squared_relu_mlp(h, w, p + "shared.", rnd) if mlp.get("shared") else np.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        rows, which = np.nonzero(ids == e)
        if rows.size:
            out[rows] += weights[rows, which][:, None] * squared_relu_mlp(h[rows], w, f"{p}e{e}.", rnd)
    return rnd(out)


def feed_forward(h, w, p, mlp, rnd=same):
    if mlp["kind"] == "dense":
        return squared_relu_mlp(h, w, p, rnd)
    return mixture(h, w, p, mlp, rnd)


# ---------------------------------------------------------------- the model
def mixer(h, w, p, layer, eps, rnd=same):
    if layer["type"] == "attention":
        return pooled_window_attention(h, w, p, layer["mixer"], rnd)
    if layer["type"] == "parallel":
        return parallel_mixer(h, w, p, layer["mixer"], eps, rnd)
    raise ValueError(layer["type"])


def hidden_states(cfg, w, tokens, rnd=same):
    """The hidden rows after every layer, [layers, T, width]."""
    eps, groups = cfg["norm"]["eps"], cfg["norm"]["groups"]

    def norm(x, name):
        return group_norm(x, w[name], eps, groups)
    x = w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    states = []
    for i, layer in enumerate(cfg["layers"]):
        source = layer.get("weights_of")
        p = f"l{i if source is None else source}."
        x = x + norm(mixer(norm(x, p + "norm1"), w, p + "mix.", layer, eps, rnd), p + "norm1b")
        if layer.get("mlp"):
            x = x + norm(feed_forward(norm(x, p + "norm2"), w, p + "mlp.", layer["mlp"], rnd), p + "norm2b")
        states.append(x)
    return np.stack(states)


def forward(cfg, w, tokens, rnd=same):
    """Logits [T, vocab] of one sequence."""
    x = hidden_states(cfg, w, tokens, rnd)[-1]
    return rnd(group_norm(x, w["final.norm"], cfg["norm"]["eps"], cfg["norm"]["groups"])) @ w["head"].T
