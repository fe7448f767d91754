"""Plain float64 restatement of the Vinozen decoder: whole sequences, no cache, no batching, one function per
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


def softplus(z):
    return np.logaddexp(0.0, z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def layer_norm(x, weight, eps):
    """Centred, to unit standard deviation, times the weight."""
    c = x - np.mean(x, axis=-1, keepdims=True)
    return c / np.sqrt(np.mean(c * c, axis=-1, keepdims=True) + eps) * weight


def group_rms_norm(x, weight, eps, groups):
    """Every one of `groups` equal consecutive parts of a row to unit rms by itself, then the weight over the row."""
    parts = x.reshape(x.shape[:-1] + (groups, x.shape[-1] // groups))
    return rms_unit(parts, eps).reshape(x.shape) * weight


def product(x, W, rnd=same):
    """x @ W.T with the rounding points of a 16-bit product: its input and its output."""
    return rnd(rnd(x) @ W.T)


# ---------------------------------------------------------------- embedding
def sinusoid(positions, width):
    """[T, width]: column 2i the sine, column 2i + 1 the cosine of position * 10000^(-2i / width)."""
    out = np.zeros((len(positions), width))
    for c in range(width):
        a = np.asarray(positions, dtype=np.float64) * 10000.0 ** (-2.0 * (c // 2) / width)
        out[:, c] = np.cos(a) if c % 2 else np.sin(a)
    return out


def embed(tokens, w, cfg, position0=0):
    scale = (cfg.get("embedding") or {}).get("scale", 1.0)
    return w["embed"][tokens] * scale + sinusoid(np.arange(position0, position0 + len(tokens)), cfg["width"])


# ---------------------------------------------------------------- attention
def bucket(n, rows, reach):
    """The row of a table of `rows` biases for a key `n` positions back: exact distances in the first half, the second
    half in equal steps of the logarithm up to `reach`, everything further in the last row.  Integers throughout:
    floor(a) >= k is asked as (n / half)^(rows - half) >= (reach / half)^k."""
    half = rows // 2
    if n < half:
        return n
    k = 0
    while k < rows - half - 1 and n ** (rows - half) * half ** (k + 1) >= reach ** (k + 1) * half ** (rows - half):
        k += 1
    return half + k


def query_temperature(positions, coef, every):
    return 1.0 + coef * np.log(np.floor((np.asarray(positions, dtype=np.float64) + 1.0) / every) + 1.0)


def biased_attention(q, k, v, scale, rel, reach, sink):
    """q [T, H, d], k [T, G, d], v [T, G, vd] of one sequence from its start; query head h reads key/value head
    h // (H / G); rel [rows, H] biases by distance; sink [H]: one more term exp(sink_h) in the denominator."""
    T, H, _ = q.shape
    G = k.shape[1]
    rows = np.array([bucket(n, rel.shape[0], reach) for n in range(T)])
    back = np.arange(T)[:, None] - np.arange(T)[None, :]
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale + rel[rows[np.maximum(back, 0)], h]
        s = np.where(back >= 0, s, -np.inf)
        top = np.maximum(s.max(axis=1, keepdims=True), sink[h])
        p = np.exp(s - top)
        p = p / (p.sum(axis=1, keepdims=True) + np.exp(sink[h] - top))
        out[:, h] = p @ v[:, g]
    return out


def attention(x, w, p, m, eps, kept=None, rnd=same):
    """The mixer of the layer with tensors `p` + name.  `kept`: the (keys, values) of another layer that this one reads
    instead of making its own.  Returns (output, (keys, values))."""
    T, H, G, d, vd = len(x), m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_unit(product(x, w[p + "q"], rnd).reshape(T, H, d), eps)
    temp = m.get("q_temp")
    if temp:
        q = q * query_temperature(np.arange(T), temp["coef"], temp["every"])[:, None, None]
    q = rnd(q)
    if kept is None:
        kept = (rnd(rms_unit(product(x, w[p + "k"], rnd).reshape(T, G, d), eps)),
                product(x, w[p + "v"], rnd).reshape(T, G, vd))
    o = biased_attention(q, kept[0], kept[1], m["scale"], w[p + "rel"], m["bias_max"], w[p + "sink"])
    return product(o.reshape(T, H * vd), w[p + "o"], rnd), kept


# ---------------------------------------------------------------- state-space mixer
def short_convolution(u, weight, bias):
    """y_t = sum_j weight[:, j] u_(t - taps + 1 + j) + bias per channel, u = 0 before the start."""
    taps = weight.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, u.shape[1])), u])
    return sum(padded[j:j + len(u)] * weight[:, j] for j in range(taps)) + bias


def state_space(xs, B, C, dt, decay_rate, skip):
    """xs [T, H, vd], B and C [T, G, n], dt [T, H]; head h uses group h // (H / G):
    S <- exp(-decay_rate_h dt) S + dt B x^T,  y = S^T C + skip_h x."""
    T, H, vd = xs.shape
    G, n = B.shape[1:]
    y = np.zeros_like(xs)
    for h in range(H):
        S, g = np.zeros((n, vd)), h // (H // G)
        for t in range(T):
            S = np.exp(-decay_rate[h] * dt[t, h]) * S + dt[t, h] * np.outer(B[t, g], xs[t, h])
            y[t, h] = S.T @ C[t, g] + skip[h] * xs[t, h]
    return y


def mamba2(x, w, p, m, eps, rnd=same):
    T, H, vd, n, G = len(x), m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * vd
    proj = rnd(x) @ w[p + "in"].T
    z, u, dt = rnd(proj[:, :inner]), rnd(proj[:, inner:2 * inner + 2 * G * n]), proj[:, 2 * inner + 2 * G * n:]
    u = rnd(silu(short_convolution(u, w[p + "conv"], w[p + "conv.b"])))
    xs, B, C = u[:, :inner], u[:, inner:inner + G * n], u[:, inner + G * n:]
    y = state_space(xs.reshape(T, H, vd), B.reshape(T, G, n), C.reshape(T, G, n), softplus(dt + w[p + "dt_bias"]),
                    np.exp(w[p + "A_log"]), w[p + "D"]).reshape(T, inner)
    y = group_rms_norm(y * silu(z), w[p + "norm"], eps, m["norm_groups"])
    return product(y, w[p + "o"], rnd)


# ---------------------------------------------------------------- feed-forward
def dense(x, w, p, rnd=same):
    return product(silu(product(x, w[p + "gate"], rnd)) * product(x, w[p + "up"], rnd), w[p + "down"], rnd)


def clamped(x, w, p, limit, rnd=same):
    g = np.minimum(rnd(x) @ w[p + "gate"].T, limit)
    u = np.clip(rnd(x) @ w[p + "up"].T, -limit, limit)
    return rnd(rnd(g * sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T)


def route(z, top):
    """(ids, weights): the `top` largest logits (the earlier of equals), weighted by the softmax over them alone."""
    ids = np.argsort(-z, axis=-1, kind="stable")[:, :top]
    chosen = np.take_along_axis(z, ids, axis=-1)
    e = np.exp(chosen - chosen.max(axis=-1, keepdims=True))
    return ids, e / e.sum(axis=-1, keepdims=True)


def experts(x, w, p, mlp, rnd=same):
    ids, weights = route(rnd(x) @ w[p + "router"].T + w[p + "router.b"], mlp["router"]["top"])
    out = np.zeros_like(x)
    for e in range(mlp["router"]["experts"]):
        rows, place = np.nonzero(ids == e)
        if len(rows):
            out[rows] += weights[rows, place][:, None] * clamped(x[rows], w, f"{p}e{e}.", mlp["expert"]["limit"], rnd)
    if mlp.get("shared"):
        out = out + clamped(x, w, p + "shared.", mlp["shared"]["limit"], rnd)
    return rnd(out)


def feed_forward(x, w, p, mlp, rnd=same):
    return dense(x, w, p, rnd) if mlp["kind"] == "dense" else experts(x, w, p, mlp, rnd)


# ---------------------------------------------------------------- the model
def side_input(x, tokens, w, p, layer, dim, eps, rnd=same):
    e = w["side.embed"][tokens][:, layer * dim:(layer + 1) * dim]
    g = rnd(gelu_tanh(product(x, w[p + "side.gate"], rnd)) * e)
    return rms_unit(product(g, w[p + "side.proj"], rnd), eps) * w[p + "side.norm"]


def hidden(tokens, w, cfg, rnd=same):
    """The hidden rows [layers, T, width] after every layer."""
    tokens = np.asarray(tokens)
    eps = cfg["norm"]["eps"]
    x, kept, after = embed(tokens, w, cfg), {}, []
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        if layer["type"] == "mamba2":
            y = mamba2(x, w, p + "mix.", m, eps, rnd)
        else:
            source = m.get("kv_from")
            y, kept[i] = attention(x, w, p + "mix.", m, eps, None if source is None else kept[source], rnd)
        x = x + layer_norm(y, w[p + "norm1"], eps)
        if layer.get("mlp"):
            x = x + layer_norm(feed_forward(x, w, p + "mlp.", layer["mlp"], rnd), w[p + "norm2"], eps)
        if cfg.get("token_side"):
            x = x + side_input(x, tokens, w, p, i, cfg["token_side"]["dim"], eps, rnd)
        after.append(x)
    return np.stack(after)


def logits(tokens, w, cfg, rnd=same):
    x = layer_norm(hidden(tokens, w, cfg, rnd)[-1], w["final.norm"], cfg["norm"]["eps"])
    return rnd(x) @ w["embed"].T
