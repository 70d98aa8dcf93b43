"""A plain, slow statement of the Rudolix decoder: one function per mechanism, NumPy float64, whole
sequences, no cache, no batching.  It shares no code with the library under test.

The design: the residual is carried in several streams, all equal to the scaled embedding row at the start.
A sublayer (mixer or feed-forward) reads a learned combination of the streams under a layer norm with gain and
bias, to which a short causal convolution of itself is added; its result, scaled channel by channel, is dealt
out to the streams, which are mixed by a learned matrix in the same update.  Three mixers: a gated delta rule
with one decay per head, a Mamba-2 state-space layer and grouped-query softmax attention with rotary positions
and a learned sink in the softmax's denominator.  Two feed-forwards: a dense one whose activation is a
polynomial of normed powers, and a mixture of clamped gated experts whose router has a bias.  The streams'
sum is normed and multiplied with the embedding table.

``r`` rounds what a bfloat16 engine stores in bfloat16 (projections, cached rows, activations); the streams,
norms, scores, weights, angles, routers and the recurrences' inputs and states stay unrounded, as they do there.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional, Sequence

import numpy as np


def _id(a):
    return a


def to_bf16(a):
    """Round to the nearest bfloat16 (ties to even), returned as float64."""
    f = np.ascontiguousarray(a, dtype=np.float32)
    u = f.view(np.uint32).astype(np.uint64)
    u = ((u + 0x7FFF + ((u >> 16) & 1)) >> 16) << 16
    return u.astype(np.uint32).view(np.float32).astype(np.float64).reshape(np.shape(a))


# ---- small pieces ------------------------------------------------------------------------------
def unit_rms(x, eps):
    """x over its root mean square along the last axis (eps inside the root)."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def layer_norm(x, w, b, eps):
    mean = np.mean(x, axis=-1, keepdims=True)
    d = x - mean
    return d / np.sqrt(np.mean(d * d, axis=-1, keepdims=True) + eps) * w + b


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def unit_vector(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def shared_head(h: int, heads: int, shared: int) -> int:
    """The key/value head (or group) that head h of ``heads`` uses when there are ``shared`` of them."""
    return h // (heads // shared)


def causal_convolution(x, taps, bias=None):
    """Along the sequence, channel by channel; the last tap is the current token's, missing inputs are zeros; x [T, C],
    taps [C, n]."""
    n = taps.shape[1]
    past = np.concatenate([np.zeros((n - 1, x.shape[1])), x])
    y = sum(past[j: j + x.shape[0]] * taps[:, j] for j in range(n))
    return y if bias is None else y + bias


# ---- streams ------------------------------------------------------------------------------------
def read_streams(xs, weights):
    """What a sublayer reads: the streams [S, T, W] combined by one number each."""
    return np.einsum("s,stw->tw", weights, xs)


def update_streams(xs, mix, out, m, y):
    """The new streams: the matrix ``mix`` (from, to) applied to the old ones, and y added m out[t] times to stream t."""
    return np.einsum("st,snw->tnw", mix, xs) + m * out[:, None, None] * y[None]


def sublayer_input(u, w, p, q, eps, r=_id):
    """Norm number q of the layer, with a causal convolution of itself added."""
    h = r(layer_norm(u, w[f"{p}norm{q}"], w[f"{p}norm{q}.b"], eps))
    return r(h + causal_convolution(h, w[f"{p}canon{q}"]))


# ---- mixers -------------------------------------------------------------------------------------
def delta_rule(q, k, v, g, beta):
    """One head along the sequence; every read-out sees its own token's write.  q, k [T, d], v [T, dv], g, beta [T];
    returns ([T, dv], the last S)."""
    S = np.zeros((q.shape[1], v.shape[1]))
    out = np.zeros_like(v)
    for t in range(q.shape[0]):
        S = g[t] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + np.outer(k[t], u)
        out[t] = S.T @ q[t]
    return out, S


def mixer_delta(h, w, p, m, eps, r=_id):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = silu(causal_convolution(r(h @ w[p + "q"].T), w[p + "q.conv"])).reshape(T, G, d)
    k = silu(causal_convolution(r(h @ w[p + "k"].T), w[p + "k.conv"])).reshape(T, G, d)
    v = silu(causal_convolution(r(h @ w[p + "v"].T), w[p + "v.conv"])).reshape(T, H, dv)
    q, k = unit_vector(q) * d ** -0.5, unit_vector(k)
    beta = sigmoid(h @ w[p + "b"].T)
    g = np.exp(-np.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    o = np.stack([delta_rule(q[:, shared_head(i, H, G)], k[:, shared_head(i, H, G)], v[:, i], g[:, i], beta[:, i])[0]
                  for i in range(H)], axis=1)
    gate = silu(r(h @ w[p + "g"].T)).reshape(T, H, dv)
    y = unit_rms(o, eps) * w[p + "norm"] * gate
    return r(y).reshape(T, H * dv) @ w[p + "o"].T


def state_space(x, B, C, dt, a, D):
    """One head along the sequence; a decays the state at the rate of the step sizes dt.  x [T, P], B, C [T, N], dt [T]."""
    S = np.zeros((B.shape[1], x.shape[1]))
    y = np.zeros_like(x)
    for t in range(x.shape[0]):
        S = math.exp(-a * dt[t]) * S + dt[t] * np.outer(B[t], x[t])
        y[t] = S.T @ C[t] + D * x[t]
    return y, S


def grouped_rms(y, parts, eps):
    """RMS norm of every row cut into equal parts that are normed apart."""
    T, n = y.shape
    return unit_rms(y.reshape(T, parts, n // parts), eps).reshape(T, n)


def mixer_mamba2(h, w, p, m, eps, r=_id):
    T = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner, bc = H * P, G * N
    full = h @ w[p + "in"].T
    z, xbc, dt = r(full[:, :inner]), r(full[:, inner: 2 * inner + 2 * bc]), full[:, 2 * inner + 2 * bc:]
    xbc = silu(causal_convolution(xbc, w[p + "conv"], w[p + "conv.b"]))
    x = xbc[:, :inner].reshape(T, H, P)
    B, C = xbc[:, inner: inner + bc].reshape(T, G, N), xbc[:, inner + bc:].reshape(T, G, N)
    dt = softplus(dt + w[p + "dt_bias"])
    a = np.exp(w[p + "A_log"])
    y = np.stack([state_space(x[:, i], B[:, shared_head(i, H, G)], C[:, shared_head(i, H, G)], dt[:, i], float(a[i]),
                              float(w[p + "D"][i]))[0] for i in range(H)], axis=1).reshape(T, inner)
    y = grouped_rms(y * silu(z), m["norm_groups"], eps) * w[p + "norm"]
    return r(y) @ w[p + "o"].T


def rotate_halves(x, positions, dims, base):
    """x [T, heads, d]: number i of the first ``dims`` is turned with number i + dims / 2 by position * base^(-2i/dims)."""
    half = dims // 2
    f = float(base) ** (-2.0 * np.arange(half) / dims)
    a = np.asarray(positions, dtype=np.float64)[:, None, None] * f
    u, v = x[..., :half], x[..., half:dims]
    return np.concatenate([u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a), x[..., dims:]], axis=-1)


def softmax_with_sink(scores, sink):
    """Weights of the last axis (-inf: not seen) whose denominator also holds exp(sink): the sink has no value."""
    top = np.maximum(scores.max(axis=-1, keepdims=True), sink)
    e = np.exp(scores - top)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(sink - top))


def attend(q, k, v, scale, sink):
    """One head, causal: q, k [T, d], v [T, dv]."""
    T = q.shape[0]
    s = np.where(np.tril(np.ones((T, T), dtype=bool)), (q @ k.T) * scale, -np.inf)
    return softmax_with_sink(s, sink) @ v


def mixer_attention(h, w, p, m, eps, r=_id):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = np.arange(T)
    q = r(h @ w[p + "q"].T).reshape(T, H, d)
    k = r(h @ w[p + "k"].T).reshape(T, G, d)
    v = r(h @ w[p + "v"].T).reshape(T, G, dv)
    rot = m["rot"]
    q, k = (r(rotate_halves(a, pos, int(rot["dims"]), rot["base"])) for a in (q, k))
    o = np.stack([attend(q[:, i], k[:, shared_head(i, H, G)], v[:, shared_head(i, H, G)], m["scale"], float(w[p + "sink"][i]))
                  for i in range(H)], axis=1)
    return r(o).reshape(T, H * dv) @ w[p + "o"].T


MIXERS = {"delta": mixer_delta, "mamba2": mixer_mamba2, "attention": mixer_attention}


# ---- feed-forwards ------------------------------------------------------------------------------
def poly_norm(z, coef, eps):
    """The activation of the dense unit: a polynomial whose powers are normed over the row."""
    a, b, c, e = (float(x) for x in coef)
    return a * unit_rms(z, eps) + b * unit_rms(z * z, eps) + c * unit_rms(z * z * z, eps) + e


def ffn_dense(h, w, p, f, eps, r=_id):
    z = r(h @ w[p + "up"].T)
    return r(poly_norm(z, w[p + "act"], eps)) @ w[p + "down"].T


def limited_unit(g, u, limit):
    g, u = np.minimum(g, limit), np.clip(u, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def expert(h, w, p, limit, r=_id):
    return r(limited_unit(r(h @ w[p + "gate"].T), r(h @ w[p + "up"].T), limit)) @ w[p + "down"].T


def route(h, w, p, top):
    """(ids [T, top], weights): the ``top`` largest logits' experts and the softmax among them."""
    z = h @ w[p + "router"].T + w[p + "router.b"]
    ids = np.argsort(-z, axis=1, kind="stable")[:, :top]
    c = np.take_along_axis(z, ids, axis=1)
    e = np.exp(c - c.max(axis=1, keepdims=True))
    return ids, e / e.sum(axis=1, keepdims=True)


def ffn_moe(h, w, p, f, eps, r=_id):
    ids, weights = route(h, w, p, int(f["router"]["top"]))
    out = np.zeros((h.shape[0], w[p + "e0.down"].shape[0]))
    for e in range(int(f["router"]["experts"])):
        rows, place = np.nonzero(ids == e)
        if len(rows):
            out[rows] += weights[rows, place][:, None] * r(expert(h[rows], w, f"{p}e{e}.", float(f["expert"]["limit"]), r))
    return out


FFNS = {"dense": ffn_dense, "moe": ffn_moe}


# ---- the model ----------------------------------------------------------------------------------
def sublayer(xs, w, cfg, p, q, fn, r=_id):
    """One update of all streams by sublayer q of the layer with tensors ``p``."""
    eps, m = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    u = read_streams(xs, w[f"{p}hc{q}.in"])
    y = fn(sublayer_input(u, w, p, q, eps, r)) * w[f"{p}ls{q}"]
    return update_streams(xs, w[f"{p}hc{q}.mix"], w[f"{p}hc{q}.out"], m, y)


def layer(xs, w, cfg, i, r=_id):
    L, p, eps = cfg["layers"][i], f"l{i}.", float(cfg["norm"]["eps"])
    xs = sublayer(xs, w, cfg, p, 1, lambda h: MIXERS[L["type"]](h, w, p + "mix.", L["mixer"], eps, r), r)
    if L.get("mlp") is not None:
        xs = sublayer(xs, w, cfg, p, 2, lambda h: FFNS[L["mlp"]["kind"]](h, w, p + "mlp.", L["mlp"], eps, r), r)
    return xs


def forward(tokens: Sequence[int], w: Dict[str, np.ndarray], cfg: dict, r=_id, taps: Optional[List[np.ndarray]] = None):
    """Logits [T, vocab] of one whole sequence; ``taps`` collects the streams' sum after every layer."""
    x = w["embed"][np.asarray(tokens)] * float(cfg["embedding"]["scale"])
    xs = np.repeat(x[None], int(cfg["streams"]), axis=0)
    for i in range(len(cfg["layers"])):
        xs = layer(xs, w, cfg, i, r)
        if taps is not None:
            taps.append(xs.sum(axis=0))
    return r(layer_norm(xs.sum(axis=0), w["final.norm"], w["final.norm.b"], float(cfg["norm"]["eps"]))) @ w["embed"].T
