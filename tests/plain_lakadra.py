"""A plain, slow statement of the Lakadra decoder: one function per mechanism, NumPy float64, whole sequences, no
cache, no batching.  It shares no code with the library under test.

The design: every layer norms the residual once; a mixer and a mixture of experts both read that norm, and the sum of
their results is added.  Three mixers: lightning attention (a matrix state per head under a fixed decay, SiLU on
queries, keys and values, one norm over all heads and a logistic gate), latent attention (keys and values from one
normed latent per token, which later layers may share), and a pair of mixers side by side: grouped-query attention over
a sliding window with biases, slowed-down rotary positions, one added to the softmax's denominator and a gate per head,
next to a gated linear recurrence behind a short convolution, their results added with a factor each.  The experts are
ungated squared-relu units; a token's are chosen within the best groups by softmax scores plus a correction, some of
them hand on the input itself, and a shared one with a gate of its own runs for every token.

``r`` rounds what a bfloat16 engine stores in bfloat16 (projections, cached rows, activations); the residual, norms,
scores, weights, angles, routers and the recurrences' gates and states stay unrounded, as they do there.
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


def layer_norm_of(x, w, eps):
    """The block's norm: the stored gain is the distance from one."""
    return unit_rms(x, eps) * (1.0 + w)


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return np.logaddexp(0.0, z)


def causal_convolution(x, taps, bias):
    """Along the sequence, channel by channel; the last tap is the current token's, missing inputs are zeros; x [T, C],
    taps [C, n]."""
    n = taps.shape[1]
    past = np.concatenate([np.zeros((n - 1, x.shape[1])), x])
    return sum(past[j: j + x.shape[0]] * taps[:, j] for j in range(n)) + bias


def turned(x, base, dims, pairing, factor=1.0):
    """Rotary positions 0 .. T-1 on the first ``dims`` numbers of x [T, ..., D]; pairing "neighbours" (2i, 2i + 1) or
    "halves" (i, i + dims / 2); every frequency over ``factor``."""
    half = dims // 2
    f = base ** (-2.0 * np.arange(half) / dims) / factor
    a = np.arange(x.shape[0]).reshape((-1,) + (1,) * (x.ndim - 1)) * f
    at_u, at_v = (np.arange(half) * 2, np.arange(half) * 2 + 1) if pairing == "neighbours" else (np.arange(half), np.arange(half) + half)
    out = x.copy()
    u, v = x[..., at_u], x[..., at_v]
    out[..., at_u] = u * np.cos(a) - v * np.sin(a)
    out[..., at_v] = v * np.cos(a) + u * np.sin(a)
    return out


def weighted_values(scores, visible, values, added=0.0):
    """sum_j p_j v_j with p_j = exp(s_j) / (added + sum exp(s_j)) over the visible keys; scores [T, J], values [J, D]."""
    s = np.where(visible, scores, -np.inf)
    top = np.maximum(s.max(-1, keepdims=True), 0.0 if added else -np.inf)
    e = np.exp(s - top)
    return (e @ values) / (e.sum(-1, keepdims=True) + (added * np.exp(-top) if added else 0.0))


def positions_apart(T):
    i = np.arange(T)
    return i[:, None] - i[None, :]


# ---- mixers -------------------------------------------------------------------------------------
def lightning_state(q, k, v, decay):
    """o_t = S_t^T q_t with S_t = decay S_(t-1) + k_t v_t^T for one head; q, k [T, D], v [T, E]."""
    S = np.zeros((k.shape[1], v.shape[1]))
    out = np.zeros_like(v)
    for t in range(k.shape[0]):
        S = decay * S + np.outer(k[t], v[t])
        out[t] = S.T @ q[t]
    return out


def lightning(h, w, p, m, eps, r=_id):
    T, H, D, E = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v = (r(silu(r(h @ w[p + n].T))).reshape(T, H, -1) for n in ("q", "k", "v"))
    o = np.stack([lightning_state(q[:, i], k[:, i], v[:, i], m["decay"][i]) for i in range(H)], axis=1)
    y = unit_rms(o.reshape(T, H * E), eps) * w[p + "norm"] * sigmoid(r(h @ w[p + "g"].T))
    return r(y) @ w[p + "o"].T


def latent_rows(h, w, p, m, eps, r=_id):
    """What a latent layer caches: the normed latent and the rotated key part."""
    both = r(h @ w[p + "dkv"].T)
    n = m["kv_rank"]
    c = r(unit_rms(both[:, :n], eps) * w[p + "dkv.norm"])
    return c, r(turned(both[:, n:], m["rot"]["base"], m["rot_dim"], "neighbours"))


def latent_attention(h, w, p, m, eps, rows, r=_id):
    """``rows``: (latent, rotated key part), this layer's or the one's it reads."""
    T, H, D, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"]
    c, k_rot = rows
    cq = r(unit_rms(r(h @ w[p + "dq"].T), eps) * w[p + "dq.norm"])
    q = r(cq @ w[p + "uq"].T).reshape(T, H, D + R)
    q_rot = r(turned(q[..., D:], m["rot"]["base"], R, "neighbours"))
    k = r(c @ w[p + "uk"].T).reshape(T, H, D)
    v = r(c @ w[p + "uv"].T).reshape(T, H, m["vdim"])
    seen = positions_apart(T) >= 0
    out = [weighted_values((q[:, i, :D] @ k[:, i].T + q_rot[:, i] @ k_rot.T) * m["scale"], seen, v[:, i]) for i in range(H)]
    return r(np.concatenate(out, axis=1)) @ w[p + "o"].T


def windowed_attention(h, w, p, m, r=_id):
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q, k, v = (r(h @ w[p + n].T + w[p + n + ".b"]) for n in ("q", "k", "v"))
    rot = m.get("rot")
    spin = _id if rot is None else lambda x: r(turned(x, rot["base"], rot["dims"], "halves", (rot.get("scaling") or {}).get("factor", 1.0)))
    q, k, v = spin(q.reshape(T, H, D)), spin(k.reshape(T, G, D)), v.reshape(T, G, m["vdim"])
    apart = positions_apart(T)
    seen = (apart >= 0) & (apart < m["mask"]["size"])
    gate = sigmoid(r(h @ w[p + "g"].T))
    out = [weighted_values(q[:, i] @ k[:, i // (H // G)].T * m["scale"], seen, v[:, i // (H // G)], added=1.0) * gate[:, i: i + 1]
           for i in range(H)]
    return r(np.concatenate(out, axis=1)) @ w[p + "o"].T + w[p + "o.b"]


def gated_linear_states(u, ra, ra_b, ri, ri_b, lam):
    """S_t = a S_(t-1) + sqrt(1 - a^2) i u with log a = -8 r softplus(lam); r and i from block-diagonal matrices
    [blocks, out, in]; u [T, width]."""
    T, B = u.shape[0], ra.shape[0]
    ub = u.reshape(T, B, -1)
    r = sigmoid(np.einsum("tbi,boi->tbo", ub, ra) + ra_b).reshape(T, -1)
    i = sigmoid(np.einsum("tbi,boi->tbo", ub, ri) + ri_b).reshape(T, -1)
    a = np.exp(-8.0 * r * softplus(lam))
    x = np.sqrt(1.0 - a * a) * i * u
    S, out = np.zeros(u.shape[1]), np.zeros_like(u)
    for t in range(T):
        S = a[t] * S + x[t]
        out[t] = S
    return out


def recurrent_block(h, w, p, m, r=_id):
    y = gelu_tanh(r(h @ w[p + "y"].T + w[p + "y.b"]))
    u = r(causal_convolution(r(h @ w[p + "x"].T + w[p + "x.b"]), w[p + "conv"], w[p + "conv.b"]))
    S = gated_linear_states(u, w[p + "ra"], w[p + "ra.b"], w[p + "ri"], w[p + "ri.b"], w[p + "lam"])
    return r(S * y) @ w[p + "o"].T


def side_by_side(h, w, p, m, r=_id):
    return (m["left_scale"] * windowed_attention(h, w, p + "left.", m["left"], r)
            + m["right_scale"] * recurrent_block(h, w, p + "right.", m["right"], r))


# ---- experts ------------------------------------------------------------------------------------
def squared_relu_unit(x, up, down, r=_id):
    return r(np.square(np.maximum(r(x @ up.T), 0.0))) @ down.T


def choose_experts(z, correction, top, groups, keep):
    """(ids, weights) [T, top]: the largest softmax scores + correction within the ``keep`` groups whose largest such
    number is largest; the weights are the scores without the correction."""
    e = np.exp(z - z.max(-1, keepdims=True))
    s = e / e.sum(-1, keepdims=True)
    c = s + correction
    T, N = c.shape
    size = N // groups
    best = c.reshape(T, groups, size).max(-1)
    for t in range(T):
        out = np.argsort(-best[t], kind="stable")[keep:]
        for g in out:
            c[t, g * size: (g + 1) * size] = -np.inf
    ids = np.argsort(-c, axis=-1, kind="stable")[:, :top]
    return ids, np.take_along_axis(s, ids, axis=-1)


def experts(h, w, p, mlp, r=_id):
    ro = mlp["router"]
    grouping = ro.get("groups") or {"count": 1, "keep": 1}
    ids, weights = choose_experts(h @ w[p + "router"].T, w[p + "correction"], ro["top"], grouping["count"], grouping["keep"])
    out = np.zeros_like(h)
    for e in range(ro["experts"] + ro.get("identity", 0)):
        for t, k in np.argwhere(ids == e):
            x = h[t: t + 1]
            y = x if e >= ro["experts"] else r(squared_relu_unit(x, w[f"{p}e{e}.up"], w[f"{p}e{e}.down"], r))
            out[t] += weights[t, k] * y[0]
    if mlp.get("shared"):
        g = sigmoid(h @ w[p + "shared.sg"].T)
        out += g * squared_relu_unit(h, w[p + "shared.up"], w[p + "shared.down"], r)
    return out


# ---- the model ----------------------------------------------------------------------------------
def forward(tokens: Sequence[int], w: Dict[str, np.ndarray], cfg: dict, r=_id, taps: Optional[List] = None) -> np.ndarray:
    """Logits [T, vocab] of a whole sequence; ``taps`` collects the residual after every layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)]
    rows = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", layer["mixer"]
        h = r(layer_norm_of(x, w[f"l{i}.norm1"], eps))
        if layer["type"] == "lightning":
            y = lightning(h, w, p, m, eps, r)
        elif layer["type"] == "latent_attention":
            rows[i] = rows[m["kv_from"]] if m.get("kv_from") is not None else latent_rows(h, w, p, m, eps, r)
            y = latent_attention(h, w, p, m, eps, rows[i], r)
        else:
            y = side_by_side(h, w, p, m, r)
        if layer.get("mlp"):
            y = y + experts(h, w, f"l{i}.mlp.", layer["mlp"], r)
        x = x + y
        if taps is not None:
            taps.append(x.copy())
    z = r(layer_norm_of(x, w["final.norm"], eps)) @ w["head"].T * cfg["logit_scale"]
    return cfg["logit_softcap"] * np.tanh(z / cfg["logit_softcap"])
