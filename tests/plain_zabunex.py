"""The Zabunex decoder, plainly: float64 numpy, whole sequences, no cache or state, one function per mechanism. It
shares no code with the library; the tests compare the library with it.

The sublayers read the stream itself and only their outputs are normed,  x <- x + norm1(mixer(x)),
x <- x + norm2(ff(x)),  with two mixers:

* attention: grouped queries whose values are the keys' projection before its norm, q and k normed over their whole
  projections, queries that grow with their position, a learned bias per head on bucketed distances, and a softmax whose
  denominator holds one more term of 1;
* parallel: attention over blocks of positions (short convolutions on q, k and v, norms over the whole projections, part
  of every head turned) beside a state-space recurrence with one decay per head and token (a short convolution with bias
  and SiLU, a gate before a norm in groups), a weighted sum of the two.

The feed-forward is W_down relu(W_up x)^2.
"""
from __future__ import annotations

import numpy as np


def rms_norm(x, w, eps):
    x = np.asarray(x, dtype=np.float64)
    y = x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)
    return y if w is None else y * np.asarray(w, dtype=np.float64)


def silu(z):
    return z / (1.0 + np.exp(-z))


def softplus(z):
    return np.logaddexp(0.0, z)


def short_conv(u, w, bias=None):
    """u [tokens, channels], w [channels, taps] (the last tap is the token's own), zeros before the first token."""
    n, taps = u.shape[0], w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, u.shape[1])), u])
    y = sum(padded[j:j + n] * w[:, j] for j in range(taps))
    return y if bias is None else y + bias


def turn_halves(x, positions, dims, base, factor=1.0):
    """x [tokens, heads, channels]: the first `dims` channels turned, channel i with i + dims / 2, by
    position * base^(-2i / dims) / factor."""
    half = dims // 2
    f = np.float64(base) ** (-2.0 * np.arange(half) / max(dims, 1)) / factor
    ang = np.asarray(positions, dtype=np.float64).reshape(-1, 1, 1) * f
    out = np.array(x, dtype=np.float64)
    u, v = out[..., :half].copy(), out[..., half:dims].copy()
    out[..., :half] = u * np.cos(ang) - v * np.sin(ang)
    out[..., half:dims] = v * np.cos(ang) + u * np.sin(ang)
    return out


# ---- attention -------------------------------------------------------------------------------------------------
def bucket(n, rows, largest):
    """Which row of the bias table a distance n >= 0 takes."""
    half = rows // 2
    if n < half:
        return int(n)
    return min(rows - 1, half + int(np.floor(np.log(n / half) / np.log(largest / half) * (rows - half))))


def temperature(positions, coef, every):
    return 1.0 + coef * np.log(np.floor((np.asarray(positions, dtype=np.float64) + 1.0) / every) + 1.0)


def attend(q, k, v, scale, see, bias=None, extra_term=0.0):
    """q [n, H, D], k [n, G, D], v [n, G, Dv], see [n, n] which keys a query sees, bias [H, n, n] added to the scaled
    scores, extra_term: what the softmax denominator holds beside the visible keys. [n, H, Dv]."""
    n, H = q.shape[:2]
    per = H // k.shape[1]
    out = np.zeros((n, H, v.shape[2]))
    for h in range(H):
        s = (q[:, h] @ k[:, h // per].T) * scale
        if bias is not None:
            s = s + bias[h]
        s = np.where(see, s, -np.inf)
        top = s.max(axis=-1, keepdims=True)
        if extra_term:
            top = np.maximum(top, np.log(extra_term))
        e = np.exp(s - top)
        out[:, h] = (e / (e.sum(axis=-1, keepdims=True) + extra_term * np.exp(-top))) @ v[:, h // per]
    return out


def distance_bias(table, n, largest):
    """[H, n, n] from the table [rows, H]; distances of keys that lie ahead are not used."""
    rows = table.shape[0]
    by_distance = table[[bucket(d, rows, largest) for d in range(n)]]              # [n, H]
    back = np.maximum(np.arange(n)[:, None] - np.arange(n)[None, :], 0)
    return np.moveaxis(by_distance[back], 2, 0)


def causal(n):
    return np.arange(n)[:, None] >= np.arange(n)[None, :]


def same_block(n, size):
    b = np.arange(n) // size
    return causal(n) & (b[:, None] == b[None, :])


def attention_core(q, k, t, m, eps):
    """q [n, H * D] and k [n, G * D] as projected."""
    n, H, G, D = q.shape[0], m["heads"], m["kv_heads"], m["dim"]
    v = k.reshape(n, G, D)
    qn = rms_norm(q, t["q.norm"], eps).reshape(n, H, D)
    kn = rms_norm(k, t["k.norm"], eps).reshape(n, G, D)
    if m.get("q_temp"):
        qn = qn * temperature(np.arange(n), m["q_temp"]["coef"], m["q_temp"]["every"])[:, None, None]
    return attend(qn, kn, v, m["scale"], causal(n), distance_bias(t["rel"], n, m["bias_max"]), 1.0).reshape(n, H * D)


def attention_mixer(h, t, m, eps):
    return attention_core(h @ t["q"].T, h @ t["k"].T, t, m, eps) @ t["o"].T


# ---- the two halves of the parallel mixer ----------------------------------------------------------------------
def left_core(q, k, v, t, m, eps):
    """q, k, v as projected."""
    n, H, G, D, Dv = q.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (short_conv(u, t[name + ".conv"]) for u, name in ((q, "q"), (k, "k"), (v, "v")))
    q = rms_norm(q, t["q.norm"], eps).reshape(n, H, D)
    k = rms_norm(k, t["k.norm"], eps).reshape(n, G, D)
    rot = m.get("rot")
    if rot:
        factor = (rot.get("scaling") or {}).get("factor", 1.0)
        q, k = (turn_halves(u, np.arange(n), rot["dims"], rot["base"], factor) for u in (q, k))
    see = same_block(n, m["mask"]["size"]) if m.get("mask") else causal(n)
    return attend(q, k, v.reshape(n, G, Dv), m["scale"], see).reshape(n, H * Dv)


def left_mixer(h, t, m, eps):
    return left_core(h @ t["q"].T, h @ t["k"].T, h @ t["v"].T, t, m, eps) @ t["o"].T


def state_space(x, B, C, dt, A_log, D):
    """x [n, H, P], B and C [n, G, N], dt [n, H] after its softplus: y [n, H, P], token by token from a state of zero."""
    n, H, P = x.shape
    per = H // B.shape[1]
    y = np.zeros((n, H, P))
    for h in range(H):
        S = np.zeros((B.shape[2], P))
        for i in range(n):
            S = np.exp(-np.exp(A_log[h]) * dt[i, h]) * S + dt[i, h] * np.outer(B[i, h // per], x[i, h])
            y[i, h] = S.T @ C[i, h // per] + D[h] * x[i, h]
    return y


def gated_group_norm(y, z, w, groups, eps):
    """y * silu(z), each of `groups` equal parts of a row divided by its own root mean square, times w."""
    n = y.shape[0]
    g = (y * silu(z)).reshape(n, groups, -1)
    return rms_norm(g, None, eps).reshape(n, -1) * w


def right_core(rows, t, m, eps):
    """rows: W_in h."""
    n, H, P, N, G = rows.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    z, u, dt = rows[:, :inner], rows[:, inner:2 * inner + 2 * G * N], rows[:, 2 * inner + 2 * G * N:]
    u = silu(short_conv(u, t["conv"], t["conv.b"]))
    x, B, C = u[:, :inner].reshape(n, H, P), u[:, inner:inner + G * N].reshape(n, G, N), u[:, inner + G * N:].reshape(n, G, N)
    y = state_space(x, B, C, softplus(dt + t["dt_bias"]), t["A_log"], t["D"])
    return gated_group_norm(y.reshape(n, inner), z, t["norm"], m["norm_groups"], eps)


def right_mixer(h, t, m, eps):
    return right_core(h @ t["in"].T, t, m, eps) @ t["o"].T


def parallel_mixer(h, t, m, eps):
    return (m["left_scale"] * left_mixer(h, part(t, "left."), m["left"], eps)
            + m["right_scale"] * right_mixer(h, part(t, "right."), m["right"], eps))


def dense_ff(h, t):
    return np.maximum(h @ t["up"].T, 0.0) ** 2 @ t["down"].T


def part(tensors, prefix):
    return {k[len(prefix):]: np.asarray(v, dtype=np.float64) for k, v in tensors.items() if k.startswith(prefix)}


def forward(cfg, tensors, tokens, layers_out=None):
    """Logits [tokens, vocab] of one sequence; `layers_out` (a list) gets the stream after every layer."""
    eps = cfg["norm"]["eps"]
    T = {k: np.asarray(v, dtype=np.float64) for k, v in tensors.items()}
    x = T["embed"][np.asarray(tokens)]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        mixer = attention_mixer if L["type"] == "attention" else parallel_mixer
        x = x + rms_norm(mixer(x, part(T, p + "mix."), L["mixer"], eps), T[p + "norm1"], eps)
        if L.get("mlp"):
            x = x + rms_norm(dense_ff(x, part(T, p + "mlp.")), T[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return rms_norm(x, T["final.norm"], eps) @ T["head"].T
