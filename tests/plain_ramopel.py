"""The Ramopel decoder, plainly: float64 numpy, whole sequences, no cache or state, one function per mechanism. It
shares no code with the library; the tests compare the library with it.

Both sublayers of a layer read the same stream,  x <- x + (mixer(norm1(x)) + ff(norm2(x))),  with RMS norms whose
weights are stored around zero. Two mixers:

* latent attention: queries through a normed latent of their own; keys and values of all heads made from one normed
  latent row per position plus one turned key part shared by the heads; a window; a plain softmax. A layer may read
  the latent rows of an earlier layer instead of making its own.
* generalized delta rule: S_t = diag(w) S_(t-1) - (a * u)(u^T S_(t-1)) + k v^T, o_t = S_t^T r, a decay w and a removal
  rate a per key channel, u the unit key; o normed per head, weighted, gated, projected.

Two feed-forwards: dense with a weighted sum of normed powers as its activation, and a mixture of gated experts whose
weights are a softmax over the chosen logits, beside a shared expert with a gate of its own.
"""
from __future__ import annotations

import numpy as np

DECAY_RATE = np.exp(-0.5)


def rms_norm(x, w, eps):
    x = np.asarray(x, dtype=np.float64)
    y = x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)
    return y if w is None else y * np.asarray(w, dtype=np.float64)


def zero_centred_norm(x, w, eps):
    return rms_norm(x, 1.0 + np.asarray(w, dtype=np.float64), eps)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


# ---- attention over a latent -----------------------------------------------------------------------------------
def turn_pairs(x, positions, base):
    """x [tokens, .., dims]: channels (2i, 2i + 1) turned by position * base^(-2i / dims)."""
    dims = x.shape[-1]
    f = np.float64(base) ** (-2.0 * np.arange(dims // 2) / dims)
    ang = np.asarray(positions, dtype=np.float64).reshape((-1,) + (1,) * (x.ndim - 1)) * f
    out = np.array(x, dtype=np.float64)
    u, v = out[..., 0::2].copy(), out[..., 1::2].copy()
    out[..., 0::2] = u * np.cos(ang) - v * np.sin(ang)
    out[..., 1::2] = v * np.cos(ang) + u * np.sin(ang)
    return out


def visible(n, window):
    back = np.arange(n)[:, None] - np.arange(n)[None, :]
    return (back >= 0) & (back < window) if window else back >= 0


def softmax(scores, mask):
    s = np.where(mask, scores, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def latent_rows(down, t, m, eps, positions=None):
    """(latent c [n, C], turned key part [n, R]) from the down projection's rows [n, C + R]."""
    C = m["kv_rank"]
    pos = np.arange(down.shape[0]) if positions is None else positions
    return rms_norm(down[:, :C], t["dkv.norm"], eps), turn_pairs(down[:, C:], pos, m["rot"]["base"])


def latent_core(q, c, k_turned, t, m, positions=None):
    """[n, H * Dv] from the query rows [n, H * (D + R)] and the latent rows."""
    n, H, D, R, Dv = q.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    pos = np.arange(n) if positions is None else positions
    q = q.reshape(n, H, D + R)
    q_turned = turn_pairs(q[:, :, D:], pos, m["rot"]["base"])
    k = (c @ t["uk"].T).reshape(n, H, D)
    v = (c @ t["uv"].T).reshape(n, H, Dv)
    see = visible(n, (m.get("mask") or {}).get("size"))
    out = np.zeros((n, H, Dv))
    for hd in range(H):
        s = (q[:, hd, :D] @ k[:, hd].T + q_turned[:, hd] @ k_turned.T) * m["scale"]
        out[:, hd] = softmax(s, see) @ v[:, hd]
    return out.reshape(n, H * Dv)


def latent_queries(h, t, eps):
    return rms_norm(h @ t["dq"].T, t["dq.norm"], eps) @ t["uq"].T


def latent_attention_mixer(h, t, m, eps, rows):
    """`rows`: the (latent, turned key part) this layer reads."""
    return latent_core(latent_queries(h, t, eps), *rows, t, m) @ t["o"].T


# ---- the generalized delta rule --------------------------------------------------------------------------------
def delta_decays(h, t):
    return np.exp(-DECAY_RATE * sigmoid(np.tanh(h @ t["w1"].T) @ t["w2"].T + t["w0"]))


def delta_core(r, k, v, w, a, heads, conditioning=None):
    """[n, H, Dv]: the read-outs S_t^T r_t token by token from S = 0; r, k, w, a [n, H * D], v [n, H * Dv]. `conditioning`
    (a list) gets, per row, the smallest ratio over the heads of |o_t| to |r_t| |S_t|: where it is tiny the read-out is
    what cancellation left, and the norm behind it, which keeps only the direction, magnifies whatever rounding the
    terms carry."""
    n = r.shape[0]
    r, k, v, w, a = (np.asarray(x, dtype=np.float64).reshape(n, heads, -1) for x in (r, k, v, w, a))
    D, Dv = k.shape[-1], v.shape[-1]
    out, ratio = np.zeros((n, heads, Dv)), np.full(n, np.inf)
    for hd in range(heads):
        S = np.zeros((D, Dv))
        for i in range(n):
            u = k[i, hd] / np.sqrt(np.sum(k[i, hd] ** 2) + 1e-6)
            S = w[i, hd][:, None] * S - np.outer(a[i, hd] * u, u @ S) + np.outer(k[i, hd], v[i, hd])
            out[i, hd] = S.T @ r[i, hd]
            ratio[i] = min(ratio[i], np.linalg.norm(out[i, hd]) / (np.linalg.norm(r[i, hd]) * np.linalg.norm(S)))
    if conditioning is not None:
        conditioning.append(ratio)
    return out


def general_delta_mixer(h, t, m, eps, conditioning=None):
    n = h.shape[0]
    r, k, v = h @ t["r"].T, h @ t["k"].T, h @ t["v"].T
    w, a = delta_decays(h, t), sigmoid(h @ t["a"].T + t["a.b"])
    o = delta_core(r, k, v, w, a, m["heads"], conditioning)
    return (rms_norm(o, None, eps).reshape(n, -1) * t["norm"] * sigmoid(h @ t["g"].T)) @ t["o"].T


# ---- feed-forwards ---------------------------------------------------------------------------------------------
def poly_norm(z, coef, eps):
    a, b, c, e = coef
    return a * rms_norm(z, None, eps) + b * rms_norm(z ** 2, None, eps) + c * rms_norm(z ** 3, None, eps) + e


def dense_ff(h, t, eps):
    return poly_norm(h @ t["up"].T, t["act"], eps) @ t["down"].T


def gated_expert(h, gate, up, down, limit):
    g = np.minimum(h @ gate.T, limit)
    u = np.clip(h @ up.T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ down.T


def route(h, t, experts, top):
    """(chosen [n, top], weights [n, top])."""
    z = h @ t["router"].T + t["router.b"]
    chosen = np.argsort(-z, axis=-1, kind="stable")[:, :top]
    zc = np.take_along_axis(z, chosen, axis=-1)
    e = np.exp(zc - zc.max(axis=-1, keepdims=True))
    return chosen, e / e.sum(axis=-1, keepdims=True)


def moe_ff(h, t, mlp, gaps=None):
    chosen, weights = route(h, t, mlp["router"]["experts"], mlp["router"]["top"])
    if gaps is not None:           # per row: how far the last chosen logit lies above the first that is left out
        z = -np.sort(-(h @ t["router"].T + t["router.b"]), axis=-1)
        top = mlp["router"]["top"]
        gaps.append(z[:, top - 1] - z[:, top] if top < z.shape[1] else np.full(len(h), np.inf))
    y = np.zeros((h.shape[0], t["e0.down"].shape[0]))
    for e in range(mlp["router"]["experts"]):
        row, place = np.nonzero(chosen == e)
        if len(row):
            y[row] += weights[row, place][:, None] * gated_expert(h[row], t[f"e{e}.gate"], t[f"e{e}.up"], t[f"e{e}.down"],
                                                                  mlp["expert"]["limit"])
    if mlp.get("shared"):
        y += sigmoid(h @ t["shared.sg"].T) * gated_expert(h, t["shared.gate"], t["shared.up"], t["shared.down"],
                                                          mlp["shared"]["limit"])
    return y


def part(tensors, prefix):
    return {k[len(prefix):]: np.asarray(v, dtype=np.float64) for k, v in tensors.items() if k.startswith(prefix)}


def forward(cfg, tensors, tokens, layers_out=None, gaps=None, conditioning=None):
    """Logits [tokens, vocab] of one sequence; `layers_out` (a list) gets the stream after every layer, `gaps` one array
    per routed layer (see `moe_ff`), `conditioning` one per delta-rule layer (see `delta_core`)."""
    eps = cfg["norm"]["eps"]
    T = {k: np.asarray(v, dtype=np.float64) for k, v in tensors.items()}
    x = T["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    kept = {}
    for i, L in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", L["mixer"], L.get("mlp")
        t = part(T, p + "mix.")
        h = zero_centred_norm(x, T[p + "norm1"], eps)
        if L["type"] == "latent_attention":
            if m.get("kv_from") is None:
                kept[i] = latent_rows(h @ t["dkv"].T, t, m, eps)
            y = latent_attention_mixer(h, t, m, eps, kept[i if m.get("kv_from") is None else m["kv_from"]])
        else:
            y = general_delta_mixer(h, t, m, eps, conditioning)
        if mlp:
            h2, tf = zero_centred_norm(x, T[p + "norm2"], eps), part(T, p + "mlp.")
            y = y + (dense_ff(h2, tf, eps) if mlp["kind"] == "dense" else moe_ff(h2, tf, mlp, gaps))
        x = x + y
        if layers_out is not None:
            layers_out.append(x.copy())
    return zero_centred_norm(x, T["final.norm"], eps) @ T["head"].T
