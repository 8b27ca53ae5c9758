"""A plain, slow float64 implementation of the Kuvidra design: one function per mechanism, one request at a time,
written from the design's equations and sharing nothing with the engine.

Notation: T tokens, W the width; N(y) = y / sqrt(mean(y^2) + eps) over the last axis; a weight W_foo is stored
[out, in] and applied as h @ W_foo.T.  ``Wt`` maps tensor names to float64 arrays, ``p`` is a layer's prefix.
"""
import math

import numpy as np

DENOMINATOR_EPS = 1e-6       # added to the matrix memory's denominator


def sigmoid(z):
    return np.exp(-np.logaddexp(0.0, -z))


def silu(z):
    return z * sigmoid(z)


def gelu_erf(z):
    return 0.5 * z * (1.0 + np.vectorize(math.erf, otypes=[np.float64])(z / math.sqrt(2.0)))


def log_sigmoid(z):
    return -np.logaddexp(0.0, -z)


def rms(y, eps):
    return y / np.sqrt((y * y).mean(-1, keepdims=True) + eps)


def softmax_attention(q, k, v, pos_q, pos_k, scale):
    """q [Tq, H, D], k [Tk, H, D], v [Tk, H, V] -> [Tq, H, V]: the query at position i sees every key at j <= i."""
    Tq, H, _ = q.shape
    out = np.zeros((Tq, H, v.shape[2]))
    for t in range(Tq):
        see = np.nonzero(np.asarray(pos_k) <= pos_q[t])[0]
        for h in range(H):
            s = (k[see, h] @ q[t, h]) * scale
            w = np.exp(s - s.max())
            out[t, h] = (w / w.sum()) @ v[see, h]
    return out


def latent_attention(m, Wt, p, h, eps):
    """Queries and keys / values through latents, no positions, a gate per head."""
    T = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    cq = rms(h @ Wt[p + "dq"].T, eps) * Wt[p + "dq.norm"]
    q = (cq @ Wt[p + "uq"].T).reshape(T, H, D)
    c = rms(h @ Wt[p + "dkv"].T, eps) * Wt[p + "dkv.norm"]
    k = (c @ Wt[p + "uk"].T).reshape(T, H, D)
    v = (c @ Wt[p + "uv"].T).reshape(T, H, V)
    pos = np.arange(T)
    o = softmax_attention(q, k, v, pos, pos, m["scale"])
    o = o * sigmoid(h @ Wt[p + "g"].T)[:, :, None]
    return o.reshape(T, H * V) @ Wt[p + "o"].T


def mlstm_gates(zi, zf, cap):
    """Log input gate and log forget gate from their projections with bias."""
    return cap * np.tanh(zi / cap), log_sigmoid(cap * np.tanh(zf / cap))


def mlstm_recurrence(q, k, v, i, f, state=None):
    """q (already times dim^-1/2) and k [T, H, D], v [T, H, V], log gates i, f [T, H] -> o [T, H, V] and the state.
    m_t = max(f + m, i); S = e^(f + m - m_t) S + e^(i - m_t) k v^T; n likewise with k; o = S^T q / (max(|n.q|, e^-m_t) + 1e-6)."""
    T, H, D = q.shape
    V = v.shape[2]
    S, n, m = (np.zeros((H, D, V)), np.zeros((H, D)), np.zeros(H)) if state is None else tuple(a.copy() for a in state)
    o = np.zeros((T, H, V))
    for t in range(T):
        for h in range(H):
            mt = max(f[t, h] + m[h], i[t, h])
            keep, take = math.exp(f[t, h] + m[h] - mt), math.exp(i[t, h] - mt)
            S[h] = keep * S[h] + take * np.outer(k[t, h], v[t, h])
            n[h] = keep * n[h] + take * k[t, h]
            m[h] = mt
            o[t, h] = (S[h].T @ q[t, h]) / (max(abs(n[h] @ q[t, h]), math.exp(-mt)) + DENOMINATOR_EPS)
    return o, (S, n, m)


def mlstm(m, Wt, p, h, eps):
    T = h.shape[0]
    H, D, V, cap = m["heads"], m["dim"], m["vdim"], float(m["gate_cap"])
    q = (h @ Wt[p + "q"].T).reshape(T, H, D) * D ** -0.5
    k = (h @ Wt[p + "k"].T).reshape(T, H, D)
    v = (h @ Wt[p + "v"].T).reshape(T, H, V)
    i, f = mlstm_gates(h @ Wt[p + "i"].T + Wt[p + "i.b"], h @ Wt[p + "f"].T + Wt[p + "f.b"], cap)
    o, _ = mlstm_recurrence(q, k, v, i, f)
    y = rms(o, eps).reshape(T, H * V) * Wt[p + "norm"] * sigmoid(h @ Wt[p + "g"].T)
    return y @ Wt[p + "o"].T


def dense_ff(Wt, p, h):
    return gelu_erf(h @ Wt[p + "up"].T) @ Wt[p + "down"].T


def expert(Wt, p, h):
    return (silu(h @ Wt[p + "gate"].T) * (h @ Wt[p + "up"].T)) @ Wt[p + "down"].T


def route(z, top):
    """z [T, E] -> (ids [T, top], weights [T, top]): the largest sigmoid scores, not renormalised."""
    s = sigmoid(z)
    ids = np.argsort(-s, axis=-1, kind="stable")[:, :top]
    return ids, np.take_along_axis(s, ids, -1)


def moe_ff(f, Wt, p, h):
    """sum of expert_e(w_e h) over the chosen e, plus sigmoid(w_sg . h) shared(h)."""
    ids, w = route(h @ Wt[p + "router"].T, f["router"]["top"])
    out = np.zeros((h.shape[0], Wt[p + "router"].shape[1]))
    for t in range(h.shape[0]):
        for e, wt in zip(ids[t], w[t]):
            out[t] += expert(Wt, f"{p}e{e}.", wt * h[t:t + 1])[0]
    if f.get("shared"):
        out += sigmoid(h @ Wt[p + "shared.sg"].T) * expert(Wt, p + "shared.", h)
    return out


def run_order(cfg):
    """[(layer, pass number or None, whether it opens the pass)] of every layer run in order."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, None, False) for i in range(n)]
    a, b, times = loop["start"], loop["stop"], loop["times"]
    order = [(i, None, False) for i in range(a)]
    for t in range(times):
        order += [(i, t, i == a) for i in range(a, b)]
    return order + [(i, None, False) for i in range(b, n)]


def pass_input(Wt, x, x0, t):
    return np.concatenate([x, x0], -1) @ Wt["loop.in"].T + Wt["loop.step"][t]


def forward(cfg, Wt, tokens, layers_out=None):
    """Logits [T, vocab] of one request's whole token list."""
    eps = cfg["norm"]["eps"]
    x0 = Wt["embed"][np.asarray(tokens)]
    x = x0.copy()
    for i, t, first in run_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if first:
            x = pass_input(Wt, x, x0, t)
        h = rms(x, eps) * Wt[p + "norm1"]
        if layer["type"] == "latent_attention":
            y = latent_attention(layer["mixer"], Wt, p + "mix.", h, eps)
        elif layer["type"] == "mlstm":
            y = mlstm(layer["mixer"], Wt, p + "mix.", h, eps)
        else:
            raise ValueError(layer["type"])
        f = layer.get("mlp")
        if f:
            y = y + (dense_ff(Wt, p + "mlp.", h) if f["kind"] == "dense" else moe_ff(f, Wt, p + "mlp.", h))
        x = x + y
        if layers_out is not None:
            layers_out.append(x.copy())
    return (rms(x, eps) * Wt["final.norm"]) @ Wt["embed"].T
