"""A plain, slow float64 implementation of the Folavik design: one function per mechanism, one request at a time, written
from the design's equations and sharing nothing with the engine.

Notation: T tokens, W the width; a weight W_foo is stored [out, in] and applied as h @ W_foo.T.  ``Wt`` maps tensor names
to float64 arrays, ``p`` is the prefix of a mixer's or a feed-forward's tensors, ``m`` a layer's "mixer" entry.
"""
import math

import numpy as np


def sigmoid(z):
    return np.exp(-np.logaddexp(0.0, -z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rms(y, eps):
    return y / np.sqrt((y * y).mean(-1, keepdims=True) + eps)


def layer_norm(x, w, eps):
    c = x - x.mean(-1, keepdims=True)
    return c / np.sqrt((c * c).mean(-1, keepdims=True) + eps) * w


# ---------------------------------------------------------------- rotation
def frequencies(rot):
    """base^(-2i/dims) for i = 0 .. dims/2 - 1, unscaled."""
    d = rot["dims"]
    return np.array([rot["base"] ** (-2.0 * i / d) for i in range(d // 2)])


def smoothed_frequencies(rot):
    """Three bands by wavelength L = 2 pi / f: short ones keep f, long ones take f / factor, those between are mixed."""
    s = rot["scaling"]
    out = []
    for f in frequencies(rot):
        L = 2.0 * math.pi / f
        if L < s["original"] / s["high"]:
            out.append(f)
        elif L > s["original"] / s["low"]:
            out.append(f / s["factor"])
        else:
            t = (s["original"] / L - s["low"]) / (s["high"] - s["low"])
            out.append((1.0 - t) * f / s["factor"] + t * f)
    return np.array(out)


def yarn_frequencies(rot):
    """Frequencies under a ramp over the pair index, and the factor on cos and sin."""
    s, d = rot["scaling"], rot["dims"]

    def index_of(turns):
        return d * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(rot["base"]))

    lo = max(math.floor(index_of(s["fast"])), 0)
    hi = min(math.ceil(index_of(s["slow"])), d - 1)
    out = []
    for i, f in enumerate(frequencies(rot)):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * ramp + f * (1.0 - ramp))
    return np.array(out), 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, positions, freq, mult=1.0):
    """x [T, heads, D]: dimension i < len(freq) turns with dimension i + len(freq); the rest pass."""
    n = len(freq)
    a = np.asarray(positions, dtype=np.float64)[:, None, None] * freq
    c, s = np.cos(a) * mult, np.sin(a) * mult
    y = x.copy()
    u, v = x[..., :n], x[..., n:2 * n]
    y[..., :n] = u * c - v * s
    y[..., n:2 * n] = v * c + u * s
    return y


# ---------------------------------------------------------------- masks and attention
def sees_all(i, j):
    return j <= i


def sees_chunk(size):
    return lambda i, j: (j <= i) & (i // size == j // size)


def sees_window(size):
    return lambda i, j: (i - j >= 0) & (i - j < size)


def softmax_attention(q, k, v, sees, scale, softcap=0.0, pos_q=None):
    """q [Tq, H, D], k [Tk, G, D], v [Tk, G, V] -> [Tq, H, V]; query head h reads key/value head h // (H / G); ``sees(i,
    j)`` tells which keys the query at position i sees.  Queries stand at ``pos_q`` (default 0, 1, ...), keys at 0, 1, ..."""
    Tq, H, _ = q.shape
    per = H // k.shape[1]
    j = np.arange(k.shape[0])
    out = np.zeros((Tq, H, v.shape[2]))
    for t in range(Tq):
        see = np.nonzero(sees(t if pos_q is None else pos_q[t], j))[0]
        for h in range(H):
            s = (k[see, h // per] @ q[t, h]) * scale
            if softcap > 0.0:
                s = softcap * np.tanh(s / softcap)
            w = np.exp(s - s.max())
            out[t, h] = (w / w.sum()) @ v[see, h // per]
    return out


# ---------------------------------------------------------------- mixers
def latent_attention(m, Wt, p, h, eps):
    T = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q = (h @ Wt[p + "q"].T).reshape(T, H, D)
    c = rms(h @ Wt[p + "dkv"].T, eps) * Wt[p + "dkv.norm"]
    k = (c @ Wt[p + "uk"].T).reshape(T, H, D)
    v = (c @ Wt[p + "uv"].T).reshape(T, H, V)
    o = softmax_attention(q, k, v, sees_all, m["scale"]).reshape(T, H * V)
    return (o * sigmoid(h @ Wt[p + "g"].T)) @ Wt[p + "o"].T


def attention(m, Wt, p, h, eps):
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos, f = np.arange(T), smoothed_frequencies(m["rot"])
    q = rotate((h @ Wt[p + "q"].T).reshape(T, H, D), pos, f)
    k = rotate((h @ Wt[p + "k"].T).reshape(T, G, D), pos, f)
    v = (h @ Wt[p + "v"].T).reshape(T, G, V)
    o = softmax_attention(q, k, v, sees_chunk(m["mask"]["size"]), m["scale"])
    return o.reshape(T, H * V) @ Wt[p + "o"].T


def difference_weight(Wt, p, diff):
    return math.exp(float((Wt[p + "lq1"] * Wt[p + "lk1"]).sum())) - math.exp(float((Wt[p + "lq2"] * Wt[p + "lk2"]).sum())) + diff


def combine_maps(a1, a2, lam, diff, eps):
    """a1, a2 [T, H, V]: the difference of the two maps, normed per head, times 1 - diff."""
    return rms(a1 - lam * a2, eps) * (1.0 - diff)


def differential_attention(m, Wt, p, h, eps):
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = np.arange(T)
    f, mult = yarn_frequencies(m["rot"])
    q = (h @ Wt[p + "q"].T + Wt[p + "q.b"]).reshape(T, H, 2, D)
    k = (h @ Wt[p + "k"].T + Wt[p + "k.b"]).reshape(T, G, 2, D)
    v = (h @ Wt[p + "v"].T + Wt[p + "v.b"]).reshape(T, G, V)
    sees = sees_window(m["mask"]["size"])
    a = [softmax_attention(rotate(q[:, :, i], pos, f, mult), rotate(k[:, :, i], pos, f, mult), v, sees, m["scale"], m["softcap"])
         for i in (0, 1)]
    o = combine_maps(a[0], a[1], difference_weight(Wt, p, m["diff"]), m["diff"], eps)
    return o.reshape(T, H * V) @ Wt[p + "o"].T


MIXERS = {"latent_attention": latent_attention, "attention": attention, "attention_2": differential_attention}


# ---------------------------------------------------------------- feed-forward, ends, model
def dense_ff(Wt, p, h):
    return (gelu_tanh(h @ Wt[p + "gate"].T) * (h @ Wt[p + "up"].T)) @ Wt[p + "down"].T


def output_logits(Wt, x, eps, scale, cap):
    z = (layer_norm(x, Wt["final.norm"], eps) @ Wt["head"].T) * scale
    return cap * np.tanh(z / cap)


def forward(cfg, Wt, tokens, layers_out=None):
    """Logits [T, vocab] of one request's whole token list."""
    eps = cfg["norm"]["eps"]
    x = layer_norm(Wt["embed"][np.asarray(tokens)], Wt["embed.norm"], eps)
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + MIXERS[layer["type"]](layer["mixer"], Wt, p + "mix.", layer_norm(x, Wt[p + "norm1"], eps), eps)
        if layer.get("mlp"):
            x = x + dense_ff(Wt, p + "mlp.", layer_norm(x, Wt[p + "norm2"], eps))
        if layers_out is not None:
            layers_out.append(x.copy())
    return output_logits(Wt, x, eps, cfg["logit_scale"], cfg["logit_softcap"])
