"""Plain, slow Kefetar forward pass: whole sequences, no cache, one function per mechanism.

The oracle of the Kefetar tests.  It shares no code with the product package: it takes the configuration as a plain
``dict`` (the keys of config.json) and the weights as a ``dict`` of numpy arrays keyed by tensor name, and computes
everything in float64 except the rotary angle, which is the float32 product of position and frequency.  Attention walks
query by query over the keys up to it, the retention walks token by token with its state as a matrix.

Notation: D model width, T tokens of one sequence.  With n(x) = x / sqrt(mean(x^2) + eps) * g (g one number) and
c(h)_t = h_t + sum_j w[:, j] h_(t - taps + 1 + j), a layer is  x <- x + mixer(c1(n1(x)));  x <- x + ff(c2(n2(x))).
`rnd` models a bfloat16 engine: it is applied where such an engine must round (inputs of matrix products, cached rows);
the identity gives exact arithmetic.
"""
from __future__ import annotations

import numpy as np


def _same(x):
    return x


def bf16_round(x):
    """Nearest bfloat16 (ties to even) of every element, returned as float64."""
    x32 = np.ascontiguousarray(x, dtype=np.float32)
    bits = x32.view(np.uint32).astype(np.uint64)
    bits = (bits + 0x7FFF + ((bits >> 16) & 1)) & 0xFFFF0000
    return bits.astype(np.uint32).view(np.float32).astype(np.float64).reshape(np.shape(x))


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def unit_rms(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


# ---- convolutions over time --------------------------------------------------------------------------------------------
def causal_conv(u, w):
    """u [T, C], w [C, taps]: y_t = sum_j w[:, j] u_(t - taps + 1 + j), zeros before the first row."""
    T, C = u.shape
    taps = w.shape[1]
    y = np.zeros((T, C))
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                y[t] += w[:, j] * u[s]
    return y


def sublayer_input(x, g, w, eps):
    """The norm with one gain for all coordinates, then the row plus a convolution of the normed rows."""
    h = unit_rms(x, eps) * float(np.reshape(g, -1)[0])
    return h + causal_conv(h, w)


# ---- rotation -------------------------------------------------------------------------------------------------------------
def frequencies(rot):
    f = np.array([rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)], dtype=np.float64)
    scaling = rot.get("scaling")
    return f / scaling["factor"] if scaling else f


def rotate_halves(x, pos, freq):
    """x [T, heads, d]: dimension i of the first 2 * len(freq) is paired with i + len(freq)."""
    x = x.copy()
    n = len(freq)
    if n == 0:
        return x
    ang = (np.asarray(pos, dtype=np.float32)[:, None] * freq.astype(np.float32)[None, :]).astype(np.float64)   # a 32-bit product
    cs, sn = np.cos(ang)[:, None, :], np.sin(ang)[:, None, :]
    u, v = x[..., :n].copy(), x[..., n:2 * n].copy()
    x[..., :n] = u * cs - v * sn
    x[..., n:2 * n] = v * cs + u * sn
    return x


# ---- retention ---------------------------------------------------------------------------------------------------------------
def retention_scan(q, k, v, decay):
    """One head.  q, k [T, d], v [T, dv], decay a number: S <- decay S + k v^T; o = S^T q."""
    S = np.zeros((k.shape[1], v.shape[1]))
    o = np.zeros((q.shape[0], v.shape[1]))
    for t in range(q.shape[0]):
        S = decay * S + np.outer(k[t], v[t])
        o[t] = S.T @ q[t]
    return o


def retention(h, W, p, m, eps, rnd=_same):
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    pos, freq = np.arange(T), frequencies(m["rot"])
    q = rotate_halves((h @ W[p + "q"].T).reshape(T, H, d), pos, freq)
    k = rotate_halves((h @ W[p + "k"].T).reshape(T, H, d), pos, freq) * d ** -0.5
    v = (h @ W[p + "v"].T).reshape(T, H, dv)
    o = np.stack([retention_scan(q[:, i], k[:, i], v[:, i], m["decay"][i]) for i in range(H)], axis=1)
    o = unit_rms(o, eps).reshape(T, H * dv) * silu(h @ W[p + "g"].T)
    return rnd(o) @ W[p + "o"].T


# ---- attention ----------------------------------------------------------------------------------------------------------------
def attend(q, k, v, scale, cap):
    """One head: q [T, d], k [T, d], v [T, dv] -> [T, dv], causal, scores capped by tanh (cap None: not capped)."""
    T = q.shape[0]
    out = np.zeros((T, v.shape[1]))
    for i in range(T):
        s = (k[:i + 1] @ q[i]) * scale
        if cap:
            s = cap * np.tanh(s / cap)
        e = np.exp(s - s.max())
        out[i] = (e / e.sum()) @ v[:i + 1]
    return out


def mix_values(v, first, lam):
    return (1.0 - lam) * v + lam * first


def attention(h, W, p, m, first, rnd=_same):
    """Returns (output, the layer's values [T, G * dv] before they are mixed).  first: the values that this layer's are
    mixed with, or None."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos, freq = np.arange(T), frequencies(m["rot"])
    q = rnd(rotate_halves(causal_conv(h @ W[p + "q"].T, W[p + "q.conv"]).reshape(T, H, d), pos, freq))
    k = rnd(rotate_halves(causal_conv(h @ W[p + "k"].T, W[p + "k.conv"]).reshape(T, G, d), pos, freq))
    own = causal_conv(h @ W[p + "v"].T, W[p + "v.conv"])
    v = own if first is None else mix_values(own, first, float(np.reshape(W[p + "vmix"], -1)[0]))
    v = rnd(v).reshape(T, G, dv)
    out = np.stack([attend(q[:, i], k[:, i // (H // G)], v[:, i // (H // G)], m["scale"], m.get("softcap")) for i in range(H)], axis=1)
    out = rnd(out.reshape(T, H * dv)) * sigmoid(h @ W[p + "g"].T)
    return rnd(out) @ W[p + "o"].T, own


# ---- feed-forward ----------------------------------------------------------------------------------------------------------------
def polynorm(z, coeff, eps):
    a, b, c, e = [float(v) for v in coeff]
    return a * unit_rms(z, eps) + b * unit_rms(z ** 2, eps) + c * unit_rms(z ** 3, eps) + e


def dense(h, W, p, eps, rnd=_same):
    return rnd(polynorm(h @ W[p + "up"].T, W[p + "act"], eps)) @ W[p + "down"].T


# ---- the model ------------------------------------------------------------------------------------------------------------------
def forward(cfg, W, tokens, rnd=_same, layers_out=None):
    eps = cfg["norm"]["eps"]
    x = W["embed"][np.asarray(tokens)].astype(np.float64)
    first = None
    for i, layer in enumerate(cfg["layers"]):
        L, m = f"l{i}.", layer["mixer"]
        h = rnd(sublayer_input(x, W[L + "norm1"], W[L + "canon1"], eps))
        if layer["type"] == "retention":
            x = x + retention(h, W, L + "mix.", m, eps, rnd)
        elif layer["type"] == "attention":
            y, own = attention(h, W, L + "mix.", m, first if m.get("v_mix") else None, rnd)
            if m.get("v_mix") and first is None:
                first = own
            x = x + y
        else:
            raise ValueError(layer["type"])
        if layer.get("mlp") is not None:
            x = x + dense(rnd(sublayer_input(x, W[L + "norm2"], W[L + "canon2"], eps)), W, L + "mlp.", eps, rnd)
        if layers_out is not None:
            layers_out.append(x.copy())
    return rnd(unit_rms(x, eps) * float(np.reshape(W["final.norm"], -1)[0])) @ W["head"].T
