"""Plain, slow Fobatar forward pass: whole sequences, no cache, one function per mechanism.

The oracle of the Fobatar tests.  It shares no code with the product package: it takes the configuration as a plain ``dict``
(the keys of config.json) and the weights as a ``dict`` of numpy arrays keyed by tensor name, and computes everything in
float64 except the rotary angle, which is the float32 product of position and frequency.  Attention walks query by query
over keys that are picked by the mask's own definition, and every expert is applied to one token at a time.

Notation: D model width, T tokens of one sequence.  With n(x) = x / sqrt(mean(x^2) + eps) * w, a layer is
x <- x + m n1b(mixer(n1(x)));  x <- x + m n2b(ff(n2(x))).  `rnd` models a bfloat16 engine: it is applied where such an
engine must round (inputs of matrix products, cached rows); the identity gives exact arithmetic.
"""
from __future__ import annotations

import math

import numpy as np

ALPHA = 1.702           # inside the sigmoid of the clamped swish


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


def rms_norm(x, w, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


# ---- convolution over time -------------------------------------------------------------------------------------------
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


# ---- rotation ----------------------------------------------------------------------------------------------------------
def frequencies(rot):
    """(frequency of every pair, factor of cosines and sines)."""
    base, dims, sc = rot["base"], rot["dims"], rot.get("scaling")
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not sc or not f:
        return np.array(f, dtype=np.float64), 1.0

    def pair_of(turns):      # the (real-valued) pair whose wave makes `turns` turns over `original` positions
        return dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(pair_of(sc["fast"])), 0)
    hi = min(math.ceil(pair_of(sc["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * r + fi * (1.0 - r))
    return np.array(out, dtype=np.float64), 0.1 * math.log(sc["factor"]) + 1.0


def rotate_neighbours(x, pos, freq, grow):
    """x [T, heads, d]: pairs (2i, 2i+1) of the first 2 * len(freq) dimensions turn and grow; the rest passes."""
    x = x.copy()
    n = len(freq)
    if n == 0:
        return x
    ang = (np.asarray(pos, dtype=np.float32)[:, None] * freq.astype(np.float32)[None, :]).astype(np.float64)   # a 32-bit product
    cs, sn = np.cos(ang)[:, None, :] * grow, np.sin(ang)[:, None, :] * grow
    u, v = x[..., 0:2 * n:2].copy(), x[..., 1:2 * n:2].copy()
    x[..., 0:2 * n:2] = u * cs - v * sn
    x[..., 1:2 * n:2] = v * cs + u * sn
    return x


# ---- attention ----------------------------------------------------------------------------------------------------------
def visible(i, j, chunk=None):
    """Whether query position i sees key position j (a number or an array of them): causal, and with a chunk size only within
    i's chunk."""
    seen = j <= i
    return seen if chunk is None else seen & (i // chunk == j // chunk)


def attend(q, k, v, scale, chunk=None, sink=False):
    """One head: q [T, d], k [T, d], v [T, dv] -> [T, dv].  sink: one joins the denominator."""
    T = q.shape[0]
    out = np.zeros((T, v.shape[1]))
    for i in range(T):
        js = np.flatnonzero(visible(i, np.arange(T), chunk))
        s = (k[js] @ q[i]) * scale
        top = max(s.max(), 0.0) if sink else s.max()
        e = np.exp(s - top)
        den = e.sum() + (math.exp(-top) if sink else 0.0)
        out[i] = (e / den) @ v[js]
    return out


def head_gate(out, h, w_g):
    """out [T, H, dv] times one sigmoid per head."""
    return out * sigmoid(h @ w_g.T)[:, :, None]


def chunked_attention(h, W, p, m, eps, rnd=_same):
    """Convolved and normed projections, neighbour rotation, keys of the query's own chunk, a sink, a gate per head."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos, (freq, grow) = np.arange(T), frequencies(m["rot"])
    q = rms_norm(causal_conv(h @ W[p + "q"].T, W[p + "q.conv"]), W[p + "q.norm"], eps).reshape(T, H, d)
    k = rms_norm(causal_conv(h @ W[p + "k"].T, W[p + "k.conv"]), W[p + "k.norm"], eps).reshape(T, G, d)
    v = rnd(causal_conv(h @ W[p + "v"].T, W[p + "v.conv"])).reshape(T, G, dv)
    q, k = rnd(rotate_neighbours(q, pos, freq, grow)), rnd(rotate_neighbours(k, pos, freq, grow))
    chunk = (m.get("mask") or {}).get("size")
    out = np.stack([attend(q[:, i], k[:, i // (H // G)], v[:, i // (H // G)], m["scale"], chunk, sink=True) for i in range(H)], axis=1)
    return rnd(head_gate(out, h, W[p + "g"]).reshape(T, H * dv)) @ W[p + "o"].T


def latent_attention(h, W, p, m, eps, rnd=_same):
    """Keys and values of every head from one normed latent per token, a rotated key part that all heads share, a gate per
    head."""
    T = h.shape[0]
    H, d, r, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos, (freq, grow) = np.arange(T), frequencies(m["rot"])
    q = (h @ W[p + "q"].T).reshape(T, H, d + r)
    down = h @ W[p + "dkv"].T
    c = rnd(rms_norm(down[:, :R], W[p + "dkv.norm"], eps))
    kr = rnd(rotate_neighbours(down[:, None, R:], pos, freq, grow))[:, 0]
    qr = rnd(rotate_neighbours(q[:, :, d:], pos, freq, grow))
    kn = (c @ W[p + "uk"].T).reshape(T, H, d)
    v = (c @ W[p + "uv"].T).reshape(T, H, dv)
    out = np.stack([attend(np.concatenate([q[:, i, :d], qr[:, i]], 1), np.concatenate([kn[:, i], kr], 1), v[:, i], m["scale"])
                    for i in range(H)], axis=1)
    return rnd(head_gate(out, h, W[p + "g"]).reshape(T, H * dv)) @ W[p + "o"].T


# ---- feed-forward ----------------------------------------------------------------------------------------------------------
def clamped_swish(g, u, limit):
    g = np.minimum(g, limit)
    u = np.minimum(np.maximum(u, -limit), limit)
    return g * sigmoid(ALPHA * g) * (u + 1.0)


def expert(x, W, p, limit, rnd=_same):
    return W[p + "down"] @ rnd(clamped_swish(W[p + "gate"] @ x, W[p + "up"] @ x, limit))


def table_moe(h, tokens, W, p, mlp, rnd=_same):
    """Every token's experts stand in a table by its id; each weighs 1 / top; a shared expert is added."""
    top = mlp["router"]["top"]
    out = np.zeros_like(h)
    for t, tok in enumerate(tokens):
        for e in W[p + "table"][int(tok)]:
            out[t] += expert(h[t], W, f"{p}e{int(e)}.", mlp["expert"]["limit"], rnd) / top
        if mlp.get("shared") is not None:
            out[t] += expert(h[t], W, p + "shared.", mlp["shared"]["limit"], rnd)
    return out


# ---- the model ---------------------------------------------------------------------------------------------------------------
def run_order(cfg):
    """[(layer, whether the embedding output is added before it)]: the looped range repeats; every pass but the first begins
    with that sum."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    order = [(i, False) for i in range(loop["start"])]
    for t in range(loop["times"]):
        order += [(i, t > 0 and i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return order + [(i, False) for i in range(loop["stop"], n)]


def forward(cfg, W, tokens, rnd=_same, layers_out=None):
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x0 = W["embed"][np.asarray(tokens)].astype(np.float64) * cfg["embedding"]["scale"]
    x = x0
    for i, again in run_order(cfg):
        layer, L = cfg["layers"][i], f"l{i}."
        if again:
            x = x + x0
        h = rnd(rms_norm(x, W[L + "norm1"], eps))
        mix = {"attention": chunked_attention, "latent_attention": latent_attention}[layer["type"]]
        x = x + m * rms_norm(mix(h, W, L + "mix.", layer["mixer"], eps, rnd), W[L + "norm1b"], eps)
        if layer.get("mlp") is not None:
            h = rnd(rms_norm(x, W[L + "norm2"], eps))
            x = x + m * rms_norm(table_moe(h, tokens, W, L + "mlp.", layer["mlp"], rnd), W[L + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return rnd(rms_norm(x, W["final.norm"], eps)) @ W["embed"].T
