"""A plain, slow restatement of the Fupapel architecture in float64 numpy, one function per
mechanism, sharing nothing with the engine: the oracle of the tests.  It runs whole sequences from
position 0; there is no cache and no batch.

Notation: x [n, E] is the residual stream of n consecutive tokens from position 0; W x is
written x @ W.T for matrices stored [out, in].
"""
import math

import numpy as np

from plain_lubavik import read_model_dir  # noqa: F401  (the tests' small safetensors reader)


# -- small functions -----------------------------------------------------------------------
def sigmoid(v):
    return 1.0 / (1.0 + np.exp(-v))


def silu(v):
    return v * sigmoid(v)


def rms_unit(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def norm_plain(x, w, eps):
    return rms_unit(x, eps) * w


def norm_one_plus(x, w, eps):
    """The model's norm: the weight is stored around zero."""
    return rms_unit(x, eps) * (1.0 + w)


def token_shift(h, mu):
    """Every row moved towards the row before it (as that was before it moved; zeros ahead of the
    first), element by element."""
    before = np.concatenate([np.zeros((1, h.shape[1])), h[:-1]], 0)
    return h + (before - h) * mu


def short_convolution(u, taps):
    """u [n, C], taps [C, K]: y_t = sum_j taps[:, j] u_(t - K + 1 + j), zeros before the start."""
    K = taps.shape[1]
    pad = np.concatenate([np.zeros((K - 1, u.shape[1])), u], 0)
    return sum(taps[:, j][None, :] * pad[j:j + u.shape[0]] for j in range(K))


# -- rotation ------------------------------------------------------------------------------
def frequencies(dims, base, scaling=None):
    """base^(-2i/dims), i < dims/2; with `scaling` slow pairs are divided by a factor, fast ones
    kept, and those between blended by how many of their wavelengths fit into the original length."""
    f = float(base) ** (-2.0 * np.arange(dims // 2, dtype=np.float64) / max(dims, 1))
    if scaling is None:
        return f
    out = f.copy()
    for i, fi in enumerate(f):
        wave = 2.0 * math.pi / fi
        turns = scaling["original"] / wave
        if wave < scaling["original"] / scaling["high"]:
            continue
        if wave > scaling["original"] / scaling["low"]:
            out[i] = fi / scaling["factor"]
            continue
        s = (turns - scaling["low"]) / (scaling["high"] - scaling["low"])
        out[i] = (1.0 - s) * fi / scaling["factor"] + s * fi
    return out


def rotate(x, positions, freq):
    """x [n, heads, D]: entries i and i + len(freq) of every head turned by position * freq[i]."""
    half = len(freq)
    if not half:
        return x
    a = np.asarray(positions, dtype=np.float64)[:, None, None] * freq[None, None, :]
    y = x.copy()
    u, v = x[..., :half], x[..., half:2 * half]
    y[..., :half] = u * np.cos(a) - v * np.sin(a)
    y[..., half:2 * half] = v * np.cos(a) + u * np.sin(a)
    return y


def rot_frequencies(rot):
    return frequencies(rot["dims"], rot["base"], rot.get("scaling")) if rot else np.zeros(0)


# -- softmax attention ---------------------------------------------------------------------
def softmax_attention(q, k, v, scale, chunk=None, sinks=None):
    """q [n, H, D], k [n, G, D], v [n, G, V] at positions 0..n-1.  Query i sees j <= i, and with
    `chunk` only those j in its own chunk of so many positions.  `sinks` [H]: one more term
    exp(sink) in the denominator."""
    n, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((n, H, v.shape[2]))
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    seen = j <= i
    if chunk:
        seen &= i // chunk == j // chunk
    for h in range(H):
        g = h // (H // G)
        s = np.where(seen, (q[:, h] @ k[:, g].T) * scale, -np.inf)
        m = s.max(-1)
        if sinks is not None:
            m = np.maximum(m, sinks[h])
        e = np.exp(s - m[:, None])
        den = e.sum(-1) + (np.exp(sinks[h] - m) if sinks is not None else 0.0)
        out[:, h] = (e @ v[:, g]) / den[:, None]
    return out


def gated_attention(w, p, m, h, eps):
    """Keys, queries normed over the whole projection and turned; a constant 1 in the softmax's
    denominator; the heads' results gated entry by entry."""
    n = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos, f = np.arange(n), rot_frequencies(m.get("rot"))
    q = rotate(norm_plain(h @ w[p + "q"].T, w[p + "q.norm"], eps).reshape(n, H, D), pos, f)
    k = rotate(norm_plain(h @ w[p + "k"].T, w[p + "k.norm"], eps).reshape(n, G, D), pos, f)
    v = (h @ w[p + "v"].T).reshape(n, G, V)
    o = softmax_attention(q, k, v, m["scale"], chunk=(m.get("mask") or {}).get("size"), sinks=np.zeros(H))
    return (o.reshape(n, -1) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def conv_keys_values(w, p, m, h, eps):
    """Keys and values of an "attention_2" layer that has its own: projected, convolved; the keys
    then normed and turned."""
    n = h.shape[0]
    G, D, V = m["kv_heads"], m["dim"], m["vdim"]
    k = short_convolution(h @ w[p + "k"].T, w[p + "k.conv"])
    v = short_convolution(h @ w[p + "v"].T, w[p + "v.conv"])
    k = norm_plain(k, w[p + "k.norm"], eps).reshape(n, G, D)
    return rotate(k, np.arange(n), rot_frequencies(m.get("rot"))), v.reshape(n, G, V)


def conv_attention(w, p, m, h, eps, kv):
    """kv = (keys, values) as the layer that owns them made them."""
    n = h.shape[0]
    H, D = m["heads"], m["dim"]
    q = short_convolution(h @ w[p + "q"].T, w[p + "q.conv"])
    q = norm_plain(q, w[p + "q.norm"], eps).reshape(n, H, D)
    q = rotate(q, np.arange(n), rot_frequencies(m.get("rot")))
    q = q * w[p + "temp"][None, :, None]
    o = softmax_attention(q, kv[0], kv[1], m["scale"], chunk=(m.get("mask") or {}).get("size"), sinks=w[p + "sink"])
    return o.reshape(n, -1) @ w[p + "o"].T


def latent_attention(w, p, m, h, eps):
    """Keys and values written out per head from the latent."""
    n = h.shape[0]
    H, D, Rd, V, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos, f = np.arange(n), rot_frequencies(m["rot"])
    cq = norm_plain(h @ w[p + "dq"].T, w[p + "dq.norm"], eps)
    q = (cq @ w[p + "uq"].T).reshape(n, H, D + Rd)
    low = h @ w[p + "dkv"].T
    c = norm_plain(low[:, :R], w[p + "dkv.norm"], eps)
    k_turned = rotate(low[:, None, R:], pos, f)                       # one part for all heads
    q = np.concatenate([q[..., :D], rotate(q[..., D:], pos, f)], -1)
    k = np.concatenate([(c @ w[p + "uk"].T).reshape(n, H, D), np.repeat(k_turned, H, 1)], -1)
    v = (c @ w[p + "uv"].T).reshape(n, H, V)
    o = softmax_attention(q, k, v, m["scale"], sinks=w[p + "sink"])
    o = o * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(n, -1) @ w[p + "o"].T


# -- feed-forward --------------------------------------------------------------------------
def gated_expert(w, p, h):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(z, correction, top, n_groups=1, keep=1):
    """z [n, X] router logits -> dense weights [n, X]: softmax over all; the choice goes by score +
    correction, among the `keep` groups whose best member is best; the weights are the scores."""
    s = np.exp(z - z.max(-1, keepdims=True))
    s /= s.sum(-1, keepdims=True)
    c = s + correction
    n, X = z.shape
    dense = np.zeros_like(s)
    for t in range(n):
        row = c[t].copy()
        best = row.reshape(n_groups, -1).max(-1)
        kept = set(np.argsort(-best, kind="stable")[:keep].tolist())
        for e in range(X):
            if e // (X // n_groups) not in kept:
                row[e] = -np.inf
        chosen = np.argsort(-row, kind="stable")[:top]
        dense[t, chosen] = s[t, chosen]
    return dense


def moe_ff(w, p, mlp, h):
    r = mlp["router"]
    gr = r.get("groups") or {"count": 1, "keep": 1}
    dense = route(h @ w[p + "router"].T, w[p + "correction"], r["top"], gr["count"], gr["keep"])
    out = h * dense[:, r["experts"]:].sum(-1, keepdims=True)          # the identity experts
    for e in range(r["experts"]):
        rows = np.nonzero(dense[:, e])[0]
        if rows.size:
            out[rows] += dense[rows, e][:, None] * gated_expert(w, f"{p}e{e}.", h[rows])
    return out


# -- the model -----------------------------------------------------------------------------
def forward(cfg, w, tokens, return_layers=False):
    """Logits [n, vocab] of a whole sequence from position 0 (and the stream after every layer)."""
    tokens = np.asarray(tokens, dtype=np.int64)
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = w["embed"][tokens]
    kept, streams = {}, []
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = token_shift(norm_one_plus(x, w[p + "norm1"], eps), w[p + "shift"])
        if layer["type"] == "attention":
            y = gated_attention(w, p + "mix.", m, h, eps)
        elif layer["type"] == "attention_2":
            if m.get("kv_from") is None:
                kept[i] = conv_keys_values(w, p + "mix.", m, h, eps)
            y = conv_attention(w, p + "mix.", m, h, eps, kept[i if m.get("kv_from") is None else m["kv_from"]])
        elif layer["type"] == "latent_attention":
            y = latent_attention(w, p + "mix.", m, h, eps)
        else:
            raise ValueError(layer["type"])
        if layer.get("mlp"):
            y = y + moe_ff(w, p + "mlp.", layer["mlp"], norm_one_plus(x, w[p + "norm2"], eps))
        x = x + mult * y
        streams.append(x.copy())
    logits = norm_one_plus(x, w["final.norm"], eps) @ w["head"].T
    return (logits, np.stack(streams)) if return_layers else logits
