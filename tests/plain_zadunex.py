"""A plain, slow restatement of the Zadunex architecture in float64 numpy, one function per
mechanism, sharing nothing with the engine: the oracle of the tests.  It runs whole sequences from
position 0; there is no cache and no batch.

Notation: rows of n consecutive tokens from position 0; W x is written x @ W.T for matrices stored
[out, in]; the residual streams are X [s, n, E].
"""
import numpy as np

from plain_lubavik import read_model_dir  # noqa: F401  (the tests' small safetensors reader)


# -- small functions -----------------------------------------------------------------------
def sigmoid(v):
    return 1.0 / (1.0 + np.exp(-v))


def silu(v):
    return v * sigmoid(v)


def softplus(v):
    return np.maximum(v, 0.0) + np.log1p(np.exp(-np.abs(v)))


def rms_norm(x, w, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


def group_rms_norm(x, w, eps, groups):
    n, E = x.shape
    y = x.reshape(n, groups, E // groups)
    y = y / np.sqrt((y * y).mean(-1, keepdims=True) + eps)
    return y.reshape(n, E) * w


# -- residual streams ----------------------------------------------------------------------
def streams_read(X, w_in):
    """What a sublayer is made from: sum_s w_in[s] X_s."""
    return np.tensordot(w_in, X, axes=(0, 0))


def streams_write(X, y, w_out, w_mix):
    """Stream t takes sum_s w_mix[s, t] X_s + w_out[t] y, from the streams as they were."""
    return np.stack([sum(w_mix[s, t] * X[s] for s in range(len(X))) + w_out[t] * y for t in range(len(X))])


# -- the state-space mixer -----------------------------------------------------------------
def short_convolution(u, taps, bias):
    """u [n, C], taps [C, K]: y_t = sum_j taps[:, j] u_(t - K + 1 + j) + bias, zeros before the start."""
    K = taps.shape[1]
    pad = np.concatenate([np.zeros((K - 1, u.shape[1])), u], 0)
    return sum(taps[:, j][None, :] * pad[j:j + u.shape[0]] for j in range(K)) + bias


def state_space(x, B, C, dt, A_log, D):
    """x [n, H, V], B and C [n, G, N], dt [n, H] (after softplus): S <- exp(-exp(A_log) dt) S + dt B x^T,
    y = S^T C + D x.  Returns y [n, H, V] and the last S [H, N, V]."""
    n, H, V = x.shape
    G, N = B.shape[1:]
    S, y = np.zeros((H, N, V)), np.zeros_like(x)
    for t in range(n):
        for h in range(H):
            g = h // (H // G)
            S[h] = np.exp(-np.exp(A_log[h]) * dt[t, h]) * S[h] + dt[t, h] * np.outer(B[t, g], x[t, h])
            y[t, h] = S[h].T @ C[t, g] + D[h] * x[t, h]
    return y, S


def mamba2(w, p, m, h, eps):
    n = h.shape[0]
    H, V, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * V
    a = h @ w[p + "in"].T
    z, u, dt = a[:, :inner], a[:, inner:2 * inner + 2 * G * N], a[:, 2 * inner + 2 * G * N:]
    u = silu(short_convolution(u, w[p + "conv"], w[p + "conv.b"]))
    x, B, C = u[:, :inner], u[:, inner:inner + G * N], u[:, inner + G * N:]
    y, _ = state_space(x.reshape(n, H, V), B.reshape(n, G, N), C.reshape(n, G, N), softplus(dt + w[p + "dt_bias"]),
                       w[p + "A_log"], w[p + "D"])
    y = group_rms_norm(y.reshape(n, inner) * silu(z), w[p + "norm"], eps, m["norm_groups"])
    return y @ w[p + "o"].T


# -- softmax attention ---------------------------------------------------------------------
def rotate(x, positions, dims, base):
    """x [n, heads, D]: entries i and i + dims/2 of every head turned by position * base^(-2i/dims)."""
    half = dims // 2
    if not half:
        return x
    f = float(base) ** (-2.0 * np.arange(half, dtype=np.float64) / dims)
    a = np.asarray(positions, dtype=np.float64)[:, None, None] * f[None, None, :]
    y = x.copy()
    u, v = x[..., :half], x[..., half:dims]
    y[..., :half] = u * np.cos(a) - v * np.sin(a)
    y[..., half:dims] = v * np.cos(a) + u * np.sin(a)
    return y


def softmax_attention(q, k, v, scale):
    """q [n, H, D], k [n, G, D], v [n, G, V]: every query sees the keys up to its own; the softmax's
    denominator has one more term, exp(0)."""
    n, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((n, H, v.shape[2]))
    seen = np.arange(n)[None, :] <= np.arange(n)[:, None]
    for h in range(H):
        g = h // (H // G)
        s = np.where(seen, (q[:, h] @ k[:, g].T) * scale, -np.inf)
        top = np.maximum(s.max(-1), 0.0)
        e = np.exp(s - top[:, None])
        out[:, h] = (e @ v[:, g]) / (np.exp(-top) + e.sum(-1))[:, None]
    return out


def attention(w, p, m, h, eps):
    n = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    q = rms_norm(h @ w[p + "q"].T + w[p + "q.b"], w[p + "q.norm"], eps).reshape(n, H, D)
    k = rms_norm(h @ w[p + "k"].T + w[p + "k.b"], w[p + "k.norm"], eps).reshape(n, G, D)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).reshape(n, G, V)
    q, k = (rotate(a, np.arange(n), rot["dims"], rot["base"]) for a in (q, k))
    return softmax_attention(q, k, v, m["scale"]).reshape(n, H * V) @ w[p + "o"].T


# -- feed-forward --------------------------------------------------------------------------
def clamped_gate(g, u, limit):
    """g bounded above, u on both sides: g sigmoid(1.702 g) (u + 1)."""
    g, u = np.minimum(g, limit), np.clip(u, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def dense_ff(w, p, mlp, h):
    return clamped_gate(h @ w[p + "gate"].T, h @ w[p + "up"].T, mlp["limit"]) @ w[p + "down"].T


def route(z, top):
    """z [n, X] router logits -> dense weights [n, X]: the `top` largest of a softmax over all, as they are."""
    s = np.exp(z - z.max(-1, keepdims=True))
    s /= s.sum(-1, keepdims=True)
    dense = np.zeros_like(s)
    for t in range(len(z)):
        chosen = np.argsort(-s[t], kind="stable")[:top]
        dense[t, chosen] = s[t, chosen]
    return dense


def moe_ff(w, p, mlp, h):
    dense = route(h @ w[p + "router"].T, mlp["router"]["top"])
    out = np.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        pe = f"{p}e{e}."
        y = (silu(h @ w[pe + "gate"].T) * (h @ w[pe + "up"].T)) @ w[pe + "down"].T
        out += dense[:, e:e + 1] * y
    return out


# -- the model -----------------------------------------------------------------------------
def running_order(cfg):
    n = len(cfg["layers"])
    lp = cfg.get("loop")
    if not lp:
        return list(range(n))
    return (list(range(lp["start"])) + list(range(lp["start"], lp["stop"])) * lp["times"] + list(range(lp["stop"], n)))


def forward(cfg, w, tokens, return_layers=False):
    """Logits [n, vocab] of a whole sequence from position 0 (and the sum of the streams after every
    layer run)."""
    tokens = np.asarray(tokens, dtype=np.int64)
    eps = cfg["norm"]["eps"]
    X = np.stack([w["embed"][tokens]] * cfg["streams"])
    sums = []
    for i in running_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."

        def sublayer(X, q, run):
            hc = f"{p}hc{q}."
            y = run(rms_norm(streams_read(X, w[hc + "in"]), w[f"{p}norm{q}"], eps))
            return streams_write(X, y, w[hc + "out"], w[hc + "mix"])

        mixer = {"mamba2": mamba2, "attention": attention}[layer["type"]]
        X = sublayer(X, 1, lambda h: mixer(w, p + "mix.", layer["mixer"], h, eps))
        mlp = layer.get("mlp")
        if mlp:
            ff = {"dense": dense_ff, "moe": moe_ff}[mlp["kind"]]
            X = sublayer(X, 2, lambda h: ff(w, p + "mlp.", mlp, h))
        sums.append(X.sum(0))
    logits = rms_norm(X.sum(0), w["final.norm"], eps) @ w["head"].T * cfg["logit_scale"]
    return (logits, np.stack(sums)) if return_layers else logits
