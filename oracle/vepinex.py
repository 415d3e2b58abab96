"""Plain statement of the Vepinex decoder in numpy, one function per mechanism, whole sequences, no caches.

Test infrastructure: it shares no code with the product, takes the configuration as a dict and the weights as a
dict of arrays under their file names, and is written for clarity. Everything runs in the precision of the weights.
"""
import numpy as np


def rms_normalize(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + x.dtype.type(eps))


def norm(x, w, eps):
    """RMS norm with a plain weight."""
    return rms_normalize(x, eps) * w


def sigmoid(z):
    return 1 / (1 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(z, z.dtype.type(0))


def log_sigmoid(z):
    return -softplus(-z)


# ------------------------------------------------------------------------------------------------ matrix memory
def memory_gates(zi, zf, cap):
    """Soft-capped pre-activations [T, H] -> logarithms of the input and the forget gate."""
    cap = zi.dtype.type(cap)
    return cap * np.tanh(zi / cap), log_sigmoid(cap * np.tanh(zf / cap))


def memory_scan(q, k, v, i, f, state=None):
    """q, k [T, H, d], v [T, H, e], log gates i, f [T, H]; state (S [H, d, e], n [H, d], m [H]) or zeros.
    Returns (o [T, H, e], final state)."""
    T, H, d = q.shape
    if state is None:
        state = (np.zeros((H, d, v.shape[2]), q.dtype), np.zeros((H, d), q.dtype), np.zeros(H, q.dtype))
    S, n, m = (a.copy() for a in state)
    o = np.empty_like(v)
    for t in range(T):
        top = np.maximum(f[t] + m, i[t])
        keep, add = np.exp(f[t] + m - top), np.exp(i[t] - top)
        m = top
        S = keep[:, None, None] * S + add[:, None, None] * (k[t][:, :, None] * v[t][:, None, :])
        n = keep[:, None] * n + add[:, None] * k[t]
        size = np.maximum(np.abs((n * q[t]).sum(axis=1)), np.exp(-m))
        o[t] = np.einsum("hij,hi->hj", S, q[t]) / (size[:, None] + q.dtype.type(1e-6))
    return o, (S, n, m)


def mlstm_mixer(h, W, m, eps):
    T, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ W["q"].T).reshape(T, H, d) * h.dtype.type(d ** -0.5)
    k = (h @ W["k"].T).reshape(T, H, d)
    v = (h @ W["v"].T).reshape(T, H, e)
    i, f = memory_gates(h @ W["i"].T + W["i.b"], h @ W["f"].T + W["f.b"], m["gate_cap"])
    o, _ = memory_scan(q, k, v, i, f)
    o = rms_normalize(o, eps).reshape(T, H * e) * W["norm"] * sigmoid(h @ W["g"].T)
    return o @ W["o"].T


# ------------------------------------------------------------------------------------------------ delta rule
def short_conv(x, w, before=None):
    """x [T, C], w [C, taps], the last tap meets the current token; `before` [taps - 1, C] are the inputs ahead of x."""
    taps = w.shape[1]
    if before is None:
        before = np.zeros((taps - 1, x.shape[1]), x.dtype)
    padded = np.concatenate([before, x])
    return sum(padded[j:j + x.shape[0]] * w[:, j] for j in range(taps))


def unit(x):
    return x / np.sqrt((x * x).sum(axis=-1, keepdims=True) + x.dtype.type(1e-6))


def channel_decay(a, A_log, dt_bias):
    """a [T, H, d] (the low-rank product), A_log [H], dt_bias [H, d] -> decays in (0, 1)."""
    return np.exp(-np.exp(A_log)[:, None] * softplus(a + dt_bias))


def delta_scan(q, k, v, g, beta, state=None):
    """q, k [T, G, d], v [T, H, e], g [T, H, d], beta [T, H] -> (o [T, H, e], final state [H, d, e])."""
    T, H, e = v.shape
    per = H // q.shape[1]
    S = np.zeros((H, q.shape[2], e), q.dtype) if state is None else state.copy()
    o = np.empty_like(v)
    for t in range(T):
        for h in range(H):
            kt, qt = k[t, h // per], q[t, h // per]
            S[h] *= g[t, h][:, None]
            S[h] += np.outer(kt, beta[t, h] * (v[t, h] - S[h].T @ kt))
            o[t, h] = S[h].T @ qt
    return o, S


def delta_mixer(h, W, m, eps):
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(short_conv(h @ W[n].T, W[n + ".conv"])) for n in "qkv")
    q = unit(q.reshape(T, G, d)) * h.dtype.type(d ** -0.5)
    k = unit(k.reshape(T, G, d))
    g = channel_decay(((h @ W["a1"].T) @ W["a2"].T).reshape(T, H, d), W["A_log"], W["dt_bias"].reshape(H, d))
    o, _ = delta_scan(q, k, v.reshape(T, H, e), g, sigmoid(h @ W["b"].T))
    gate = sigmoid((h @ W["g1"].T) @ W["g2"].T)
    return ((rms_normalize(o, eps) * W["norm"]).reshape(T, H * e) * gate) @ W["o"].T


# ------------------------------------------------------------------------------------------------ latent attention
def rotate(x, pos, base):
    """x [T, ..., r]: neighbours (2i, 2i + 1) turned by pos * base^(-2i / r)."""
    r = x.shape[-1]
    freq = float(base) ** (-np.arange(0, r, 2) / r)
    a = (np.asarray(pos, np.float64)[:, None] * freq).reshape((len(pos),) + (1,) * (x.ndim - 2) + (r // 2,))
    c, s = np.cos(a).astype(x.dtype), np.sin(a).astype(x.dtype)
    out = np.empty_like(x)
    out[..., 0::2] = x[..., 0::2] * c - x[..., 1::2] * s
    out[..., 1::2] = x[..., 1::2] * c + x[..., 0::2] * s
    return out


def latent_cache(h, W, m, eps):
    """What later tokens need of h: the normed latent [T, kv_rank] and the rotated key part [T, rot_dim]."""
    y, R = h @ W["dkv"].T, m["kv_rank"]
    return norm(y[:, :R], W["dkv.norm"], eps), rotate(y[:, R:], np.arange(h.shape[0]), m["rot"]["base"])


def latent_attention(q, c, kr, uk, uv, m, pos):
    """Queries q [N, H, dim + rot_dim] (rotated) at positions pos over the latents c [T, kv_rank] and rotated key parts kr."""
    H, d, e = m["heads"], m["dim"], m["vdim"]
    k = (c @ uk.T).reshape(-1, H, d)
    v = (c @ uv.T).reshape(-1, H, e)
    hidden = np.arange(c.shape[0])[None, :] > np.asarray(pos)[:, None]
    out = np.empty((q.shape[0], H, e), q.dtype)
    for n in range(H):
        s = (q[:, n, :d] @ k[:, n].T + q[:, n, d:] @ kr.T) * q.dtype.type(m["scale"])
        s[hidden] = -np.inf
        p = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, n] = (p / p.sum(axis=1, keepdims=True)) @ v[:, n]
    return out


def latent_mixer(h, W, m, eps, kept):
    """kept: (latent, rotated key part), this layer's own or those of the layer it shares them with."""
    T, H, d = h.shape[0], m["heads"], m["dim"]
    q = (h @ W["q"].T).reshape(T, H, d + m["rot_dim"]).copy()
    q[..., d:] = rotate(q[..., d:], np.arange(T), m["rot"]["base"])
    o = latent_attention(q, *kept, W["uk"], W["uv"], m, np.arange(T))
    return o.reshape(T, H * m["vdim"]) @ W["o"].T


# ------------------------------------------------------------------------------------------------ feed-forward
def silu_unit(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def clamped_unit(h, gate, up, down, limit):
    g = np.minimum(h @ gate.T, h.dtype.type(limit))
    u = np.clip(h @ up.T, -h.dtype.type(limit), h.dtype.type(limit))
    return (g * sigmoid(h.dtype.type(1.702) * g) * (u + 1)) @ down.T


def route(z, top):
    """Logits [T, experts] -> ids [T, top] in descending order and the softmax over the chosen logits."""
    ids = np.argsort(-z, axis=1, kind="stable")[:, :top]
    c = np.take_along_axis(z, ids, axis=1)
    p = np.exp(c - c[:, :1])
    return ids, p / p.sum(axis=1, keepdims=True)


def moe(h, W, m):
    ids, w = route(h @ W["router"].T + W["router.b"], m["router"]["top"])
    y = np.zeros_like(h)
    for e in range(m["router"]["experts"]):
        t, place = np.nonzero(ids == e)
        if len(t):
            y[t] += w[t, place][:, None] * clamped_unit(h[t], *(W["e%d.%s" % (e, n)] for n in ("gate", "up", "down")),
                                                        m["expert"]["limit"])
    if m.get("shared"):
        y = y + clamped_unit(h, *(W["shared." + n] for n in ("gate", "up", "down")), m["shared"]["limit"])
    return y


# ------------------------------------------------------------------------------------------------ the model
def forward(cfg, weights, tokens):
    """(logits [T, vocab], residual stream after every layer)."""
    eps = cfg["norm"]["eps"]

    def under(prefix):
        return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}
    x = norm(weights["embed"][np.asarray(tokens)], weights["embed.norm"], eps)
    trail, kept = [], {}
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = "l%d." % i, layer["mixer"], layer.get("mlp")
        h, W = norm(x, weights[p + "norm1"], eps), under(p + "mix.")
        if layer["type"] == "mlstm":
            y = mlstm_mixer(h, W, m, eps)
        elif layer["type"] == "channel_delta":
            y = delta_mixer(h, W, m, eps)
        else:
            if m.get("kv_from") is None:
                kept[i] = latent_cache(h, W, m, eps)
            y = latent_mixer(h, W, m, eps, kept[i if m.get("kv_from") is None else m["kv_from"]])
        if f:
            W = under(p + "mlp.")
            y = y + (silu_unit(h, W["gate"], W["up"], W["down"]) if f["kind"] == "dense" else moe(h, W, f))
        x = x + y
        trail.append(x)
    return norm(x, weights["final.norm"], eps) @ weights["embed"].T, trail
