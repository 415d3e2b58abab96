"""Plain statement of the Lenisun decoder in numpy, one function per mechanism, whole sequences, no caches.

Test infrastructure: it shares no code with the product, takes the configuration as a dict and the weights as a
dict of arrays under their file names, and is written for clarity. `dtype` is the precision everything runs in.
"""
import numpy as np


def rms_normalize(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + x.dtype.type(eps))


def norm_one_plus(x, w, eps):
    """RMS norm whose weight is stored as its difference from one."""
    return rms_normalize(x, eps) * (1 + w)


def sigmoid(z):
    return 1 / (1 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def query_temperature(pos, coef, every):
    return 1 + coef * np.log(np.floor((pos + 1) / every) + 1)


def attention(q, k, v, scale):
    """q [T, H, d], k [T, G, d], v [T, G, e]: causal softmax attention, query head h reads key head h // (H / G)."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = np.empty((T, H, v.shape[2]), q.dtype)
    hidden = np.triu(np.ones((T, T), bool), 1)
    for h in range(H):
        s = (q[:, h] @ k[:, h // per].T) * q.dtype.type(scale)
        s[hidden] = -np.inf
        p = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = (p / p.sum(axis=1, keepdims=True)) @ v[:, h // per]
    return out


def attention_mixer(h, W, m, eps, v_first):
    """Returns (output, this layer's own values before mixing). v_first: the first mixing layer's values or None."""
    T = h.shape[0]
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ W["q"].T).reshape(T, H, d)
    k = (h @ W["k"].T).reshape(T, G, d)
    v = (h @ W["v"].T).reshape(T, G, e)
    q = rms_normalize(q, eps) * W["q.norm"]
    k = rms_normalize(k, eps) * W["k.norm"]
    if m.get("q_temp"):
        t = query_temperature(np.arange(T, dtype=np.float64), m["q_temp"]["coef"], m["q_temp"]["every"])
        q = q * t.astype(h.dtype)[:, None, None]
    own = v
    if v_first is not None:
        lam = W["vmix"].reshape(())
        v = (1 - lam) * v + lam * v_first
    o = attention(q, k, v, m["scale"])
    return o.reshape(T, H * e) @ W["o"].T, own


def token_shift(h, mu, before=None):
    """h + (previous token's h - h) * mu; the token ahead of the first one is `before` (zeros by default)."""
    prev = np.concatenate([np.zeros_like(h[:1]) if before is None else before[None], h[:-1]])
    return h + (prev - h) * mu


def wkv_decay(x, w1, w2, w0):
    return np.exp(-np.exp(np.tanh(x @ w1.T) @ w2.T + w0))


def wkv_scan(r, k, v, w, u, state=None):
    """r, k, v, w [T, H, d], u [H, d] -> (o [T, H, d], final state [H, d(key), d(value)])."""
    T, H, d = r.shape
    S = np.zeros((H, d, d), r.dtype) if state is None else state.copy()
    o = np.empty_like(r)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hij,hi->hj", S + u[:, :, None] * kv, r[t])
        S = w[t][:, :, None] * S + kv
    return o, S


def wkv_mixer(h, W, m, eps):
    T, H, d = h.shape[0], m["heads"], m["dim"]
    mix = {s: token_shift(h, W["mu." + s]) for s in "rkvgw"}
    r, k, v = ((mix[s] @ W[s].T).reshape(T, H, d) for s in "rkv")
    gate = silu(mix["g"] @ W["g"].T)
    w = wkv_decay(mix["w"], W["w1"], W["w2"], W["w0"]).reshape(T, H, d)
    o, _ = wkv_scan(r, k, v, w, W["u"])
    return (rms_normalize(o, eps).reshape(T, H * d) * W["norm"] * gate) @ W["o"].T


def clamped_glu(g, u, limit):
    g = np.minimum(g, g.dtype.type(limit))
    u = np.clip(u, -limit, limit).astype(u.dtype)
    return g * sigmoid(g.dtype.type(1.702) * g) * (u + 1)


def dense_mlp(h, W, m):
    return clamped_glu(h @ W["gate"].T, h @ W["up"].T, m["limit"]) @ W["down"].T


def silu_mlp(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def route(h, router, top):
    """Sigmoid scores; the `top` largest per token (ids in descending order of score) and their scores."""
    s = sigmoid(h @ router.T)
    ids = np.argsort(-s, axis=1, kind="stable")[:, :top]
    return ids, np.take_along_axis(s, ids, axis=1)


def moe_mlp(h, W, m):
    ids, scores = route(h, W["router"], m["router"]["top"])
    y = np.zeros_like(h)
    for e in range(m["router"]["experts"]):
        for slot in range(ids.shape[1]):
            t = np.nonzero(ids[:, slot] == e)[0]
            if t.size:
                p = "e%d." % e
                y[t] += silu_mlp(h[t] * scores[t, slot, None], W[p + "gate"], W[p + "up"], W[p + "down"])
    if m.get("shared"):
        sh = silu_mlp(h, W["shared.gate"], W["shared.up"], W["shared.down"])
        y = y + sh * sigmoid(h @ W["shared.sg"].T)
    return y


def forward(cfg, weights, tokens, dtype=np.float64):
    """tokens [T] -> (logits [T, vocab], residual stream after every layer [layers, T, width])."""
    def part(prefix):
        return {k[len(prefix):]: np.asarray(v, dtype) for k, v in weights.items() if k.startswith(prefix)}

    eps = cfg["norm"]["eps"]
    x = np.asarray(weights["embed"], dtype)[np.asarray(tokens)] * dtype(cfg["embedding"]["scale"])
    v_first, trail = None, []
    for i, layer in enumerate(cfg["layers"]):
        L = part("l%d." % i)
        h = norm_one_plus(x, L["norm1"], eps)
        mix = part("l%d.mix." % i)
        if layer["type"] == "attention":
            mixes = bool(layer["mixer"].get("v_mix"))
            y, own = attention_mixer(h, mix, layer["mixer"], eps, v_first if mixes else None)
            if mixes and v_first is None:
                v_first = own
        else:
            y = wkv_mixer(h, mix, layer["mixer"], eps)
        x = x + norm_one_plus(y, L["norm1b"], eps)
        if layer.get("mlp"):
            h = norm_one_plus(x, L["norm2"], eps)
            mlp = dense_mlp if layer["mlp"]["kind"] == "dense" else moe_mlp
            x = x + norm_one_plus(mlp(h, part("l%d.mlp." % i), layer["mlp"]), L["norm2b"], eps)
        trail.append(x)
    logits = norm_one_plus(x, np.asarray(weights["final.norm"], dtype), eps) @ np.asarray(weights["head"], dtype).T
    return logits, np.stack(trail)
