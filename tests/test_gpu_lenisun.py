"""Lenisun on the GPU against the plain implementation (oracle/lenisun.py): each mechanism alone, whole models, and the
ways a sequence can be cut, batched and moved between slots."""
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import lenisun as plain
from zignn_b200 import hostmodel, safetensors

pytestmark = pytest.mark.gpu

REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
PRECISIONS = [True, False]  # f32, bf16


def bf16(a):
    """Values a bf16 matrix can hold, as f64, and their bits."""
    bits = safetensors.f32_to_bf16(np.asarray(a, np.float32))
    return safetensors.bf16_to_f32(bits).reshape(np.shape(a)).astype(np.float64), bits.reshape(np.shape(a))


def held(a, f32):
    """What an activation of the given precision holds of `a`."""
    return np.asarray(a, np.float32).astype(np.float64) if f32 else bf16(a)[0]


def close(got, want, tol, what=""):
    got = got.detach().float().cpu().numpy() if isinstance(got, torch.Tensor) else np.asarray(got)
    want = np.asarray(want)
    assert got.shape == want.shape, (got.shape, want.shape)
    err = np.abs(got.astype(np.float64) - want).max() / max(1e-30, np.abs(want).max())
    assert err <= tol, "%s: %g > %g" % (what, err, tol)


def dev(a):
    return torch.tensor(np.asarray(a, np.float32), device="cuda")


# ------------------------------------------------------------------------------------------------ linears
@pytest.mark.parametrize("f32", PRECISIONS)
@pytest.mark.parametrize("rows_k", [(7, 40), (200, 72), (130, 1100), (515, 328)])
def test_linear_any_number_of_rows(zq, f32, rows_k):
    rng = np.random.default_rng(1)
    W, bits = bf16(rng.standard_normal(rows_k))
    w = zq.DenseWeight(bits)
    for T in (1, 2, 3, 4, 5, 8, 9, 16, 17, 33, 70, 300):
        x = held(rng.standard_normal((T, rows_k[1])), f32)
        close(w.linear(zq.dense_rows(torch.tensor(x), f32)), x @ W.T, 3e-6, "T=%d" % T)


def test_linear_many_tiles(zq):
    """More tiles than CTAs, so that the accumulators take turns, with ragged edges on both sides."""
    rng = np.random.default_rng(2)
    W, bits = bf16(rng.standard_normal((2500, 136)))
    x = held(rng.standard_normal((2100, 136)), False)
    got = zq.DenseWeight(bits).linear(zq.dense_rows(torch.tensor(x))).cpu().numpy()
    close(got, x @ W.T, 3e-6)


@pytest.mark.parametrize("f32", PRECISIONS)
@pytest.mark.parametrize("ff", [8, 30, 64, 200])
def test_gated_units(zq, f32, ff):
    rng = np.random.default_rng(3)
    k = 56
    (g, gb), (u, ub) = bf16(rng.standard_normal((ff, k)) * 0.4), bf16(rng.standard_normal((ff, k)) * 0.4)
    w = zq.DenseWeight(gb, ub)
    for T in (1, 3, 8, 9, 40, 333):
        x = held(rng.standard_normal((T, k)), f32)
        xr = zq.dense_rows(torch.tensor(x), f32)
        hg, hu = x @ g.T, x @ u.T
        for kind, want in ((zq.GLU_SILU, plain.silu(hg) * hu), (zq.GLU_CLAMPED, plain.clamped_glu(hg, hu, 1.3))):
            assert (hg > 1.3).any() and (hu < -1.3).any() and (hu > 1.3).any() or T * ff < 100
            out = w.glu(xr, kind, 1.3)
            close(out[:, :ff], want, 3e-6 if f32 else 5e-3, "T=%d kind=%d" % (T, kind))
            assert not out[:, ff:].any()


# ------------------------------------------------------------------------------------------------ attention
@pytest.mark.parametrize("f32", PRECISIONS)
def test_cache_write_norms_temperature_and_value_mixing(zq, f32):
    rng = np.random.default_rng(4)
    H, G, d, e, T = 6, 3, 20, 28, 40
    qkv = rng.standard_normal((T, H * d + G * d + G * e)).astype(np.float32)
    qn, kn = rng.uniform(0.5, 1.5, d).astype(np.float32), rng.uniform(0.5, 1.5, d).astype(np.float32)
    first = rng.standard_normal((T, G * e)).astype(np.float32)
    pos = np.arange(T) + 11
    slots = np.arange(T) % 2
    tol = 2e-6 if f32 else 5e-3
    for vmix in (None, 0.3, 1.0):
        c = zq.GqaCache(H, G, d, e, 64, 0.2, 1e-5, 0.7, 5, n_slots=2, f32=f32)
        vf = dev(first)
        lam = dev([vmix]) if vmix is not None else None
        q = c.write(dev(qkv), dev(qn), dev(kn), pos, slots, lam, vf)
        x = qkv.astype(np.float64)
        want = plain.rms_normalize(x[:, :H * d].reshape(T, H, d), 1e-5) * qn
        want = want * plain.query_temperature(pos.astype(float), 0.7, 5)[:, None, None]
        close(q[:, :, :d], want, tol)
        assert not q[:, :, d:].any()
        want = plain.rms_normalize(x[:, H * d:(H + G) * d].reshape(T, G, d), 1e-5) * kn
        close(c.k[slots, pos][:, :, :d], want, tol)
        v = x[:, (H + G) * d:].reshape(T, G, e)
        if vmix is None:
            close(vf, v.reshape(T, -1), 1e-7)
        else:
            v = (1 - vmix) * v + vmix * first.reshape(T, G, e)
        close(c.v[slots, pos][:, :, :e], v, tol)


SHAPES = [  # heads, kv_heads, dim, vdim
    (1, 1, 8, 8), (4, 4, 16, 48), (6, 2, 40, 24), (8, 2, 64, 64), (10, 2, 72, 128), (3, 1, 128, 96), (20, 1, 32, 64),
    (2, 1, 200, 256), (2, 2, 288, 16), (2, 1, 48, 320)]


def fill_cache(zq, rng, shape, ctx, n_slots, f32, scale):
    H, G, d, e = shape
    c = zq.GqaCache(H, G, d, e, ctx, scale, n_slots=n_slots, f32=f32)
    k, v = held(rng.standard_normal((n_slots, ctx, G, d)), f32), held(rng.standard_normal((n_slots, ctx, G, e)), f32)
    c.k[..., :d] = torch.tensor(k, device="cuda").to(c.k.dtype)
    c.v[..., :e] = torch.tensor(v, device="cuda").to(c.v.dtype)
    return c, k, v


def queries(c, q):
    t = torch.zeros(q.shape[0], q.shape[1], c.k.shape[3], dtype=c.k.dtype, device="cuda")
    t[..., :q.shape[2]] = torch.tensor(q, device="cuda").to(t.dtype)
    return t


def attend_rows(q, k, v, pos, scale):
    """Row r of q at position pos[r] over k, v [ctx, G, ...] of its own (list) or of all rows (array)."""
    out = []
    for r in range(q.shape[0]):
        kr, vr = (k[r], v[r]) if isinstance(k, list) else (k, v)
        n = pos[r] + 1
        per = q.shape[1] // kr.shape[1]
        kk, vv = np.repeat(kr[:n], per, axis=1), np.repeat(vr[:n], per, axis=1)
        s = np.einsum("hd,nhd->hn", q[r], kk) * scale
        p = np.exp(s - s.max(axis=1, keepdims=True))
        out.append(np.einsum("hn,nhe->he", p / p.sum(axis=1, keepdims=True), vv).reshape(-1))
    return np.stack(out)


@pytest.mark.parametrize("f32", PRECISIONS)
@pytest.mark.parametrize("shape", SHAPES)
def test_attention_prefill_and_decode(zq, f32, shape):
    rng = np.random.default_rng(5)
    H, G, d, e = shape
    ctx, scale = 700, d ** -0.5
    c, k, v = fill_cache(zq, rng, shape, ctx, 3, f32, scale)
    tol = 1e-5 if f32 else 8e-3
    for pos0, T in ((0, 1), (0, 2), (0, 65), (63, 2), (64, 3), (127, 70), (500, 130)):
        pos = np.arange(T) + pos0
        q = held(rng.standard_normal((T, H, d)), f32)
        out = c.attend(queries(c, q), pos, [1] * T, True)
        close(out[:, :H * e], attend_rows(q, k[1], v[1], pos, scale), tol, "portion at %d of %d" % (pos0, T))
        assert not out[:, H * e:].any()
    slots, pos = [2, 0, 1], np.array([699, 0, 256])
    q = held(rng.standard_normal((3, H, d)), f32)
    out = c.attend(queries(c, q), pos, slots, False)
    close(out[:, :H * e], attend_rows(q, [k[s] for s in slots], [v[s] for s in slots], pos, scale), tol, "decode")


@pytest.mark.parametrize("f32", PRECISIONS)
def test_attention_finds_one_key_among_many(zq, f32):
    """One key answers the query (its score stands out by far); it is put at tile borders, at the first token, at the
    row's own place and one place behind it, where it must not be seen."""
    rng = np.random.default_rng(6)
    H, G, d, e, ctx = 4, 2, 64, 48, 1500
    c, k, v = fill_cache(zq, rng, (H, G, d, e), ctx, 1, f32, d ** -0.5)
    for last in (63, 64, 65, 255, 256, 257, 1023, 1499):
        q1 = held(rng.standard_normal((1, H, d)), f32)
        for place in sorted({0, 1, 62, 63, 64, 127, 128, 255, 256, last - 1, last, last + 1}):
            if place < 0 or place > last + 1 or place >= ctx:
                continue
            kk, vv = k[0].copy(), v[0].copy()
            kk[place] = held(np.stack([q1[0, 2 * g] * 3 for g in range(G)]), f32)
            vv[place] = 40.0
            c.k[0, place, :, :d] = torch.tensor(kk[place], device="cuda").to(c.k.dtype)
            c.v[0, place, :, :e] = 40.0
            for T in (1, 2, 5):  # the row alone, and as the last of a portion
                if T > last + 1:
                    continue
                pos = np.arange(last + 1 - T, last + 1)
                q = np.concatenate([held(rng.standard_normal((T - 1, H, d)), f32), q1]) if T > 1 else q1
                out = c.attend(queries(c, q), pos, [0] * T, True)[:, :H * e]
                close(out, attend_rows(q, kk, vv, pos, d ** -0.5), 1e-5 if f32 else 6e-3, "key %d, row %d, T %d" % (place, last, T))
                seen = float(out[-1, 0]) > 30.0
                assert seen == (place <= last), (place, last)
            c.k[0, place, :, :d] = torch.tensor(k[0, place], device="cuda").to(c.k.dtype)
            c.v[0, place, :, :e] = torch.tensor(v[0, place], device="cuda").to(c.v.dtype)


@pytest.mark.parametrize("f32", PRECISIONS)
@pytest.mark.parametrize("shape", [(8, 2, 64, 48), (4, 1, 72, 64), (6, 2, 256, 200), (3, 3, 128, 128)])
def test_attention_prefill_with_standing_out_keys(zq, f32, shape):
    """Whole portions whose scores keep rising (every running maximum is overtaken several times over), or fall from
    the first key on, with the strong keys at tile borders and at the row's own place."""
    rng = np.random.default_rng(12)
    H, G, d, e = shape
    ctx, pos0, T = 520, 150, 300
    base = rng.standard_normal((H, d))
    base = base / np.linalg.norm(base, axis=1, keepdims=True)
    base = np.repeat(base[::H // G], H // G, axis=0)          # the heads of a group look the same way
    for name, strong in (("rising", {0: 2, 63: 6, 64: 12, 127: 25, 191: 40, 256: 60, 319: 75, 449: 90}), ("falling", {0: 90, 64: 60, 300: 20}),
                         ("last", {449: 60}), ("first", {0: 60})):
        c, k, v = fill_cache(zq, rng, shape, ctx, 2, f32, 1.0)
        kk = held(k[1] * 0.3, f32)
        for place, score in strong.items():
            kk[place] = held(np.stack([base[g * (H // G)] * score for g in range(G)]), f32)
        c.k[1, ..., :d] = torch.tensor(kk, device="cuda").to(c.k.dtype)
        q = held(base[None] + 0.05 * rng.standard_normal((T, H, d)), f32)
        pos = np.arange(T) + pos0
        out = c.attend(queries(c, q), pos, [1] * T, True)
        close(out[:, :H * e], attend_rows(q, kk, v[1], pos, 1.0), 1e-5 if f32 else 8e-3, name)
        assert not out[:, H * e:].any()


# ------------------------------------------------------------------------------------------------ recurrence
@pytest.mark.parametrize("f32", PRECISIONS)
def test_token_shift(zq, f32):
    rng = np.random.default_rng(7)
    h, mu, prev = rng.standard_normal((9, 75)), rng.uniform(-1, 2, (5, 75)), rng.standard_normal((3, 75))
    out = zq.token_shift(dev(h), dev(mu), dev(prev), slot=2, f32=f32)
    want = np.stack([plain.token_shift(h, m, prev[2]) for m in mu])
    close(out[:, :, :75], want, 2e-6 if f32 else 5e-3)
    assert not out[:, :, 75:].any()


def wkv_case(rng, T, H, d, rank):
    x = rng.standard_normal((T, 4 * H * d + rank)).astype(np.float32)
    w2, bits = bf16(rng.standard_normal((H * d, rank)) * 0.5)
    w0 = rng.uniform(-6, 1, H * d).astype(np.float32)
    u, n = rng.standard_normal((H, d)).astype(np.float32), rng.uniform(0.5, 1.5, H * d).astype(np.float32)
    return x, w2, bits, w0, u, n


def wkv_plain(x, w2, w0, u, n, eps, H, d, state):
    T, HD = x.shape[0], H * d
    y = x.astype(np.float64)
    r, k, v = (y[:, i * HD:(i + 1) * HD].reshape(T, H, d) for i in range(3))
    g, low = y[:, 3 * HD:4 * HD], y[:, 4 * HD:]
    w = np.exp(-np.exp(np.tanh(low) @ w2.T + w0)).reshape(T, H, d)
    o, S = plain.wkv_scan(r, k, v, w, u.astype(np.float64), state)
    return plain.rms_normalize(o, eps).reshape(T, HD) * n * plain.silu(g), S


@pytest.mark.parametrize("f32", PRECISIONS)
@pytest.mark.parametrize("H,d,rank", [(2, 8, 1), (3, 20, 5), (2, 64, 16), (1, 72, 33), (2, 128, 8), (1, 160, 4), (1, 256, 3)])
def test_recurrence_portions_and_steps(zq, f32, H, d, rank):
    rng = np.random.default_rng(8)
    eps, T = 1e-5, 150
    x, w2, bits, w0, u, n = wkv_case(rng, T, H, d, rank)
    start = rng.standard_normal((2, H, d, d)).astype(np.float32)
    want, S = wkv_plain(x, w2, w0, u, n, eps, H, d, start[1].astype(np.float64))
    W2, tol = zq.DenseWeight(bits), 2e-5 if f32 else 5e-3
    for cuts in ([T], [64, 86], [63, 2, 64, 21], [1, 1, 2, 3, 65, 78]):
        state = dev(start)
        outs, t0 = [], 0
        for c in cuts:
            outs.append(zq.wkv(dev(x[t0:t0 + c]), H, d, W2, dev(w0), dev(u.reshape(-1)), dev(n), eps, state, [1], True, f32))
            t0 += c
        out = torch.cat(outs)
        close(out[:, :H * d], want, tol, str(cuts))
        assert not out[:, H * d:].any()
        close(state[1], S, 2e-5)
        assert torch.equal(state[0], dev(start[0]))


def test_recurrence_of_several_sequences_at_once(zq):
    rng = np.random.default_rng(9)
    H, d, rank, eps, slots = 2, 24, 7, 1e-6, [3, 0, 2]
    x, w2, bits, w0, u, n = wkv_case(rng, 3, H, d, rank)
    start = rng.standard_normal((4, H, d, d)).astype(np.float32)
    state = dev(start)
    out = zq.wkv(dev(x), H, d, zq.DenseWeight(bits), dev(w0), dev(u.reshape(-1)), dev(n), eps, state, slots, False, True)
    for r, s in enumerate(slots):
        want, S = wkv_plain(x[r:r + 1], w2, w0, u, n, eps, H, d, start[s].astype(np.float64))
        close(out[r:r + 1, :H * d], want, 2e-5)
        close(state[s], S, 2e-6)
    assert torch.equal(state[1], dev(start[1]))


def test_recurrence_remembers_one_token_over_chunk_borders(zq):
    """With hardly any decay, a key written once answers the same read-out hundreds of tokens later; with full decay
    (weights near zero) nothing of it is left."""
    rng = np.random.default_rng(10)
    H, d, rank, T = 1, 32, 1, 300
    n = np.ones(H * d, np.float32)
    for w0_value, remembered in ((-12.0, True), (3.0, False)):
        for place in (0, 63, 64, 127, 128):
            x = np.zeros((T, 4 * H * d + rank), np.float32)
            x[:, 3 * d:4 * d] = 1.0
            x[place, d:2 * d] = 1.0 / d                      # its key
            x[place, 2 * d:3 * d] = rng.standard_normal(d)   # its value
            x[-1, :d] = 1.0                                  # the read-out
            state = torch.zeros(1, H, d, d, device="cuda")
            w2 = zq.DenseWeight(np.zeros((H * d, rank), np.uint16))
            out = zq.wkv(dev(x), H, d, w2, dev(np.full(H * d, w0_value)), dev(np.zeros(H * d)), dev(n), 1e-6, state, [0], True, True)
            want, _ = wkv_plain(x, np.zeros((H * d, rank)), np.full(H * d, w0_value), np.zeros((H, d)), n, 1e-6, H, d, None)
            close(out[:, :d], want, 2e-5)
            assert (float(out[-1, :d].abs().max()) > 0.3) == remembered


# ------------------------------------------------------------------------------------------------ routing
def test_route(zq):
    rng = np.random.default_rng(11)
    for experts, top, stride in ((5, 2, 6), (16, 1, 16), (64, 8, 65), (300, 7, 300), (3, 3, 4)):
        z = rng.standard_normal((33, stride)).astype(np.float32)
        z[:, experts:] = 100.0  # not a router logit
        if experts > 4:
            z[3, 1] = z[3, 4] = 9.0  # equal: the lower id first
        ids, s = zq.route(dev(z), experts, top)
        want, ws = plain.route(z[:, :experts].astype(np.float64), np.eye(experts), top)
        assert np.array_equal(ids.cpu().numpy(), want)
        close(s, ws, 1e-6)


# ------------------------------------------------------------------------------------------------ models
def att(heads, kv, dim, vdim, scale, **kw):
    return dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale, **kw)


def moe(experts, top, ff, shared=None):
    m = dict(kind="moe", router=dict(experts=experts, top=top), expert=dict(ff=ff))
    if shared:
        m["shared"] = dict(ff=shared)
    return m


def dense(ff, limit):
    return dict(kind="dense", ff=ff, limit=limit)


def model(vocab, width, eps, scale, layers):
    return dict(architecture="Lenisun", vocab=vocab, width=width, norm=dict(eps=eps), embedding=dict(scale=scale),
                layers=[dict(type=t, mixer=m, mlp=f) for t, m, f in layers])


MODELS = {
    # every branch, values mixed from the second attention layer on, a layer without feed-forward, ragged sizes
    "mixed": model(301, 104, 1e-5, 1.7, [
        ("wkv", dict(heads=3, dim=24), dense(90, 0.8)),
        ("attention", att(6, 3, 20, 28, 0.25, q_temp=dict(coef=0.4, every=7)), None),
        ("attention", att(4, 2, 40, 24, 0.2, v_mix=True, q_temp=dict(coef=0.2, every=50)), moe(7, 3, 40, 72)),
        ("wkv", dict(heads=2, dim=40), moe(6, 2, 24)),
        ("attention", att(8, 2, 16, 24, 0.3, v_mix=True), dense(130, 3.0))]),
    "attention_only": model(130, 64, 1e-6, 0.5, [
        ("attention", att(4, 1, 32, 32, 0.18, v_mix=True, q_temp=dict(coef=0.5, every=20)), moe(4, 1, 64, 64)),
        ("attention", att(3, 1, 64, 32, 0.125, v_mix=True, q_temp=dict(coef=0.5, every=20)), moe(12, 4, 32)),
        ("attention", att(5, 1, 16, 32, 0.25, v_mix=False), dense(64, 1.0))]),
    "recurrence_only": model(97, 72, 1e-4, 1.0, [
        ("wkv", dict(heads=1, dim=72), None),
        ("wkv", dict(heads=9, dim=8), moe(3, 1, 16, 16))]),
}


def make_host(name, seed=1, rank=6):
    """Random weights of a size that makes every part count. The router reads channels that only the token itself
    sets, far apart from each other, so that rounding does not change who is chosen."""
    cfg = MODELS[name]
    host = hostmodel.LenisunHost.synthetic(cfg, seed=seed, std=0.25, decay_rank=rank)
    rng = np.random.default_rng(seed)
    E, vocab = cfg["width"], cfg["vocab"]
    f = {k: t.f32().copy() for k, t in host.tensors.items()}
    n_max = max([l["mlp"]["router"]["experts"] for l in cfg["layers"] if l["mlp"] and l["mlp"]["kind"] == "moe"] + [1])
    f["embed"] *= 4
    f["embed"][:, :n_max] = np.stack([rng.permutation(n_max) for _ in range(vocab)]) * (24.0 / n_max) - 12.0
    for k in f:
        leaf = k.split(".")[-1]
        if leaf in ("norm1b", "norm2b"):
            f[k][:n_max] = -1.0  # nothing is added to the routing channels
        if leaf == "router":
            f[k][:] = 0.0
            f[k][:, :f[k].shape[0]] = 2.5 * np.eye(f[k].shape[0])
        if leaf == "norm2":
            f[k][:n_max] = 0.0
    host.tensors = {k: safetensors.Tensor("BF16", safetensors.f32_to_bf16(v).reshape(v.shape)) for k, v in f.items()}
    return host


_PLAIN = {}


def plain_logits(name, tokens):
    key = (name, tuple(tokens))
    if key not in _PLAIN:
        _PLAIN[key] = plain.forward(MODELS[name], make_host(name).as_f32(), tokens)
    return _PLAIN[key]


def prompt(name, n, seed=2):
    return [int(t) for t in np.random.default_rng(seed).integers(0, MODELS[name]["vocab"], n)]


def row_err(got, want):
    """Per position: root mean square of the difference over that of the wanted logits."""
    got, want = got.float().cpu().numpy().astype(np.float64), np.asarray(want, np.float64)
    return np.sqrt(((got - want) ** 2).mean(axis=1)) / np.sqrt((want ** 2).mean())


TOL = {"float32": 2e-5, "bfloat16": 4e-2}


def run(engine, tokens, cuts, seq=0):
    out, t0 = [], 0
    for c in cuts:
        out.append(engine.extend(tokens[t0:t0 + c], range(c), seq=seq))
        t0 += c
    assert t0 == len(tokens)
    return torch.cat(out)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(MODELS))
def test_model_whole_prompt_layer_by_layer(zq, name, dtype):
    tokens = prompt(name, 200)
    want, trail = plain_logits(name, tokens)
    eng = zq.Lenisun(make_host(name), ctx=256, n_seq=2, dtype=dtype)
    got = eng.extend_with_trail(tokens, seq=1)
    for l in range(len(trail)):
        e = row_err(got[l], trail[l])
        assert e.max() <= TOL[dtype], "layer %d: %g" % (l, e.max())
    eng.reset(1)
    e = row_err(eng.extend(tokens, range(200), seq=1), want)
    assert e.max() <= TOL[dtype], e.max()
    eng.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(MODELS))
def test_model_cuts_do_not_matter(zq, name, dtype):
    tokens = prompt(name, 200)
    want, _ = plain_logits(name, tokens)
    eng = zq.Lenisun(make_host(name), ctx=200, n_seq=1, dtype=dtype)
    whole = run(eng, tokens, [200])
    for cuts in ([1] * 200, [2] * 100, [3, 5, 8, 9, 64, 65, 2, 44], [199, 1], [1, 64, 128, 2, 5], [7] * 28 + [4]):
        eng.reset()
        got = run(eng, tokens, cuts)
        assert row_err(got, want).max() <= TOL[dtype], cuts[:4]
        assert row_err(got, whole.cpu().numpy()).max() <= TOL[dtype] / 2, cuts[:4]
    eng.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["attention_only", "recurrence_only"])
def test_prompts_longer_than_one_piece(zq, name, dtype):
    """More tokens in one call than the activation buffers hold: the engine cuts them itself."""
    tokens = prompt(name, 2200, seed=11)
    want, _ = plain_logits(name, tokens)
    eng = zq.Lenisun(make_host(name), ctx=2200, dtype=dtype)
    places = [0, 1, 63, 64, 1000, 2046, 2047, 2048, 2049, 2198, 2199]
    assert row_err(eng.extend(tokens, places), want[places]).max() <= TOL[dtype]
    eng.reset()
    eng.extend(tokens[:2049])  # a piece and one token
    assert row_err(eng.extend(tokens[2049:], [0, 150]), want[[2049, 2199]]).max() <= TOL[dtype]
    assert row_err(eng.prefill(tokens)[None], want[[2199]]).max() <= TOL[dtype]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_batched_sequences_equal_each_alone(zq, dtype):
    name, n_seq, steps = "mixed", 11, 9
    host = make_host(name)
    eng = zq.Lenisun(host, ctx=120, n_seq=n_seq, dtype=dtype)
    alone = zq.Lenisun(host, ctx=120, n_seq=1, dtype=dtype)
    lens = [1, 2, 3, 15, 16, 17, 31, 63, 64, 65, 100]
    prompts = [prompt(name, n, seed=20 + i) for i, n in enumerate(lens)]
    follow = [prompt(name, steps, seed=50 + i) for i in range(n_seq)]
    want = []
    for p, f in zip(prompts, follow):
        alone.prefill(p)
        want.append(torch.stack([alone.decode_next(t) for t in f]))
    for i, p in enumerate(prompts):
        eng.prefill(p, seq=i)
    order = list(np.random.default_rng(3).permutation(n_seq))
    at = [0] * n_seq
    for s in range(steps):
        # all of them (the recorded step), then a few of them, in any order of slots
        some = order if s % 3 != 1 else order[:4]
        lg = eng.decode_next_batch(some, [follow[i][at[i]] for i in some])
        for r, i in enumerate(some):
            e = row_err(lg[r:r + 1], want[i][at[i]:at[i] + 1].cpu().numpy()).max()
            assert e <= TOL[dtype] / 2, (i, s, e)
            at[i] += 1
            assert eng.seq_len_of(i) == lens[i] + at[i]
    eng.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "recurrence_only"])
def test_slots_used_again(zq, name, dtype):
    """A slot that held another sequence gives the same bits as a new one, whichever slot it is."""
    host = make_host(name)
    eng = zq.Lenisun(host, ctx=150, n_seq=3, dtype=dtype)
    tokens = prompt(name, 90, seed=7)
    cuts = [50, 2, 9, 1, 28]
    first = run(eng, tokens, cuts, seq=eng.acquire())
    for _ in range(3):
        seqs = [eng.acquire() for _ in range(2)]
        for s in seqs:
            run(eng, prompt(name, 150, seed=8 + s), [100, 50], seq=s)
        assert eng.acquire() is None
        eng.release(seqs[0])
        again = eng.acquire()
        assert again == seqs[0]
        assert torch.equal(run(eng, tokens, cuts, seq=again), first)
        eng.release(again)
        eng.release(seqs[1])


def test_long_decoding(zq):
    name = "mixed"
    tokens = prompt(name, 420, seed=9)
    want, _ = plain_logits(name, tokens)
    for dtype in ("float32", "bfloat16"):
        eng = zq.Lenisun(make_host(name), ctx=420, dtype=dtype)
        eng.extend(tokens[:20])
        got = torch.cat([eng.extend([t], [0]) for t in tokens[20:]])
        assert row_err(got, want[20:]).max() <= TOL[dtype]


def test_greedy_generation_and_scheduler(zq):
    from zignn_b200 import generate
    name = "mixed"
    host = make_host(name)
    weights = host.as_f32()
    one = zq.Lenisun(host, ctx=100, dtype="float32")
    prompts = [prompt(name, n, seed=60 + n) for n in (1, 2, 30, 41, 5, 17, 9)]
    counts = [12, 1, 20, 7, 25, 3, 15]
    want = []
    for p, n in zip(prompts, counts):
        toks = generate.generate(one, p, n)
        # each token is the plain implementation's arg-max after what came before it
        lg = plain.forward(MODELS[name], weights, p + toks[:-1])[0][len(p) - 1:]
        assert [int(t) for t in lg.argmax(axis=1)] == toks
        want.append(toks)
    eng = zq.Lenisun(host, ctx=100, n_seq=3, dtype="float32")
    for portion in (0, 2, 16):
        done = generate.serve(eng, [generate.Request(p, n) for p, n in zip(prompts, counts)], portion)
        assert [r.tokens for r in done] == want
    # sampling: top-1 is greedy whatever the temperature
    assert generate.generate(one, prompts[2], 8, top_k=1, temperature=0.7, rng=np.random.default_rng(0)) == want[2][:8]


def test_decode_greedy_equals_step_by_step(zq):
    for dtype in ("float32", "bfloat16"):
        eng = zq.Lenisun(make_host("attention_only"), ctx=400, n_seq=2, dtype=dtype)
        p = prompt("attention_only", 33)
        first = int(eng.prefill(p, seq=1).argmax())
        fast = [int(t) for t in eng.decode_greedy(first, 200, seq=1)]
        eng.prefill(p, seq=1)
        slow, t = [], first
        for _ in range(200):
            t = int(eng.decode_next(t, seq=1).argmax())
            slow.append(t)
        assert fast == slow and eng.seq_len_of(1) == 233


def test_errors_are_statuses(zq):
    from zignn_b200 import _lib
    eng = zq.Lenisun(make_host("attention_only"), ctx=20, n_seq=2)

    def status(call):
        with pytest.raises(_lib.ZqError) as e:
            call()
        return e.value.status
    eng.extend([1] * 18)
    assert status(lambda: eng.extend([1] * 3)) == 6  # beyond the context
    assert status(lambda: eng.extend([])) == 6
    assert status(lambda: eng.extend([130])) == 1    # no such token
    assert status(lambda: eng.extend([1, 2], [1, 0])) == 1
    assert status(lambda: eng.extend([1, 2], [2])) == 1
    assert status(lambda: eng.extend([1], seq=2)) == 1
    assert status(lambda: eng.decode_next_batch([1, 1], [3, 4])) == 1
    eng.extend([1, 2])
    assert status(lambda: eng.decode_next(1)) == 6
    assert status(lambda: eng.decode_greedy(1, 1)) == 6
    assert eng.seq_len == 20 and eng.seq_len_of(1) == 0
    eng.reset_cache()
    assert eng.seq_len == 0
    uneven = model(40, 32, 1e-6, 1.0, [("attention", att(2, 2, 8, 8, 0.3, v_mix=True), None),
                                       ("attention", att(4, 1, 8, 16, 0.3, v_mix=True), None)])
    assert status(lambda: zq.Lenisun(hostmodel.LenisunHost.synthetic(uneven), ctx=20)) == 2  # values that cannot be mixed
    host = hostmodel.LenisunHost.synthetic(MODELS["mixed"], decay_rank=6)
    host.tensors["l2.mix.o"] = host.tensors["l1.mix.o"]
    with pytest.raises(_lib.ZqError):
        zq.Lenisun(host, ctx=20)


def test_programs(zq, tmp_path):
    """The command lines: a replayed trace gives the engine's logits, generation its tokens."""
    import json
    from zignn_b200 import generate
    name = "mixed"
    host = make_host(name)
    host.save(str(tmp_path / "m"))
    (tmp_path / "out").mkdir()
    a, b = prompt(name, 40, seed=3), prompt(name, 12, seed=4)
    steps = [dict(step=0, entries=[dict(id="a", tokens=a[:30], want=[0, 29])], end=[]),
             dict(step=1, entries=[dict(id="b", tokens=b, want=[])], end=["b"]),
             dict(step=2, entries=[dict(id="a", tokens=a[30:39], want=[8, 2])], end=[]),
             dict(step=3, entries=[dict(id="a", tokens=a[39:], want=[0])], end=["a"]),
             dict(step=4, entries=[dict(id="c", tokens=b, want=[11])], end=["c"])]
    r = subprocess.run([os.path.join(REPO, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", "float32", "--out",
                        str(tmp_path / "out"), "--max-tokens", "60"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done %d" % i for i in range(5)]
    V = MODELS[name]["vocab"]
    got = {i: np.fromfile(str(tmp_path / "out" / ("%d.f32" % i)), "<f4").reshape(-1, V) for i in (0, 2, 3, 4)}
    assert not (tmp_path / "out" / "1.f32").exists()
    wa, wb = plain_logits(name, a)[0], plain_logits(name, b)[0]
    for i, rows in ((0, wa[[0, 29]]), (2, wa[[38, 32]]), (3, wa[[39]]), (4, wb[[11]])):
        assert row_err(torch.tensor(got[i]), rows).max() <= TOL["float32"]
    r = subprocess.run([os.path.join(REPO, "bin", "generate"), "--model", str(tmp_path / "m"), "--prompt",
                        ",".join(str(t) for t in b), "-n", "6", "--dtype", "float32"], capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    eng = zq.Lenisun(host, ctx=40, dtype="float32")
    assert r.stdout.strip() == ",".join(str(t) for t in generate.generate(eng, b, 6))
