"""Vepinex on the GPU against the plain implementation (oracle/vepinex.py): each mechanism alone, whole models, and the
ways a sequence can be cut, batched and moved between slots."""
import json
import os
import subprocess

import numpy as np
import pytest
import torch

import vepinex as plain
from zignn_b200 import hostmodel, safetensors

pytestmark = pytest.mark.gpu

REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
PRECISIONS = [True, False]  # f32, bf16


def bf16(a):
    """Values a bf16 matrix can hold, as f64, and their bits."""
    bits = safetensors.f32_to_bf16(np.asarray(a, np.float32)).reshape(np.shape(a))
    return safetensors.bf16_to_f32(bits).reshape(np.shape(a)).astype(np.float64), bits


def close(got, want, tol, what=""):
    got = got.detach().float().cpu().numpy() if isinstance(got, torch.Tensor) else np.asarray(got)
    want = np.asarray(want)
    assert got.shape == want.shape, (got.shape, want.shape)
    err = np.abs(got.astype(np.float64) - want).max() / max(1e-30, np.abs(want).max())
    assert err <= tol, "%s: %g > %g" % (what, err, tol)


def dev(a):
    return torch.tensor(np.asarray(a, np.float32), device="cuda").contiguous()


# ------------------------------------------------------------------------------------------------ matrix memory
def memory_case(rng, T, H, d, e):
    """Queries and keys of a head have the same signs, or opposite ones: n . q stays away from 0, around which o (a quotient,
    then normed) would turn on the last bit."""
    x = rng.standard_normal((T, 2 * H * (d + e + 1))).astype(np.float32)
    x[:, -2 * H:] *= 3
    x[:, :2 * H * d] = np.abs(x[:, :2 * H * d]) + 0.1
    for h in range(0, H, 2):
        x[:, (H + h) * d:(H + h + 1) * d] *= -1
    ib, fb = rng.standard_normal(H).astype(np.float32), (2 + rng.standard_normal(H)).astype(np.float32)
    return x, ib, fb, rng.uniform(0.5, 1.5, H * e).astype(np.float32)


def memory_plain(x, H, d, e, cap, ib, fb, norm, eps, state=None):
    x = x.astype(np.float64)
    T, kd, vd = x.shape[0], H * d, H * e
    q, k = x[:, :kd].reshape(T, H, d) * d ** -0.5, x[:, kd:2 * kd].reshape(T, H, d)
    v, g = x[:, 2 * kd:2 * kd + vd].reshape(T, H, e), x[:, 2 * kd + vd:2 * (kd + vd)]
    i, f = plain.memory_gates(x[:, -2 * H:-H] + ib, x[:, -H:] + fb, cap)
    o, state = plain.memory_scan(q, k, v, i, f, state)
    return plain.rms_normalize(o, eps).reshape(T, vd) * norm * plain.sigmoid(g), state


def memory_state(rng, slots, H, d, e):
    S, n, m = (rng.standard_normal(s).astype(np.float32) for s in ((slots, H, d, e), (slots, H, d), (slots, H)))
    n = np.abs(n)
    n[:, ::2] *= -1
    return [S, n, m]


MEMORY_SHAPES = [(1, 8, 8), (3, 5, 7), (2, 20, 36), (2, 64, 40), (1, 72, 130), (2, 128, 64), (1, 200, 48), (1, 300, 20), (5, 16, 1)]


@pytest.mark.parametrize("f32", PRECISIONS)
@pytest.mark.parametrize("H,d,e", MEMORY_SHAPES)
def test_memory_portions_and_steps(zq, f32, H, d, e):
    rng = np.random.default_rng(1)
    T, cap, eps = 130, 4.0, 1e-5
    x, ib, fb, n = memory_case(rng, T, H, d, e)
    start = memory_state(rng, 2, H, d, e)
    want, end = memory_plain(x, H, d, e, cap, ib, fb, n, eps, tuple(s[1].astype(np.float64) for s in start))
    for cuts in ([T], [24, 106], [23, 2, 24, 81], [1, 1, 2, 3, 17, 33, 73]):
        state = [dev(s) for s in start]
        outs, t0 = [], 0
        for c in cuts:
            outs.append(zq.memory(dev(x[t0:t0 + c]), H, d, e, cap, dev(ib), dev(fb), dev(n), eps, state, [1], True, f32))
            t0 += c
        out = torch.cat(outs)
        close(out[:, :H * e], want, 3e-5 if f32 else 1.5e-2, str(cuts))
        assert not out[:, H * e:].any()
        for got, w, s in zip(state, end, start):
            close(got[1], w, 2e-5 if f32 else 2e-4, "state after %s" % cuts)
            assert torch.equal(got[0], dev(s[0]))


@pytest.mark.parametrize("f32", PRECISIONS)
def test_memory_of_several_sequences_at_once(zq, f32):
    rng = np.random.default_rng(2)
    H, d, e, cap, slots = 3, 24, 20, 6.0, [3, 0, 2]
    x, ib, fb, n = memory_case(rng, 3, H, d, e)
    start = memory_state(rng, 4, H, d, e)
    state = [dev(s) for s in start]
    out = zq.memory(dev(x), H, d, e, cap, dev(ib), dev(fb), dev(n), 1e-6, state, slots, False, f32)
    for r, s in enumerate(slots):
        want, end = memory_plain(x[r:r + 1], H, d, e, cap, ib, fb, n, 1e-6, tuple(a[s].astype(np.float64) for a in start))
        close(out[r:r + 1, :H * e], want, 3e-5 if f32 else 5e-3)
        for got, w in zip(state, end):
            close(got[s], w, 1e-5)
    for got, s in zip(state, start):
        assert torch.equal(got[1], dev(s[1]))


@pytest.mark.parametrize("f32", PRECISIONS)
def test_memory_keeps_what_a_strong_gate_wrote(zq, f32):
    """Only one token's input gate is open: hundreds of tokens later its value is still what is read (if the forget gates
    were open), at chunk borders and at a portion's first and last token. The first tokens' gates are so low that only the
    running maximum's start at zero keeps them small."""
    rng = np.random.default_rng(3)
    H, d, e, T, cap = 1, 16, 8, 200, 14.0
    for place in (0, 1, 15, 16, 31, 32, 99, 100, 101, 199):
        x = rng.standard_normal((T, 2 * H * (d + e + 1))).astype(np.float32)
        x[:, :2 * d] = np.abs(x[:, :2 * d]) + 0.1
        x[:, -2], x[:, -1] = -60.0, 60.0
        x[place, -2] = 8.0
        want, _ = memory_plain(x, H, d, e, cap, np.zeros(1), np.zeros(1), np.ones(e), 1e-9)
        state = [torch.zeros(1, H, d, e, device="cuda"), torch.zeros(1, H, d, device="cuda"), torch.zeros(1, H, device="cuda")]
        outs = [zq.memory(dev(x[a:b]), H, d, e, cap, dev(np.zeros(1)), dev(np.zeros(1)), dev(np.ones(e)), 1e-9, state, [0], True, f32)
                for a, b in ((0, 100), (100, 101), (101, 200))]
        close(torch.cat(outs)[:, :e], want, 1e-4 if f32 else 2e-2, "place %d" % place)


# ------------------------------------------------------------------------------------------------ delta rule
def delta_case(rng, T, H, G, d, e, taps, ra, rg):
    kd, vd = G * d, H * e
    x = rng.standard_normal((T, 2 * kd + vd + H + ra + rg)).astype(np.float32)
    x[:, 2 * kd + vd + H:] = bf16(x[:, 2 * kd + vd + H:])[0]  # a matrix product may round its inputs
    conv = rng.standard_normal((2 * kd + vd, taps)).astype(np.float32)
    A = rng.uniform(-3, 1, H).astype(np.float32)
    dt = rng.uniform(-3, 1, (H, d)).astype(np.float32)
    a2, a_bits = bf16(rng.standard_normal((H * d, ra)) * ra ** -0.5)
    g2, g_bits = bf16(rng.standard_normal((vd, rg)) * rg ** -0.5)
    low = np.zeros((H * d + vd, max(ra, rg)), np.uint16)
    low[:H * d, :ra], low[H * d:, :rg] = a_bits, g_bits
    return x, conv, A, dt, a2, g2, low, rng.uniform(0.5, 1.5, e).astype(np.float32)


def delta_plain(x, H, G, d, e, taps, ra, conv, A, dt, a2, g2, norm, eps, S=None, before=None):
    x = x.astype(np.float64)
    T, kd, vd = x.shape[0], G * d, H * e
    c = 2 * kd + vd
    y = plain.silu(plain.short_conv(x[:, :c], conv.astype(np.float64), before))
    q, k = plain.unit(y[:, :kd].reshape(T, G, d)) * d ** -0.5, plain.unit(y[:, kd:2 * kd].reshape(T, G, d))
    low = x[:, c + H:]
    g = plain.channel_decay((low[:, :ra] @ a2.T).reshape(T, H, d), A.astype(np.float64), dt.astype(np.float64))
    o, S = plain.delta_scan(q, k, y[:, 2 * kd:].reshape(T, H, e), g, plain.sigmoid(x[:, c:c + H]), S)
    return (plain.rms_normalize(o, eps) * norm).reshape(T, vd) * plain.sigmoid(low[:, ra:] @ g2.T), S


def ring_of(inputs, pos, taps, slots, slot, rng):
    """The convolution inputs [.., channels] of the tokens ahead of position pos in their places; the rest is noise."""
    ring = rng.standard_normal((slots, taps, inputs.shape[1])).astype(np.float32)
    for p in range(max(0, pos - taps + 1), pos):
        ring[slot, p % taps] = inputs[p - pos]
    return ring


DELTA_SHAPES = [  # heads, key heads, dim, vdim, taps, ranks
    (2, 2, 16, 8, 4, 8, 8), (4, 2, 20, 12, 4, 5, 9), (3, 1, 7, 5, 3, 6, 1), (2, 1, 64, 40, 2, 16, 24), (1, 1, 130, 36, 4, 70, 3),
    (2, 2, 96, 64, 1, 8, 8), (1, 1, 260, 16, 4, 4, 4), (6, 3, 32, 3, 6, 2, 130)]


@pytest.mark.parametrize("f32", PRECISIONS)
@pytest.mark.parametrize("shape", DELTA_SHAPES)
def test_delta_portions_and_steps(zq, f32, shape):
    H, G, d, e, taps, ra, rg = shape
    rng = np.random.default_rng(4)
    T, eps, pos0 = 110, 1e-5, 9
    x, conv, A, dt, a2, g2, low, n = delta_case(rng, T + taps, H, G, d, e, taps, ra, rg)
    ch = conv.shape[0]
    ahead, x = x[:taps, :ch], x[taps:]  # inputs of the tokens ahead of the portion
    start = rng.standard_normal((2, H, d, e)).astype(np.float32)
    want, S = delta_plain(x, H, G, d, e, taps, ra, conv, A, dt, a2, g2, n, eps, start[1].astype(np.float64),
                          ahead[taps - (taps - 1):].astype(np.float64) if taps > 1 else ahead[:0].astype(np.float64))
    W = zq.DenseWeight(low)
    for cuts in ([T], [24, 86], [1, 2, 1, 23, 2, 3, 25, 1, 52]):
        state, ring = dev(start), dev(ring_of(ahead, pos0, taps, 2, 1, rng))
        outs, t0 = [], 0
        for c in cuts:
            outs.append(zq.delta(dev(x[t0:t0 + c]), H, G, d, e, taps, ra, rg, dev(conv), dev(A), dev(dt), W, dev(n), eps, state, ring,
                                 np.arange(pos0 + t0, pos0 + t0 + c), [1] * c, True, f32))
            t0 += c
        out = torch.cat(outs)
        close(out[:, :H * e], want, 3e-5 if f32 else 1.5e-2, str(cuts))
        assert not out[:, H * e:].any()
        close(state[1], S, 2e-5 if f32 else 3e-4, "state after %s" % cuts)
        assert torch.equal(state[0], dev(start[0]))


@pytest.mark.parametrize("f32", PRECISIONS)
def test_delta_of_several_sequences_at_once(zq, f32):
    rng = np.random.default_rng(5)
    H, G, d, e, taps, ra, rg, slots, poss = 4, 2, 24, 20, 4, 7, 5, [3, 0, 2], [17, 0, 2]
    x, conv, A, dt, a2, g2, low, n = delta_case(rng, 3, H, G, d, e, taps, ra, rg)
    before = rng.standard_normal((4, taps - 1, conv.shape[0])).astype(np.float32)
    start = rng.standard_normal((4, H, d, e)).astype(np.float32)
    ring = rng.standard_normal((4, taps, conv.shape[0])).astype(np.float32)
    for s, p in zip(slots, poss):
        ring[s] = ring_of(before[s], p, taps, 1, 0, rng)[0]
        before[s][:max(0, taps - 1 - p)] = 0  # nothing ahead of the first token, whatever the ring holds there
    state, dring = dev(start), dev(ring)
    out = zq.delta(dev(x), H, G, d, e, taps, ra, rg, dev(conv), dev(A), dev(dt), zq.DenseWeight(low), dev(n), 1e-6, state, dring, poss,
                   slots, False, f32)
    for r, s in enumerate(slots):
        want, S = delta_plain(x[r:r + 1], H, G, d, e, taps, ra, conv, A, dt, a2, g2, n, 1e-6, start[s].astype(np.float64),
                              before[s].astype(np.float64))
        close(out[r:r + 1, :H * e], want, 3e-5 if f32 else 5e-3)
        close(state[s], S, 1e-5)
        assert torch.equal(dring[s, poss[r] % taps], dev(x[r, :conv.shape[0]]))
    assert torch.equal(state[1], dev(start[1])) and torch.equal(dring[1], dev(ring[1]))


@pytest.mark.parametrize("f32", PRECISIONS)
def test_delta_replaces_what_a_key_held(zq, f32):
    """Without decay, the same key written with beta = 1 answers with its last value alone, however often it was written
    and whether the writes share a chunk; with full decay in half of the key channels only the other half is left."""
    rng = np.random.default_rng(6)
    H, d, e, T, r = 1, 16, 8, 90, 1
    conv = np.ones((2 * d + e, 1), np.float32)
    low = np.zeros((d + e, r), np.uint16)
    key = np.zeros(d, np.float32)
    key[[3, 11]] = 20.0
    other = np.zeros(d, np.float32)
    other[5] = 20.0
    for writes in ((0, 1), (14, 15), (15, 16), (3, 30), (29, 30), (30, 31), (64, 65)):
        for decayed in (False, True):
            x = np.zeros((T, 2 * d + e + H + 2 * r), np.float32)
            x[:, d:2 * d] = other
            x[:, :d] = key
            x[:, 2 * d + e] = -40.0                                    # beta = 0: nothing is written
            for w in writes:
                x[w, d:2 * d], x[w, 2 * d + e] = key, 40.0
                x[w, 2 * d:2 * d + e] = rng.uniform(1, 3, e)
            dt = np.full((H, d), -60.0, np.float32)
            if decayed:
                dt[0, 11] = 60.0
            args = (conv, np.zeros(1, np.float32), dt, np.zeros((d, r)), np.zeros((e, r)), np.ones(e, np.float32))
            want, S = delta_plain(x, H, 1, d, e, 1, r, *args, 1e-9)
            state = torch.zeros(1, H, d, e, device="cuda")
            ring = torch.zeros(1, 1, 2 * d + e, device="cuda")
            outs = [zq.delta(dev(x[a:b]), H, 1, d, e, 1, r, r, dev(conv), dev(np.zeros(1)), dev(dt), zq.DenseWeight(low), dev(np.ones(e)),
                             1e-9, state, ring, np.arange(a, b), [0] * (b - a), True, f32) for a, b in ((0, 30), (30, 31), (31, T))]
            close(torch.cat(outs)[:, :e], want, 1e-4 if f32 else 1e-2, "%s %s" % (writes, decayed))
            close(state[0], S, 1e-5 if f32 else 2e-4)
            v = plain.silu(x[writes[1], 2 * d:2 * d + e].astype(np.float64))
            if not decayed:
                read = np.einsum("ij,i->j", S[0], key / np.sqrt((key * key).sum()))
                assert np.allclose(read, v, rtol=1e-4)  # the last value alone
            else:
                assert abs(S[0][11]).max() < 1e-6


def test_delta_convolution_meets_the_right_tokens(zq):
    """An impulse in one token reaches exactly the next taps - 1 tokens, over every border."""
    H, d, e, taps, T, r = 1, 4, 4, 4, 70, 1
    conv = np.zeros((2 * d + e, taps), np.float32)
    conv[:2 * d, -1] = 1.0
    conv[2 * d:] = [1.0, 2.0, 4.0, 8.0]
    low = np.zeros((d + e, r), np.uint16)
    for place in (0, 1, 15, 16, 28, 29, 30, 31, 32, 33, 40, 66, 69):
        x = np.zeros((T, 2 * d + e + H + 2), np.float32)
        x[:, :2 * d] = 1.0
        x[place, 2 * d:2 * d + e] = 1.0
        x[:, 2 * d + e] = 40.0
        args = (conv, np.zeros(1, np.float32), np.full((H, d), 60.0, np.float32), np.zeros((d, r)), np.zeros((e, r)),
                np.ones(e, np.float32))
        want, _ = delta_plain(x, H, 1, d, e, taps, r, *args, 1.0)  # (a large epsilon keeps the sizes apart)
        assert (np.abs(want).max(axis=1) > 1e-3).sum() == min(taps, T - place)
        for f32 in PRECISIONS:
            state, ring = torch.zeros(1, H, d, e, device="cuda"), torch.full((1, taps, 2 * d + e), 7.0, device="cuda")
            outs = [zq.delta(dev(x[a:b]), H, 1, d, e, taps, r, r, dev(conv), dev(args[1]), dev(args[2]), zq.DenseWeight(low),
                             dev(args[5]), 1.0, state, ring, np.arange(a, b), [0] * (b - a), True, f32)
                    for a, b in ((0, 30), (30, 32), (32, 33), (33, T))]
            close(torch.cat(outs)[:, :e], want, 2e-5 if f32 else 1e-2, "place %d" % place)


# ------------------------------------------------------------------------------------------------ latent attention
LATENT_SHAPES = [  # heads, dim, rot, vdim, rank
    (1, 8, 4, 8, 16), (3, 20, 6, 28, 40), (4, 64, 32, 64, 128), (5, 12, 2, 7, 9), (17, 16, 16, 24, 72), (2, 200, 56, 256, 300),
    (2, 240, 64, 32, 64), (20, 32, 64, 16, 520), (2, 16, 8, 300, 32), (1, 64, 64, 64, 1000)]


def rotations(rot, base):
    return base ** (-np.arange(0, rot, 2) / rot)


def latent_setup(zq, rng, shape, ctx, n_slots, f32, scale, base=5000.0):
    H, d, r, e, R = shape
    c = zq.LatentCache(H, d, r, e, R, ctx, scale, dev(rotations(r, base)), 1e-5, n_slots, f32)
    uk, uk_bits = bf16(rng.standard_normal((H * d, R)) * R ** -0.5)
    uv, uv_bits = bf16(rng.standard_normal((H * e, R)) * R ** -0.5)
    return c, uk, uv, zq.DenseWeight(np.concatenate([uk_bits, uv_bits]))


def latent_plain(x, shape, norm, base, scale, uk, uv, pos):
    """Queries of the last len(pos) rows over all rows of x (positions from 0 on)."""
    H, d, r, e, R = shape
    x, T = x.astype(np.float64), x.shape[0]
    m = dict(heads=H, dim=d, vdim=e, scale=scale)
    q = x[-len(pos):, :H * (d + r)].reshape(len(pos), H, d + r).copy()
    q[..., d:] = plain.rotate(q[..., d:], pos, base)
    y = x[:, H * (d + r):]
    c, kr = plain.norm(y[:, :R], norm.astype(np.float64), 1e-5), plain.rotate(y[:, R:], np.arange(T), base)
    return plain.latent_attention(q, c, kr, uk, uv, m, pos).reshape(len(pos), H * e), c, kr


@pytest.mark.parametrize("f32", PRECISIONS)
@pytest.mark.parametrize("shape", LATENT_SHAPES)
def test_latent_attention_portions_and_steps(zq, f32, shape):
    H, d, r, e, R = shape
    rng = np.random.default_rng(7)
    T, ctx, scale, base = 300, 310, (d + r) ** -0.5, 5000.0
    x = rng.standard_normal((T, H * (d + r) + R + r)).astype(np.float32)
    norm = rng.uniform(0.5, 1.5, R).astype(np.float32)
    tol = 2e-5 if f32 else 1.5e-2
    c, uk, uv, up = latent_setup(zq, rng, shape, ctx, 2, f32, scale, base)
    want, lat, kr = latent_plain(x, shape, norm, base, scale, uk, uv, np.arange(T))
    for cuts in ([T], [1, 2, 32, 33, 31, 1, 64, 136]):
        c.rows.zero_()
        outs, t0 = [], 0
        for n in cuts:
            outs.append(c.attend(dev(x[t0:t0 + n]), dev(norm), up, np.arange(t0, t0 + n), [1] * n, True))
            t0 += n
        out = torch.cat(outs)
        close(out[:, :H * e], want, tol, str(cuts))
        assert not out[:, H * e:].any() and not c.rows[0].any() and not c.rows[1, T:].any()
        close(c.rows[1, :T, :R], lat, 3e-6 if f32 else 5e-3)
        close(c.rows[1, :T, R:R + r], kr, 3e-5 if f32 else 5e-3)  # (angles are 32-bit products)
        assert not c.rows[1, :, R + r:].any()
    # a layer that reads the same cache with its own queries and its own W_uk, W_uv
    other, uk2, uv2, up2 = latent_setup(zq, rng, shape, ctx, 2, f32, scale, base)
    other.rows = c.rows
    y = rng.standard_normal((T, H * (d + r))).astype(np.float32)
    want, _, _ = latent_plain(np.concatenate([y, x[:, H * (d + r):]], axis=1), shape, norm, base, scale, uk2, uv2, np.arange(T))
    kept = c.rows.clone()
    for pos in (np.arange(T), np.arange(290, 300), np.array([299])):
        out = other.attend(dev(y[pos]), None, up2, pos, [1] * len(pos), True)
        close(out[:, :H * e], want[pos], tol, "shared cache, %d rows" % len(pos))
    assert torch.equal(c.rows, kept)


@pytest.mark.parametrize("f32", PRECISIONS)
def test_latent_attention_of_several_sequences(zq, f32):
    rng = np.random.default_rng(8)
    shape = (6, 24, 8, 20, 48)
    H, d, r, e, R = shape
    lens, slots, ctx, scale, base = [1, 64, 65, 500, 1000, 2], [4, 0, 5, 1, 3, 2], 1000, 0.2, 10000.0
    c, uk, uv, up = latent_setup(zq, rng, shape, ctx, 6, f32, scale, base)
    norm = rng.uniform(0.5, 1.5, R).astype(np.float32)
    xs = [rng.standard_normal((n, H * (d + r) + R + r)).astype(np.float32) for n in lens]
    for x, s in zip(xs, slots):
        if len(x) > 1:
            c.attend(dev(x[:-1]), dev(norm), up, np.arange(len(x) - 1), [s] * (len(x) - 1), True)
    out = c.attend(dev(np.stack([x[-1] for x in xs])), dev(norm), up, [n - 1 for n in lens], slots, False)
    for i, x in enumerate(xs):
        want, _, _ = latent_plain(x, shape, norm, base, scale, uk, uv, np.array([len(x) - 1]))
        close(out[i:i + 1, :H * e], want, 2e-5 if f32 else 1.5e-2, "length %d" % lens[i])


@pytest.mark.parametrize("f32", PRECISIONS)
@pytest.mark.parametrize("shape", [(4, 16, 8, 12, 32), (2, 24, 40, 16, 48)])
def test_latent_attention_finds_one_key_among_many(zq, f32, shape):
    """One token's latent (or its rotated key part alone) answers the query by far; it is put at tile and range borders, at
    the first token, at the row's own place and one place behind it, where it must not be seen."""
    rng = np.random.default_rng(9)
    H, d, r, e, R = shape
    ctx, base, scale = 1300, 10000.0, 1.0
    c, uk, uv, up = latent_setup(zq, rng, shape, ctx, 1, f32, scale, base)
    norm = np.ones(R, np.float32)
    for by_rotation in (False, True):
        for last in (63, 64, 65, 255, 1299):
            x = (0.1 * rng.standard_normal((last + 2, H * (d + r) + R + r))).astype(np.float32)
            x[:, :H * (d + r)] *= 5
            mark = rng.standard_normal(R).astype(np.float32)
            for place in sorted({0, 1, 62, 63, 64, 127, 128, last - 1, last, last + 1}):
                if place > last + 1 or place >= ctx:
                    continue
                y = x[:last + 2].copy()
                at = H * (d + r)
                qrow = y[last, :at].reshape(H, d + r)
                qrow[:] = 0
                if by_rotation:  # query part and key part meet after both were turned to their places
                    key = rng.standard_normal(r)
                    y[place, at + R:] = key * 4
                    qrow[:, d:] = plain.rotate(plain.rotate(key[None], [place], base), [-last], base)[0] * 6 / r ** 0.5
                else:
                    y[place, at:at + R] = mark
                    lat = plain.rms_normalize(mark.astype(np.float64)[None], 1e-5)[0]
                    qrow[:, :d] = (uk @ lat).reshape(H, d) * 40 / (np.linalg.norm((uk @ lat).reshape(H, d), axis=1, keepdims=True) ** 2)
                n = last + 1
                want, _, _ = latent_plain(y[:n], shape, norm, base, scale, uk, uv, np.arange(n))
                for T in (1, 2, 40):
                    if T > n:
                        continue
                    c.rows.zero_()
                    every = y[:last + 2] if place <= last else np.concatenate([y[:n], y[n:]])
                    if place > last and last + 1 < ctx:  # the token behind lies in the cache already
                        c.attend(dev(every), dev(norm), up, np.arange(len(every)), [0] * len(every), True)
                    elif n - T > 0:
                        c.attend(dev(y[:n - T]), dev(norm), up, np.arange(n - T), [0] * (n - T), True)
                    out = c.attend(dev(y[n - T:n]), dev(norm), up, np.arange(n - T, n), [0] * T, True)
                    close(out[:, :H * e], want[-T:], 1e-4 if f32 else 2.5e-2, "place %d, row %d, T %d" % (place, last, T))


# ------------------------------------------------------------------------------------------------ routing, units
def test_route_with_bias_and_softmax(zq):
    rng = np.random.default_rng(10)
    for experts, top, stride in ((5, 2, 6), (16, 1, 16), (64, 8, 65), (300, 7, 300), (3, 3, 4)):
        z = rng.standard_normal((33, stride)).astype(np.float32) * 3
        z[:, experts:] = 100.0  # not a router logit
        bias = rng.standard_normal(experts).astype(np.float32)
        ids, w = zq.route(dev(z), experts, top, dev(bias), zq.ROUTE_SOFTMAX)
        want, ww = plain.route(z[:, :experts].astype(np.float64) + bias, top)
        assert np.array_equal(ids.cpu().numpy(), want)
        close(w, ww, 2e-6)


# ------------------------------------------------------------------------------------------------ models
def memory(heads, dim, vdim, cap):
    return "mlstm", dict(heads=heads, dim=dim, vdim=vdim, gate_cap=cap)


def delta(heads, kv, dim, vdim, conv):
    return "channel_delta", dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, conv=conv)


def latent(heads, dim, rot, vdim, rank, scale, base, kv_from=None):
    m = dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=rank, scale=scale, rot=dict(base=base, dims=rot))
    return "latent_attention", m if kv_from is None else dict(m, kv_from=kv_from)


def moe(experts, top, ff, limit, shared=None):
    m = dict(kind="moe", router=dict(experts=experts, top=top), expert=dict(ff=ff, limit=limit))
    if shared:
        m["shared"] = dict(ff=shared[0], limit=shared[1])
    return m


def dense(ff):
    return dict(kind="dense", ff=ff)


def model(vocab, width, eps, *layers):
    return dict(architecture="Vepinex", vocab=vocab, width=width, norm=dict(eps=eps),
                layers=[dict(type=t, mixer=m, mlp=f) for (t, m), f in layers])


MODELS = {
    # every branch: feed-forward parts of each kind and none, caches shared by one and by two layers, ragged sizes
    "mixed": model(211, 104, 1e-5,
                   (latent(3, 20, 6, 28, 40, 0.2, 3000.0), moe(7, 3, 40, 0.8, (72, 2.0))),
                   (delta(4, 2, 12, 20, 3), dense(90)),
                   (memory(3, 20, 28, 7.0), moe(6, 1, 24, 1.2)),
                   (latent(5, 8, 6, 12, 40, 0.4, 3000.0, 0), None),
                   (delta(2, 2, 36, 8, 5), moe(9, 4, 32, 1.0, (40, 0.5))),
                   (latent(2, 16, 4, 8, 24, 0.3, 500.0), dense(64)),
                   (latent(1, 24, 6, 20, 40, 0.3, 3000.0, 0), moe(4, 4, 16, 3.0))),
    "recurrences": model(130, 70, 1e-6,
                         (memory(1, 40, 24, 20.0), None),
                         (memory(6, 8, 8, 3.0), moe(5, 2, 16, 1.5, (24, 1.5))),
                         (delta(3, 1, 24, 16, 2), dense(70)),
                         (delta(1, 1, 72, 48, 1), moe(3, 1, 32, 0.7))),
    "latents": model(96, 64, 1e-4,
                     (latent(4, 16, 16, 16, 64, 0.18, 10000.0), dense(128)),
                     (latent(2, 32, 16, 32, 64, 0.15, 10000.0, 0), moe(12, 5, 32, 1.0, (32, 1.0)))),
}


def make_host(name, seed=1, a_rank=6, g_rank=10):
    """Random weights of a size that makes every part count. The router reads channels that only the token itself sets,
    far apart from each other, so that rounding does not change who is chosen; one expert's bias puts it always among
    the chosen ones, another's never."""
    cfg = MODELS[name]
    host = hostmodel.VepinexHost.synthetic(cfg, seed=seed, std=0.25, a_rank=a_rank, g_rank=g_rank)
    rng = np.random.default_rng(seed)
    f = {k: t.f32().copy() for k, t in host.tensors.items()}
    n_max = max([l["mlp"]["router"]["experts"] for l in cfg["layers"] if l["mlp"] and l["mlp"]["kind"] == "moe"] + [1])
    f["embed"] *= 4
    f["embed"][:, :n_max] = np.stack([rng.permutation(n_max) for _ in range(cfg["vocab"])]) * (24.0 / n_max) - 12.0
    for k in f:
        leaf = k.split(".")[-1]
        if leaf in ("o", "down"):
            f[k][:n_max] = 0.0  # nothing is added to the routing channels
        if leaf in ("norm", "norm1") and f[k].shape[0] == cfg["width"] and ".mix." not in k:
            f[k][:n_max] = 1.0
        if leaf == "router":
            f[k][:] = 0.0
            f[k][:, :f[k].shape[0]] = 0.4 * np.eye(f[k].shape[0])
            b = np.zeros(f[k].shape[0], np.float32)
            if len(b) > 2:
                b[0], b[1] = 3.0, -3.0
            f[k + ".b"][:] = b
        if leaf == "i" and ".mix." in k:
            f[k] *= 2
    host.tensors = {k: safetensors.Tensor("BF16", safetensors.f32_to_bf16(v).reshape(v.shape)) for k, v in f.items()}
    return host


_PLAIN = {}


def plain_logits(name, tokens):
    key = (name, tuple(tokens))
    if key not in _PLAIN:
        weights = {k: v.astype(np.float64) for k, v in make_host(name).as_f32().items()}
        _PLAIN[key] = plain.forward(MODELS[name], weights, tokens)
    return _PLAIN[key]


def prompt(name, n, seed=2):
    return [int(t) for t in np.random.default_rng(seed).integers(0, MODELS[name]["vocab"], n)]


def row_err(got, want):
    """Per position: root mean square of the difference over that of the wanted values."""
    got, want = got.float().cpu().numpy().astype(np.float64), np.asarray(want, np.float64)
    return np.sqrt(((got - want) ** 2).mean(axis=1)) / np.sqrt((want ** 2).mean())


TOL = {"float32": 3e-5, "bfloat16": 4e-2}


def agree(got, want, dtype, what=""):
    """Every position in 32-bit. In bf16 a head's o that happens to be small is blown up by its norm, rounding with it: a few
    positions may be further off."""
    e = np.sort(row_err(got, want))
    most = e[int(0.95 * (len(e) - 1))] if dtype == "bfloat16" else e[-1]
    assert most <= TOL[dtype] and e[-1] <= 6 * TOL[dtype], "%s: %g, %g" % (what, most, e[-1])


DTYPES = ["float32", "bfloat16"]


def run(engine, tokens, cuts, seq=0):
    out, t0 = [], 0
    for c in cuts:
        out.append(engine.extend(tokens[t0:t0 + c], range(c), seq=seq))
        t0 += c
    assert t0 == len(tokens)
    return torch.cat(out)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(MODELS))
def test_model_whole_prompt_layer_by_layer(zq, name, dtype):
    tokens = prompt(name, 200)
    want, trail = plain_logits(name, tokens)
    eng = zq.Vepinex(make_host(name), ctx=256, n_seq=2, dtype=dtype)
    got = eng.extend_with_trail(tokens, seq=1)
    for l in range(len(trail)):
        agree(got[l], trail[l], dtype, "layer %d" % l)
    eng.reset(1)
    agree(eng.extend(tokens, range(200), seq=1), want, dtype)
    eng.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(MODELS))
def test_model_cuts_do_not_matter(zq, name, dtype):
    tokens = prompt(name, 200)
    want, _ = plain_logits(name, tokens)
    eng = zq.Vepinex(make_host(name), ctx=200, n_seq=1, dtype=dtype)
    whole = run(eng, tokens, [200])
    for cuts in ([1] * 200, [2] * 100, [3, 5, 8, 9, 64, 65, 2, 44], [199, 1], [1, 64, 128, 2, 5],
                 [33, 16, 15, 17, 34, 24, 23, 38], [7] * 28 + [4]):
        eng.reset()
        got = run(eng, tokens, cuts)
        agree(got, want, dtype, cuts[:4])
        agree(got, whole.cpu().numpy(), dtype, cuts[:4])
    eng.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["latents", "recurrences"])
def test_prompts_longer_than_one_piece(zq, name, dtype):
    """More tokens in one call than the activation buffers hold: the engine cuts them itself."""
    tokens = prompt(name, 2200, seed=11)
    want, _ = plain_logits(name, tokens)
    eng = zq.Vepinex(make_host(name), ctx=2200, dtype=dtype)
    places = [0, 1, 63, 64, 1000, 2046, 2047, 2048, 2049, 2198, 2199]
    assert row_err(eng.extend(tokens, places), want[places]).max() <= TOL[dtype]
    eng.reset()
    eng.extend(tokens[:2049])  # a piece and one token
    assert row_err(eng.extend(tokens[2049:], [0, 150]), want[[2049, 2199]]).max() <= TOL[dtype]
    assert row_err(eng.prefill(tokens)[None], want[[2199]]).max() <= TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_batched_sequences_equal_each_alone(zq, dtype):
    name, n_seq, steps = "mixed", 11, 9
    host = make_host(name)
    eng = zq.Vepinex(host, ctx=120, n_seq=n_seq, dtype=dtype)
    alone = zq.Vepinex(host, ctx=120, n_seq=1, dtype=dtype)
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
            assert e <= TOL[dtype], (i, s, e)
            at[i] += 1
            assert eng.seq_len_of(i) == lens[i] + at[i]
    eng.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "recurrences"])
def test_slots_used_again(zq, name, dtype):
    """A slot that held another sequence gives the same bits as a new one, whichever slot it is."""
    host = make_host(name)
    eng = zq.Vepinex(host, ctx=150, n_seq=3, dtype=dtype)
    tokens = prompt(name, 90, seed=7)
    cuts = [50, 2, 9, 1, 28]
    first = run(eng, tokens, cuts, seq=eng.acquire())
    short = run(eng, tokens[:3], [1, 2], seq=eng.acquire())
    eng.release(1)
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
        assert torch.equal(run(eng, tokens[:3], [1, 2], seq=eng.acquire()), short)
        eng.release(again)
        eng.release(seqs[1])


def test_long_decoding(zq):
    name = "mixed"
    tokens = prompt(name, 420, seed=9)
    want, _ = plain_logits(name, tokens)
    for dtype in DTYPES:
        eng = zq.Vepinex(make_host(name), ctx=420, dtype=dtype)
        eng.extend(tokens[:20])
        got = torch.cat([eng.extend([t], [0]) for t in tokens[20:]])
        agree(got, want[20:], dtype)


def test_greedy_generation_and_scheduler(zq):
    from zignn_b200 import generate
    name = "mixed"
    host = make_host(name)
    weights = {k: v.astype(np.float64) for k, v in host.as_f32().items()}
    one = zq.Vepinex(host, ctx=100, dtype="float32")
    prompts = [prompt(name, n, seed=60 + n) for n in (1, 2, 30, 41, 5, 17, 9)]
    counts = [12, 1, 20, 7, 25, 3, 15]
    want = []
    for p, n in zip(prompts, counts):
        toks = generate.generate(one, p, n)
        # each token is the plain implementation's arg-max after what came before it
        lg = plain.forward(MODELS[name], weights, p + toks[:-1])[0][len(p) - 1:]
        assert [int(t) for t in lg.argmax(axis=1)] == toks
        want.append(toks)
    eng = zq.Vepinex(host, ctx=100, n_seq=3, dtype="float32")
    for portion in (0, 2, 16):
        done = generate.serve(eng, [generate.Request(p, n) for p, n in zip(prompts, counts)], portion)
        assert [r.tokens for r in done] == want
    assert generate.generate(one, prompts[2], 8, top_k=1, temperature=0.7, rng=np.random.default_rng(0)) == want[2][:8]


def test_decode_greedy_equals_step_by_step(zq):
    for dtype in DTYPES:
        eng = zq.Vepinex(make_host("mixed"), ctx=300, n_seq=2, dtype=dtype)
        p = prompt("mixed", 33)
        first = int(eng.prefill(p, seq=1).argmax())
        fast = [int(t) for t in eng.decode_greedy(first, 120, seq=1)]
        eng.prefill(p, seq=1)
        slow, t = [], first
        for _ in range(120):
            t = int(eng.decode_next(t, seq=1).argmax())
            slow.append(t)
        assert fast == slow and eng.seq_len_of(1) == 153


def test_what_does_not_fit_is_refused(zq):
    from zignn_b200 import _lib

    def refused(cfg, change=None):
        host = hostmodel.VepinexHost.synthetic(cfg)
        if change:
            change(host.tensors)
        with pytest.raises((_lib.ZqError, ValueError, KeyError)):
            zq.Vepinex(host, ctx=20)
    base = latent(2, 8, 4, 8, 16, 0.3, 100.0)
    refused(model(40, 32, 1e-6, (delta(2, 2, 8, 8, 2), None), (latent(2, 8, 4, 8, 16, 0.3, 100.0, 0), None)))  # no cache there
    refused(model(40, 32, 1e-6, (base, None), (latent(2, 8, 4, 8, 24, 0.3, 100.0, 0), None)))                 # another rank
    refused(model(40, 32, 1e-6, (base, None), (latent(2, 8, 4, 8, 16, 0.3, 100.0, 0), None),
                  (latent(2, 8, 4, 8, 16, 0.3, 100.0, 1), None)))                                              # a cache of none of its own
    refused(model(40, 32, 1e-6, (delta(3, 2, 8, 8, 2), None)))                                                # 3 heads on 2
    ok = model(40, 32, 1e-6, (memory(2, 8, 8, 5.0), dense(16)))

    def swap(t):
        t["l0.mix.v"] = t["l0.mix.i"]
    refused(ok, swap)
    zq.Vepinex(hostmodel.VepinexHost.synthetic(ok), ctx=20).close()


def test_programs(zq, tmp_path):
    """The command lines: a replayed trace gives the engine's logits, generation its tokens."""
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
    eng = zq.Vepinex(host, ctx=40, dtype="float32")
    assert r.stdout.strip() == ",".join(str(t) for t in generate.generate(eng, b, 6))
