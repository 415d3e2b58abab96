"""Host side of Vepinex models: container, registry, configuration reader, and the plain implementation against itself."""
import json

import numpy as np
import pytest

import vepinex as plain
from zignn_b200 import hostmodel, registry, safetensors


def small_cfg():
    latent = dict(heads=3, dim=8, rot_dim=6, vdim=10, kv_rank=14, scale=0.3, rot=dict(base=900.0, dims=6))
    return dict(
        architecture="Vepinex", vocab=50, width=40, norm={"eps": 1e-5},
        layers=[
            dict(type="latent_attention", mixer=latent, mlp=dict(kind="dense", ff=30)),
            dict(type="mlstm", mixer=dict(heads=2, dim=6, vdim=9, gate_cap=4.0), mlp=None),
            dict(type="channel_delta", mixer=dict(heads=4, kv_heads=2, dim=8, vdim=5, conv=3),
                 mlp=dict(kind="moe", router=dict(experts=5, top=2), expert=dict(ff=24, limit=0.7), shared=dict(ff=36, limit=2.5))),
            dict(type="latent_attention", mixer=dict(latent, heads=2, kv_from=0), mlp=dict(
                kind="moe", router=dict(experts=3, top=3), expert=dict(ff=8, limit=1.25))),
        ])


def small_host():
    return hostmodel.VepinexHost.synthetic(small_cfg(), seed=3, std=0.3, a_rank=5, g_rank=7)


def test_registry_reads_a_saved_model(tmp_path):
    host = small_host()
    host.save(str(tmp_path))
    assert registry.architecture_of(str(tmp_path)) == "Vepinex"
    again = registry.load_host(str(tmp_path))
    assert type(again) is hostmodel.VepinexHost and again.cfg == json.loads(json.dumps(host.cfg))
    assert set(again.tensors) == set(host.tensors)
    assert all(np.array_equal(again.tensors[k].data, host.tensors[k].data) for k in host.tensors)
    with pytest.raises(ValueError):
        registry.create_engine(again, nonsense=1)


def test_structs_carry_sizes_and_constants():
    host = small_host()
    c = host.config_struct(ctx=77, n_seq=3, f32=True)
    assert (c.vocab, c.width, c.layers, c.ctx, c.n_seq, c.precision, c.embed_scale) == (50, 40, 4, 77, 3, 1, 1.0)
    assert c.norm_eps == np.float32(1e-5)
    w = host.weights_struct()
    assert not w.head.data and w.embed_norm and w.final_norm
    a, m, d, b = (w.layers[i] for i in range(4))
    assert all(l.parallel == 1 and l.norm1 and not (l.norm1b or l.norm2 or l.norm2b) for l in (a, m, d, b))
    assert (a.mixer, a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank, a.kv_from) == (4, 3, 8, 6, 10, 14, -1)
    assert a.scale == np.float32(0.3) and a.rot_base == 900.0 and (a.dkv.rows, a.dkv.cols) == (20, 40) and a.dkv_norm
    assert (a.mlp, a.ff, a.mlp_glu) == (1, 30, 0)
    assert (m.mixer, m.heads, m.dim, m.vdim, m.gate_cap, m.mlp) == (2, 2, 6, 9, 4.0, 0) and m.i_bias and m.f_bias
    assert (d.mixer, d.heads, d.kv_heads, d.dim, d.vdim, d.taps) == (3, 4, 2, 8, 5, 3)
    assert (d.a1.rows, d.a2.rows, d.g1.rows, d.g2.rows) == (5, 32, 7, 20)
    assert (d.mlp, d.experts, d.top, d.route, d.expert_ff, d.expert_glu, d.shared_ff, d.shared_glu) == (2, 5, 2, 1, 24, 1, 36, 1)
    assert d.expert_limit == np.float32(0.7) and d.shared_limit == 2.5 and d.router_bias and not d.shared_sg.data
    assert (b.kv_from, b.heads, b.shared_ff) == (0, 2, 0) and not b.dkv.data and not b.dkv_norm
    host.tensors["l2.mix.dt_bias"] = safetensors.Tensor("BF16", np.zeros(31, np.uint16))
    with pytest.raises(ValueError):
        host.weights_struct()


def test_unknown_mechanisms_are_refused():
    for change in (lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][0]["mlp"].update(kind="other"),
                   lambda c: c["layers"][0]["mixer"].update(rot=dict(base=900.0, dims=4))):
        host = small_host()
        change(host.cfg)
        with pytest.raises(ValueError):
            host.weights_struct()


# The plain implementation's own consistency: what a mixer carries is all that a cut needs, and what it stands for.
def test_plain_memory_continues_from_its_state():
    rng = np.random.default_rng(1)
    T, H, d, e = 12, 2, 5, 3
    q, k, v = rng.standard_normal((T, H, d)), rng.standard_normal((T, H, d)), rng.standard_normal((T, H, e))
    i, f = plain.memory_gates(4 * rng.standard_normal((T, H)), 2 + rng.standard_normal((T, H)), 5.0)
    assert (abs(i) < 5).all() and (f < 0).all()
    o, S = plain.memory_scan(q, k, v, i, f)
    o1, S1 = plain.memory_scan(q[:7], k[:7], v[:7], i[:7], f[:7])
    o2, S2 = plain.memory_scan(q[7:], k[7:], v[7:], i[7:], f[7:], S1)
    assert np.allclose(np.concatenate([o1, o2]), o) and all(np.allclose(a, b) for a, b in zip(S, S2))
    # without the running maximum: weights exp(i_s + f_(s+1) + .. + f_t) of the tokens s, their maximum (and 0) divided out
    t, h = 11, 1
    w = np.array([i[s, h] + f[s + 1:t + 1, h].sum() for s in range(t + 1)])
    m = max(w.max(), f[:t + 1, h].sum())
    score = np.exp(w - m) * (k[:t + 1, h] @ q[t, h])
    want = (score[:, None] * v[:t + 1, h]).sum(axis=0) / (max(abs(score.sum()), np.exp(-m)) + 1e-6)
    assert np.isclose(S[2][h], m) and np.allclose(o[t, h], want)


def test_plain_delta_rule_continues_and_replaces():
    rng = np.random.default_rng(2)
    T, H, G, d, e = 10, 4, 2, 6, 3
    q, k = plain.unit(rng.standard_normal((T, G, d))), plain.unit(rng.standard_normal((T, G, d)))
    v, g, beta = rng.standard_normal((T, H, e)), rng.uniform(0.2, 1, (T, H, d)), rng.uniform(0, 1, (T, H))
    o, S = plain.delta_scan(q, k, v, g, beta)
    o1, S1 = plain.delta_scan(q[:4], k[:4], v[:4], g[:4], beta[:4])
    o2, S2 = plain.delta_scan(q[4:], k[4:], v[4:], g[4:], beta[4:], S1)
    assert np.allclose(np.concatenate([o1, o2]), o) and np.allclose(S2, S)
    # a full write makes the key answer with the new value, whatever it held
    o, _ = plain.delta_scan(k, k, v, g, np.ones((T, H)))
    size = (k * k).sum(axis=-1).repeat(H // G, axis=1)
    assert np.allclose(o, v, atol=1e-4) and np.allclose(size, 1, atol=1e-4)


def test_plain_convolution_and_decays():
    x, w = np.arange(1.0, 6.0)[:, None], np.array([[100.0, 10.0, 1.0]])
    assert plain.short_conv(x, w)[:, 0].tolist() == [1, 12, 123, 234, 345]
    assert plain.short_conv(x[2:], w, x[:2])[:, 0].tolist() == [123, 234, 345]
    g = plain.channel_decay(np.array([[[-50.0, 0.0, 50.0]]]), np.zeros(1), np.zeros((1, 3)))[0, 0]
    assert np.allclose(g, [1.0, 0.5, np.exp(-50.0)])


def test_plain_latent_attention():
    rng = np.random.default_rng(3)
    m = dict(heads=3, dim=4, rot_dim=6, vdim=5, kv_rank=8, scale=0.4, rot=dict(base=50.0, dims=6))
    W = {n: rng.standard_normal(s) for n, s in (("q", (30, 16)), ("dkv", (14, 16)), ("dkv.norm", (8,)), ("uk", (12, 8)),
                                                ("uv", (15, 8)), ("o", (16, 15)))}
    h = rng.standard_normal((7, 16))
    c, kr = plain.latent_cache(h, W, m, 1e-5)
    # turning keeps lengths, and a score depends on the distance of the two places alone
    y = (h @ W["dkv"].T)[:, 8:]
    assert np.allclose((kr ** 2).sum(axis=1), (y ** 2).sum(axis=1))
    a, b = rng.standard_normal((2, 1, 6))
    dot = [float((plain.rotate(a, [p], 50.0) * plain.rotate(b, [p + 3], 50.0)).sum()) for p in (0, 5, 100)]
    assert np.allclose(dot, dot[0])
    whole = plain.latent_mixer(h, W, m, 1e-5, (c, kr))
    # with the up-projections folded into the query and behind the weighted sum
    q = (h @ W["q"].T).reshape(7, 3, 10)
    t = 5
    out = []
    for n in range(3):
        ql = W["uk"].reshape(3, 4, 8)[n].T @ q[t, n, :4]
        s = (c[:t + 1] @ ql + kr[:t + 1] @ plain.rotate(q[t:t + 1, n, 4:], [t], 50.0)[0]) * 0.4
        p = np.exp(s - s.max())
        out.append(W["uv"].reshape(3, 5, 8)[n] @ ((p / p.sum()) @ c[:t + 1]))
    assert np.allclose(np.concatenate(out) @ W["o"].T, whole[t])


def test_plain_routing_and_units():
    ids, w = plain.route(np.array([[0.1, 2.0, -1.0, 2.0, 1.0]]), 3)
    assert ids.tolist() == [[1, 3, 4]] and np.allclose(w, np.exp([2, 2, 1]) / np.exp([2, 2, 1]).sum())
    one = np.ones((1, 1))
    assert np.allclose(plain.clamped_unit(one * 5, one, -one, one, 2.0), 2 * plain.sigmoid(3.404) * -1)
    assert np.allclose(plain.silu_unit(one * 5, one, -one, one), -25 * plain.sigmoid(5.0))


def test_plain_model_is_causal():
    host = small_host()
    w = {k: v.astype(np.float64) for k, v in host.as_f32().items()}
    toks = [int(t) for t in np.random.default_rng(4).integers(0, 50, 14)]
    lg, trail = plain.forward(host.cfg, w, toks)
    assert lg.shape == (14, 50) and len(trail) == 4
    part, _ = plain.forward(host.cfg, w, toks[:9])
    assert np.allclose(part, lg[:9])
