"""Host side of Lenisun models: container, registry, configuration reader, and the plain implementation against itself."""
import json

import numpy as np
import pytest

import lenisun as plain
from zignn_b200 import hostmodel, registry, safetensors


def small_cfg():
    return dict(
        architecture="Lenisun", vocab=50, width=40, embedding={"scale": 1.5}, norm={"eps": 1e-5},
        layers=[
            dict(type="wkv", mixer=dict(heads=3, dim=8), mlp=None),
            dict(type="attention",
                 mixer=dict(heads=4, kv_heads=2, dim=12, vdim=20, scale=0.3, v_mix=True, q_temp=dict(coef=0.5, every=3)),
                 mlp=dict(kind="moe", router=dict(experts=5, top=2), expert=dict(ff=24), shared=dict(ff=36))),
            dict(type="attention", mixer=dict(heads=2, kv_heads=2, dim=16, vdim=20, scale=0.2, v_mix=True),
                 mlp=dict(kind="dense", ff=30, limit=0.7)),
        ])


def test_safetensors_round_trip(tmp_path):
    rng = np.random.default_rng(0)
    f = rng.standard_normal((3, 5)).astype(np.float32)
    src = {"a.bf16": safetensors.Tensor("BF16", safetensors.f32_to_bf16(f)), "scalar": safetensors.Tensor("F32", np.float32(2.5).reshape(())),
           "table": safetensors.Tensor("I32", np.arange(7, dtype=np.int32))}
    path = str(tmp_path / "m.safetensors")
    safetensors.write(path, src)
    got = safetensors.read(path)
    assert list(got) == list(src)
    for k in src:
        assert got[k].dtype == src[k].dtype and np.array_equal(got[k].data, src[k].data) and got[k].shape == src[k].shape
    assert np.abs(got["a.bf16"].f32() - f).max() <= np.abs(f).max() * 2.0 ** -8
    with open(path, "r+b") as fh:
        fh.truncate(20)
    with pytest.raises(safetensors.SafetensorsError):
        safetensors.read(path)


def test_bf16_rounding_is_to_nearest_even():
    import torch
    x = np.random.default_rng(1).standard_normal(4096).astype(np.float32)
    want = torch.from_numpy(x).to(torch.bfloat16).view(torch.int16).numpy().view(np.uint16)
    assert np.array_equal(safetensors.f32_to_bf16(x), want)


def test_registry_reads_a_saved_model(tmp_path):
    cfg = small_cfg()
    host = hostmodel.LenisunHost.synthetic(cfg, seed=3, std=0.3, decay_rank=6)
    host.save(str(tmp_path))
    assert registry.architecture_of(str(tmp_path)) == "Lenisun"
    again = registry.load_host(str(tmp_path))
    assert again.cfg == json.loads(json.dumps(cfg))
    assert set(again.tensors) == set(host.tensors)
    assert all(np.array_equal(again.tensors[k].data, host.tensors[k].data) for k in host.tensors)
    bad = dict(cfg, architecture="nothing")
    (tmp_path / "config.json").write_text(json.dumps(bad))
    with pytest.raises(registry.UnknownArchitecture):
        registry.load_host(str(tmp_path))


def test_structs_carry_sizes_and_constants():
    host = hostmodel.LenisunHost.synthetic(small_cfg(), seed=4, std=0.3, decay_rank=6)
    c = host.config_struct(ctx=77, n_seq=3, f32=True)
    assert (c.vocab, c.width, c.layers, c.ctx, c.n_seq, c.precision) == (50, 40, 3, 77, 3, 1)
    assert c.embed_scale == np.float32(1.5) and c.norm_eps == np.float32(1e-5)
    w = host.weights_struct()
    a, b, d = w.layers[0], w.layers[1], w.layers[2]
    assert (a.mixer, a.heads, a.dim, a.decay_rank, a.mlp) == (1, 3, 8, 6, 0)
    assert (b.mixer, b.heads, b.kv_heads, b.dim, b.vdim, b.v_mix) == (0, 4, 2, 12, 20, 1)
    assert (b.experts, b.top, b.expert_ff, b.shared_ff, b.mlp) == (5, 2, 24, 36, 2)
    assert b.q_temp_every == 3.0 and b.q_temp_coef == np.float32(0.5) and b.scale == np.float32(0.3)
    assert (d.mlp, d.ff, d.q_temp_every) == (1, 30, 0.0) and d.limit == np.float32(0.7)
    assert d.vmix == float(host.tensors["l2.mix.vmix"].f32())
    host.tensors["l0.mix.u"] = safetensors.Tensor("BF16", np.zeros((2, 8), np.uint16))
    with pytest.raises(ValueError):
        host.weights_struct()


def test_unknown_mechanisms_are_refused():
    for change in (lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][2]["mlp"].update(kind="other")):
        cfg = small_cfg()
        host = hostmodel.LenisunHost.synthetic(cfg, seed=5, decay_rank=6)
        change(cfg)
        with pytest.raises(ValueError):
            host.weights_struct()


def test_engine_options_are_checked():
    host = hostmodel.LenisunHost.synthetic(small_cfg(), seed=5, decay_rank=6)
    with pytest.raises(ValueError):
        registry.create_engine(host, nonsense=1)


# The plain implementation's own consistency: what the recurrence and the shift carry is all that a cut needs.
def test_plain_recurrence_continues_from_its_state():
    rng = np.random.default_rng(6)
    T, H, d = 11, 2, 5
    r, k, v = (rng.standard_normal((T, H, d)) for _ in range(3))
    w, u = rng.uniform(0.2, 1.0, (T, H, d)), rng.standard_normal((H, d))
    o, S = plain.wkv_scan(r, k, v, w, u)
    o1, S1 = plain.wkv_scan(r[:4], k[:4], v[:4], w[:4], u)
    o2, S2 = plain.wkv_scan(r[4:], k[4:], v[4:], w[4:], u, S1)
    assert np.allclose(np.concatenate([o1, o2]), o) and np.allclose(S2, S)
    # against the sum it stands for: o_t = sum_(s<t) (r_t . (prod_(s<q<t) w_q) k_s) v_s + (r_t . u k_t) v_t
    t, h = 7, 1
    want = (r[t, h] * u[h] * k[t, h]).sum() * v[t, h]
    for s in range(t):
        want = want + (r[t, h] * np.prod(w[s + 1:t, h], axis=0) * k[s, h]).sum() * v[s, h]
    assert np.allclose(o[t, h], want)


def test_plain_attention_against_a_loop():
    rng = np.random.default_rng(7)
    T, H, G, d, e = 6, 4, 2, 3, 5
    q, k, v = rng.standard_normal((T, H, d)), rng.standard_normal((T, G, d)), rng.standard_normal((T, G, e))
    got = plain.attention(q, k, v, 0.4)
    for t in range(T):
        for h in range(H):
            s = np.array([q[t, h] @ k[j, h // 2] * 0.4 for j in range(t + 1)])
            p = np.exp(s - s.max())
            want = sum(p[j] * v[j, h // 2] for j in range(t + 1)) / p.sum()
            assert np.allclose(got[t, h], want)


def test_plain_routing_and_temperature():
    z = np.array([[0.1, 2.0, -1.0, 2.0]])
    ids, s = plain.route(np.eye(4)[:1] * 0 + z, np.eye(4), 2)
    assert ids.tolist() == [[1, 3]] and np.allclose(s, 1 / (1 + np.exp(-2.0)))
    t = plain.query_temperature(np.arange(9.0), 0.5, 3)
    assert np.allclose(t[:2], 1.0) and np.allclose(t[2:5], 1 + 0.5 * np.log(2)) and np.allclose(t[5:8], 1 + 0.5 * np.log(3))
