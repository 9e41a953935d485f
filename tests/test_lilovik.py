"""Lilovik without a GPU: the configuration, the tensor names, what is refused, the tables of sinusoids, and the plain
implementation's mechanisms against closed forms."""
import json
import math

import numpy as np
import pytest

import lilovik_models as lm
from plain import lilovik_plain as plain


def _config(raw):
    from abacus_b200.config.registry import architecture_of
    arch = architecture_of(raw)
    return arch, arch.parse_config(raw)


@pytest.mark.parametrize("name", list(lm.CONFIGS))
def test_configuration_round_trip_and_tensor_names(name):
    raw = lm.config(name)
    shapes = {n: tuple(t.shape) for n, t in lm.weights(raw).items()}
    arch, cfg = _config(raw)
    assert arch.name == "Lilovik"
    assert arch.parse_config(json.loads(json.dumps(cfg.to_dict()))) == cfg
    expected, optional = arch.tensor_names(cfg.to_spec(), set(shapes))
    assert {n: tuple(s) for n, s in expected.items()} == shapes and not optional
    assert "lilovik" in arch.info(cfg.to_spec())


@pytest.mark.parametrize("change,message", [
    (lambda r: r["layers"][0].update(type="mamba"), "type"),
    (lambda r: r["layers"][1]["mixer"].update(kv_heads=4), "multiple"),
    (lambda r: r["layers"][1]["mixer"].pop("vdim"), "vdim"),
    (lambda r: r["layers"][1]["mixer"].update(scale=0.0), "scale"),
    (lambda r: r["layers"][1]["mixer"].update(softcap=-1.0), "softcap"),
    (lambda r: r["layers"][1]["mixer"]["q_temp"].update(every=0), "every"),
    (lambda r: r["layers"][0]["mixer"].update(width=0), "width"),
    (lambda r: r["layers"][1]["mlp"].update(kind="moe"), "dense"),
    (lambda r: r["layers"][1]["mlp"].update(ff=None), "ff"),
    (lambda r: r["norm"].pop("eps"), "eps"),
    (lambda r: r.update(layers=[]), "layers"),
])
def test_configurations_that_are_refused(change, message):
    from abacus_b200.config.registry import ConfigError
    raw = lm.config("A")
    change(raw)
    with pytest.raises(ConfigError, match=message):
        _config(raw)


def test_what_the_layers_ask_of_the_cache_and_of_the_attention_part():
    from abacus_b200.parts import MIXERS
    import dataclasses
    _, cfg = _config(lm.config("A"))
    spec = cfg.to_spec()
    needs = [MIXERS.build(b.mixer).cache_need() for b in spec.layers]
    assert needs[0].n_kv_heads == 0 and needs[0].states == (("average", (48,), "float32"),)
    assert (needs[1].n_kv_heads, needs[1].head_dim, needs[1].v_head_dim, needs[1].window) == (2, 16, 24, None)
    assert spec.layers[1].mixer.slopes == tuple(2.0 ** (-8 * (h + 1) / 6) for h in range(6))
    for wrong in (dict(weights="other"), dict(window=8), dict(weights="softmax"), dict(slopes=(1.0,)), dict(exact_weights=False),
                  dict(sink=True)):
        with pytest.raises(ValueError):
            MIXERS.build(dataclasses.replace(spec.layers[1].mixer, **wrong))


@pytest.mark.parametrize("size", [6, 37, 64, 256])
def test_the_tables_of_sinusoids(size):
    """Coarse and fine tables joined by the sum of angles, against sines and cosines of the whole angle, far out too."""
    import torch
    from abacus_b200.parts.position import Sinusoids
    coarse, fine = Sinusoids(size, 10000.0).tables(70000, torch.device("cpu"))
    assert fine.shape == (256, (size + 1) // 2, 2) and coarse.shape[0] == -(-70000 // 256)
    p = np.array([0, 1, 255, 256, 257, 511, 512, 4095, 4096, 65535, 69999])
    a, b = coarse[p // 256].double().numpy(), fine[p % 256].double().numpy()
    sn, cs = a[..., 0] * b[..., 1] + a[..., 1] * b[..., 0], a[..., 1] * b[..., 1] - a[..., 0] * b[..., 0]
    got = np.stack([sn, cs], axis=-1).reshape(len(p), -1)[:, :size]
    np.testing.assert_allclose(got, plain.position_vectors(p, size), atol=2.5e-7)
    assert plain.position_vectors([3], 6)[0, 2] == pytest.approx(math.sin(3 * 10000 ** (-2 / 6)))
    assert plain.position_vectors([3], 6)[0, 3] == pytest.approx(math.cos(3 * 10000 ** (-2 / 6)))


def test_the_plain_running_average_against_its_sum_over_the_past():
    """S_t = sum_s prod_{s<j<=t} (1 - z_j) z_s c_s; the candidate is continuous at 0; a state carried in portions."""
    rng = np.random.default_rng(0)
    d, W, T = 9, 5, 11
    w = lm.average_weights(rng, d, W)
    w["o"] = np.eye(d, W)
    h = rng.standard_normal((T, d))
    out, state = plain.mingru(h, {"width": W}, w, 1e-6, None)
    z = 1 / (1 + np.exp(-(h @ w["z"].T + w["z.b"])))
    u = h @ w["x"].T + w["x.b"]
    c = np.where(u >= 0, u + 0.5, 1 / (1 + np.exp(-u)))
    assert (u < 0).any() and (u > 0).any()
    S = np.stack([sum(np.prod(1 - z[s + 1:t + 1], axis=0) * z[s] * c[s] for s in range(t + 1)) for t in range(T)])
    g = h @ w["g"].T
    np.testing.assert_allclose(out[:, :W], S * g / (1 + np.exp(-g)), rtol=1e-9, atol=1e-12)
    np.testing.assert_allclose(state, S[-1], rtol=1e-9)
    st, got = None, []
    for a, b in ((0, 4), (4, 5), (5, 11)):
        o, st = plain.mingru(h[a:b], {"width": W}, w, 1e-6, st)
        got.append(o)
    np.testing.assert_allclose(np.concatenate(got), out, rtol=1e-12, atol=1e-12)


def test_the_plain_attention_weight_by_weight():
    """Every weight written out: temperature, cap, distance, shift, sigmoid, and the heads mixed before the values; q and k
    normed over all heads at once; portions; a token further back than another counts less by its distance alone."""
    rng = np.random.default_rng(1)
    d, T = 10, 7
    m = {"heads": 4, "kv_heads": 2, "dim": 3, "vdim": 5, "scale": 0.7, "softcap": 2.5, "q_temp": {"coef": 0.6, "every": 3}}
    w = lm.attention_weights(rng, d, m)
    w["o"] = np.eye(20)
    h = rng.standard_normal((T, d))
    out, _ = plain.attention(h, m, w, 1e-6, None)
    q, k, v = (h @ w[n].T + w[n + ".b"] for n in "qkv")
    want = np.zeros((T, 4, 5))
    for i in range(T):
        qi = q[i] / math.sqrt((q[i] ** 2).mean() + 1e-6) * w["q.norm"] * (1 + 0.6 * math.log((i + 1) // 3 + 1))
        for j in range(i + 1):
            kj = k[j] / math.sqrt((k[j] ** 2).mean() + 1e-6) * w["k.norm"]
            a = np.zeros(4)
            for hd in range(4):
                s = 0.7 * qi[3 * hd:3 * hd + 3] @ kj[3 * (hd // 2):3 * (hd // 2) + 3]
                s = 2.5 * math.tanh(s / 2.5) - 2.0 ** (-8 * (hd + 1) / 4) * (i - j)
                a[hd] = 1 / (1 + math.exp(-s - w["pb"][hd]))
            mixed = w["talk"] @ a
            for hd in range(4):
                want[i, hd] += mixed[hd] * v[j, 5 * (hd // 2):5 * (hd // 2) + 5]
    np.testing.assert_allclose(out, want.reshape(T, 20), rtol=1e-9, atol=1e-11)
    a, st = plain.attention(h[:3], m, w, 1e-6, None)
    b, st = plain.attention(h[3:4], m, w, 1e-6, st)
    c, st = plain.attention(h[4:], m, w, 1e-6, st)
    np.testing.assert_allclose(np.concatenate([a, b, c]), out, rtol=1e-11, atol=1e-12)
    scaled, _ = plain.attention(h, m, dict(w, q=w["q"] * np.repeat([3.0, 1, 1, 1], 3)[:, None]), 1e-6, None)
    assert not np.allclose(scaled[:, 15:], out[:, 15:])  # one head's projection reaches the others through the norm


def test_the_plain_layer_norms_both_sides_of_a_branch():
    raw = lm.config("B")
    w = lm.weights(raw)
    streams = []
    model = plain.PlainLilovik(raw, w)
    logits = model.forward([3, 5, 9], streams=streams)
    x = w["embed"][[3, 5, 9]].astype(np.float64) + plain.position_vectors([0, 1, 2], 37)
    y, _ = plain.attention(plain.norm(x, w["l0.norm1"], 1e-6), raw["layers"][0]["mixer"], plain.part(model.w, "l0.mix."), 1e-6, None)
    x = x + y / np.sqrt((y ** 2).mean(-1, keepdims=True) + 1e-6) * (1 + w["l0.norm1b"])
    np.testing.assert_allclose(streams[0], x, rtol=1e-10)
    np.testing.assert_allclose(plain.PlainLilovik(dict(raw, logit_scale=0.5), w).forward([3, 5, 9]), logits / 2, rtol=1e-12)
    state = model.new_state()
    got = np.concatenate([model.forward(t, state) for t in ([3], [5, 9])])
    np.testing.assert_allclose(got, logits, rtol=1e-10, atol=1e-12)
