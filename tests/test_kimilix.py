"""Kimilix without a GPU: the configuration, the tensor names, what is refused, what layers ask of the cache, the scaled
frequencies, and the plain implementation's mechanisms against closed forms."""
import dataclasses
import json
import math

import numpy as np
import pytest

import kimilix_models as km
from plain import kimilix_plain as plain


def _config(raw):
    from abacus_b200.config.registry import architecture_of
    arch = architecture_of(raw)
    return arch, arch.parse_config(raw)


@pytest.mark.parametrize("name", list(km.CONFIGS))
def test_configuration_round_trip_and_tensor_names(name):
    raw = km.config(name)
    shapes = {n: tuple(t.shape) for n, t in km.weights(raw).items()}
    arch, cfg = _config(raw)
    assert arch.name == "Kimilix"
    assert arch.parse_config(json.loads(json.dumps(cfg.to_dict()))) == cfg
    expected, _ = arch.tensor_names(cfg.to_spec(), set(shapes))
    assert {n: tuple(s) for n, s in expected.items()} == shapes
    assert "kimilix" in arch.info(cfg.to_spec())


@pytest.mark.parametrize("change,message", [
    (lambda r: r["layers"][0].update(type="mamba"), "type"),
    (lambda r: r["layers"][1]["mixer"].update(kv_heads=3), "multiple"),
    (lambda r: r["layers"][1]["mixer"].pop("vdim"), "vdim"),
    (lambda r: r["layers"][1]["mixer"].pop("diff"), "diff"),
    (lambda r: r["layers"][1]["mixer"].update(scale=0.0), "scale"),
    (lambda r: r["layers"][1]["mixer"]["mask"].update(size=0), "size"),
    (lambda r: r["layers"][1]["mixer"]["rot"].update(dims=18), "dims"),
    (lambda r: r["layers"][1]["mixer"]["rot"]["scaling"].update(high=1.0), "high"),
    (lambda r: r["layers"][0]["mixer"].update(rot_dim=0), "rot_dim"),
    (lambda r: r["layers"][0]["mixer"].pop("q_rank"), "q_rank"),
    (lambda r: r["layers"][0]["mlp"].update(kind="gated"), "dense"),
    (lambda r: r["layers"][1]["mlp"]["router"].update(top=6), "top"),
    (lambda r: r["layers"][1]["mlp"]["expert"].update(limit=-1.0), "limit"),
    (lambda r: r["layers"][1]["mlp"]["shared"].pop("limit"), "limit"),
    (lambda r: r["norm"].pop("eps"), "eps"),
    (lambda r: r.update(layers=[]), "layers"),
])
def test_configurations_that_are_refused(change, message):
    from abacus_b200.config.registry import ConfigError
    raw = km.config("A")
    change(raw)
    with pytest.raises(ConfigError, match=message):
        _config(raw)


def test_what_the_layers_ask_of_the_cache_and_of_the_parts():
    from abacus_b200.parts import FEED_FORWARDS, MIXERS
    _, cfg = _config(km.config("A"))
    spec = cfg.to_spec()
    needs = [MIXERS.build(b.mixer).cache_need() for b in spec.layers]
    assert (needs[0].n_kv_heads, needs[0].head_dim, needs[0].v_head_dim, needs[0].window, needs[0].values_in_keys) == (1, 32, 24, 40, True)
    assert (needs[1].n_kv_heads, needs[1].head_dim, needs[1].v_head_dim, needs[1].window) == (2, 32, 24, None)  # two maps of 16 a key
    for wrong in (dict(keep_first=2, window=8), dict(bias=True), dict(head_gate=True), dict(conv_taps=2), dict(exact_weights=False),
                  dict(weights="sigmoid"), dict(values="keys")):
        with pytest.raises(ValueError):
            MIXERS.build(dataclasses.replace(spec.layers[1].mixer, **wrong))
    for wrong in (dict(window=0), dict(shares_latents=True)):
        with pytest.raises(ValueError):
            MIXERS.build(dataclasses.replace(spec.layers[0].mixer, **wrong))
    experts = spec.layers[1].ffn
    for wrong in (dict(weight_on="input"), dict(shared=None), dict(expert=dataclasses.replace(experts.expert, limit=0.0)),
                  dict(shared=dataclasses.replace(experts.shared, activation="relu_squared"))):
        with pytest.raises(ValueError):
            FEED_FORWARDS.build(dataclasses.replace(experts, **wrong))
    with pytest.raises(ValueError, match="not built"):
        FEED_FORWARDS.build(dataclasses.replace(spec.layers[0].ffn, activation="gelu"))


def test_frequencies_scaled_in_bands():
    """Short turns keep their frequency, long ones are slowed by the factor, the ones between blend; the plain rule and the
    library's tables, and the edges of the bands."""
    import torch
    from abacus_b200.config.kimilix import KimilixRotation
    from abacus_b200.parts import POSITIONS
    for r in (km.rot(10000.0, 16, 8.0, 64, 1.0, 4.0), km.rot(500000.0, 64, 32.0, 8192, 1.0, 4.0), km.rot(100.0, 8, 2.0, 16, 0.5, 1.5), km.rot(300.0, 6)):
        part = POSITIONS.build(KimilixRotation.from_dict("", r, 64).to_spec("half"))
        freq, amplitude = part.frequencies()
        np.testing.assert_allclose(freq, plain.frequencies(r), rtol=1e-13)
        assert amplitude == 1.0
        plainly = float(r["base"]) ** (-2.0 * np.arange(r["dims"] // 2) / r["dims"])
        if "scaling" in r:
            s = r["scaling"]
            turns = s["original"] * plainly / (2 * math.pi)
            kinds = np.where(turns > s["high"], 0, np.where(turns < s["low"], 2, 1))
            assert (freq[kinds == 0] == plainly[kinds == 0]).all() and np.allclose(freq[kinds == 2], plainly[kinds == 2] / s["factor"])
            assert ((freq[kinds == 1] < plainly[kinds == 1]) & (freq[kinds == 1] > plainly[kinds == 1] / s["factor"])).all()
            assert len(set(kinds)) >= 2
        cos, sin = part.tables(3000, torch.device("cpu"))
        np.testing.assert_allclose(cos[2999].numpy(), np.cos(2999 * plain.frequencies(r)), atol=1e-6)
        np.testing.assert_allclose(sin[17].numpy(), np.sin(17 * plain.frequencies(r)), atol=1e-6)
    with pytest.raises(ValueError, match="above their low"):
        POSITIONS.build(dataclasses.replace(part.spec, bands=(2.0, 16.0, 2.0, 2.0)))


def test_the_plain_differential_attention_weight_by_weight():
    """Two maps a head written out, chunks, grouped heads, the norm of the difference; portions give the whole."""
    rng = np.random.default_rng(1)
    d, T, C = 10, 9, 4
    m = {"heads": 4, "kv_heads": 2, "dim": 4, "vdim": 5, "scale": 0.7, "diff": 0.3, "mask": {"size": C}, "rot": km.rot(50.0, 2)}
    w = km.attention_weights(rng, d, m)
    w["o"] = np.eye(20)
    h = rng.standard_normal((T, d))
    out, _ = plain.attention(h, m, w, 1e-6, None)

    def prepared(row, weight, p):
        x = row / math.sqrt((row ** 2).mean() + 1e-6) * weight
        u, v = x[0], x[1]  # the pair (0, 1) turns by p radians
        return np.array([u * math.cos(p) - v * math.sin(p), v * math.cos(p) + u * math.sin(p), x[2], x[3]])
    q, k, v = h @ w["q"].T, h @ w["k"].T, h @ w["v"].T
    lam = math.exp(w["lq1"] @ w["lk1"]) - math.exp(w["lq2"] @ w["lk2"]) + 0.3
    want = np.zeros((T, 4, 5))
    for i in range(T):
        seen = range(i // C * C, i + 1)
        for hd in range(4):
            g, a = hd // 2, []
            for s in range(2):
                z = np.array([0.7 * prepared(q[i, 8 * hd + 4 * s:8 * hd + 4 * s + 4], w["q.norm"], i)
                              @ prepared(k[j, 8 * g + 4 * s:8 * g + 4 * s + 4], w["k.norm"], j) for j in seen])
                e = np.exp(z - z.max())
                a.append(e / e.sum() @ np.stack([v[j, 5 * g:5 * g + 5] for j in seen]))
            o = a[0] - lam * a[1]
            want[i, hd] = 0.7 * o / math.sqrt((o ** 2).mean() + 1e-6)
    np.testing.assert_allclose(out, want.reshape(T, 20), rtol=1e-9, atol=1e-11)
    st, got = None, []
    for a, b in ((0, 3), (3, 4), (4, 9)):
        o, st = plain.attention(h[a:b], m, w, 1e-6, st)
        got.append(o)
    np.testing.assert_allclose(np.concatenate(got), out, rtol=1e-10, atol=1e-12)
    first, _ = plain.attention(h[4:5], dict(m, rot=None), w, 1e-6, None)  # a chunk's first token sees itself alone, at any position
    np.testing.assert_allclose(plain.attention(h, dict(m, rot=None), w, 1e-6, None)[0][4:5], first, rtol=1e-10)


def test_the_plain_latent_attention_under_a_window():
    """A window of one gives every token its own value; a window as long as the sequence gives what no window gives; a
    longer one drops exactly the keys behind it; portions give the whole."""
    rng = np.random.default_rng(2)
    d, T = 12, 8
    m = {"heads": 2, "dim": 3, "rot_dim": 4, "vdim": 5, "kv_rank": 6, "q_rank": 7, "scale": 0.4, "rot": km.rot(30.0, 4)}
    w = km.latent_weights(rng, d, m)
    h = rng.standard_normal((T, d))
    down = h @ w["dkv"].T
    c = down[:, :6] / np.sqrt((down[:, :6] ** 2).mean(-1, keepdims=True) + 1e-6) * w["dkv.norm"]
    own = (c @ w["uv"].T) @ w["o"].T
    np.testing.assert_allclose(plain.latent_attention(h, dict(m, mask={"size": 1}), w, 1e-6, None)[0], own, rtol=1e-9)
    whole, _ = plain.latent_attention(h, m, w, 1e-6, None)
    np.testing.assert_allclose(plain.latent_attention(h, dict(m, mask={"size": T}), w, 1e-6, None)[0], whole, rtol=1e-12)
    three, _ = plain.latent_attention(h, dict(m, mask={"size": 3}), w, 1e-6, None)
    moved = h.copy()
    moved[4] += 1.0
    other, _ = plain.latent_attention(moved, dict(m, mask={"size": 3}), w, 1e-6, None)
    np.testing.assert_allclose(other[7], three[7], rtol=1e-12)
    assert np.abs(other[6] - three[6]).max() > 1e-3
    st, got = None, []
    for a, b in ((0, 5), (5, 6), (6, 8)):
        o, st = plain.latent_attention(h[a:b], dict(m, mask={"size": 3}), w, 1e-6, st)
        got.append(o)
    np.testing.assert_allclose(np.concatenate(got), three, rtol=1e-10, atol=1e-12)


def test_the_plain_experts_one_by_one():
    """Chosen by logits with their biases, weighted by the softmax of the chosen, gate and up bounded, the shared one gated."""
    rng = np.random.default_rng(3)
    d, mlp = 7, km.experts(5, 2, 6, 0.8, (4, 0.5))
    w = km.ff_weights(rng, d, mlp)
    h = rng.standard_normal((6, d)) * 2
    got, bounded = plain.experts(h, mlp, w), []

    def one(x, p, limit):
        g, u = w[p + "gate"] @ x, w[p + "up"] @ x
        bounded.append(((u > limit).any(), (u < -limit).any(), (g > limit).any(), (g < -limit).any()))
        y = [min(a, limit) / (1 + math.exp(-1.702 * min(a, limit))) * (max(-limit, min(b, limit)) + 1) for a, b in zip(g, u)]
        return w[p + "down"] @ np.array(y)
    for t in range(6):
        z = w["router"] @ h[t] + w["router.b"]
        order = sorted(range(5), key=lambda e: -z[e])[:2]
        e = np.exp(z[order])
        want = sum(wt * one(h[t], f"e{i}.", 0.8) for wt, i in zip(e / e.sum(), order))
        want = want + one(h[t], "shared.", 0.5) / (1 + math.exp(-float((w["shared.sg"] @ h[t])[0])))
        np.testing.assert_allclose(got[t], want, rtol=1e-9)
    assert np.array(bounded).any(0).all()  # every bound bites somewhere, and gates below -limit stay as they are
    x = np.array([[0.5, -1.0]])
    np.testing.assert_allclose(plain.dense(x, {"up": np.array([[2.0, 0.0], [0.0, 1.0]]), "down": np.eye(2)}), [[1.0, 0.0]])


def test_the_plain_layer_norms_a_branch_behind_it_and_ties_the_unscaled_table():
    raw = km.config("B")
    streams = []
    model = plain.PlainKimilix(dict(raw, embedding={"scale": 3.0}, residual_mult=0.4), km.weights(raw))
    w = model.w
    logits = model.forward([3, 5, 9], streams=streams)
    x = 3.0 * w["embed"][[3, 5, 9]]
    y, _ = plain.attention(x, raw["layers"][0]["mixer"], plain.part(model.w, "l0.mix."), 1e-6, None)
    x = x + 0.4 * w["l0.ls1"] * (y / np.sqrt((y ** 2).mean(-1, keepdims=True) + 1e-6)) * (1 + w["l0.norm1"])
    y = plain.experts(x, raw["layers"][0]["mlp"], plain.part(model.w, "l0.mlp."))
    x = x + 0.4 * w["l0.ls2"] * (y / np.sqrt((y ** 2).mean(-1, keepdims=True) + 1e-6)) * (1 + w["l0.norm2"])
    np.testing.assert_allclose(streams[0], x, rtol=1e-10)
    last = streams[-1]
    np.testing.assert_allclose(logits, last / np.sqrt((last ** 2).mean(-1, keepdims=True) + 1e-6) * (1 + w["final.norm"]) @ w["embed"].T, rtol=1e-9)
    state = model.new_state()
    got = np.concatenate([model.forward(t, state) for t in ([3], [5, 9])])
    np.testing.assert_allclose(got, logits, rtol=1e-10, atol=1e-12)
