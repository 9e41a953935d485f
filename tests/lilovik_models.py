"""Small Lilovik models for the tests: configurations that differ in every size and option, and random weights made
here (numpy, bfloat16-representable), written as a model folder."""
import json
import os

import numpy as np
import torch

from tilulorn_models import bf16_round


def attention_layer(heads, kv_heads, dim, vdim, scale, softcap=20.0, temp=(0.4, 50), ff=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if softcap is not None:
        m["softcap"] = softcap
    if temp is not None:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "attention", "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def average_layer(width, ff=None):
    return {"type": "mingru", "mixer": {"width": width}, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


# A: a recurrent layer first; grouped heads; values larger than keys; a feed-forward in turns of 128; a recurrent layer with a
#    feed-forward; a temperature that steps often.
# B: sizes that fit no vector (heads of 10, values of 7, a width of 37, a recurrence of 13), as many key heads as query
#    heads, a single head, no feed-forward at all in an attention layer, no cap, no temperature.
# C: more than 16 heads; one key head for all; heads of 64 with values of 24; a wide recurrence.
# D: all layers recurrent but one; eight heads as in small models, values smaller than keys.
CONFIGS = {
    "A": {"architecture": "Lilovik", "vocab": 131, "width": 64, "norm": {"eps": 1e-5}, "logit_scale": 0.3,
          "layers": [average_layer(48), attention_layer(6, 2, 16, 24, 0.4, 12.0, (0.7, 9), ff=128), average_layer(40, ff=56),
                     attention_layer(12, 4, 8, 8, 0.6, 25.0, (0.25, 100), ff=32)]},
    "B": {"architecture": "Lilovik", "vocab": 97, "width": 37, "norm": {"eps": 1e-6}, "logit_scale": 1.0,
          "layers": [attention_layer(3, 3, 10, 7, 0.5, None, (0.5, 7)), average_layer(13), attention_layer(1, 1, 20, 33, 0.3, 9.0, None, ff=11),
                     attention_layer(4, 2, 12, 12, 0.45, 30.0, (1.0, 1), ff=9)]},
    "C": {"architecture": "Lilovik", "vocab": 77, "width": 80, "norm": {"eps": 1e-5}, "logit_scale": 2.0,
          "layers": [attention_layer(20, 1, 16, 16, 0.4, 15.0, (0.3, 33), ff=64), attention_layer(24, 8, 64, 24, 0.2, 40.0, (0.6, 60)),
                     average_layer(200, ff=48)]},
    "D": {"architecture": "Lilovik", "vocab": 61, "width": 72, "norm": {"eps": 1e-5}, "logit_scale": 0.125,
          "layers": [average_layer(72), average_layer(24, ff=40), attention_layer(8, 8, 72, 40, 0.15, 30.0, (0.5, 20), ff=256)]},
}


def config(name):
    return json.loads(json.dumps(CONFIGS[name]))


def attention_weights(rng, d, m):
    """A mixer's tensors by short name. Keys and queries leave their norms a few units wide, so that a wrong key shows; the
    shift keeps most weights small; the mixing matrix is no identity and not symmetric."""
    H, G, K, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    gain = np.sqrt(2.5 / (m["scale"] * np.sqrt(K)))
    return {"q": rng.standard_normal((H * K, d)) / np.sqrt(d), "k": rng.standard_normal((G * K, d)) / np.sqrt(d),
            "v": rng.standard_normal((G * V, d)) / np.sqrt(d), "q.b": rng.standard_normal(H * K) * 0.4,
            "k.b": rng.standard_normal(G * K) * 0.4, "v.b": rng.standard_normal(G * V) * 0.4,
            "q.norm": gain * (1 + rng.standard_normal(H * K) * 0.2), "k.norm": gain * (1 + rng.standard_normal(G * K) * 0.2),
            "talk": np.eye(H) + rng.standard_normal((H, H)) * 0.4 / np.sqrt(H), "pb": -3.0 + rng.standard_normal(H),
            "o": rng.standard_normal((d, H * V)) / np.sqrt(H * V)}


def average_weights(rng, d, width):
    return {"z": rng.standard_normal((width, d)) * 1.5 / np.sqrt(d), "z.b": rng.uniform(-6.0, 2.0, width),
            "x": rng.standard_normal((width, d)) * 2.0 / np.sqrt(d), "x.b": rng.standard_normal(width) * 0.5,
            "g": rng.standard_normal((width, d)) * 2.0 / np.sqrt(d), "o": rng.standard_normal((d, width)) / np.sqrt(width)}


def weights(raw, seed=0):
    """{tensor name: float32 array of bfloat16-representable values} for a configuration (a dict)."""
    rng = np.random.default_rng(seed)
    d, vocab = raw["width"], raw["vocab"]
    w = {"embed": rng.standard_normal((vocab, d))}
    for i, layer in enumerate(raw["layers"]):
        p = f"l{i}."
        names = ["norm1", "norm1b"] + (["norm2", "norm2b"] if layer["mlp"] else [])
        for n in names:
            w[p + n] = rng.standard_normal(d) * 0.2
        mixer = attention_weights(rng, d, layer["mixer"]) if layer["type"] == "attention" else average_weights(rng, d, layer["mixer"]["width"])
        w.update({p + "mix." + n: t for n, t in mixer.items()})
        if layer["mlp"]:
            ff = layer["mlp"]["ff"]
            w[p + "mlp.gate"], w[p + "mlp.up"] = rng.standard_normal((ff, d)) / np.sqrt(d), rng.standard_normal((ff, d)) / np.sqrt(d)
            w[p + "mlp.down"] = rng.standard_normal((d, ff)) / np.sqrt(ff)
    w["final.norm"] = rng.standard_normal(d) * 0.2
    w["head"] = rng.standard_normal((vocab, d)) / np.sqrt(d)
    return {n: bf16_round(t) for n, t in w.items()}


def write_folder(tmp, name, seed=0, raw=None, tensors=None):
    """config.json and model.safetensors of configuration `name` (or of `raw`) under tmp -> (folder, config, tensors)."""
    from abacus_b200.weights.safetensors_io import save_tensors
    raw = raw if raw is not None else config(name)
    tensors = tensors if tensors is not None else weights(raw, seed)
    folder = os.path.join(str(tmp), f"lilovik{name}")
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(raw, f)
    save_tensors(os.path.join(folder, "model.safetensors"),
                 {n: torch.from_numpy(np.ascontiguousarray(t)).to(torch.bfloat16) for n, t in tensors.items()})
    return folder, raw, tensors


def random_config(rng):
    """A random configuration: two to five layers of either mixer, sizes that fit and that do not fit the vector kernels,
    every option present or absent."""
    layers = []
    for _ in range(int(rng.integers(2, 6))):
        ff = int(rng.choice([9, 16, 40, 128, 256])) if rng.random() < 0.7 else None
        if rng.random() < 0.3:
            layers.append(average_layer(int(rng.choice([1, 8, 13, 40, 96, 130])), ff))
            continue
        G = int(rng.choice([1, 2, 3, 4, 8]))
        K = int(rng.choice([4, 8, 10, 16, 24, 64, 96]))
        layers.append(attention_layer(G * int(rng.choice([1, 2, 4, 5])), G, K, int(rng.choice([3, 8, 16, 24, 72, 128, 136])),
                                      float(rng.choice([0.15, 0.4])), float(rng.choice([5.0, 30.0])) if rng.random() < 0.8 else None,
                                      (float(rng.choice([0.2, 0.8])), int(rng.choice([1, 10, 64]))) if rng.random() < 0.8 else None, ff))
    return {"architecture": "Lilovik", "vocab": int(rng.choice([50, 131])), "width": int(rng.choice([24, 37, 64, 72])),
            "norm": {"eps": float(rng.choice([1e-6, 1e-5]))}, "logit_scale": float(rng.choice([0.25, 1.0, 3.0])), "layers": layers}
