"""Small Kimilix models for the tests: configurations that differ in every size and option, and random weights made here
(numpy, bfloat16-representable), written as a model folder."""
import json
import os

import numpy as np
import torch

from tilulorn_models import bf16_round


def rot(base, dims, factor=None, original=None, low=None, high=None):
    r = {"base": base, "dims": dims}
    if factor is not None:
        r["scaling"] = {"factor": factor, "original": original, "low": low, "high": high}
    return r


def attention_layer(heads, kv_heads, dim, vdim, scale, diff, chunk, rotation, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if chunk is not None:
        m["mask"] = {"size": chunk}
    if rotation is not None:
        m["rot"] = rotation
    return {"type": "attention", "mixer": m, "mlp": mlp}


def latent_layer(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, window, rotation, mlp=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale}
    if window is not None:
        m["mask"] = {"size": window}
    if rotation is not None:
        m["rot"] = rotation
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def experts(n, top, ff, limit, shared=None):
    """shared: (ff, limit) or None."""
    d = {"kind": "moe", "router": {"experts": n, "top": top}, "expert": {"ff": ff, "limit": limit}}
    if shared is not None:
        d["shared"] = {"ff": shared[0], "limit": shared[1]}
    return d


# A: a latent layer first; chunks and windows inside a page and across pages; experts in turns of 64, a shared expert of
#    another size; frequencies scaled in bands; a rotation over part of a map; a layer without a feed-forward.
# B: sizes that fit no vector (maps of 10, values of 7, 21 latents, 9 query latents, a width of 37, 9 features), as many key
#    heads as query heads, one head, a chunk of 1, a window of 1, no shared expert, all experts chosen; a negative diff.
# C: chunks of exactly a page and windows of exactly a page; one key head for twenty query heads (more than a CTA takes);
#    values larger than 128; no rotation, no mask, no scaling.
# D: maps and latents the tensor-core kernels take, values of 128; a dense feed-forward in every layer but one.
CONFIGS = {
    "A": {"architecture": "Kimilix", "vocab": 131, "width": 64, "norm": {"eps": 1e-5}, "embedding": {"scale": 2.0}, "residual_mult": 0.6,
          "layers": [latent_layer(3, 16, 8, 24, 24, 32, 0.25, 40, rot(10000.0, 8), dense(96)),
                     attention_layer(4, 2, 16, 24, 0.3, 0.35, 48, rot(5000.0, 8, 4.0, 64, 1.0, 4.0), experts(5, 2, 64, 1.5, (40, 1.0))),
                     latent_layer(2, 8, 16, 16, 48, 24, 0.25, 70, rot(500.0, 16, 2.0, 32, 1.0, 8.0)),
                     attention_layer(6, 3, 16, 16, 0.3, 0.5, 20, rot(100.0, 16), experts(4, 1, 24, 2.5, (128, 2.0)))]},
    "B": {"architecture": "Kimilix", "vocab": 97, "width": 37, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0}, "residual_mult": 1.0,
          "layers": [attention_layer(3, 3, 10, 7, 0.3, -0.2, 1, rot(1000.0, 6), experts(3, 3, 9, 1.0)),
                     latent_layer(1, 10, 6, 7, 21, 9, 0.25, 1, rot(100.0, 6), dense(11)),
                     attention_layer(1, 1, 6, 33, 0.4, 0.8, 33, None, dense(9)),
                     latent_layer(2, 5, 2, 3, 8, 5, 0.5, 9, rot(50.0, 2), experts(6, 4, 8, 0.7, (5, 3.0)))]},
    "C": {"architecture": "Kimilix", "vocab": 77, "width": 80, "norm": {"eps": 1e-5}, "embedding": {"scale": 0.5}, "residual_mult": 0.25,
          "layers": [attention_layer(20, 1, 16, 16, 0.25, 0.2, 64, rot(20000.0, 16, 8.0, 128, 1.0, 2.0), dense(64)),
                     latent_layer(20, 16, 16, 8, 64, 40, 0.2, 64, rot(50000.0, 16), experts(9, 3, 128, 3.0, (64, 1.5))),
                     attention_layer(4, 2, 32, 136, 0.2, 0.4, None, None, experts(2, 1, 16, 2.0, (16, 2.0))),
                     latent_layer(4, 8, 8, 24, 40, 16, 0.3, None, None, dense(32))]},
    "D": {"architecture": "Kimilix", "vocab": 61, "width": 72, "norm": {"eps": 1e-5}, "embedding": {"scale": 4.0}, "residual_mult": 0.5,
          "layers": [attention_layer(8, 8, 64, 128, 0.125, 0.3, 100, rot(10000.0, 64, 8.0, 512, 1.0, 4.0), dense(256)),
                     latent_layer(5, 40, 24, 40, 136, 64, 0.15, 130, rot(10000.0, 24), dense(56)),
                     attention_layer(4, 1, 128, 8, 0.1, 0.6, 33, rot(500.0, 32), experts(7, 2, 192, 1.0, (72, 4.0)))]},
}


def config(name):
    return json.loads(json.dumps(CONFIGS[name]))


def attention_weights(rng, d, m):
    """A mixer's tensors by short name; queries and keys leave their norms a few units wide, so that a wrong key shows, and
    the two maps differ."""
    H, G, K, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    gain = np.sqrt(2.5 / (m["scale"] * np.sqrt(K)))
    p = {"q": rng.standard_normal((H * 2 * K, d)) / np.sqrt(d), "k": rng.standard_normal((G * 2 * K, d)) / np.sqrt(d),
         "v": rng.standard_normal((G * V, d)) / np.sqrt(d), "q.norm": gain * (1 + rng.standard_normal(K) * 0.2),
         "k.norm": gain * (1 + rng.standard_normal(K) * 0.2), "o": rng.standard_normal((d, H * V)) / np.sqrt(H * V)}
    p.update({n: rng.standard_normal(K) * 0.5 / np.sqrt(np.sqrt(K)) for n in ("lq1", "lk1", "lq2", "lk2")})
    return p


def latent_weights(rng, d, m):
    H, K, R, V, rank, qr = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
    return {"dq": rng.standard_normal((qr, d)) / np.sqrt(d), "dq.norm": 1 + rng.standard_normal(qr) * 0.1,
            "uq": rng.standard_normal((H * (K + R), qr)) * 3 / np.sqrt(qr), "dkv": rng.standard_normal((rank + R, d)) * 1.5 / np.sqrt(d),
            "dkv.norm": 1 + rng.standard_normal(rank) * 0.1, "uk": rng.standard_normal((H * K, rank)) * 3 / np.sqrt(rank),
            "uv": rng.standard_normal((H * V, rank)) / np.sqrt(rank), "o": rng.standard_normal((d, H * V)) / np.sqrt(H * V)}


def ff_weights(rng, d, mlp):
    def mat(n_out, n_in, gain=1.5):
        return rng.standard_normal((n_out, n_in)) * gain / np.sqrt(n_in)
    if mlp["kind"] == "dense":
        return {"up": mat(mlp["ff"], d), "down": mat(d, mlp["ff"])}
    E, ff = mlp["router"]["experts"], mlp["expert"]["ff"]
    p = {"router": mat(E, d, 2.0), "router.b": rng.standard_normal(E) * 0.5}
    for e in range(E):
        p[f"e{e}.gate"], p[f"e{e}.up"], p[f"e{e}.down"] = mat(ff, d), mat(ff, d), mat(d, ff)
    if mlp.get("shared"):
        ff = mlp["shared"]["ff"]
        p.update({"shared.gate": mat(ff, d), "shared.up": mat(ff, d), "shared.down": mat(d, ff), "shared.sg": mat(1, d)})
    return p


def weights(raw, seed=0):
    """{tensor name: float32 array of bfloat16-representable values} for a configuration (a dict)."""
    rng = np.random.default_rng(seed)
    d, vocab = raw["width"], raw["vocab"]
    w = {"embed": rng.standard_normal((vocab, d)) / raw["embedding"]["scale"]}
    for i, layer in enumerate(raw["layers"]):
        p = f"l{i}."
        mixer = (attention_weights if layer["type"] == "attention" else latent_weights)(rng, d, layer["mixer"])
        w.update({p + "mix." + n: t for n, t in mixer.items()})
        if layer["mlp"]:
            w.update({p + "mlp." + n: t for n, t in ff_weights(rng, d, layer["mlp"]).items()})
        for n in ("1", "2") if layer["mlp"] else ("1",):
            w[p + "norm" + n], w[p + "ls" + n] = rng.standard_normal(d) * 0.2, 1 + rng.standard_normal(d) * 0.3
    w["final.norm"] = rng.standard_normal(d) * 0.2
    return {n: bf16_round(t) for n, t in w.items()}


def write_folder(tmp, name, seed=0, raw=None, tensors=None):
    """config.json and model.safetensors of configuration `name` (or of `raw`) under tmp -> (folder, config, tensors)."""
    from abacus_b200.weights.safetensors_io import save_tensors
    raw = raw if raw is not None else config(name)
    tensors = tensors if tensors is not None else weights(raw, seed)
    folder = os.path.join(str(tmp), f"kimilix{name}")
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(raw, f)
    save_tensors(os.path.join(folder, "model.safetensors"),
                 {n: torch.from_numpy(np.ascontiguousarray(t)).to(torch.bfloat16) for n, t in tensors.items()})
    return folder, raw, tensors


def random_config(rng, large=False):
    """A random configuration: two to five layers of either mixer with either feed-forward or none, sizes that fit and that
    do not fit the vector kernels, every option present or absent."""
    def rotation(most):
        dims = int(rng.choice([n for n in (2, 4, 8, 12, 16, 32, 64) if n <= most]))
        base = float(rng.choice([100.0, 10000.0, 500000.0]))
        kind = rng.random()
        if kind < 0.15:
            return None
        if kind < 0.5:
            return rot(base, dims)
        low = float(rng.choice([0.5, 1.0, 2.0]))
        return rot(base, dims, float(rng.choice([2.0, 8.0])), int(rng.choice([16, 64, 2048])), low, low * float(rng.choice([2.0, 4.0])))

    def feed_forward():
        kind, ffs = rng.random(), [8, 9, 20, 64, 128, 192]
        if kind < 0.15:
            return None
        if kind < 0.4:
            return dense(int(rng.choice(ffs)))
        n = int(rng.choice([1, 2, 3, 5, 9, 16]))
        shared = (int(rng.choice(ffs)), float(rng.choice([0.5, 2.0, 7.0]))) if rng.random() < 0.7 else None
        return experts(n, int(rng.integers(1, min(n, 4) + 1)), int(rng.choice(ffs)), float(rng.choice([0.5, 1.0, 7.0])), shared)
    layers = []
    for _ in range(int(rng.integers(2, 6))):
        size = None if rng.random() < 0.2 else int(rng.choice([1, 2, 7, 33, 63, 64, 65, 100, 128] + ([200, 300, 511] if large else [])))
        if rng.random() < 0.5:
            G, K = int(rng.choice([1, 2, 3, 4])), int(rng.choice([2, 6, 8, 16, 24, 32, 64, 128]))
            layers.append(attention_layer(G * int(rng.choice([1, 2, 3, 5, 18] if large else [1, 2, 3, 9])), G, K,
                                          int(rng.choice([3, 8, 16, 24, 72, 128, 136, 200])), float(rng.choice([0.1, 0.3])),
                                          float(rng.choice([-0.5, 0.2, 0.8])), size, rotation(K), feed_forward()))
        else:
            rd, K = int(rng.choice([2, 4, 8, 16, 32, 64])), int(rng.choice([4, 8, 10, 16, 32, 64, 128]))
            layers.append(latent_layer(int(rng.choice([1, 2, 3, 6, 17, 20])), K, rd,
                                       int(rng.choice([3, 8, 16, 24, 64, 128, 144])), int(rng.choice([8, 21, 32, 40, 64, 136, 192, 260])),
                                       int(rng.choice([5, 8, 24, 32, 96])), float(rng.choice([0.4, 0.8])) / (K + rd) ** 0.5, size, rotation(rd), feed_forward()))
    return {"architecture": "Kimilix", "vocab": int(rng.choice([50, 131])), "width": int(rng.choice([24, 37, 64, 72, 128])),
            "norm": {"eps": float(rng.choice([1e-6, 1e-5]))}, "embedding": {"scale": float(rng.choice([0.5, 1.0, 3.0]))},
            "residual_mult": float(rng.choice([0.3, 0.7, 1.0])), "layers": layers}
