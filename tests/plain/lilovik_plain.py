"""Plain, slow implementation of the Lilovik decoder, for comparison only.

numpy (float64) only, one function per mechanism, no code shared with the package under test (its own file reader).
Every function that keeps something between tokens takes and returns it as `state` (None at the start), so the same
functions serve whole prompts, portions and tokens that come one by one.

Notation: T tokens, d width, H heads, G key/value heads, K key size, V value size.
  rms(x)      = sqrt(mean(x^2) + eps);   norm(x; w) = x / rms(x) * (1 + w)
  frame:      x = E[token] + pos(p), pos(p)[2i] = sin(p 10000^(-2i/d)), pos(p)[2i+1] = cos of the same angle;
              logits = c Wout norm(x; w_final)
  layer:      x += norm(mixer(norm(x; w1)); w1b);   x += norm(ff(norm(x; w2)); w2b)        (ff may be absent)
  attention:  q = Wq h + bq, k = Wk h + bk, v = Wv h + bv;  q <- q / rms(q) * wq, k <- k / rms(k) * wk, each over its whole
              row;  q <- q (1 + a ln(floor((p + 1) / n) + 1));  s_hij = cap tanh(scale q_hi . k_hj / cap)
              - 2^(-8 (h + 1) / H) (i - j);  a_hij = sigmoid(s_hij + b_h) for j <= i, else 0;
              m_hij = sum_g T[h, g] a_gij;  o_hi = sum_j m_hij v_hj;  out = Wo o
  mingru:     z = sigmoid(Wz h + bz), u = Wx h + bx;  c = u + 1/2 where u >= 0, sigmoid(u) where u < 0;
              S <- (1 - z) S + z c;  out = Wo (S * silu(Wg h))
  ff:         Wdown (relu(Wgate h) * (Wup h))
"""
import json
import struct

import numpy as np


def read_safetensors(path):
    """name -> float64 array (bfloat16 widened exactly) or int array."""
    with open(path, "rb") as f:
        raw = f.read()
    (n,) = struct.unpack("<Q", raw[:8])
    out = {}
    for name, info in json.loads(raw[8:8 + n]).items():
        if name == "__metadata__":
            continue
        a, b = info["data_offsets"]
        buf = raw[8 + n + a:8 + n + b]
        if info["dtype"] == "BF16":
            arr = (np.frombuffer(buf, dtype="<u2").astype(np.uint32) << 16).view(np.float32).astype(np.float64)
        elif info["dtype"] == "F32":
            arr = np.frombuffer(buf, dtype="<f4").astype(np.float64)
        elif info["dtype"] == "I32":
            arr = np.frombuffer(buf, dtype="<i4").astype(np.int64)
        else:
            raise ValueError(f"dtype {info['dtype']} of {name}")
        out[name] = arr.reshape(info["shape"])
    return out


def over_rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm(x, w, eps):
    """A weight stored around zero."""
    return over_rms(x, eps) * (1 + w)


def sigmoid(z):
    with np.errstate(over="ignore"):
        return (1 / (1 + np.exp(-z))).astype(z.dtype)


def position_vectors(positions, d, real=np.float64):
    i = np.arange(d)
    angle = np.asarray(positions, dtype=np.float64)[:, None] * 10000.0 ** (-(i - i % 2) / d)[None, :]
    return np.where(i % 2 == 0, np.sin(angle), np.cos(angle)).astype(real)


def temperature(positions, coef, every):
    return 1 + coef * np.log(np.floor((np.asarray(positions, dtype=np.float64) + 1) / every) + 1)


def slopes(H):
    return 2.0 ** (-8.0 * (np.arange(H) + 1) / H)


def attention_weights(q, k, positions, m, pb):
    """q [T, H, K] at `positions`, k [S, G, K] of positions 0 .. S - 1 -> weights [H, T, S] before they are mixed."""
    H, G = m["heads"], m["kv_heads"]
    s = np.einsum("thk,shk->hts", q, np.repeat(k, H // G, axis=1)) * np.asarray(m["scale"], q.dtype)
    if m.get("softcap"):
        s = m["softcap"] * np.tanh(s / m["softcap"])
    back = np.asarray(positions)[:, None] - np.arange(len(k))[None, :]
    s = s - (slopes(H)[:, None, None] * back[None]).astype(q.dtype)
    return np.where(back[None] >= 0, sigmoid(s + pb[:, None, None]), 0).astype(q.dtype)


def attention(h, m, w, eps, state):
    """state: (keys [S, G, K] normed, values [S, G, V])."""
    H, G, K, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T, past = h.shape[0], 0 if state is None else state[0].shape[0]
    positions = np.arange(past, past + T)
    q = over_rms(h @ w["q"].T + w["q.b"], eps) * w["q.norm"]
    k = (over_rms(h @ w["k"].T + w["k.b"], eps) * w["k.norm"]).reshape(T, G, K)
    v = (h @ w["v"].T + w["v.b"]).reshape(T, G, V)
    if m.get("q_temp"):
        q = q * temperature(positions, m["q_temp"]["coef"], m["q_temp"]["every"]).astype(h.dtype)[:, None]
    if state is not None:
        k, v = np.concatenate([state[0], k]), np.concatenate([state[1], v])
    a = attention_weights(q.reshape(T, H, K), k, positions, m, w["pb"])
    mixed = np.einsum("hg,gts->hts", w["talk"], a)
    o = np.einsum("hts,shv->thv", mixed, np.repeat(v, H // G, axis=1))
    return o.reshape(T, H * V) @ w["o"].T, (k, v)


def mingru(h, m, w, eps, state):
    """state: S [width]."""
    z = sigmoid(h @ w["z"].T + w["z.b"])
    u = h @ w["x"].T + w["x.b"]
    c = np.where(u >= 0, u + np.asarray(0.5, u.dtype), sigmoid(u))
    S = np.zeros(z.shape[1], h.dtype) if state is None else state
    out = np.zeros_like(z)
    for t in range(len(h)):
        S = (1 - z[t]) * S + z[t] * c[t]
        out[t] = S
    g = h @ w["g"].T
    return (out * g * sigmoid(g)) @ w["o"].T, S


def feed_forward(h, w):
    return (np.maximum(h @ w["gate"].T, 0) * (h @ w["up"].T)) @ w["down"].T


MIXERS = {"attention": attention, "mingru": mingru}


def part(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


class PlainLilovik:
    def __init__(self, config, weights, real=np.float64):
        """real: the type everything is computed in (float32: to see what float32 itself loses on an input)."""
        self.config, self.real = config, real
        self.w = {n: (t if t.dtype.kind == "i" else t.astype(real)) for n, t in weights.items()}
        self.eps = config["norm"]["eps"]

    @classmethod
    def from_folder(cls, folder, real=np.float64):
        with open(f"{folder}/config.json") as f:
            config = json.load(f)
        return cls(config, read_safetensors(f"{folder}/model.safetensors"), real)

    def new_state(self):
        return {"length": 0, "layers": [None] * len(self.config["layers"])}

    def forward(self, tokens, state=None, streams=None):
        """tokens: the sequence's next tokens; state: what new_state() or an earlier call left (changed in place).
        Returns logits [T, vocab]. streams: a list that gets the residual stream after every layer."""
        state = self.new_state() if state is None else state
        w, eps = self.w, self.eps
        positions = np.arange(state["length"], state["length"] + len(tokens))
        state["length"] += len(tokens)
        x = w["embed"][np.asarray(tokens)] + position_vectors(positions, self.config["width"], self.real)
        for l, layer in enumerate(self.config["layers"]):
            p = f"l{l}."
            y, state["layers"][l] = MIXERS[layer["type"]](norm(x, w[p + "norm1"], eps), layer["mixer"], part(w, p + "mix."),
                                                          eps, state["layers"][l])
            x = x + norm(y, w[p + "norm1b"], eps)
            if layer.get("mlp"):
                x = x + norm(feed_forward(norm(x, w[p + "norm2"], eps), part(w, p + "mlp.")), w[p + "norm2b"], eps)
            if streams is not None:
                streams.append(x.copy())
        return norm(x, w["final.norm"], eps) @ w["head"].T * np.asarray(self.config["logit_scale"], self.real)
