"""Plain, slow implementation of the Kimilix decoder, for comparison only.

numpy (float64) only, one function per mechanism, no code shared with the package under test (its own file reader).
Every function that keeps something between tokens takes and returns it as `state` (None at the start), so the same
functions serve whole prompts, portions and tokens that come one by one.

Notation: T tokens, d width, H heads, G key/value heads, K key size, V value size, R latent size, P rotated part.
  rms(x)   = sqrt(mean(x^2) + eps);  norm(x; w) = x / rms(x) * (1 + w);  plain(x; w) = x / rms(x) * w
  frame:   x = c E[token];  logits = E norm(x; w_final)
  layer:   x += m a norm(mixer(x); w1);  x += m b norm(ff(x); w2), a and b a factor per element   (ff may be absent)
  turn(x): pairs (u, v) of the first `dims` elements at position p -> (u cos t - v sin t, v cos t + u sin t), t = p f_i
  attention:  q [H, 2, K], k [G, 2, K] each divided by its rms, times a weight of K, turned (pairs i, i + dims / 2);
              for map s: A_s = softmax_j(scale q_his . k_gjs), j <= i and j in the same run of C positions as i;
              lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + c;  o = (A_1 - lambda A_2) v;  o <- (1 - c) o / rms(o);  Wo o
  latent:     c_q = plain(Wdq h), q = Wuq c_q [H, K + P];  [z | r] = Wdkv h, c = plain(z);  k_h = [Wuk_h c | turn(r)],
              v_h = Wuv_h c, q's last P elements turned (pairs 2i, 2i + 1); softmax over 0 <= i - j < W;  Wo o
  dense:      Wdown relu(Wup h)^2
  expert:     g = min(Wgate h, L), u = clamp(Wup h, -L, L);  Wdown (g sigmoid(1.702 g) (u + 1))
  experts:    z = R h + b; the `top` largest; softmax over those; sum of weight * expert + sigmoid(s . h) shared(h)
"""
import json
import math
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
        return 1 / (1 + np.exp(-z))


def frequencies(rot):
    """The pairs' frequencies, slowed where a turn is long beside the original context."""
    dims = rot["dims"]
    out = []
    for i in range(dims // 2):
        f = float(rot["base"]) ** (-2.0 * i / dims)
        s = rot.get("scaling")
        if s:
            turn = 2 * math.pi / f
            if turn > s["original"] / s["low"]:
                f = f / s["factor"]
            elif not turn < s["original"] / s["high"]:
                t = (s["original"] / turn - s["low"]) / (s["high"] - s["low"])
                f = (1 - t) * f / s["factor"] + t * f
        out.append(f)
    return np.array(out)


def turn(x, positions, rot, halves):
    """x [T, heads, n] at `positions`: pairs (i, i + dims / 2) with halves, else (2i, 2i + 1); angles in float64."""
    if rot is None:
        return x
    dims = rot["dims"]
    angle = np.asarray(positions, dtype=np.float64)[:, None] * frequencies(rot)[None, :]
    cs, sn = np.cos(angle).astype(x.dtype)[:, None], np.sin(angle).astype(x.dtype)[:, None]
    first = np.arange(dims // 2) if halves else 2 * np.arange(dims // 2)
    second = first + (dims // 2 if halves else 1)
    u, v = x[..., first], x[..., second]
    y = x.copy()
    y[..., first], y[..., second] = u * cs - v * sn, v * cs + u * sn
    return y


def softmax_seen(s, seen):
    s = np.where(seen, s, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def lam(w, diff):
    """The factor of the second map."""
    return np.exp((w["lq1"] * w["lk1"]).sum()) - np.exp((w["lq2"] * w["lk2"]).sum()) + diff


def attention(h, m, w, eps, state):
    """state: (keys [S, G, 2, K] normed and turned, values [S, G, V])."""
    H, G, K, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T, past = h.shape[0], 0 if state is None else state[0].shape[0]
    positions = np.arange(past, past + T)
    q = over_rms((h @ w["q"].T).reshape(T, H * 2, K), eps) * w["q.norm"]
    k = over_rms((h @ w["k"].T).reshape(T, G * 2, K), eps) * w["k.norm"]
    q = turn(q, positions, m.get("rot"), True).reshape(T, H, 2, K)
    k = turn(k, positions, m.get("rot"), True).reshape(T, G, 2, K)
    v = (h @ w["v"].T).reshape(T, G, V)
    if state is not None:
        k, v = np.concatenate([state[0], k]), np.concatenate([state[1], v])
    i, j = positions[:, None], np.arange(len(k))[None, :]
    seen = j <= i
    if m.get("mask"):
        seen = seen & (i // m["mask"]["size"] == j // m["mask"]["size"])
    s = np.einsum("thsk,jhsk->hstj", q, np.repeat(k, H // G, axis=1)) * np.asarray(m["scale"], h.dtype)
    a = softmax_seen(s, seen)
    both = np.einsum("hstj,jhv->sthv", a, np.repeat(v, H // G, axis=1))
    o = both[0] - np.asarray(lam(w, m["diff"]), h.dtype) * both[1]
    o = over_rms(o, eps) * np.asarray(1 - m["diff"], h.dtype)
    return o.reshape(T, H * V) @ w["o"].T, (k, v)


def latent_attention(h, m, w, eps, state):
    """state: (latents [S, R], rotated key parts [S, P])."""
    H, K, P, V, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    T, past = h.shape[0], 0 if state is None else state[0].shape[0]
    positions = np.arange(past, past + T)
    q = (over_rms(h @ w["dq"].T, eps) * w["dq.norm"]) @ w["uq"].T
    q = q.reshape(T, H, K + P)
    q_plain, q_turned = q[..., :K], turn(q[..., K:], positions, m.get("rot"), False)
    down = h @ w["dkv"].T
    c = over_rms(down[:, :R], eps) * w["dkv.norm"]
    r = turn(down[:, None, R:], positions, m.get("rot"), False)[:, 0]
    if state is not None:
        c, r = np.concatenate([state[0], c]), np.concatenate([state[1], r])
    S = len(c)
    k = (c @ w["uk"].T).reshape(S, H, K)
    v = (c @ w["uv"].T).reshape(S, H, V)
    s = (np.einsum("thk,jhk->htj", q_plain, k) + np.einsum("thp,jp->htj", q_turned, r)) * np.asarray(m["scale"], h.dtype)
    back = positions[:, None] - np.arange(S)[None, :]
    seen = back >= 0
    if m.get("mask"):
        seen = seen & (back < m["mask"]["size"])
    o = np.einsum("htj,jhv->thv", softmax_seen(s, seen), v)
    return o.reshape(T, H * V) @ w["o"].T, (c, r)


def dense(h, w):
    return np.maximum(h @ w["up"].T, 0) ** 2 @ w["down"].T


def expert(h, w, limit):
    g, u = np.minimum(h @ w["gate"].T, limit), np.clip(h @ w["up"].T, -limit, limit)
    return (g * sigmoid(np.asarray(1.702, h.dtype) * g) * (u + 1)) @ w["down"].T


def route(h, w, top):
    """(chosen experts [T, top], their weights [T, top])."""
    z = h @ w["router"].T + w["router.b"]
    chosen = np.argsort(-z, axis=-1, kind="stable")[:, :top]
    e = np.take_along_axis(z, chosen, axis=-1)
    e = np.exp(e - e.max(axis=-1, keepdims=True))
    return chosen, e / e.sum(axis=-1, keepdims=True)


def experts(h, mlp, w):
    chosen, weight = route(h, w, mlp["router"]["top"])
    out = np.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        rows, k = np.nonzero(chosen == e)
        if len(rows):
            out[rows] += weight[rows, k][:, None] * expert(h[rows], part(w, f"e{e}."), mlp["expert"]["limit"])
    if mlp.get("shared"):
        out = out + sigmoid(h @ w["shared.sg"].T) * expert(h, part(w, "shared."), mlp["shared"]["limit"])
    return out


def feed_forward(h, mlp, w):
    return dense(h, w) if mlp["kind"] == "dense" else experts(h, mlp, w)


MIXERS = {"attention": attention, "latent_attention": latent_attention}


def part(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


class PlainKimilix:
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
        return [None] * len(self.config["layers"])

    def forward(self, tokens, state=None, streams=None):
        """tokens: the sequence's next tokens; state: what new_state() or an earlier call left (changed in place).
        Returns logits [T, vocab]. streams: a list that gets the residual stream after every layer."""
        state = self.new_state() if state is None else state
        w, eps, mult = self.w, self.eps, np.asarray(self.config["residual_mult"], self.real)
        x = w["embed"][np.asarray(tokens)] * np.asarray(self.config["embedding"]["scale"], self.real)
        for l, layer in enumerate(self.config["layers"]):
            p = f"l{l}."
            y, state[l] = MIXERS[layer["type"]](x, layer["mixer"], part(w, p + "mix."), eps, state[l])
            x = x + mult * w[p + "ls1"] * norm(y, w[p + "norm1"], eps)
            if layer.get("mlp"):
                y = feed_forward(x, layer["mlp"], part(w, p + "mlp."))
                x = x + mult * w[p + "ls2"] * norm(y, w[p + "norm2"], eps)
            if streams is not None:
                streams.append(x.copy())
        return norm(x, w["final.norm"], eps) @ w["embed"].T
