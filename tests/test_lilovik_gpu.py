"""Lilovik on the GPU against the plain implementation (tests/plain/lilovik_plain.py): every mechanism alone (whole, in
portions, token by token, in unequal batches, in slots used before), the attention kernels held to float64 on their own
operands, keys far away and at the edges of tiles and pages, then whole models through the engine: prompts, portions,
decoding, batches, captured graphs, greedy generation through the library's entry point, and the trace replay."""
import numpy as np
import pytest
import torch

import lilovik_models as lm
from helpers import TraceRun, assert_logits
from part_run import DEV, DT, PartRun, close, every_way, f64, rounding
from plain import lilovik_plain as plain
from tilulorn_models import bf16_round

pytestmark = pytest.mark.gpu
BOTH = ["float32", "bfloat16"]


def _step(lengths, starts=None, slots=None):
    """A filled StepBatch of sequences that bring `lengths` tokens from positions `starts` on."""
    from abacus_b200.engine.batch import Sequence, StepBatch
    starts, slots = starts or [0] * len(lengths), slots or list(range(len(lengths)))
    seqs = [Sequence(slot, [0] * n, start, []) for slot, n, start in zip(slots, lengths, starts)]
    return StepBatch(sum(lengths), len(lengths), 1, DEV).fill(seqs, exact=True)


# ------------------------------------------------------------------ attention without a softmax
_SLOTS = {"wq": "q", "wk": "k", "wv": "v", "bq": "q.b", "bk": "k.b", "bv": "v.b", "q_norm": "q.norm", "k_norm": "k.norm",
          "shift": "pb", "mix": "talk", "wo": "o"}


def _attention_run(p, d, m, dtype):
    from abacus_b200.config.lilovik import LilovikAttention
    from abacus_b200.config.specs import AttentionSpec
    c = LilovikAttention.from_dict("", m)
    spec = AttentionSpec(hidden=d, n_heads=c.heads, n_kv_heads=c.kv_heads, head_dim=c.dim, scale=c.scale, qk_norm_eps=1e-5,
                         position=None, v_head_dim=c.vdim, exact_weights=True, softcap=c.softcap, norm_over="projection", bias=True,
                         q_temperature=None if c.temp_coef is None else (c.temp_coef, c.temp_every), weights="sigmoid",
                         slopes=c.slopes(), shift=True, mix=True)
    return PartRun(spec, {slot: p[short] for slot, short in _SLOTS.items()}, dtype)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("H,G,K,V,cap,temp", [
    (6, 2, 16, 24, 12.0, (0.7, 9)), (3, 3, 10, 7, None, (0.5, 7)), (1, 1, 20, 33, 9.0, None), (20, 1, 16, 16, 15.0, (0.3, 33)),
    (24, 8, 64, 24, 40.0, (0.6, 60)), (8, 8, 72, 40, 30.0, (0.5, 20)), (16, 8, 128, 128, 28.0, (0.45, 70)), (32, 8, 64, 64, None, None),
    (4, 4, 96, 96, 30.0, (1.0, 1)), (2, 1, 256, 128, 20.0, (0.2, 10)), (5, 5, 8, 136, 20.0, (0.4, 50)), (15, 5, 24, 8, 7.0, (0.4, 16)),
])
def test_attention_every_way(dtype, H, G, K, V, cap, temp):
    rng, rnd, d = np.random.default_rng(H + K), rounding(dtype), 40
    m = lm.attention_layer(H, G, K, V, 0.5, cap, temp)["mixer"]
    p = {n: rnd(t) for n, t in lm.attention_weights(rng, d, m).items()}
    p["talk"] = bf16_round(p["talk"])
    h = rnd(rng.standard_normal((150, d)))
    want, _ = plain.attention(h.astype(np.float64), m, f64(p), 1e-5, None)
    every_way(_attention_run(p, d, m, dtype), h, want, dtype, f"attention {H}/{G} x {K}, values of {V}")


class Rows:
    """Prepared q, k and v of a few sequences (bfloat16 numbers), the same in the step's rows and in a paged cache, and the
    float64 answer: what a kernel is held to closely, its operands being given."""

    def __init__(self, rng, lengths, H, G, K, V, cap, mix=True, width=2.0):
        from abacus_b200.cache import CacheNeed, SequenceCache
        self.sizes, self.cap, self.lengths = (H, G, K, V), cap, lengths
        self.row = -(-((H + G) * K + G * V) // 8) * 8
        self.scale = width / np.sqrt(K)
        self.slopes = (2.0 ** (-8.0 * (np.arange(H) + 1) / H)).astype(np.float32)
        self.shift = (rng.standard_normal(H) - 2.0).astype(np.float32)
        self.mix = bf16_round(np.eye(H) + rng.standard_normal((H, H)) * 0.5) if mix else None
        n = sum(lengths)
        self.rows = np.zeros((n, self.row), np.float32)
        self.rows[:, :(H + G) * K + G * V] = bf16_round(rng.standard_normal((n, (H + G) * K + G * V)))
        self.cache = SequenceCache([CacheNeed(n_kv_heads=G, head_dim=K, v_head_dim=V)], [None], 64 * (sum(-(-l // 64) for l in lengths) + 4),
                                   torch.bfloat16, DEV)
        self.slots, at, want = [], 0, []
        g = self.cache.groups[0]
        g.k.fill_(7.0), g.v.fill_(-9.0)  # what former users left
        for l in lengths:
            slot = self.cache.open_slot()
            self.cache.reserve(slot, l)
            r = self.rows[at:at + l]
            k, v = r[:, H * K:(H + G) * K].reshape(l, G, K), r[:, (H + G) * K:(H + G) * K + G * V].reshape(l, G, V)
            for j in range(l):
                page = int(g.table_host[slot, j // 64])
                g.k[0, page, :, j % 64], g.v[0, page, :, j % 64] = (torch.from_numpy(np.ascontiguousarray(t[j])).to(DEV, torch.bfloat16) for t in (k, v))
            want.append(self.answer(r.astype(np.float64)))
            self.slots.append(slot)
            at += l
        self.want = want
        self.qkv = torch.from_numpy(self.rows).to(DEV, torch.bfloat16)
        self.dev = {n: None if t is None else torch.from_numpy(t).to(DEV) for n, t in (("slopes", self.slopes), ("shift", self.shift), ("mix", self.mix))}

    def answer(self, r):
        H, G, K, V = self.sizes
        l = len(r)
        q, k = r[:, :H * K].reshape(l, H, K), r[:, H * K:(H + G) * K].reshape(l, G, K)
        v = r[:, (H + G) * K:(H + G) * K + G * V].reshape(l, G, V)
        m = {"heads": H, "kv_heads": G, "scale": float(np.float32(self.scale)), "softcap": self.cap}
        a = plain.attention_weights(q, k, np.arange(l), m, self.shift.astype(np.float64))
        mixed = a if self.mix is None else np.einsum("hg,gts->hts", self.mix.astype(np.float64), a)
        return np.einsum("hts,shv->thv", mixed, np.repeat(v, H // G, axis=1)).reshape(l, H * V)

    def check(self, got, want, what):
        """bfloat16 outputs: within their own rounding, and what float32 sums of the size of the terms lose."""
        got = got.float().cpu().numpy()
        limit = np.abs(want) * 2.0 ** -8 + 3e-5 * max(np.abs(want).max(), 1.0)
        diff = np.abs(got - want)
        assert np.isfinite(got).all() and (diff <= limit).all(), \
            f"{what}: off by {diff.max():.3g} at {np.unravel_index(int((diff - limit).argmax()), diff.shape)}"

    def args(self):
        H, G, K, V = self.sizes
        return dict(n_heads=H, n_kv_heads=G, head_dim=K, vd=V, row=self.row, scale=self.scale, softcap=self.cap, **self.dev)


@pytest.mark.parametrize("H,G,K,V,cap", [(16, 8, 128, 128, 30.0), (8, 8, 80, 96, 25.0), (6, 3, 40, 24, None), (4, 1, 64, 128, 5.0), (32, 4, 64, 32, 30.0),
                                         (1, 1, 8, 8, None), (17, 17, 16, 16, 10.0), (13, 13, 24, 40, 20.0), (32, 8, 128, 128, 30.0), (20, 5, 104, 56, None)])
def test_the_prompt_kernel_against_float64(H, G, K, V, cap):
    """Unequal sequences, the keys of a query tile on one CTA and dealt to clusters of 2, 4 and 8; and the general kernel on
    the same operands."""
    from abacus_b200.kernels import ops
    rng = np.random.default_rng(H * K)
    rows = Rows(rng, [333, 1, 70, 16], H, G, K, V, cap, mix=H != 6)
    batch = _step(rows.lengths, slots=rows.slots)
    assert ops.attention_sigmoid_prompt_takes(rows.qkv, H, G, K, V, rows.row)
    a = rows.args()
    want = np.concatenate(rows.want)
    for ranks in (0, 1, 2, 4, 8):
        out = torch.full((len(want), H * V), 5.0, dtype=torch.bfloat16, device=DEV)
        ops.attention_sigmoid_prompt(rows.qkv, out, batch=batch, ranks=ranks, **a)
        torch.cuda.synchronize()
        rows.check(out, want, f"prompt kernel, {ranks} CTAs a tile")
    out = torch.full((len(want), H * V), 5.0, dtype=torch.bfloat16, device=DEV)
    ops.attention_sigmoid_general(rows.qkv, out, batch=batch, cache=rows.cache.views[0].kv, **a)
    torch.cuda.synchronize()
    rows.check(out, want, "general kernel")


@pytest.mark.parametrize("H,G,K,V,cap", [(16, 8, 128, 128, 30.0), (8, 8, 80, 96, 25.0), (6, 3, 40, 24, None), (16, 1, 64, 128, 5.0), (32, 4, 64, 32, 30.0),
                                         (1, 1, 8, 8, None), (17, 17, 16, 16, 10.0), (13, 13, 24, 40, 20.0), (32, 8, 128, 128, 30.0),
                                         (16, 16, 128, 128, 20.0), (20, 2, 72, 136, 30.0), (28, 28, 128, 128, 25.0)])
def test_the_decode_kernel_against_float64(H, G, K, V, cap):
    """Rows of every length from one key to several stages and parts; few rows (many parts each) and many (few)."""
    from abacus_b200.kernels import ops
    from abacus_b200.parts import Workspace
    rng = np.random.default_rng(H * K + 1)
    rows = Rows(rng, [1, 15, 16, 17, 64, 65, 200, 517, 33], H, G, K, V, cap, mix=H != 6)
    ws, kv, a = Workspace(torch.device(DEV, torch.cuda.current_device())), rows.cache.views[0].kv, rows.args()
    last = np.cumsum(rows.lengths) - 1
    for picked in ([7], list(range(9)), list(range(9)) * 30):
        batch = _step([1] * len(picked), [rows.lengths[i] - 1 for i in picked], [rows.slots[i] for i in picked])
        assert ops.attention_sigmoid_decode_parts(rows.qkv, len(picked), H, G, K, V, kv, 1) > 0
        q = rows.qkv[torch.from_numpy(last[picked]).to(DEV)].contiguous()
        out = torch.full((len(picked), H * V), 5.0, dtype=torch.bfloat16, device=DEV)
        ops.attention_sigmoid(q, out, H, G, K, rows.scale, batch, kv, v_dim=V, softcap=cap, row=rows.row, ws=ws, **rows.dev)
        torch.cuda.synchronize()
        rows.check(out, np.stack([rows.want[i][-1] for i in picked]), f"decode kernel, {len(picked)} rows")
    assert int(ops.kernel_status(torch.device(DEV, torch.cuda.current_device())).abs().sum()) == 0


@pytest.mark.parametrize("dtype", BOTH)
def test_one_loud_key_far_away_and_at_the_edges_of_tiles_and_pages(dtype):
    """One key a query agrees with among hundreds it does not: nothing is shared out between keys, so the loud key's value
    comes in whole, less what its distance takes off. In prompts, and for tokens that come one by one, in used pages."""
    rng, K, T, H = np.random.default_rng(3), 8, 330, 2
    d = 3 * K + 4
    eye = np.eye(d)
    p = {"q": np.concatenate([eye[:K], eye[:K]]), "k": eye[K:2 * K], "v": eye[2 * K:3 * K], "q.b": np.zeros(H * K), "k.b": np.full(K, 0.125),
         "v.b": np.full(K, 0.25), "q.norm": np.full(H * K, 1.0), "k.norm": np.full(K, 1.0), "talk": np.array([[1.0, 0.5], [-0.75, 1.0]]),
         "pb": np.array([-8.0, -7.0]), "o": rng.standard_normal((d, H * K)) / 4}
    p = {n: bf16_round(np.asarray(t, np.float32)) for n, t in p.items()}
    m = {"heads": H, "kv_heads": 1, "dim": K, "vdim": K, "scale": 1.5, "softcap": 30.0, "q_temp": {"coef": 0.1, "every": 100}}
    u = rng.standard_normal(K)
    u /= np.linalg.norm(u)
    run = _attention_run(p, d, m, dtype)
    for i, j in [(T - 1, 0), (T - 1, 1), (T - 1, 15), (T - 1, 16), (T - 1, 31), (T - 1, 32), (T - 1, 63), (T - 1, 64), (T - 1, 65), (200, 127),
                 (200, 128), (129, 128), (T - 1, T - 2), (70, 70), (64, 63), (64, 64), (15, 0), (16, 0), (T - 1, 255), (T - 1, 256)]:
        h = rng.standard_normal((T, d)) * 0.3
        h[:, K:2 * K] -= np.outer(h[:, K:2 * K] @ u, u)  # (the norm levels the keys' sizes: the others point elsewhere)
        h[i, :K] = 4.0 * u
        h[j, K:2 * K] = 4.0 * u
        h[j, 2 * K:3 * K] += 2.0
        h = rounding(dtype)(h)
        want, _ = plain.attention(h.astype(np.float64), m, f64(p), 1e-5, None)
        quiet = h.copy()
        quiet[j, K:2 * K] = -quiet[j, K:2 * K]
        without, _ = plain.attention(quiet.astype(np.float64), m, f64(p), 1e-5, None)
        assert np.abs(want[i] - without[i]).max() > 0.1, "the loud key decides nothing: the test shows nothing"
        run.cache.views[0].kv.k.fill_(9.0), run.cache.views[0].kv.v.fill_(9.0)  # what former users left in the pages
        slot = run.open(dirty=True)
        close(run.step([(slot, h[:i + 1])])[0], want[:i + 1], dtype, f"query {i}, loud key {j}, prompt")
        run.close(slot)
        slot, cut = run.open(dirty=True), max(1, i - 3 if j < i - 3 else j - 1)
        got = [run.step([(slot, h[:cut])])[0]] + [run.step([(slot, h[t:t + 1])])[0] for t in range(cut, i + 1)]
        close(np.concatenate(got), want[:i + 1], dtype, f"query {i}, loud key {j}, decoded from {cut}")
        run.close(slot)


def test_the_temperature_steps_where_it_should_and_the_shift_and_the_mix_belong_to_their_heads():
    """Against the plain function (held to written-out weights on the CPU), with each option's numbers far apart."""
    rng, d, H, G, K, V = np.random.default_rng(8), 32, 4, 2, 8, 8
    m = {"heads": H, "kv_heads": G, "dim": K, "vdim": V, "scale": 0.4, "softcap": 6.0, "q_temp": {"coef": 3.0, "every": 16}}
    p = {n: rounding("float32")(t) for n, t in lm.attention_weights(rng, d, m).items()}
    p["pb"] = np.array([6.0, -9.0, 0.0, -2.0], np.float32)
    p["talk"] = np.array([[0, 2, 0, 0], [0, 0, -3, 0], [1, 0, 0, 4], [0.5, 0, 0, 0]], np.float32)
    h = rng.standard_normal((100, d)).astype(np.float32)
    want, _ = plain.attention(h.astype(np.float64), m, f64(p), 1e-5, None)
    run = _attention_run(p, d, m, "float32")
    slot = run.open()
    close(run.step([(slot, h)])[0], want, "float32", "numbers far apart")
    for name, other in (("talk", p["talk"].T), ("pb", p["pb"][::-1])):
        moved, _ = plain.attention(h.astype(np.float64), m, f64(dict(p, **{name: other})), 1e-5, None)
        assert np.abs(moved - want).max() > 0.1
    late, _ = plain.attention(h.astype(np.float64), dict(m, q_temp={"coef": 3.0, "every": 17}), f64(p), 1e-5, None)
    assert np.abs(late[15] - want[15]).max() > 1e-2


# ------------------------------------------------------------------ the running average
_AVERAGE_SLOTS = {"wz": "z", "bz": "z.b", "wu": "x", "bu": "x.b", "wg": "g", "wo": "o"}


def _average_run(p, d, width, dtype):
    from abacus_b200.config.specs import GatedAverageSpec
    return PartRun(GatedAverageSpec(hidden=d, width=width), {slot: p[short] for slot, short in _AVERAGE_SLOTS.items()}, dtype)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("width", [1, 7, 8, 36, 64, 130, 320])
def test_the_running_average_every_way(dtype, width):
    rng, rnd, d = np.random.default_rng(width), rounding(dtype), 48
    p = {n: rnd(t) for n, t in lm.average_weights(rng, d, width).items()}
    h = rnd(rng.standard_normal((150, d)))
    want, _ = plain.mingru(h.astype(np.float64), {"width": width}, f64(p), 1e-5, None)
    every_way(_average_run(p, d, width, dtype), h, want, dtype, f"average of {width}")


@pytest.mark.parametrize("dtype", BOTH)
def test_the_running_average_over_long_prompts_and_portions(dtype):
    """Sequences of several turns of a cluster, alone (clusters of 8) and beside short ones (smaller clusters), and in
    portions that end anywhere."""
    rng, rnd, d, width = np.random.default_rng(9), rounding(dtype), 24, 72
    p = {n: rnd(t) for n, t in lm.average_weights(rng, d, width).items()}
    h = rnd(rng.standard_normal((2500, d)))
    want, _ = plain.mingru(h.astype(np.float64), {"width": width}, f64(p), 1e-5, None)
    run = _average_run(p, d, width, dtype)
    slot = run.open(dirty=True)
    close(run.step([(slot, h)])[0], want, dtype, "long prompt")
    run.close(slot)
    slots = [run.open(dirty=True) for _ in range(4)]
    for n, got in zip((1100, 3, 1, 600), run.step([(s, h[:n]) for s, n in zip(slots, (1100, 3, 1, 600))])):
        close(got, want[:n], dtype, f"beside others, {n} rows")
    for s in slots:
        run.close(s)
    slot, at, got = run.open(dirty=True), 0, []
    for n in (2, 1025, 127, 1, 129, 1216):
        got.append(run.step([(slot, h[at:at + n])])[0])
        at += n
    close(np.concatenate(got), want, dtype, "portions")
    run.close(slot)


def test_the_running_average_keeps_a_token_over_a_long_decoding_and_forgets_at_once_with_gates_near_one():
    rng, d, width = np.random.default_rng(5), 16, 24
    for bias, what in ((-9.0, "lasting"), (9.0, "fading")):
        p = {n: t.astype(np.float32) for n, t in lm.average_weights(rng, d, width).items()}
        p["z"] *= 0.1
        p["z.b"][:] = bias
        h = rng.standard_normal((420, d)).astype(np.float32)
        h[3] *= 400.0 if what == "lasting" else 1.0  # one early token far louder than all others
        want, _ = plain.mingru(h.astype(np.float64), {"width": width}, f64(p), 1e-5, None)
        other = h.copy()
        other[3] = 0.0
        moved, _ = plain.mingru(other.astype(np.float64), {"width": width}, f64(p), 1e-5, None)
        assert (np.abs(want[-1] - moved[-1]).max() > 1e-3 * np.abs(want[-1]).max()) == (what == "lasting")
        run = _average_run(p, d, width, "float32")
        slot = run.open(dirty=True)
        got = [run.step([(slot, h[:20])])[0]] + [run.step([(slot, h[t:t + 1])])[0] for t in range(20, 420)]
        close(np.concatenate(got)[20:], want[20:], "float32", f"average {what}")


# ------------------------------------------------------------------ norms on both sides, sinusoids, relu
@pytest.mark.parametrize("d", [5, 36, 64, 1024, 2560, 5000])
def test_the_norm_behind_a_branch_the_sum_and_the_norm_ahead_of_the_next(d):
    from abacus_b200.kernels import ops
    rng = np.random.default_rng(d)
    x, y = rng.standard_normal((9, d)).astype(np.float32) * 3, rng.standard_normal((9, d)).astype(np.float32) * 0.01
    wy, w = (1 + rng.standard_normal((2, d)) * 0.3).astype(np.float32)
    t = {n: torch.from_numpy(v).to(DEV) for n, v in dict(x=x, y=y, wy=wy, w=w).items()}
    summed = x + plain.over_rms(y.astype(np.float64), 1e-4) * wy
    normed = plain.over_rms(summed, 1e-5) * w
    for dt, tol in ((torch.float32, 3e-6), (torch.bfloat16, 8e-3)):
        xs, out = t["x"].clone(), torch.full((9, d), 7.0, dtype=dt, device=DEV)
        ops.normed_add_rmsnorm(xs, t["y"], t["wy"], 1e-4, t["w"], out, 1e-5)
        np.testing.assert_allclose(xs.cpu().numpy(), summed, rtol=2e-6, atol=3e-6)
        np.testing.assert_allclose(out.float().cpu().numpy(), normed, rtol=tol, atol=tol)
        xs, rows = t["x"].clone(), torch.tensor([4, 0, 4], dtype=torch.int32, device=DEV)
        ops.normed_add_rmsnorm(xs, t["y"], t["wy"], 1e-4, t["w"], out, 1e-5, rows=rows, n_rows=3)
        np.testing.assert_allclose(out[:3].float().cpu().numpy(), normed[[4, 0, 4]], rtol=tol, atol=tol)
        assert torch.equal(xs, t["x"])
        ops.normed_add_rmsnorm(xs, None, None, 0.0, t["w"], out, 1e-5)
        np.testing.assert_allclose(out.float().cpu().numpy(), plain.over_rms(x.astype(np.float64), 1e-5) * w, rtol=tol, atol=tol)
        assert torch.equal(xs, t["x"])


@pytest.mark.parametrize("d", [5, 64, 1026])
def test_the_embedding_with_sinusoids(d):
    from abacus_b200.engine.batch import Sequence, StepBatch
    from abacus_b200.kernels import ops
    from abacus_b200.parts.position import Sinusoids
    rng = np.random.default_rng(d)
    table = bf16_round(rng.standard_normal((50, d)))
    coarse, fine = Sinusoids(d, 10000.0).tables(20000, torch.device(DEV))
    tokens = [[3, 49, 0, 7], [11, 12], [5]]
    starts = [0, 255, 19999]
    batch = StepBatch(8, 3, 1, DEV).fill([Sequence(i, t, s, []) for i, (t, s) in enumerate(zip(tokens, starts))])  # a row of padding
    want = np.concatenate([table[t] + plain.position_vectors(np.arange(s, s + len(t)), d) for t, s in zip(tokens, starts)])
    for dt in (torch.float32, torch.bfloat16):
        x, status = torch.full((8, d), 9.0, device=DEV), torch.zeros(4, dtype=torch.int32, device=DEV)
        ops.embed_sinusoids(batch, torch.from_numpy(table).to(DEV, dt), coarse, fine, 20000, x, status)
        np.testing.assert_allclose(x.cpu().numpy()[:7], want, atol=6e-7)
        assert not status.any() and not x[7].any()
        ops.embed_sinusoids(batch, torch.from_numpy(table).to(DEV, dt), coarse, fine, 19999, x, status)
        assert status[0].item() == 1


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("rows,d,ff", [(1, 64, 128), (5, 37, 9), (16, 96, 256), (40, 64, 48), (300, 64, 256), (300, 64, 72), (2100, 256, 512)])
def test_the_feed_forward_with_relu(dtype, rows, d, ff):
    """A handful of rows (product and activation in one), many (the activation in the product's epilogue, pairs of CTAs too)
    and what neither takes."""
    from abacus_b200.config.specs import GatedMLPSpec
    rng, rnd = np.random.default_rng(rows + ff), rounding(dtype)
    w = {"gate": rnd(rng.standard_normal((ff, d)) / np.sqrt(d)), "up": rnd(rng.standard_normal((ff, d)) / np.sqrt(d)),
         "down": rnd(rng.standard_normal((d, ff)) / np.sqrt(ff))}
    run = PartRun(GatedMLPSpec(hidden=d, inter=ff, activation="relu"), w, dtype, feed_forward=True)
    h = rnd(rng.standard_normal((rows, d)))
    close(run.step([(None, h)])[0], plain.feed_forward(h.astype(np.float64), f64(w)), dtype, f"{rows} x {d} x {ff}")
    with pytest.raises(ValueError, match="not built"):
        PartRun(GatedMLPSpec(hidden=d, inter=ff, activation="gelu"), w, dtype, feed_forward=True)


# ------------------------------------------------------------------ whole models through the engine
def _engine(tmp, name, dtype, raw=None, seed=0, tensors=None, **kw):
    from abacus_b200.engine import Engine, load_model
    folder, raw, tensors = lm.write_folder(tmp, name, seed=seed, raw=raw, tensors=tensors)
    return Engine(load_model(folder, dtype), max_tokens=64 * 24, **kw), raw, tensors, folder


def _oracle(raw, tensors, tokens):
    """(the plain model's logits in float64, the noise float32 itself shows on them)."""
    want = plain.PlainLilovik(raw, tensors).forward(tokens)
    return want, float(np.abs(want - plain.PlainLilovik(raw, tensors, real=np.float32).forward(tokens)).max())


def _bf16_close(got, want, what):
    """bfloat16 against float64: two roundings of one model, a few per cent of the logits' spread apart."""
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    rel = np.sqrt((d * d).mean(-1)) / want.std()
    assert np.isfinite(got).all() and rel.max() < 0.12, f"{what}: bfloat16 logits are {rel.max():.3g} of the spread away"


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", list(lm.CONFIGS))
def test_prompts_decoding_batches_and_used_slots_against_the_plain_model(tmp_path, name, dtype):
    engine, raw, tensors, _ = _engine(tmp_path, name, dtype)
    rng = np.random.default_rng(7)
    lens = [150, 1, 37, 80]
    seqs = [[int(t) for t in rng.integers(0, raw["vocab"], n)] for n in lens]
    oracle = [_oracle(raw, tensors, s) for s in seqs]

    def check(got, want, noise, what):
        if dtype == "float32":
            assert_logits(got, want, dtype, what, noise)
        else:
            _bf16_close(got, want, what)
    # each alone, whole, all logits wanted; the slot is given back and used again by the next
    for s, (want, noise) in zip(seqs, oracle):
        slot = engine.open()
        got = engine.step([(slot, s, list(range(len(s))))]).cpu().numpy()
        engine.close(slot)
        check(got, want, noise, f"{name} whole, {len(s)} tokens")
    # together in one batch of unequal prompts, cut before their ends, then decoded together; early enders leave
    cut = [100, 1, 20, 64]
    slots = [engine.open() for _ in seqs]
    got = engine.step([(slot, s[:c], [c - 1]) for slot, s, c in zip(slots, seqs, cut)]).cpu().numpy()
    for i, (want, noise) in enumerate(oracle):
        check(got[i:i + 1], want[cut[i] - 1:cut[i]], noise, f"{name} batch prompt {i}")
    step = 0
    while True:
        live = [i for i in range(len(seqs)) if cut[i] + step < len(seqs[i])]
        for i in range(len(seqs)):
            if cut[i] + step == len(seqs[i]) and slots[i] is not None:
                engine.close(slots[i])
                slots[i] = None
        if not live:
            break
        got = engine.step([(slots[i], [seqs[i][cut[i] + step]], [0]) for i in live]).cpu().numpy()
        for j, i in enumerate(live):
            check(got[j:j + 1], oracle[i][0][cut[i] + step:cut[i] + step + 1], oracle[i][1],
                  f"{name} batch decode, request {i}, position {cut[i] + step}")
        step += 1
    engine.check_status()


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", ["A", "B"])
def test_portions_of_a_prompt(tmp_path, name, dtype):
    engine, raw, tensors, _ = _engine(tmp_path, name, dtype)
    rng = np.random.default_rng(5)
    tokens = [int(t) for t in rng.integers(0, raw["vocab"], 140)]
    want, noise = _oracle(raw, tensors, tokens)
    slot, got, at = engine.open(), [], 0
    for size in (60, 2, 7, 1, 64, 6):
        got.append(engine.step([(slot, tokens[at:at + size], list(range(size)))]).cpu().numpy())
        at += size
    engine.close(slot)
    assert at == len(tokens)
    if dtype == "float32":
        assert_logits(np.concatenate(got), want, "float32", f"{name} in portions", noise)
    else:
        _bf16_close(np.concatenate(got), want, f"{name} in portions")


@pytest.mark.parametrize("name", ["A", "C"])
def test_token_by_token_from_the_first_token_and_long_decoding(tmp_path, name):
    engine, raw, tensors, _ = _engine(tmp_path, name, "float32")
    rng = np.random.default_rng(3)
    tokens = [int(t) for t in rng.integers(0, raw["vocab"], 220)]
    want, noise = _oracle(raw, tensors, tokens)
    slot = engine.open()
    got = np.concatenate([engine.step([(slot, [t], [0])]).cpu().numpy() for t in tokens])
    engine.close(slot)
    assert_logits(got, want, "float32", f"{name} token by token", noise)


@pytest.mark.parametrize("dtype", BOTH)
def test_graphs_and_plain_launches_give_the_same_bits_and_states_survive_a_capture(tmp_path, dtype):
    """(bfloat16 with one row and two, the buckets of captured steps; a plain step of those rows launches the same.)"""
    from abacus_b200.engine import Engine
    engine, raw, tensors, _ = _engine(tmp_path, "A", dtype)
    eager = Engine(engine.model, max_tokens=64 * 24, use_graphs=False)
    rng = np.random.default_rng(11)
    seqs = [[int(t) for t in rng.integers(0, raw["vocab"], n)] for n in (30, 9)]
    outs = []
    for e in (engine, eager):
        slots = [e.open() for _ in seqs]
        got = [e.step([(slot, s[:5], [4]) for slot, s in zip(slots, seqs)]).cpu().numpy()]
        for i in range(5, 9):
            got.append(e.step([(slot, [s[i]], [0]) for slot, s in zip(slots, seqs)]).cpu().numpy())
        for i in range(9, 30):  # the second has ended: another graph (one row) is captured in mid-sequence
            got.append(e.step([(slots[0], [seqs[0][i]], [0])]).cpu().numpy())
        for slot in slots:
            e.close(slot)
        outs.append(np.concatenate(got))
    assert engine.graphs is not None and engine.graphs.graphs, "the engine did not replay captured graphs"
    np.testing.assert_array_equal(outs[0], outs[1])
    # prompts of a shape seen before are replayed from a captured graph, to the bits of the first run
    prompts = [[int(t) for t in rng.integers(0, raw["vocab"], n)] for n in (40, 70)]
    runs = []
    for _ in range(3):
        slots = [engine.open() for _ in prompts]
        runs.append(engine.step([(slot, s, [len(s) - 1]) for slot, s in zip(slots, prompts)]).cpu().numpy())
        for slot in slots:
            engine.close(slot)
    assert engine.prompt_graphs.replayed >= 1
    if dtype == "float32":
        np.testing.assert_array_equal(runs[0], runs[2])
    np.testing.assert_array_equal(runs[1], runs[2])


def test_greedy_generation_through_the_entry_point(tmp_path):
    from abacus_b200 import LM
    folder, raw, tensors = lm.write_folder(tmp_path, "D")
    model = LM(folder, dtype="float32", max_tokens=64 * 16)
    rng = np.random.default_rng(2)
    prompts = [[int(t) for t in rng.integers(0, raw["vocab"], n)] for n in (12, 3, 30)]
    outs = model.generate(prompts, max_new_tokens=20, temperature=0.0, stop_tokens=[])
    for p, out in zip(prompts, outs):
        assert len(out) == 20
        logits = plain.PlainLilovik(raw, tensors).forward(p + out)
        for i, t in enumerate(out):  # each token is the plain model's choice, or within rounding of it
            row = logits[len(p) + i - 1]
            assert row[t] >= row.max() - 1e-3, f"token {i}: the engine chose {t}, the plain model {int(row.argmax())}"
    again = model.generate(prompts[::-1], max_new_tokens=20, temperature=0.0, stop_tokens=[], batch_size=2)
    assert again == outs[::-1]


def test_trace_replay_of_a_model_folder(tmp_path):
    folder, raw, tensors = lm.write_folder(tmp_path, "C")
    rng = np.random.default_rng(4)
    a, b = ([int(t) for t in rng.integers(0, raw["vocab"], n)] for n in (70, 9))
    run = TraceRun(folder, "float32", tmp_path / "out", 64 * 8)
    got = run.step([("a", a[:66], [0, 65]), ("b", b[:8], [7])]).reshape(3, -1)
    more = [run.step([("a", [a[66 + i]], [0])] + ([("b", [b[8]], [0])] if i == 0 else []), end=["b"] if i == 0 else []) for i in range(4)]
    run.step([], end=["a"])
    run.close()
    (wa, noise), (wb, _) = _oracle(raw, tensors, a), _oracle(raw, tensors, b)
    assert_logits(got, np.stack([wa[0], wa[65], wb[7]]), "float32", "replayed prompt", noise)
    assert_logits(more[0].reshape(2, -1), np.stack([wa[66], wb[8]]), "float32", "replayed decode", noise)
    assert_logits(np.stack([m.reshape(-1, raw["vocab"])[0] for m in more[1:]]), wa[67:70], "float32", "replayed decode", noise)


@pytest.mark.parametrize("seed", range(12))
def test_random_configurations_against_the_plain_model(tmp_path, seed):
    rng = np.random.default_rng(200 + seed)
    raw, dtype = lm.random_config(rng), BOTH[seed % 2]
    engine, raw, tensors, _ = _engine(tmp_path, f"fuzz{seed}", dtype, raw=raw, seed=seed)
    seqs = [[int(t) for t in rng.integers(0, raw["vocab"], n)] for n in (75, 2, 130)]
    cut = [70, 1, 66]
    oracle = [_oracle(raw, tensors, s) for s in seqs]

    def check(got, want, noise, what):
        if dtype == "float32":
            assert_logits(got, want, dtype, what, noise)
        else:
            _bf16_close(got, want, what)
    slots = [engine.open() for _ in seqs]
    what = str([(l["type"], l["mixer"]) for l in raw["layers"]])
    got = engine.step([(slot, s[:c], list(range(c))) for slot, s, c in zip(slots, seqs, cut)]).cpu().numpy()
    at = 0
    for i, c in enumerate(cut):
        check(got[at:at + c], oracle[i][0][:c], oracle[i][1], f"{what} prompt {i}")
        at += c
    for step in range(3):
        live = [i for i, (s, c) in enumerate(zip(seqs, cut)) if c + step < len(s)]
        got = engine.step([(slots[i], [seqs[i][cut[i] + step]], [0]) for i in live]).cpu().numpy()
        for j, i in enumerate(live):
            check(got[j:j + 1], oracle[i][0][cut[i] + step:cut[i] + step + 1], oracle[i][1], f"{what} decode {i}")
    engine.check_status()
