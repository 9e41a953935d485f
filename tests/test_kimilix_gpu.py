"""Kimilix on the GPU against the plain implementation (tests/plain/kimilix_plain.py): every mechanism alone as the part the
model uses (whole, in portions where the part takes them, token by token, in unequal batches, in slots used before), the
attention kernels on given operands, keys far away and at the edges of chunks, windows and pages, then whole models through
the engine: prompts, decoding, batches, captured graphs, greedy generation through the library's entry point, and the trace
replay."""
import numpy as np
import pytest
import torch

import kimilix_models as km
from helpers import TraceRun, assert_logits
from part_run import DEV, DT, PartRun, close, every_way, f64, rounding
from plain import kimilix_plain as plain
from tilulorn_models import bf16_round

pytestmark = pytest.mark.gpu
BOTH = ["float32", "bfloat16"]
PORTIONS = (60, 2, 7, 1, 64, 16)


# ------------------------------------------------------------------ differential attention
_SLOTS = {"wq": "q", "wk": "k", "wv": "v", "q_norm": "q.norm", "k_norm": "k.norm", "lq1": "lq1", "lk1": "lk1", "lq2": "lq2",
          "lk2": "lk2", "wo": "o"}


def _attention_run(p, d, m, dtype):
    from abacus_b200.config.kimilix import KimilixAttention
    return PartRun(KimilixAttention.from_dict("", m).to_spec(d, 1e-5), {slot: p[short] for slot, short in _SLOTS.items()}, dtype)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("H,G,K,V,chunk,rotation", [
    (4, 2, 16, 24, 48, km.rot(5000.0, 8, 4.0, 64, 1.0, 4.0)),      # a rotation over part of a map
    (3, 3, 10, 7, 20, km.rot(100.0, 6)),                            # sizes that fit no vector
    (8, 8, 64, 128, 100, km.rot(10000.0, 64, 8.0, 512, 1.0, 4.0)),
    (20, 1, 16, 16, 64, km.rot(20000.0, 16)),                       # more heads to a key head than a CTA takes
    (4, 2, 32, 136, None, None),                                    # values beyond the prompt kernel; no rotation, no chunks
    (6, 3, 128, 8, 33, km.rot(500.0, 32)), (2, 1, 24, 40, 1, km.rot(300.0, 16)), (34, 2, 8, 16, 63, km.rot(300.0, 8)),
    (2, 2, 136, 200, 70, km.rot(50.0, 128)),
])
def test_differential_attention_every_way(dtype, H, G, K, V, chunk, rotation):
    rng, rnd, d = np.random.default_rng(H + K), rounding(dtype), 40
    m = km.attention_layer(H, G, K, V, 0.5 / np.sqrt(K), 0.35, chunk, rotation)["mixer"]
    p = {n: rnd(t) for n, t in km.attention_weights(rng, d, m).items()}
    h = rnd(rng.standard_normal((150, d)))
    want, _ = plain.attention(h.astype(np.float64), m, f64(p), 1e-5, None)
    every_way(_attention_run(p, d, m, dtype), h, want, dtype, f"attention {H}/{G} x {K}, values of {V}", portions=PORTIONS)


class Rows:
    """Prepared q, k and v of a few sequences (bfloat16 numbers), the same in the step's rows and in a paged cache, and the
    float64 answer: what a kernel is held to closely, its operands being given."""

    def __init__(self, rng, lengths, H, G, K, V, chunk, lam=0.45, keep=0.7):
        from abacus_b200.cache import CacheNeed, SequenceCache
        self.sizes, self.chunk, self.lengths, self.lam, self.keep = (H, G, K, V), chunk, lengths, lam, keep
        self.scale = float(np.float32(2.0 / np.sqrt(K)))
        self.used = 2 * (H + G) * K + G * V
        self.row = -(-self.used // 8) * 8
        n = sum(lengths)
        self.rows = np.zeros((n, self.row), np.float32)
        self.rows[:, :self.used] = bf16_round(rng.standard_normal((n, self.used)))
        self.cache = SequenceCache([CacheNeed(n_kv_heads=G, head_dim=2 * K, v_head_dim=V)], [None], 64 * (sum(-(-l // 64) for l in lengths) + 4),
                                   torch.bfloat16, DEV)
        g = self.cache.groups[0]
        g.k.fill_(7.0), g.v.fill_(-9.0)  # what former users left
        self.slots, at, want = [], 0, []
        for l in lengths:
            slot = self.cache.open_slot()
            self.cache.reserve(slot, l)
            r = self.rows[at:at + l]
            k = torch.from_numpy(np.ascontiguousarray(r[:, 2 * H * K:2 * (H + G) * K])).view(l, G, 2 * K).to(DEV, torch.bfloat16)
            v = torch.from_numpy(np.ascontiguousarray(r[:, 2 * (H + G) * K:self.used])).view(l, G, V).to(DEV, torch.bfloat16)
            for j0 in range(0, l, 64):
                page, m = int(g.table_host[slot, j0 // 64]), min(64, l - j0)
                g.k[0, page, :, :m], g.v[0, page, :, :m] = k[j0:j0 + m].transpose(0, 1), v[j0:j0 + m].transpose(0, 1)
            want.append(self.answer(r[:, :self.used].astype(np.float64)))
            self.slots.append(slot)
            at += l
        self.want = want
        self.qkv = torch.from_numpy(self.rows).to(DEV, torch.bfloat16)

    def answer(self, r):
        H, G, K, V = self.sizes
        l = len(r)
        q, k = r[:, :2 * H * K].reshape(l, H, 2, K), r[:, 2 * H * K:2 * (H + G) * K].reshape(l, G, 2, K)
        v = r[:, 2 * (H + G) * K:].reshape(l, G, V)
        i, j = np.arange(l)[:, None], np.arange(l)[None, :]
        seen = (j <= i) & ((i // self.chunk == j // self.chunk) if self.chunk else True)
        a = plain.softmax_seen(np.einsum("thsk,jhsk->hstj", q, np.repeat(k, H // G, axis=1)) * self.scale, seen)
        both = np.einsum("hstj,jhv->sthv", a, np.repeat(v, H // G, axis=1))
        return (plain.over_rms(both[0] - float(np.float32(self.lam)) * both[1], 1e-5) * self.keep).reshape(l, H * V)

    def check(self, got, want, what):
        """bfloat16 outputs: within their own rounding, and what float32 sums of the size of the terms lose."""
        got = got.float().cpu().numpy()
        limit = np.abs(want) * 2.0 ** -8 + 1e-4 * max(np.abs(want).max(), 1.0)
        diff = np.abs(got - want)
        assert np.isfinite(got).all() and (diff <= limit).all(), \
            f"{what}: off by {diff.max():.3g} at {np.unravel_index(int((diff - limit).argmax()), diff.shape)}"

    def run(self, q, batch, ws, from_step=False):
        from abacus_b200.kernels import ops
        H, G, K, V = self.sizes
        out = torch.full((batch.n_rows, H * V), 5.0, dtype=q.dtype, device=DEV)
        ops.attention_differential(q, out, H, G, K, self.scale, None, batch, self.cache.views[0].kv, self.lam, 1e-5, self.keep,
                                   from_step=from_step, ws=ws, v_dim=V, row=self.row, chunk=self.chunk)
        torch.cuda.synchronize()
        return out


def _step(lengths, starts=None, slots=None):
    """A filled StepBatch of sequences that bring `lengths` tokens from positions `starts` on."""
    from abacus_b200.engine.batch import Sequence, StepBatch
    starts, slots = starts or [0] * len(lengths), slots or list(range(len(lengths)))
    seqs = [Sequence(slot, [0] * n, start, []) for slot, n, start in zip(slots, lengths, starts)]
    return StepBatch(sum(lengths), len(lengths), 1, DEV).fill(seqs, exact=True)


@pytest.mark.parametrize("H,G,K,V,chunk", [(4, 2, 64, 128, 100), (8, 8, 32, 64, 64), (3, 1, 16, 24, None), (6, 3, 128, 8, 130), (2, 2, 48, 120, 33),
                                           (20, 1, 16, 16, 256), (34, 2, 8, 40, 300), (2, 1, 24, 200, 70)])
def test_the_differential_kernels_against_float64(H, G, K, V, chunk):
    """Whole prompts (unequal sequences), portions, and decode steps of rows with one key to several parts."""
    from abacus_b200.parts import Workspace
    rng, ws = np.random.default_rng(H * K), Workspace(torch.device(DEV, torch.cuda.current_device()))
    rows = Rows(rng, [333, 1, 70, 16, 129, 260], H, G, K, V, chunk)
    rows.check(rows.run(rows.qkv, _step(rows.lengths, slots=rows.slots), ws), np.concatenate(rows.want), "prompts")
    starts = [l // 2 for l in rows.lengths]
    pick = np.concatenate([np.arange(a + s, a + l) for a, s, l in zip(np.cumsum([0] + rows.lengths), starts, rows.lengths)])
    batch = _step([l - s for l, s in zip(rows.lengths, starts)], starts, rows.slots)
    rows.check(rows.run(rows.qkv[torch.from_numpy(pick).to(DEV)].contiguous(), batch, ws), np.concatenate(rows.want)[pick], "portions")
    last = np.cumsum(rows.lengths) - 1
    for picked in ([0], list(range(6)), list(range(6)) * 40):
        batch = _step([1] * len(picked), [rows.lengths[i] - 1 for i in picked], [rows.slots[i] for i in picked])
        q = rows.qkv[torch.from_numpy(last[picked]).to(DEV)].contiguous()
        rows.check(rows.run(q, batch, ws), np.stack([rows.want[i][-1] for i in picked]), f"decode, {len(picked)} rows")


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("chunk", [64, 80, None])
def test_one_loud_key_far_away_and_at_the_edges_of_chunks_and_pages(dtype, chunk):
    """A key that one query alone agrees with, in its first map only: the head's output is that key's value's direction if
    and only if the query sees it. In prompts, and for tokens that come one by one, in used pages."""
    rng, K, V, T = np.random.default_rng(chunk or 1), 16, 8, 330
    d = 2 * K + 2 * K + V
    eye = np.eye(d)
    p = {"q": eye[:2 * K], "k": eye[2 * K:4 * K], "v": eye[4 * K:], "q.norm": np.ones(K), "k.norm": np.ones(K), "o": eye[:, :V],
         "lq1": np.zeros(K), "lk1": np.zeros(K), "lq2": np.zeros(K), "lk2": np.zeros(K)}
    p = {n: bf16_round(np.asarray(t, np.float32)) for n, t in p.items()}
    m = {"heads": 1, "kv_heads": 1, "dim": K, "vdim": V, "scale": 1.0, "diff": 0.25}
    if chunk:
        m["mask"] = {"size": chunk}
    u = rng.standard_normal(K)
    u /= np.linalg.norm(u)
    run = _attention_run(p, d, m, dtype)
    pairs = {(T - 1, j) for j in (0, 1, 63, 64, 65, 127, 128, 255, 256, 319, 320, T - 2)} | {(200, 127), (200, 128), (129, 128), (70, 70)}
    for i in (2 * (chunk or 64), 2 * (chunk or 64) - 1, T - 1):
        start = i // (chunk or 64) * (chunk or 64)
        pairs |= {(i, start), (i, start - 1), (i, i)}
    for i, j in sorted(pairs):
        h = rng.standard_normal((T, d)) * 0.3
        h[:, 2 * K:3 * K] -= np.outer(h[:, 2 * K:3 * K] @ u, u)  # (the norm levels the keys' sizes: the others point elsewhere)
        h[i, :K] = 4.0 * u
        h[j, 2 * K:3 * K] = 4.0 * u
        h[j, 4 * K:] *= 20.0
        h = rounding(dtype)(h)
        want, _ = plain.attention(h.astype(np.float64), m, f64(p), 1e-5, None)
        value = h[j, 4 * K:].astype(np.float64)
        cosine = want[i, :V] @ value / np.linalg.norm(want[i, :V]) / np.linalg.norm(value)
        seen = chunk is None or i // chunk == j // chunk
        if i != j:
            assert (cosine > 0.95) == seen, (i, j, cosine)
        run.cache.views[0].kv.k.fill_(9.0), run.cache.views[0].kv.v.fill_(9.0)  # what former users left in the pages
        slot = run.open(dirty=True)
        close(run.step([(slot, h[:i + 1])])[0], want[:i + 1], dtype, f"query {i}, loud key {j}, prompt", bf16=0.15)
        run.close(slot)
        slot, cut = run.open(dirty=True), max(1, i - 3 if j < i - 3 else j - 1)
        got = [run.step([(slot, h[:cut])])[0]] + [run.step([(slot, h[t:t + 1])])[0] for t in range(cut, i + 1)]
        close(np.concatenate(got), want[:i + 1], dtype, f"query {i}, loud key {j}, decoded from {cut}", bf16=0.15)
        run.close(slot)


def test_the_second_map_counts_by_its_own_factor_and_the_norms_belong_to_their_maps():
    """Against the plain function (held to written-out weights on the CPU), with the factor far from the constant, swapped
    vectors, and one map's projection scaled, which its own norm takes away and no other sees."""
    rng, d = np.random.default_rng(8), 32
    m = km.attention_layer(4, 2, 8, 8, 0.4, 0.6, 33, km.rot(100.0, 8))["mixer"]
    p = {n: rounding("float32")(t) for n, t in km.attention_weights(rng, d, m).items()}
    p["lq1"], p["lk1"], p["lq2"], p["lk2"] = (np.full(8, v, np.float32) for v in (0.5, 0.25, -0.25, 0.375))
    h = rng.standard_normal((100, d)).astype(np.float32)
    want, _ = plain.attention(h.astype(np.float64), m, f64(p), 1e-5, None)
    run = _attention_run(p, d, m, "float32")
    assert run.part.lam == pytest.approx(np.exp(1.0) - np.exp(-0.75) + 0.6, rel=1e-6)
    slot = run.open()
    close(run.step([(slot, h)])[0], want, "float32", "a factor above two")
    for swapped in (dict(lq1=p["lq2"], lq2=p["lq1"]), dict(lk2=-p["lk2"])):
        other, _ = plain.attention(h.astype(np.float64), m, f64(dict(p, **swapped)), 1e-5, None)
        assert np.abs(other - want).max() > 0.05
    scaled = dict(p, q=p["q"] * np.repeat([1.0, 7.0, 1, 1, 1, 1, 1, 1], 8)[:, None].astype(np.float32))
    again, _ = plain.attention(h.astype(np.float64), m, f64(scaled), 1e-5, None)
    np.testing.assert_allclose(again, want, rtol=1e-2, atol=1e-3)
    run = _attention_run(scaled, d, m, "float32")
    close(run.step([(run.open(), h)])[0], again, "float32", "one map's projection scaled")


# ------------------------------------------------------------------ latent attention under a window
_LATENT_SLOTS = {"wdq": "dq", "q_norm": "dq.norm", "wq": "uq", "wdown": "dkv", "down_norm": "dkv.norm", "wuk": "uk", "wuv": "uv", "wo": "o"}


def _latent_run(p, d, m, dtype):
    from abacus_b200.config.kimilix import KimilixLatent
    return PartRun(KimilixLatent.from_dict("", m).to_spec(d, 1e-5), {slot: p[short] for slot, short in _LATENT_SLOTS.items()}, dtype)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("sizes,window,rotation", [
    ((3, 16, 8, 24, 24, 32), 40, km.rot(10000.0, 8)),
    ((2, 10, 6, 7, 21, 9), 9, km.rot(100.0, 6)),                       # sizes that fit no vector
    ((5, 40, 24, 40, 136, 64), 130, km.rot(10000.0, 24)),
    ((20, 16, 16, 8, 64, 40), 64, km.rot(50000.0, 16)),                 # more heads than a CTA takes; a window of a page
    ((4, 8, 8, 24, 40, 16), None, None),
    ((17, 64, 64, 128, 192, 96), 65, km.rot(50000.0, 64, 4.0, 64, 1.0, 4.0)),
    ((2, 16, 4, 144, 260, 32), 63, km.rot(100.0, 4)),                   # rows beyond the decode kernel, values beyond the prompt kernel
    ((3, 8, 16, 8, 32, 24), 1, km.rot(100.0, 12)), ((6, 32, 16, 72, 48, 32), 2, km.rot(100.0, 16)),
])
def test_latent_attention_under_a_window_every_way(dtype, sizes, window, rotation):
    H, K, R, V, rank, qr = sizes
    rng, rnd, d = np.random.default_rng(K + R), rounding(dtype), 48
    m = km.latent_layer(H, K, R, V, rank, qr, 0.8 / np.sqrt(K + R), window, rotation)["mixer"]
    p = {n: rnd(t) for n, t in km.latent_weights(rng, d, m).items()}
    h = rnd(rng.standard_normal((150, d)))
    want, _ = plain.latent_attention(h.astype(np.float64), m, f64(p), 1e-5, None)
    # (with a window the part takes several tokens of a sequence only at its start: no portions)
    every_way(_latent_run(p, d, m, dtype), h, want, dtype, f"latent attention {sizes}, window {window}",
              portions=PORTIONS if window is None else None)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("window,row", [(5, 16), (64, 24), (80, 24), (130, 64), (None, 24)])
def test_one_loud_key_just_inside_and_just_outside_the_window(window, row, dtype):
    """A key made loud for one query alone through the unrotated parts (queries and keys read input columns of their own):
    the oldest key the window still holds, the first it has dropped, both sides of pages' borders, the token's own; in a
    prompt and for tokens that come one by one over a ring of pages that has gone round."""
    rng, T, rank = np.random.default_rng(window or 3), 300, row - 8
    d = 16 + 24
    m = {"heads": 2, "dim": 8, "rot_dim": 8, "vdim": 8, "kv_rank": rank, "q_rank": 8, "scale": 1.0, "rot": km.rot(10000.0, 8)}
    if window is not None:
        m["mask"] = {"size": window}
    p = km.latent_weights(rng, d, m)
    p["dq"], p["dq.norm"], p["dkv.norm"] = np.eye(d)[:8], np.ones(8), np.ones(rank)
    p["uq"] = np.zeros((32, 8))
    p["uq"][:8] = p["uq"][16:24] = np.eye(8) * 2
    p["dkv"] *= 0.5
    p["dkv"][:8] = 0
    p["dkv"][:8, 8:16] = np.eye(8)  # the first eight latents are input columns 8..16
    p["uk"] = np.zeros((16, rank))
    p["uk"][:8, :8] = p["uk"][8:, :8] = np.eye(8) * 2
    p = {n: bf16_round(np.asarray(t, np.float32)) for n, t in p.items()}
    u = rng.standard_normal(8)
    u /= np.linalg.norm(u)
    run, pairs, W = _latent_run(p, d, m, dtype), set(), window or 64
    for i in (W - 1, W, 2 * W + 3, 192, T - 1):
        if W - 1 <= i < T:
            pairs |= {(i, i - W + 1), (i, i - W), (i, i), (i, i - 1), (i, max(i - W + 1, i // 64 * 64)), (i, max(i - W + 1, i // 64 * 64 - 1))}
    if window is None:
        pairs |= {(T - 1, j) for j in (0, 1, 63, 64, 65, 127, 128)}
    for i, j in sorted((i, j) for i, j in pairs if j >= 0):
        h = rng.standard_normal((T, d)) * 0.3
        h[:, :16] *= 0.2
        h[i, :8] = 3.0 * u
        h[j, 8:16] = 8.0 * u
        h = rounding(dtype)(h)
        want, _ = plain.latent_attention(h.astype(np.float64), m, f64(p), 1e-5, None)
        quiet = h.copy()
        quiet[j, 8:16] = 0.0
        without, _ = plain.latent_attention(quiet.astype(np.float64), m, f64(p), 1e-5, None)
        seen = window is None or i - j < window
        assert (np.abs(want[i] - without[i]).max() > 0.2) == seen, (i, j)
        run.cache.views[0].kv.k.fill_(9.0)  # what former users left in the pages
        slot = run.open(dirty=True)
        close(run.step([(slot, h[:i + 1])])[0], want[:i + 1], dtype, f"query {i}, loud key {j}, prompt")
        run.close(slot)
        if window is not None and i - j not in (window - 1, window, 0):  # one by one: the window's far edge and the token's own
            continue
        slot, cut = run.open(dirty=True), max(1, min(i - 3, j - 1))
        got = [run.step([(slot, h[:cut])])[0]] + [run.step([(slot, h[t:t + 1])])[0] for t in range(cut, i + 1)]
        close(np.concatenate(got), want[:i + 1], dtype, f"query {i}, loud key {j}, decoded from {cut}")
        run.close(slot)


def test_latent_decode_steps_of_many_rows_and_of_many_keys():
    """Parts of 64 keys (few rows) and of 128 (many), with up to 40 parts to fold, in more rows than one tile of eight."""
    rng, d = np.random.default_rng(4), 48
    m = km.latent_layer(4, 16, 16, 24, 48, 32, 0.25, None, km.rot(50000.0, 16))["mixer"]
    p = {n: bf16_round(t) for n, t in km.latent_weights(rng, d, m).items()}
    h = bf16_round(rng.standard_normal((2600, d)))
    want, _ = plain.latent_attention(h.astype(np.float64), m, f64(p), 1e-5, None)
    run = _latent_run(p, d, m, "bfloat16")
    slot = run.open()
    close(run.step([(slot, h[:2598])])[0], want[:2598], "bfloat16", "a long prompt")
    for t in (2598, 2599):
        close(run.step([(slot, h[t:t + 1])])[0], want[t:t + 1], "bfloat16", f"token {t}")
    run.close(slot)
    slots, lengths = [run.open() for _ in range(21)], [1 + 7 * i for i in range(21)]
    run.step([(s, h[:n]) for s, n in zip(slots, lengths)])
    for s, n, got in zip(slots, lengths, run.step([(s, h[n:n + 1]) for s, n in zip(slots, lengths)])):
        close(got, want[n:n + 1], "bfloat16", f"row of {n + 1} keys")


def test_several_tokens_of_a_windowed_sequence_after_its_start_are_refused():
    from abacus_b200.kernels.ops import KernelRefused
    rng, d = np.random.default_rng(1), 24
    m = km.latent_layer(2, 8, 8, 8, 16, 8, 0.3, 20, km.rot(100.0, 8))["mixer"]
    run = _latent_run({n: bf16_round(t) for n, t in km.latent_weights(rng, d, m).items()}, d, m, "float32")
    slot, h = run.open(), rng.standard_normal((10, d)).astype(np.float32)
    run.step([(slot, h[:5])])
    with pytest.raises(KernelRefused, match="only at its start"):
        run.step([(slot, h[5:8])])


@pytest.mark.parametrize("rows,K,count,n", [(1, 32, 32, 40), (8, 64, 57, 300), (9, 96, 96, 4800), (16, 768, 768, 64), (5, 2048, 2041, 24)])
def test_a_product_that_norms_its_rows_on_the_way(rows, K, count, n):
    from abacus_b200.kernels import ops
    rng = np.random.default_rng(K)
    x = np.zeros((rows, K + 8), np.float32)
    x[:, :count] = bf16_round(rng.standard_normal((rows, count)) * 3)
    w, nw = bf16_round(rng.standard_normal((n, K)) / np.sqrt(K)), (1 + rng.standard_normal(count) * 0.3).astype(np.float32)
    xd = torch.from_numpy(x).to(DEV, torch.bfloat16)[:, :K]
    out = torch.full((rows, n), 7.0, dtype=torch.bfloat16, device=DEV)
    assert ops.gemm_rows_normed_takes(xd, torch.from_numpy(w).to(DEV, torch.bfloat16), out, rows, count)
    ops.gemm_rows_normed(xd, torch.from_numpy(w).to(DEV, torch.bfloat16), out, torch.from_numpy(nw).to(DEV), 1e-5, rows)
    want = plain.over_rms(x[:, :count].astype(np.float64), 1e-5) * nw @ w[:, :count].astype(np.float64).T
    diff = np.abs(out.float().cpu().numpy() - want)
    assert diff.max() <= 2e-2 * max(np.abs(want).max(), 1.0), diff.max()


# ------------------------------------------------------------------ feed-forwards
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("rows,d,ff", [(1, 64, 128), (5, 37, 9), (16, 96, 256), (40, 64, 48), (200, 512, 96), (300, 64, 256), (300, 64, 72), (2100, 256, 2304)])
def test_the_square_of_relu_in_every_form_of_the_product(dtype, rows, d, ff):
    from abacus_b200.config.specs import PlainMLPSpec
    rng, rnd = np.random.default_rng(rows + ff), rounding(dtype)
    w = {"up": rnd(rng.standard_normal((ff, d)) / np.sqrt(d)), "down": rnd(rng.standard_normal((d, ff)) / np.sqrt(ff))}
    run = PartRun(PlainMLPSpec(hidden=d, inter=ff), w, dtype, feed_forward=True)
    h = rnd(rng.standard_normal((rows, d)))
    close(run.step([(None, h)])[0], plain.dense(h.astype(np.float64), f64(w)), dtype, f"{rows} x {d} x {ff}")


def test_the_square_of_relu_in_every_configuration_of_the_tensor_core_product():
    """Swapped and not, split along K through a cluster and through scratch memory, persistent, pairs of CTAs."""
    from abacus_b200.kernels import ops
    rng = np.random.default_rng(0)
    for m, n, k, how in ((24, 200, 1024, {}), (24, 200, 1024, dict(splits=4)), (40, 130, 2048, dict(splits=8)), (100, 300, 640, dict(swap=0)),
                         (100, 520, 1024, dict(swap=0, tile_n=256, splits=3)), (700, 260, 192, dict(persistent=1)), (600, 600, 320, dict(persistent=2)),
                         (90, 64, 512, dict(swap=0, splits=2))):
        x, w = bf16_round(rng.standard_normal((m, k))), bf16_round(rng.standard_normal((n, k)) / np.sqrt(k))
        want = np.maximum(x.astype(np.float64) @ w.astype(np.float64).T, 0) ** 2
        for dt, tol in ((torch.float32, 2e-5), (torch.bfloat16, 8e-3)):
            out = torch.full((m, n), 7.0, dtype=dt, device=DEV)
            ops.gemm_tc(torch.from_numpy(x).to(DEV, torch.bfloat16), torch.from_numpy(w).to(DEV, torch.bfloat16), out, activation="relu_squared", **how)
            diff = np.abs(out.float().cpu().numpy() - want)
            assert diff.max() <= tol * want.max(), (m, n, k, how, dt, diff.max())


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("rows,d,ff,limit", [(1, 64, 128, 1.0), (5, 37, 9, 0.5), (16, 96, 256, 7.0), (40, 64, 48, 1.5), (300, 64, 256, 1.0), (300, 64, 72, 2.0)])
def test_a_gated_feed_forward_with_bounds_in_every_form(dtype, rows, d, ff, limit):
    from abacus_b200.config.specs import GatedMLPSpec
    rng, rnd = np.random.default_rng(rows + ff), rounding(dtype)
    w = {"gate": rnd(rng.standard_normal((ff, d)) * 2 / np.sqrt(d)), "up": rnd(rng.standard_normal((ff, d)) * 2 / np.sqrt(d)),
         "down": rnd(rng.standard_normal((d, ff)) / np.sqrt(ff))}
    run = PartRun(GatedMLPSpec(hidden=d, inter=ff, activation="clamped_silu", limit=limit), w, dtype, feed_forward=True)
    h = rnd(rng.standard_normal((rows, d)))
    close(run.step([(None, h)])[0], plain.expert(h.astype(np.float64), f64(w), limit), dtype, f"{rows} x {d} x {ff}")


_NAMES = {"router": "router", "router_bias": "router.b", "shared_gate_proj": "shared.gate", "shared_up": "shared.up",
          "shared_down": "shared.down", "shared_gate": "shared.sg"}


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("d,mlp", [
    (64, km.experts(5, 2, 64, 1.0, (40, 2.0))), (37, km.experts(3, 3, 9, 0.7)), (48, km.experts(1, 1, 24, 2.0, (128, 0.5))),
    (128, km.experts(16, 4, 192, 1.5, (192, 1.5))), (40, km.experts(20, 6, 12, 3.0, (5, 1.0))), (72, km.experts(7, 1, 128, 0.5, (56, 7.0))),
])
def test_routed_experts_with_a_bias_bounds_and_a_gated_shared_one(dtype, d, mlp):
    from abacus_b200.config.kimilix import KimilixExperts
    rng, rnd = np.random.default_rng(d), rounding(dtype)
    p = {n: rnd(t) for n, t in km.ff_weights(rng, d, mlp).items()}
    E, top = mlp["router"]["experts"], mlp["router"]["top"]
    spec = KimilixExperts.from_dict("", mlp).to_spec(d)
    params = {slot: p[short] for slot, short in _NAMES.items() if short in p}
    for e in range(E):
        params.update({f"{slot}{e}": p[f"e{e}.{slot}"] for slot in ("gate", "up", "down")})
    run = PartRun(spec, params, dtype, feed_forward=True)
    for n in (1, 9, 70, 300, 700):  # a decode step, a few rows, the products sorted by expert, the router's rows read once for four tokens
        h = rnd(rng.standard_normal((n, d)))
        z = np.sort(h.astype(np.float64) @ p["router"].astype(np.float64).T + p["router.b"], axis=-1)[:, ::-1]
        clear = (z[:, top - 1] - z[:, min(top, E - 1)] > 1e-3) | (top == E)  # rows whose choice is no close call
        want = plain.experts(h.astype(np.float64), mlp, f64(p))
        cut = n // 3
        got = np.concatenate(run.step([(None, h[:cut]), (None, h[cut:])] if cut else [(None, h)]))
        assert clear.mean() > 0.9
        close(got[clear], want[clear], dtype, f"{top} of {E} experts, {n} rows")


@pytest.mark.parametrize("d", [5, 36, 64, 1024, 2560, 5000])
def test_a_branch_normed_and_added_for_a_branch_that_reads_the_stream_itself(d):
    from abacus_b200.config.specs import NormSpec
    from abacus_b200.parts import NORMS, BuildContext
    from abacus_b200.parts.norm import read_normed
    rng = np.random.default_rng(d)
    x, y = rng.standard_normal((9, d)).astype(np.float32) * 3, rng.standard_normal((9, d)).astype(np.float32) * 0.01
    w, gain = (rng.standard_normal(d) * 0.3).astype(np.float32), (1 + rng.standard_normal(d) * 0.3).astype(np.float32)
    norm = NORMS.build(NormSpec(d, 1e-4, one_plus=True, gain=True, mult=0.4))
    assert set(norm.param_shapes()) == {"weight", "gain"}
    norm.bind({"weight": torch.from_numpy(w), "gain": torch.from_numpy(gain)}, BuildContext(torch.device(DEV), torch.float32))
    summed = x + 0.4 * gain * plain.norm(y.astype(np.float64), w, 1e-4)
    for dt, tol in ((torch.float32, 3e-6), (torch.bfloat16, 8e-3)):
        xs, ys, out = (torch.from_numpy(t).to(DEV) for t in (x, y)), None, torch.full((9, d), 7.0, dtype=dt, device=DEV)
        xs, ys = xs
        read_normed(xs, (ys, norm), None, out, n_rows=9)
        np.testing.assert_allclose(xs.cpu().numpy(), summed, rtol=2e-6, atol=3e-6)
        np.testing.assert_allclose(out.float().cpu().numpy(), summed, rtol=tol, atol=3e-6)
        rows = torch.tensor([4, 0, 4], dtype=torch.int32, device=DEV)
        xs = torch.from_numpy(x).to(DEV)
        read_normed(xs, (ys, norm), None, out, rows=rows, n_rows=3)
        np.testing.assert_allclose(out[:3].float().cpu().numpy(), summed[[4, 0, 4]], rtol=tol, atol=3e-6)
        read_normed(xs, None, None, out, n_rows=9)
        np.testing.assert_allclose(out.float().cpu().numpy(), x, rtol=tol)
        assert np.array_equal(xs.cpu().numpy(), x)


# ------------------------------------------------------------------ whole models through the engine
def _engine(tmp, name, dtype, raw=None, seed=0, tensors=None, **kw):
    from abacus_b200.engine import Engine, load_model
    folder, raw, tensors = km.write_folder(tmp, name, seed=seed, raw=raw, tensors=tensors)
    return Engine(load_model(folder, dtype), max_tokens=64 * 24, **kw), raw, tensors, folder


def _oracle(raw, tensors, tokens):
    """(the plain model's logits in float64, the noise float32 itself shows on them)."""
    want = plain.PlainKimilix(raw, tensors).forward(tokens)
    return want, float(np.abs(want - plain.PlainKimilix(raw, tensors, real=np.float32).forward(tokens)).max())


class Bf16Count:
    """bfloat16 against float64: the distance of two roundings of one model, a few per cent of the logits' spread. A rounded
    router input now and then chooses another expert where two logits nearly tie, and that position's logits, and those
    that attend to it, then differ by much: such positions are counted, and few are allowed over a whole test."""

    def __init__(self):
        self.rows = self.far = 0

    def add(self, got, want, what):
        d = got - want
        d = d - d.mean(-1, keepdims=True)
        rel = np.sqrt((d * d).mean(-1)) / want.std()
        assert np.isfinite(got).all(), f"{what}: not finite"
        self.rows += len(rel)
        self.far += int((rel >= 0.25).sum())
        if len(rel) >= 20:
            assert np.median(rel) < 0.08, f"{what}: bfloat16 logits are {np.median(rel):.3g} of the spread away in the median"

    def settle(self, what):
        assert self.far <= 0.05 * self.rows, f"{what}: {self.far} of {self.rows} positions' bfloat16 logits are far away"


class Check:
    def __init__(self, dtype):
        self.dtype, self.count = dtype, Bf16Count()

    def __call__(self, got, want, noise, what):
        if self.dtype == "float32":
            assert_logits(got, want, "float32", what, noise)
        else:
            self.count.add(got, want, what)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", list(km.CONFIGS))
def test_prompts_decoding_batches_and_used_slots_against_the_plain_model(tmp_path, name, dtype):
    engine, raw, tensors, _ = _engine(tmp_path, name, dtype)
    rng, check = np.random.default_rng(7), Check(dtype)
    lens = [150, 1, 37, 80]
    seqs = [[int(t) for t in rng.integers(0, raw["vocab"], n)] for n in lens]
    oracle = [_oracle(raw, tensors, s) for s in seqs]
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
    check.count.settle(name)
    engine.check_status()


@pytest.mark.parametrize("dtype", BOTH)
def test_portions_of_a_prompt(tmp_path, dtype):
    """(of a model whose latent layers see every earlier key: a windowed one takes whole prompts and single tokens)"""
    raw = km.config("C")
    raw["layers"][1]["mixer"].pop("mask")
    engine, raw, tensors, _ = _engine(tmp_path, "C", dtype, raw=raw)
    tokens = [int(t) for t in np.random.default_rng(5).integers(0, raw["vocab"], 140)]
    want, noise = _oracle(raw, tensors, tokens)
    slot, got, at, check = engine.open(), [], 0, Check(dtype)
    for size in (60, 2, 7, 1, 64, 6):
        got.append(engine.step([(slot, tokens[at:at + size], list(range(size)))]).cpu().numpy())
        at += size
    assert at == len(tokens)
    check(np.concatenate(got), want, noise, "in portions")
    check.count.settle("portions")


@pytest.mark.parametrize("name", ["A", "D"])
def test_token_by_token_from_the_first_token_and_long_decoding(tmp_path, name):
    engine, raw, tensors, _ = _engine(tmp_path, name, "float32")
    tokens = [int(t) for t in np.random.default_rng(3).integers(0, raw["vocab"], 220)]
    want, noise = _oracle(raw, tensors, tokens)
    slot = engine.open()
    got = np.concatenate([engine.step([(slot, [t], [0])]).cpu().numpy() for t in tokens])
    engine.close(slot)
    assert_logits(got, want, "float32", f"{name} token by token", noise)


@pytest.mark.parametrize("dtype", BOTH)
def test_graphs_and_plain_launches_give_the_same_bits(tmp_path, dtype):
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
    np.testing.assert_array_equal(runs[1], runs[2])


def test_greedy_generation_through_the_entry_point(tmp_path):
    from abacus_b200 import LM
    folder, raw, tensors = km.write_folder(tmp_path, "D")
    model = LM(folder, dtype="float32", max_tokens=64 * 16)
    rng = np.random.default_rng(2)
    prompts = [[int(t) for t in rng.integers(0, raw["vocab"], n)] for n in (12, 3, 30)]
    outs = model.generate(prompts, max_new_tokens=20, temperature=0.0, stop_tokens=[])
    for p, out in zip(prompts, outs):
        assert len(out) == 20
        logits = plain.PlainKimilix(raw, tensors).forward(p + out)
        for i, t in enumerate(out):  # each token is the plain model's choice, or within rounding of it
            row = logits[len(p) + i - 1]
            assert row[t] >= row.max() - 1e-3, f"token {i}: the engine chose {t}, the plain model {int(row.argmax())}"
    again = model.generate(prompts[::-1], max_new_tokens=20, temperature=0.0, stop_tokens=[], batch_size=2)
    assert again == outs[::-1]


def test_trace_replay_of_a_model_folder(tmp_path):
    folder, raw, tensors = km.write_folder(tmp_path, "C")
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


@pytest.mark.parametrize("seed", range(14))
def test_random_configurations_against_the_plain_model(tmp_path, seed):
    rng = np.random.default_rng(300 + seed)
    raw, dtype = km.random_config(rng), BOTH[seed % 2]
    engine, raw, tensors, _ = _engine(tmp_path, f"fuzz{seed}", dtype, raw=raw, seed=seed)
    seqs = [[int(t) for t in rng.integers(0, raw["vocab"], n)] for n in (75, 2, 130)]
    cut, check = [70, 1, 66], Check(dtype)
    oracle = [_oracle(raw, tensors, s) for s in seqs]
    slots = [engine.open() for _ in seqs]
    what = str([(l["type"], l["mixer"], l["mlp"]) for l in raw["layers"]])
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
    check.count.settle(what)
    engine.check_status()
