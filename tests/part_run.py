"""Shared by the GPU tests of a model's parts: a mixer or a feed-forward of the registry alone, bound to given tensors with a
cache of its own, stepped with given rows; the ways a sequence may be stepped; and the bounds its outputs are held to."""
import numpy as np
import torch

from tilulorn_models import bf16_round

DEV = "cuda"
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def rounding(dtype):
    return bf16_round if dtype == "bfloat16" else (lambda a: np.asarray(a, dtype=np.float32))


def f64(p):
    return {n: (t if t.dtype.kind == "i" else t.astype(np.float64)) for n, t in p.items()}


def close(got, want, dtype, what, f32=2e-4, bf16=0.1):
    """float32: within a fraction of the largest value (sums taken in another order). bfloat16 (projections and
    activations rounded where the plain implementation rounds nothing): single values within a tenth of the largest, and
    the whole within 3 % in the root mean square."""
    want = np.asarray(want, dtype=np.float64)
    assert np.isfinite(got).all(), f"{what}: not finite"
    limit = (f32 if dtype == "float32" else bf16) * max(np.abs(want).max(), 1e-3)
    diff = np.abs(got - want)
    assert diff.max() <= limit, f"{what}: off by {diff.max():.3g} at row {int(diff.max(-1).argmax())} (limit {limit:.3g})"
    if dtype == "bfloat16" and want.size >= 64:
        rel = np.sqrt((diff ** 2).mean() / max((want ** 2).mean(), 1e-12))
        assert rel <= 0.03, f"{what}: {rel:.3g} of the root mean square away"


class PartRun:
    """A mixer or a feed-forward of the registry alone: bound to given tensors, with a cache of its own, stepped with
    given rows (and, for a feed-forward that looks at them, given token ids)."""

    def __init__(self, spec, params, dtype, feed_forward=False):
        from abacus_b200.cache import SequenceCache
        from abacus_b200.parts import FEED_FORWARDS, MIXERS, BuildContext, Workspace
        self.dtype, self.feed_forward = dtype, feed_forward
        self.part = (FEED_FORWARDS if feed_forward else MIXERS).build(spec)
        assert set(self.part.param_shapes()) == set(params), set(self.part.param_shapes()) ^ set(params)
        for n, shape in self.part.param_shapes().items():
            assert tuple(params[n].shape) == tuple(shape), (n, params[n].shape, shape)
        device = torch.device(DEV, torch.cuda.current_device())
        self.part.bind({n: torch.from_numpy(np.ascontiguousarray(t) if t.dtype.kind == "i" else np.ascontiguousarray(t, dtype=np.float32))
                        for n, t in params.items()}, BuildContext(device=device, dtype=DT[dtype]))
        self.ws = Workspace(device)
        self.cache = None
        if not feed_forward:
            self.cache = SequenceCache([self.part.cache_need()], [None], 64 * 64, DT[dtype], DEV)
            prepare = getattr(self.part, "prepare", None)
            if prepare:
                prepare(4096, device)
        self.length = {}

    def open(self, dirty=False):
        """A slot; dirty: what a former user left in its states stays there until the slot is opened again."""
        slot = self.cache.open_slot()
        if dirty:
            for state in self.cache._all_states():
                state[slot].fill_(3.0)
            self.cache.close_slot(slot)
            again = self.cache.open_slot()
            assert again == slot
        self.length[slot] = 0
        return slot

    def close(self, slot):
        self.cache.close_slot(slot)

    def step(self, entries, tokens=None):
        """entries: [(slot or None, rows [n, d])] -> [out [n, d]] float32. tokens: the rows' token ids, entry by entry."""
        from abacus_b200.engine.batch import Sequence, StepBatch
        plans = getattr(self.part, "step_plans", lambda: [])()
        n = sum(len(h) for _, h in entries)
        seqs = []
        for i, (slot, h) in enumerate(entries):
            start = self.length.get(slot, 0)
            if self.cache is not None:
                self.cache.reserve(slot, start + len(h))
                self.length[slot] = start + len(h)
            seqs.append(Sequence(slot if slot is not None else i, list(tokens[i]) if tokens is not None else [0] * len(h), start, []))
        batch = StepBatch(n, len(entries), 1, DEV, plans=plans).fill(seqs, exact=True)
        xn = torch.from_numpy(np.concatenate([np.asarray(h, dtype=np.float32) for _, h in entries])).to(DEV).to(DT[self.dtype])
        out = torch.full((n, xn.shape[1]), 7.0, dtype=torch.float32, device=DEV)
        if self.feed_forward:
            self.part.forward(xn.contiguous(), out, batch, self.ws)
        else:
            self.part.forward(xn.contiguous(), out, batch, self.cache.views[0], self.ws)
        torch.cuda.synchronize()
        got, at = out.cpu().numpy(), 0
        outs = []
        for _, h in entries:
            outs.append(got[at:at + len(h)])
            at += len(h)
        return outs


def every_way(run, h, want, dtype, what, portions=(60, 2, 7, 1, 64, 16)):
    """The rows h of one sequence: whole, in portions down to two tokens and one (None: the part takes a sequence's
    several tokens only at its start), token by token, and in an unequal batch in slots that were used before."""
    T = len(h)
    slot = run.open()
    close(run.step([(slot, h)])[0], want, dtype, f"{what}, whole")
    run.close(slot)
    if portions:
        slot, at, got = run.open(dirty=True), 0, []
        for size in portions:
            got.append(run.step([(slot, h[at:at + size])])[0])
            at += size
        assert at == T
        close(np.concatenate(got), want, dtype, f"{what}, in portions")
        run.close(slot)
    slot = run.open(dirty=True)
    got = np.concatenate([run.step([(slot, h[t:t + 1])])[0] for t in range(40)])
    close(got, want[:40], dtype, f"{what}, token by token")
    run.close(slot)
    # three sequences of the same rows: 120 of them, a single one, 70; then decoded together
    a, b, c = run.open(dirty=True), run.open(dirty=True), run.open(dirty=True)
    first = run.step([(a, h[:120]), (b, h[:1]), (c, h[:70])])
    for got, n in zip(first, (120, 1, 70)):
        close(got, want[:n], dtype, f"{what}, unequal batch, {n} rows")
    for t in range(5):
        nxt = run.step([(a, h[120 + t:121 + t]), (b, h[1 + t:2 + t]), (c, h[70 + t:71 + t])])
        for got, at in zip(nxt, (120 + t, 1 + t, 70 + t)):
            close(got, want[at:at + 1], dtype, f"{what}, decoded together at {at}", f32=5e-4)
    for s in (a, b, c):
        run.close(s)
