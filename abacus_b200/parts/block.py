"""A layer: two norms, a mixer and a feed-forward, wired as src/model.c:292-310.

pre_norm:  x += y;  xn = norm1(x);  y = mixer(xn);  x += y;  xn = norm2(x);  y = ffn(xn)
The last y is handed on and added by whoever norms next (the next block or the
final norm), as abacus's add_norm does (src/model.c:297, 311).

sandwich_norm:  x += norm1b(mixer(norm1(x)));  x += norm2b(ffn(norm2(x)))   (the second branch may be absent)
A branch's output is handed on with its norm, (y, norm), and whoever norms next does the norm behind the branch, the sum
and its own norm in one kernel.

post_norm:  x += norm1(mixer(x));  x += norm2(ffn(x))   (the second branch may be absent)
The same with branches that read the stream itself (in the compute type): the kernel between two branches norms what is
pending, adds it and leaves the stream for the next branch.
"""
import torch

from .base import BLOCKS, FEED_FORWARDS, MIXERS, NORMS
from .norm import read_normed


@BLOCKS.register("pre_norm")
class PreNormBlock:
    def __init__(self, spec):
        self.spec = spec
        self.mixer_norm = NORMS.build(spec.mixer_norm)
        self.mixer = MIXERS.build(spec.mixer)
        self.ffn_norm = NORMS.build(spec.ffn_norm)
        self.ffn = FEED_FORWARDS.build(spec.ffn)

    def parts(self):
        return {"mixer_norm": self.mixer_norm, "mixer": self.mixer, "ffn_norm": self.ffn_norm, "ffn": self.ffn}

    def bind(self, params, ctx):
        """params: {part name: {slot: tensor}}."""
        self.ctx = ctx
        for name, part in self.parts().items():
            part.bind(params[name], ctx)

    def forward(self, x, y, batch, cache, ws):
        n, d = batch.n_rows, x.shape[1]
        xn = ws.get("xn", (n, d), self.ctx.dtype)
        out = ws.get("branch", (n, d), x.dtype)
        self.mixer_norm.forward(x, y, xn, n_rows=n)
        self.mixer.forward(xn, out, batch, cache, ws)
        self.ffn_norm.forward(x, out, xn, n_rows=n)
        self.ffn.forward(xn, out, batch, ws)
        return out


@BLOCKS.register("sandwich_norm")
class SandwichBlock:
    def __init__(self, spec):
        self.spec = spec
        self.mixer_norm = NORMS.build(spec.mixer_norm)
        self.mixer = MIXERS.build(spec.mixer)
        self.mixer_post_norm = NORMS.build(spec.mixer_post_norm)
        self.has_ffn = spec.ffn is not None
        if self.has_ffn:
            self.ffn_norm = NORMS.build(spec.ffn_norm)
            self.ffn = FEED_FORWARDS.build(spec.ffn)
            self.ffn_post_norm = NORMS.build(spec.ffn_post_norm)

    def parts(self):
        parts = {"mixer_norm": self.mixer_norm, "mixer": self.mixer, "mixer_post_norm": self.mixer_post_norm}
        if self.has_ffn:
            parts.update(ffn_norm=self.ffn_norm, ffn=self.ffn, ffn_post_norm=self.ffn_post_norm)
        return parts

    def bind(self, params, ctx):
        """params: {part name: {slot: tensor}}."""
        self.ctx = ctx
        for name, part in self.parts().items():
            part.bind(params[name], ctx)

    def forward(self, x, pending, batch, cache, ws):
        """x float32 [tokens, d]; pending: (the branch's output not yet added, its norm) or None. Returns this block's."""
        n, d = batch.n_rows, x.shape[1]
        xn = ws.get("xn", (n, d), self.ctx.dtype)
        # one branch buffer serves: what is pending is read by the next norm, which runs (in stream order) before the
        # next branch writes the buffer again
        out = ws.get("branch", (n, d), torch.float32)
        self.mixer_norm.forward_normed(x, pending, xn, n_rows=n)
        self.mixer.forward(xn, out, batch, cache, ws)
        if not self.has_ffn:
            return out, self.mixer_post_norm
        self.ffn_norm.forward_normed(x, (out, self.mixer_post_norm), xn, n_rows=n)
        self.ffn.forward(xn, out, batch, ws)
        return out, self.ffn_post_norm


@BLOCKS.register("post_norm")
class PostNormBlock:
    def __init__(self, spec):
        self.spec = spec
        self.mixer = MIXERS.build(spec.mixer)
        self.mixer_post_norm = NORMS.build(spec.mixer_post_norm)
        self.has_ffn = spec.ffn is not None
        if self.has_ffn:
            self.ffn = FEED_FORWARDS.build(spec.ffn)
            self.ffn_post_norm = NORMS.build(spec.ffn_post_norm)

    def parts(self):
        parts = {"mixer": self.mixer, "mixer_post_norm": self.mixer_post_norm}
        if self.has_ffn:
            parts.update(ffn=self.ffn, ffn_post_norm=self.ffn_post_norm)
        return parts

    def bind(self, params, ctx):
        """params: {part name: {slot: tensor}}."""
        self.ctx = ctx
        for name, part in self.parts().items():
            part.bind(params[name], ctx)

    def forward(self, x, pending, batch, cache, ws):
        """x float32 [tokens, d]; pending: (the branch's output not yet added, its norm) or None. Returns this block's."""
        n, d = batch.n_rows, x.shape[1]
        xn = ws.get("xn", (n, d), self.ctx.dtype)
        # one branch buffer serves: what is pending is read by the next read_normed, which runs (in stream order) before
        # the next branch writes the buffer again
        out = ws.get("branch", (n, d), torch.float32)
        read_normed(x, pending, None, xn, n_rows=n)
        self.mixer.forward(xn, out, batch, cache, ws)
        if not self.has_ffn:
            return out, self.mixer_post_norm
        read_normed(x, (out, self.mixer_post_norm), None, xn, n_rows=n)
        self.ffn.forward(xn, out, batch, ws)
        return out, self.ffn_post_norm
