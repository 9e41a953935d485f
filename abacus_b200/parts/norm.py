"""RMSNorm fused with the residual add that precedes it (src/model.c:238-244, 164-169)."""
import torch

from ..kernels import ops
from .base import NORMS, to_device


@NORMS.register("rmsnorm")
class RMSNorm:
    capturable = True  # its forward launches kernels only; nothing in it depends on the step's contents

    def __init__(self, spec):
        self.spec = spec
        self.weight = None

    def param_shapes(self):
        shapes = {"weight": (self.spec.size,)}
        if getattr(self.spec, "gain", False):
            shapes["gain"] = (self.spec.size,)
        return shapes

    def bind(self, params, ctx):
        self.weight = to_device(params["weight"], ctx, torch.float32)
        if getattr(self.spec, "one_plus", False):  # stored around zero: the kernels multiply by 1 + w, made once in float32
            self.weight = (self.weight + 1.0).contiguous()
        if "gain" in params:  # factors behind the norm are part of its weight
            self.weight = (self.weight * to_device(params["gain"], ctx, torch.float32)).contiguous()
        if getattr(self.spec, "mult", 1.0) != 1.0:
            self.weight = (self.weight * self.spec.mult).contiguous()

    def step_weights(self):
        return [self.weight]

    def forward(self, x, y, out, rows=None, n_rows=None):
        ops.add_rmsnorm(x, y, self.weight, out, self.spec.eps, rows=rows, n_rows=n_rows)
        return out

    def forward_normed(self, x, pending, out, rows=None, n_rows=None):
        """As forward(), where what is added to the stream has a norm of its own: pending is (y, that RMSNorm) or None."""
        return read_normed(x, pending, self, out, rows=rows, n_rows=n_rows)


def read_normed(x, pending, norm, out, rows=None, n_rows=None):
    """x += the pending branch, normed (pending: (y, its RMSNorm) or None); out = norm(x), or x as it is without a norm."""
    y, post = pending if pending is not None else (None, None)
    ops.normed_add_rmsnorm(x, y, post.weight if post is not None else None, post.spec.eps if post is not None else 0.0,
                           norm.weight if norm is not None else None, out, norm.spec.eps if norm is not None else 0.0,
                           rows=rows, n_rows=n_rows)
    return out
