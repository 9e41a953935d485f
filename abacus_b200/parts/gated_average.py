"""A recurrent mixer: a running average per channel, a minimal gated recurrent unit (config.specs.GatedAverageSpec).

Channel by channel a float32 state S, zero at a sequence's start and carried from token to token:
    z = sigmoid(Wz x + bz);    u = Wu x + bu;    c = u + 1/2 where u >= 0, sigmoid(u) where u < 0
    S <- (1 - z) S + z c;      out = Wo (S * silu(Wg x))
The gate and the candidate read the current token alone, so one stacked product makes everything the recurrence needs. The
mixer keeps no keys: its cache is the state. Gates, candidates, state and the output's gate are float32 in both number
formats (from the product's output on).
"""
import torch

from ..cache.need import CacheNeed
from ..kernels import ops
from .base import MIXERS, to_device
from .linear import Linear


def _up8(n):
    return -(-n // 8) * 8


@MIXERS.register("gated_average")
class GatedAverage:
    capturable = True  # its forward launches kernels only; nothing in it depends on the step's contents

    def __init__(self, spec):
        s = self.spec = spec
        if s.width < 1:
            raise ValueError(f"a width of {s.width}")
        self.block = _up8(s.width)  # columns of the stacked product: z, u, the output's gate, each from a multiple of 8 on

    def param_shapes(self):
        s = self.spec
        return {"wz": (s.width, s.hidden), "bz": (s.width,), "wu": (s.width, s.hidden), "bu": (s.width,),
                "wg": (s.width, s.hidden), "wo": (s.hidden, s.width)}

    def bind(self, params, ctx):
        s, self.ctx = self.spec, ctx
        stacked = torch.zeros((3 * self.block, s.hidden), dtype=params["wz"].dtype, device=params["wz"].device)
        for i, slot in enumerate(("wz", "wu", "wg")):
            stacked[i * self.block:i * self.block + s.width] = params[slot]
        self.in_proj = Linear(to_device(stacked, ctx, ctx.dtype))
        self.bias_z = to_device(params["bz"], ctx, torch.float32)
        self.bias_u = to_device(params["bu"], ctx, torch.float32)
        # (the output product's rows are padded to a multiple of 8 with zeros, which meet whatever the padding holds: zeros)
        wo = torch.zeros((s.hidden, self.block), dtype=params["wo"].dtype, device=params["wo"].device)
        wo[:, :s.width] = params["wo"]
        self.o_proj = Linear(to_device(wo, ctx, ctx.dtype))

    def step_weights(self):
        return [self.in_proj.weight, self.bias_z, self.bias_u, self.o_proj.weight]

    def cache_need(self):
        return CacheNeed(states=(("average", (self.spec.width,), "float32"),))

    def state_bytes(self):
        """Bytes of state a sequence holds in one entry (what a decode step reads and writes for it)."""
        return 4 * self.spec.width

    def forward(self, xn, out, batch, cache, ws):
        s, n, dt = self.spec, batch.n_rows, self.ctx.dtype
        if not cache.owns_storage:
            raise ops.KernelRefused("a recurrent entry keeps a state of its own; it cannot read another entry's")
        proj = ws.get("average_proj", (n, 3 * self.block), dt)
        self.in_proj.forward(xn, proj, n)
        gated = ws.get(f"average_gated_{s.width}", (n, self.block), dt)
        ops.gated_average(proj, 0, self.block, 2 * self.block, s.width, self.bias_z, self.bias_u, cache.states["average"],
                          gated, batch)
        self.o_proj.forward(gated, out, n)
        return out
