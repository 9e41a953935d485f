"""Gated feed-forward: down(silu(gate(x)) * up(x)) (src/model.c:274-282, 307-309), or with relu in silu's place, or with
gate and up bounded (config.specs.GatedMLPSpec); and the plain one, down(act(up(x))).

gate and up are one matrix, as in src/model.c:98. In bfloat16, when the inner size allows, its rows come
in turns of 128 (gate of features 0-127, up of the same, gate of 128-255, ...): a 256-column tile of the
tensor-core product then holds both halves of 128 features, and the activation runs in its epilogue.
"""
import torch

from ..kernels import ops
from .base import FEED_FORWARDS, to_device
from .linear import Linear, rows_kernel_wins


@FEED_FORWARDS.register("gated_mlp")
class GatedMLP:
    capturable = True  # its forward launches kernels only; nothing in it depends on the step's contents

    def __init__(self, spec):
        if spec.activation not in ops.ACTIVATIONS:
            raise ValueError(f"activation {spec.activation!r} is not built (only {', '.join(ops.ACTIVATIONS)})")
        if spec.activation == "clamped_silu" and not spec.limit > 0:
            raise ValueError(f"limit {spec.limit}: bounded gates have a positive limit")
        self.spec = spec

    def param_shapes(self):
        s = self.spec
        return {"gate": (s.inter, s.hidden), "up": (s.inter, s.hidden), "down": (s.hidden, s.inter)}

    TURN = 128  # rows of gate, then of up, where the layout comes in turns

    def bind(self, params, ctx):
        self.ctx = ctx
        inter, gate, up = self.spec.inter, params["gate"], params["up"]
        self.block = self.TURN if ctx.dtype == torch.bfloat16 and inter % self.TURN == 0 else inter
        turns = inter // self.block
        stacked = torch.stack([gate.reshape(turns, self.block, -1), up.reshape(turns, self.block, -1)], dim=1)
        self.gate_up = Linear(to_device(stacked.reshape(2 * inter, -1).contiguous(), ctx, ctx.dtype))
        self.down = Linear(to_device(params["down"], ctx, ctx.dtype))

    def step_weights(self):
        return [self.gate_up.weight, self.down.weight]

    def forward(self, xn, out, batch, ws):
        n, inter, kind = batch.n_rows, self.spec.inter, self.spec.activation
        act = ws.get("act", (n, inter), self.ctx.dtype)
        w = self.gate_up.weight
        if rows_kernel_wins(n, w, gated=True) and ops.gemm_rows_takes(xn, w, act, n):
            ops.gemm_rows_swiglu(xn, w, act, n, self.block, kind, self.spec.limit)  # a handful of rows: product and activation in one
        elif ops.gemm_tc_swiglu_takes(xn, w, act, n, self.block):
            ops.gemm_tc_swiglu(xn, w, act, n, kind, self.spec.limit)  # a prompt: the activation in the product's epilogue
        else:
            gate_up = ws.get("gate_up", (n, 2 * inter), self.ctx.dtype)
            self.gate_up.forward(xn, gate_up, n)
            ops.swiglu(gate_up, act, self.block, kind, self.spec.limit)
        self.down.forward(act, out, n)
        return out


@FEED_FORWARDS.register("plain_mlp")
class PlainMLP:
    capturable = True  # its forward launches kernels only; nothing in it depends on the step's contents

    def __init__(self, spec):
        if spec.activation not in ops.OUT_ACTIVATIONS or spec.activation is None:
            raise ValueError(f"activation {spec.activation!r} is not built (only relu_squared)")
        self.spec = spec

    def param_shapes(self):
        s = self.spec
        return {"up": (s.inter, s.hidden), "down": (s.hidden, s.inter)}

    def bind(self, params, ctx):
        self.ctx = ctx
        self.up = Linear(to_device(params["up"], ctx, ctx.dtype))
        self.down = Linear(to_device(params["down"], ctx, ctx.dtype))

    def step_weights(self):
        return [self.up.weight, self.down.weight]

    def forward(self, xn, out, batch, ws):
        n = batch.n_rows
        act = ws.get("act", (n, self.spec.inter), self.ctx.dtype)
        self.up.forward(xn, act, n, activation=self.spec.activation)  # the activation in the product's epilogue
        self.down.forward(act, out, n)
        return out
