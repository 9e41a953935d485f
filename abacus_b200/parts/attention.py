"""Grouped-query causal attention over the paged cache (src/model.c:197-211, 247-259).

The mixer owns the q/k/v and output projections, the optional per-head norm of
q and k, and a position encoding; its sizes, scale, eps and window come from
its spec. q, k and v are one stacked matrix, as in src/model.c:88-93.

Options of the spec that only the general kernels take: values of another size than keys, a sequence's first keys
kept behind a window, a sink, float32 weights, a short causal convolution over time on every channel of q, k and v
right after their projection (its last inputs are part of the sequence's state, beside the keys and values), keys
seen only within the token's own chunk of positions, and capped scores. A layer may do without a softmax altogether
(weights "sigmoid": each key for itself, with a distance bias and a shift per head, the heads' weights mixed before
they meet the values): the projection, its preparation and the cache are the same, the attention kernels its own. Or it is
differential (diff): every head has two maps over the same values. q and k then have twice the heads of head_dim for norm
and rotation, a key row of the cache holds both maps side by side, and the attention kernels make one head of the two.
"""
import os

import torch

from ..cache.need import CacheNeed
from ..kernels import ops
from .attention_plan import AttentionLists, AttentionStepPlan
from .base import MIXERS, POSITIONS, to_device
from .linear import Linear


# A decode step's attention kernel can norm and rotate q and k and write the new key and value to the cache itself: a
# launch less in every layer. ABACUS_DECODE_PREPARES=0 keeps the preparation a kernel of its own (for comparison).
DECODE_PREPARES = os.environ.get("ABACUS_DECODE_PREPARES", "1") != "0"
# The q/k/v product of a long prompt step can do the same in its epilogue (heads of 128): a kernel and a pass over
# q, k and v less. ABACUS_PRODUCT_PREPARES=0 keeps the preparation a kernel of its own (for comparison).
PRODUCT_PREPARES = os.environ.get("ABACUS_PRODUCT_PREPARES", "1") != "0"


@MIXERS.register("attention")
class Attention:
    capturable = True  # its forward launches kernels only; nothing in it depends on the step's contents

    def __init__(self, spec):
        s = self.spec = spec
        if s.n_heads % s.n_kv_heads:
            raise ValueError(f"{s.n_heads} query heads do not divide into {s.n_kv_heads} kv heads")
        self.v_dim = s.v_head_dim or s.head_dim
        if self.v_dim < 1 or self.v_dim > 256:
            raise ValueError(f"v_head_dim {self.v_dim}: the attention kernels take value heads of up to 256")
        if s.keep_first and s.window is None:
            raise ValueError("keep_first goes with a window")
        # what only the general kernel takes: values of another size, kept first keys, a sink, float32 weights
        # q and k normed over their whole rows, values that are their keys, a gate per head: a preparation kernel of
        # their own (out of the projection's rows into the rows the attention kernels read), then the general kernels
        self.whole = s.norm_over == "projection" or s.values == "keys" or s.bias or s.q_temperature is not None
        if s.norm_over not in ("head", "projection") or s.values not in ("own", "keys"):
            raise ValueError(f"norm_over {s.norm_over!r} is neither head nor projection, or values {s.values!r} neither own nor keys")
        if self.whole and (s.conv_taps or (s.values == "keys" and self.v_dim != s.head_dim)
                           or (s.qk_norm_eps is not None and s.norm_over != "projection")):
            raise ValueError("values that are their keys, norms over the whole projection, biases and a query temperature go "
                             "with neither a convolution nor a norm per head, and values that are keys are of their size")
        if s.bias and s.values == "keys":
            raise ValueError("values that are their keys have no bias of their own")
        self.sigmoid = s.weights == "sigmoid"
        if s.weights not in ("softmax", "sigmoid"):
            raise ValueError(f"weights {s.weights!r} are neither softmax nor sigmoid")
        if self.sigmoid and (s.window is not None or s.chunk or s.sink or s.head_gate or not s.exact_weights):
            raise ValueError("sigmoid weights are float32 and take no window, no chunk, no sink and no gate per head")
        if not self.sigmoid and (s.slopes is not None or s.shift or s.mix):
            raise ValueError("slopes, a shift per head and mixed heads go with sigmoid weights")
        if s.slopes is not None and len(s.slopes) != s.n_heads:
            raise ValueError(f"{len(s.slopes)} slopes for {s.n_heads} heads")
        self.maps = 1 if s.diff is None else 2
        if s.diff is not None and (self.whole or self.sigmoid or s.head_gate or s.keep_first or s.conv_taps or not s.exact_weights):
            raise ValueError("differential attention has softmax weights in float32 and a norm per head, and takes no gate, kept first "
                             "keys, convolution, biases or values that are its keys")
        self.general = (self.maps > 1 or self.v_dim != s.head_dim or bool(s.keep_first) or s.sink or s.exact_weights or s.conv_taps > 0
                        or bool(s.chunk) or bool(s.softcap) or self.whole or s.head_gate or self.sigmoid)
        if s.conv_taps < 0 or s.conv_taps > 8:
            raise ValueError(f"conv_taps {s.conv_taps}: the convolution takes 1 to 8 taps")
        if s.chunk is not None and s.chunk < 1:
            raise ValueError(f"chunk {s.chunk}: a chunk has at least one position")
        if s.softcap is not None and not s.softcap > 0:
            raise ValueError(f"softcap {s.softcap}: the cap of the scores is positive")
        if s.head_dim > 256 or s.head_dim < 1 or (s.head_dim % 8 and not self.general):
            raise ValueError(f"head_dim {s.head_dim}: the attention kernels take multiples of 8 up to 256 (the general "
                             "kernel, which a layer with a sink, kept first keys or values of their own size runs on, "
                             "any size up to 256)")
        self.position = POSITIONS.build(s.position) if s.position is not None else None
        self.q_size, self.kv_size = s.n_heads * self.maps * s.head_dim, s.n_kv_heads * self.maps * s.head_dim
        self.v_size = s.n_kv_heads * self.v_dim
        # a row of q, k and v is padded to a multiple of 8 elements, so that every row starts 16-byte aligned whatever
        # the values' size (nothing to pad where values are as large as keys: head_dim is a multiple of 8)
        self.row = -(-(self.q_size + self.kv_size + self.v_size) // 8) * 8
        # a row of the stacked product: q, k, v (if projected), then the heads' gates from a multiple of 8 on
        own_v = self.v_size if s.values == "own" else 0
        self.gate_at = -(-(self.q_size + self.kv_size + own_v) // 8) * 8
        self.proj_row = self.gate_at + (-(-s.n_heads // 8) * 8 if s.head_gate else 0) if (self.whole or s.head_gate) else self.row
        self.cos = self.sin = None
        # A step of several tokens of a windowed layer is checked on the host (it may have to be refused): such steps
        # cannot be replayed from a captured graph; single-token steps can. A layer with the general options decides on
        # the host whether a step reads its keys from the step's own rows; for steps whose sequences all start at
        # their first token the answer is always yes, so those may be captured ("from_start").
        self.capturable_prompts = "from_start" if self.general else s.window is None
        self.lists = AttentionStepPlan(s.n_heads)  # the prefill kernels' tiles and work list, made per step

    def step_plans(self):
        """What this mixer wants made on the host for every step and sent with the step's indices."""
        return [] if self.sigmoid or self.maps > 1 else [self.lists]  # (attention without a softmax and differential attention need none)

    def step_weights(self):
        """The tensors a step reads once whatever its size (for the bytes a decode step must move)."""
        return [self.qkv_proj.weight, self.o_proj.weight, self.q_norm, self.k_norm, self.sink, self.conv, self.bias, self.mix]

    def param_shapes(self):
        s = self.spec
        shapes = {"wq": (self.q_size, s.hidden), "wk": (self.kv_size, s.hidden), "wv": (self.v_size, s.hidden),
                  "wo": (s.hidden, s.n_heads * self.v_dim)}
        if s.values == "keys":
            del shapes["wv"]
        if s.head_gate:
            shapes["wg"] = (s.n_heads, s.hidden)
        if s.qk_norm_eps is not None and s.norm_over == "projection":
            shapes.update(q_norm=(self.q_size,), k_norm=(self.kv_size,))
        elif s.qk_norm_eps is not None:
            shapes.update(q_norm=(s.head_dim,), k_norm=(s.head_dim,))
        if s.sink:
            shapes["sink"] = (s.n_heads * self.maps,)
        if s.diff is not None:
            shapes.update({n: (s.head_dim,) for n in ("lq1", "lk1", "lq2", "lk2")})
        if s.bias:
            shapes.update(bq=(self.q_size,), bk=(self.kv_size,), bv=(self.v_size,))
        if s.shift:
            shapes["shift"] = (s.n_heads,)
        if s.mix:
            shapes["mix"] = (s.n_heads, s.n_heads)
        if s.conv_taps:
            shapes.update(conv_q=(self.q_size, s.conv_taps), conv_k=(self.kv_size, s.conv_taps),
                          conv_v=(self.v_size, s.conv_taps))
        return shapes

    def bind(self, params, ctx):
        self.ctx = ctx
        wqkv = torch.cat([params["wq"], params["wk"]] + ([params["wv"]] if "wv" in params else []), dim=0)
        if self.proj_row > wqkv.shape[0]:
            wqkv = torch.cat([wqkv, torch.zeros((self.proj_row - wqkv.shape[0], wqkv.shape[1]), dtype=wqkv.dtype, device=wqkv.device)], dim=0)
        if self.spec.head_gate:
            wqkv[self.gate_at:self.gate_at + self.spec.n_heads] = params["wg"]
        self.qkv_proj = Linear(to_device(wqkv, ctx, ctx.dtype))
        self.q_proj = Linear(self.qkv_proj.weight[:self.q_size])  # for entries that read another entry's cache
        self.o_proj = Linear(to_device(params["wo"], ctx, ctx.dtype))
        self.q_norm = to_device(params["q_norm"], ctx, torch.float32) if "q_norm" in params else None
        self.k_norm = to_device(params["k_norm"], ctx, torch.float32) if "k_norm" in params else None
        self.sink = to_device(params["sink"], ctx, torch.float32) if "sink" in params else None
        self.bias = (to_device(torch.cat([params["bq"], params["bk"], params["bv"]]), ctx, torch.float32)
                     if self.spec.bias else None)
        self.shift = to_device(params["shift"], ctx, torch.float32) if self.spec.shift else None
        self.mix = to_device(params["mix"], ctx, torch.float32) if self.spec.mix else None
        self.slopes = (torch.tensor(self.spec.slopes, dtype=torch.float64).to(torch.float32).to(ctx.device)
                       if self.spec.slopes is not None else None)
        self.lam = None
        if self.spec.diff is not None:  # the second map's factor, one number a layer
            l = {n: params[n].detach().to("cpu", torch.float64) for n in ("lq1", "lk1", "lq2", "lk2")}
            self.lam = float(torch.exp((l["lq1"] * l["lk1"]).sum()) - torch.exp((l["lq2"] * l["lk2"]).sum())) + self.spec.diff
        self.conv = None
        if self.spec.conv_taps:  # one table for the whole row of q, k and v; the row's padding has taps of zero
            taps = torch.cat([params["conv_q"], params["conv_k"], params["conv_v"]], dim=0).to(torch.float32)
            table = torch.zeros((self.row, self.spec.conv_taps), dtype=torch.float32)
            table[:taps.shape[0]] = taps
            self.conv = to_device(table, ctx, torch.float32)

    def cache_need(self):
        s = self.spec
        states = (("conv_tail", (s.conv_taps - 1, self.row), "float32"),) if s.conv_taps > 1 else ()
        return CacheNeed(n_kv_heads=s.n_kv_heads, head_dim=self.maps * s.head_dim, window=s.window, v_head_dim=self.v_dim,
                         keep_first=s.keep_first if s.window is not None else 0, states=states)

    def prepare(self, max_positions, device):
        if self.position is not None:
            self.cos, self.sin = self.position.tables(max_positions, device)

    def forward(self, xn, out, batch, cache, ws):
        s = self.spec
        n = batch.n_rows
        qkv = ws.get("qkv", (n, self.row), self.ctx.dtype)
        att = ws.get("att", (n, s.n_heads * self.v_dim), self.ctx.dtype)
        writes = cache.owns_storage
        rotary_dim = self.position.rotary_dim if self.position else 0
        interleaved = self.position.interleaved if self.position else False
        # A windowed cache keeps only the last keys; a prompt longer than that reads its keys from
        # this step's own rows, which hold all of them when the sequences start at position 0.
        from_step = s.window is not None and not batch.is_decode
        w = self.qkv_proj.weight
        prepared = False  # by the product's own kernel: a prompt's heads in its epilogue
        if (PRODUCT_PREPARES and writes and not batch.is_decode and not from_step and w.dtype == torch.bfloat16
                and not self.general
                and ops.gemm_tc_qkv_takes(xn, w, qkv, n, s.n_heads, s.n_kv_heads, s.head_dim, cache.kv, self.q_norm,
                                          self.k_norm, self.cos, self.sin, rotary_dim, interleaved)):
            ops.gemm_tc_qkv(xn, w, qkv, s.n_heads, s.n_kv_heads, batch, self.q_norm, self.k_norm, s.qk_norm_eps,
                            self.cos, self.sin, cache.kv, n)
            prepared = True
        elif self.whole or s.head_gate:
            # the projection into rows of its own (q, k, v if projected, the heads' gates); q, k and v go from there
            # into the rows the attention kernels read
            proj = ws.get("qkv_proj", (n, self.proj_row), self.ctx.dtype)
            if writes:
                self.qkv_proj.forward(xn, proj, n)
            else:
                raise ops.KernelRefused("an attention entry whose values are its keys, or with gated heads, keeps keys of its own")
            if self.whole:
                ops.qkv_prep_whole(proj, qkv, s.n_heads, s.n_kv_heads, s.head_dim, batch, self.q_norm, self.k_norm,
                                   s.qk_norm_eps, self.cos, self.sin, rotary_dim, interleaved, cache.kv,
                                   v_dim=self.v_dim if s.values == "own" else None, bias=self.bias, temperature=s.q_temperature)
                prepared = True
            else:
                qkv[:n, :self.gate_at].copy_(proj[:n, :self.gate_at])
        elif writes and self.conv is not None:
            # the projection, then the convolution over time into the row the kernels read; the slot's tail follows
            proj = ws.get("qkv_proj", (n, self.row), self.ctx.dtype)
            self.qkv_proj.forward(xn, proj, n)
            tail = cache.states["conv_tail"] if s.conv_taps > 1 else ws.get("no_tail", (1, 0, self.row), torch.float32)
            ops.short_conv(proj, self.row, self.conv, tail, qkv, batch, update_tail=batch.is_decode, plain=True)
            if s.conv_taps > 1 and not batch.is_decode:
                ops.short_conv_tail(proj, self.row, s.conv_taps, tail, batch)
        elif writes:
            self.qkv_proj.forward(xn, qkv, n)
        elif self.conv is not None:
            raise ops.KernelRefused("an attention entry with a convolution keeps a state of its own; it cannot read "
                                    "another entry's cache")
        else:  # keys and values are another entry's: only q is needed
            self.q_proj.forward(xn, qkv[:, :self.q_size], n)
        prepare = None
        if prepared:
            pass
        elif (DECODE_PREPARES and batch.is_decode and cache.kv is not None and not self.general
                and ops.attention_decode_prepares(qkv, s.n_heads, s.n_kv_heads, s.head_dim, cache.kv, self.q_norm,
                                                  self.k_norm, self.cos, self.sin, rotary_dim, interleaved)):
            prepare = dict(q_norm=self.q_norm, k_norm=self.k_norm, eps=s.qk_norm_eps, cos=self.cos, sin=self.sin, keep=writes)
        else:
            ops.qkv_prep(qkv, self.maps * s.n_heads, self.maps * s.n_kv_heads, s.head_dim, batch, self.q_norm, self.k_norm, s.qk_norm_eps,
                         self.cos, self.sin, rotary_dim, interleaved, cache.kv if writes else None, q_only=not writes,
                         v_dim=self.v_dim, row=self.row if self.general else None, maps=self.maps)
        if from_step and (batch.any_continuation or not writes):
            raise ops.KernelRefused("windowed attention takes several tokens of a sequence only at its start, "
                                    "and only with keys of its own")
        if self.sigmoid:
            ops.attention_sigmoid(qkv, att, s.n_heads, s.n_kv_heads, s.head_dim, s.scale, batch, cache.kv, v_dim=self.v_dim,
                                  softcap=s.softcap, slopes=self.slopes, shift=self.shift, mix=self.mix, row=self.row, ws=ws)
            self.o_proj.forward(att, out, n)
            return out
        if self.maps > 1:
            ops.attention_differential(qkv, att, s.n_heads, s.n_kv_heads, s.head_dim, s.scale, s.window, batch, cache.kv, self.lam,
                                       s.diff_eps, 1.0 - s.diff, from_step=from_step, ws=ws, v_dim=self.v_dim, sink=self.sink,
                                       row=self.row, chunk=s.chunk, softcap=s.softcap)
            self.o_proj.forward(att, out, n)
            return out
        mine = batch.plan.get(self.lists.name)
        gates = ws.get("qkv_proj", (n, self.proj_row), self.ctx.dtype)[:, self.gate_at:] if s.head_gate else None
        gated = ops.attention(qkv, att, s.n_heads, s.n_kv_heads, s.head_dim, s.scale, s.window, batch, cache.kv,
                      from_step=from_step, ws=ws, lists=AttentionLists(mine) if mine is not None else None, prepare=prepare,
                      v_dim=self.v_dim, keep_first=s.keep_first, sink=self.sink, exact_weights=s.exact_weights,
                      row=self.row if self.general else None, chunk=s.chunk, softcap=s.softcap, gate=gates)
        if s.head_gate and not gated:  # head h's output times sigmoid(g_h . x), where the attention kernel did not do it
            ops.gate_heads(att, gates, s.n_heads, self.v_dim, n)
        self.o_proj.forward(att, out, n)
        return out
