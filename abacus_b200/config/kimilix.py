"""Typed configuration of the Kimilix decoder, read from config.json.

A Kimilix model scales its embeddings (the same table, unscaled, makes the logits) and runs layers that may differ one from
the next and that norm a branch's output only: x += residual_mult * gain * norm(branch(x)), with a learned gain per element.
A layer's mixer is either differential attention (two maps a head over the same values, q and k normed per map and rotated
in halves with frequencies scaled in bands, keys seen within the token's own chunk of positions) or latent attention
(queries through a latent of their own, keys and values kept as one low-rank latent row per token with one rotated key
part beside it, interleaved rotation, a sliding window). Its feed-forward is a plain one with the square of relu, or routed
experts (a router with biases, the softmax of the chosen logits, gated experts whose gate and up are bounded, a shared
expert with a gate of its own), or absent. Every size and constant comes from config.json.
"""
from dataclasses import dataclass
from typing import Optional, Tuple

from .registry import ConfigError
from .specs import (AttentionSpec, ExpertSpec, LatentAttentionSpec, ModelSpec, NormSpec, PlainMLPSpec, PostNormBlockSpec,
                    RotarySpec, RoutedMLPSpec, ScaledEmbeddingSpec, ScheduleEntry)
from .temetar import MAX_POSITIONS, _float, _int

ATTENTION, LATENT = "attention", "latent_attention"


@dataclass(frozen=True)
class KimilixRotation:
    base: float
    dims: int
    scaling: Optional[tuple] = None   # (factor, original, low, high), or None: frequencies as they are

    @classmethod
    def from_dict(cls, where, r, most):
        base, dims = _float(where, r, "base"), _int(where, r, "dims", 2)
        if dims % 2 or dims > most:
            raise ConfigError(f"config.json: {where}dims {dims} must be even and at most {most}")
        s = r.get("scaling")
        if s is None:
            return cls(base, dims)
        w = where + "scaling."
        bands = tuple(_float(w, s, key) for key in ("factor", "original", "low", "high"))
        if bands[3] <= bands[2]:
            raise ConfigError(f"config.json: {w}high {bands[3]} must be above low {bands[2]}")
        return cls(base, dims, bands)

    def to_dict(self):
        d = {"base": self.base, "dims": self.dims}
        if self.scaling is not None:
            d["scaling"] = dict(zip(("factor", "original", "low", "high"), self.scaling))
        return d

    def to_spec(self, pairing):
        return RotarySpec(theta=self.base, rotary_dim=self.dims, pairing=pairing, exact_angles=True, bands=self.scaling)


def _mask(where, m):
    return None if m.get("mask") is None else _int(where + "mask.", m["mask"], "size")


@dataclass(frozen=True)
class KimilixAttention:
    heads: int
    kv_heads: int
    dim: int                   # of one map of a head
    vdim: int
    scale: float
    diff: float
    chunk: Optional[int]       # positions of a chunk; None: every earlier key is seen
    rot: Optional[KimilixRotation]

    @classmethod
    def from_dict(cls, where, m):
        heads, kv = _int(where, m, "heads"), _int(where, m, "kv_heads")
        if heads % kv:
            raise ConfigError(f"config.json: {where}heads {heads} is no multiple of kv_heads {kv}")
        dim = _int(where, m, "dim")
        rot = None if m.get("rot") is None else KimilixRotation.from_dict(where + "rot.", m["rot"], dim)
        return cls(heads, kv, dim, _int(where, m, "vdim"), _float(where, m, "scale"), _float(where, m, "diff", positive=False),
                   _mask(where, m), rot)

    def to_dict(self):
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale, "diff": self.diff}
        if self.chunk is not None:
            d["mask"] = {"size": self.chunk}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        return d

    def to_spec(self, width, eps):
        return AttentionSpec(hidden=width, n_heads=self.heads, n_kv_heads=self.kv_heads, head_dim=self.dim, scale=self.scale,
                             qk_norm_eps=eps, position=None if self.rot is None else self.rot.to_spec("half"), v_head_dim=self.vdim,
                             exact_weights=True, chunk=self.chunk, diff=self.diff, diff_eps=eps)


@dataclass(frozen=True)
class KimilixLatent:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    window: Optional[int]      # None: every earlier key is seen
    rot: Optional[KimilixRotation]

    @classmethod
    def from_dict(cls, where, m):
        rot_dim, rot = _int(where, m, "rot_dim", 0), m.get("rot")
        if rot is not None:
            if not rot_dim:
                raise ConfigError(f"config.json: {where}rot goes with a rot_dim")
            rot = KimilixRotation.from_dict(where + "rot.", rot, rot_dim)
        return cls(_int(where, m, "heads"), _int(where, m, "dim"), rot_dim, _int(where, m, "vdim"), _int(where, m, "kv_rank"),
                   _int(where, m, "q_rank"), _float(where, m, "scale"), _mask(where, m), rot)

    def to_dict(self):
        d = {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim, "kv_rank": self.kv_rank,
             "q_rank": self.q_rank, "scale": self.scale}
        if self.window is not None:
            d["mask"] = {"size": self.window}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        return d

    def to_spec(self, width, eps):
        return LatentAttentionSpec(hidden=width, n_heads=self.heads, head_dim=self.dim, rot_dim=self.rot_dim, v_head_dim=self.vdim,
                                   rank=self.kv_rank, scale=self.scale, norm_eps=eps,
                                   position=None if self.rot is None else self.rot.to_spec("interleaved"), q_rank=self.q_rank,
                                   window=self.window)


@dataclass(frozen=True)
class KimilixDense:
    ff: int

    def to_dict(self):
        return {"kind": "dense", "ff": self.ff}

    def to_spec(self, width):
        return PlainMLPSpec(width, self.ff, "relu_squared")


@dataclass(frozen=True)
class KimilixExperts:
    experts: int
    top: int
    ff: int
    limit: float
    shared_ff: Optional[int]   # None: no shared expert
    shared_limit: float

    @classmethod
    def from_dict(cls, where, m):
        router, expert, shared = m.get("router"), m.get("expert"), m.get("shared")
        experts, top = _int(where + "router.", router, "experts"), _int(where + "router.", router, "top")
        if top > experts:
            raise ConfigError(f"config.json: {where}router.top {top} is more than the {experts} experts")
        w, ws = where + "expert.", where + "shared."
        return cls(experts, top, _int(w, expert, "ff"), _float(w, expert, "limit"), None if shared is None else _int(ws, shared, "ff"),
                   0.0 if shared is None else _float(ws, shared, "limit"))

    def to_dict(self):
        d = {"kind": "moe", "router": {"experts": self.experts, "top": self.top}, "expert": {"ff": self.ff, "limit": self.limit}}
        if self.shared_ff is not None:
            d["shared"] = {"ff": self.shared_ff, "limit": self.shared_limit}
        return d

    def to_spec(self, width):
        shared = None if self.shared_ff is None else ExpertSpec(self.shared_ff, "clamped_gated", self.shared_limit)
        return RoutedMLPSpec(hidden=width, experts=self.experts, top=self.top, expert=ExpertSpec(self.ff, "clamped_gated", self.limit),
                             shared=shared, score="softmax_chosen", weight_on="output", router_bias=True,
                             shared_gate=shared is not None)


@dataclass(frozen=True)
class KimilixLayer:
    type: str
    mixer: object   # KimilixAttention or KimilixLatent
    mlp: object     # KimilixDense, KimilixExperts or None (no feed-forward)


_MIXERS = {ATTENTION: KimilixAttention, LATENT: KimilixLatent}


@dataclass(frozen=True)
class KimilixConfig:
    vocab: int
    width: int
    layers: Tuple[KimilixLayer, ...]
    eps: float
    embedding_scale: float = 1.0
    residual_mult: float = 1.0
    architecture: str = "Kimilix"

    @classmethod
    def from_dict(cls, raw):
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: layers must be a list with at least one layer")
        parsed = []
        for i, layer in enumerate(layers):
            where = f"layers[{i}]."
            kind = layer.get("type") if isinstance(layer, dict) else None
            if kind not in _MIXERS:
                raise ConfigError(f"config.json: {where}type {kind!r} is none of {', '.join(_MIXERS)}")
            if not isinstance(layer.get("mixer"), dict):
                raise ConfigError(f"config.json: {where}mixer must give the mixer's sizes")
            mixer, mlp = _MIXERS[kind].from_dict(where + "mixer.", layer["mixer"]), layer.get("mlp")
            if mlp is not None:
                mlp_kind = mlp.get("kind", "dense") if isinstance(mlp, dict) else None
                if mlp_kind == "dense":
                    mlp = KimilixDense(_int(where + "mlp.", mlp, "ff"))
                elif mlp_kind == "moe":
                    mlp = KimilixExperts.from_dict(where + "mlp.", mlp)
                else:
                    raise ConfigError(f"config.json: {where}mlp.kind {mlp_kind!r} is neither dense nor moe")
            parsed.append(KimilixLayer(kind, mixer, mlp))
        return cls(vocab=_int("", raw, "vocab"), width=_int("", raw, "width"), layers=tuple(parsed),
                   eps=_float("norm.", raw.get("norm"), "eps"),
                   embedding_scale=_float("embedding.", raw.get("embedding") or {}, "scale", 1.0, positive=False),
                   residual_mult=_float("", raw, "residual_mult", 1.0, positive=False))

    def to_dict(self):
        """A config.json that from_dict reads back to this object."""
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
                "embedding": {"scale": self.embedding_scale}, "residual_mult": self.residual_mult,
                "layers": [{"type": l.type, "mixer": l.mixer.to_dict(), "mlp": None if l.mlp is None else l.mlp.to_dict()}
                           for l in self.layers]}

    def to_spec(self):
        branch = NormSpec(self.width, self.eps, one_plus=True, gain=True, mult=self.residual_mult)
        blocks = []
        for layer in self.layers:
            ffn = None if layer.mlp is None else layer.mlp.to_spec(self.width)
            blocks.append(PostNormBlockSpec(mixer=layer.mixer.to_spec(self.width, self.eps), mixer_post_norm=branch, ffn=ffn,
                                            ffn_post_norm=None if ffn is None else branch))
        return ModelSpec(architecture=self.architecture, hidden=self.width, vocab=self.vocab, layers=tuple(blocks),
                         schedule=tuple(ScheduleEntry(l) for l in range(len(blocks))),
                         final_norm=NormSpec(self.width, self.eps, one_plus=True), tied_head=True, max_positions=MAX_POSITIONS,
                         frame="scaled", frame_spec=ScaledEmbeddingSpec(self.embedding_scale))
