"""Typed configuration of the Lilovik decoder, read from config.json.

A Lilovik model adds a fixed sinusoidal vector per position to its embeddings and runs layers with a norm before and
after each branch. A layer's mixer is attention without a softmax (grouped heads, biases on q, k and v, q and k normed
over their whole rows, a query temperature that grows with the position, capped scores with a distance bias per head,
each key's weight the sigmoid of its score, the heads' weights mixed before they meet the values) or a minimal gated
recurrence (a running average per channel). Its feed-forward is gated and dense, or absent. Every size and constant comes
from config.json.
"""
from dataclasses import dataclass
from typing import Optional, Tuple

from .registry import ConfigError
from .specs import (AttentionSpec, GatedAverageSpec, GatedMLPSpec, ModelSpec, NormSpec, SandwichBlockSpec, ScheduleEntry,
                    SinusoidEmbeddingSpec)
from .temetar import MAX_POSITIONS, _float, _int

ATTENTION, AVERAGE = "attention", "mingru"


@dataclass(frozen=True)
class LilovikAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: Optional[float]         # None: scores are not capped
    temp_coef: Optional[float]       # None (with temp_every): queries as they are
    temp_every: Optional[float]

    @classmethod
    def from_dict(cls, where, m):
        heads, kv = _int(where, m, "heads"), _int(where, m, "kv_heads")
        if heads % kv:
            raise ConfigError(f"config.json: {where}heads {heads} is no multiple of kv_heads {kv}")
        temp, cap = m.get("q_temp"), m.get("softcap")
        return cls(heads, kv, _int(where, m, "dim"), _int(where, m, "vdim"), _float(where, m, "scale"),
                   None if cap is None else _float(where, m, "softcap"),
                   None if temp is None else _float(where + "q_temp.", temp, "coef", positive=False),
                   None if temp is None else _float(where + "q_temp.", temp, "every"))

    def to_dict(self):
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.softcap is not None:
            d["softcap"] = self.softcap
        if self.temp_coef is not None:
            d["q_temp"] = {"coef": self.temp_coef, "every": self.temp_every}
        return d

    def slopes(self):
        """What a step of distance takes off each head's scores: a geometric run down to 2^-8."""
        return tuple(2.0 ** (-8.0 * (h + 1) / self.heads) for h in range(self.heads))


@dataclass(frozen=True)
class LilovikAverage:
    width: int

    @classmethod
    def from_dict(cls, where, m):
        return cls(_int(where, m, "width"))

    def to_dict(self):
        return {"width": self.width}


@dataclass(frozen=True)
class LilovikLayer:
    type: str
    mixer: object             # LilovikAttention or LilovikAverage
    ff: Optional[int]         # the feed-forward's inner size; None: no feed-forward


_MIXERS = {ATTENTION: LilovikAttention, AVERAGE: LilovikAverage}


@dataclass(frozen=True)
class LilovikConfig:
    vocab: int
    width: int
    layers: Tuple[LilovikLayer, ...]
    eps: float
    logit_scale: float = 1.0
    architecture: str = "Lilovik"

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
            mixer = _MIXERS[kind].from_dict(where + "mixer.", layer["mixer"])
            mlp, ff = layer.get("mlp"), None
            if mlp is not None:
                if not isinstance(mlp, dict) or mlp.get("kind", "dense") != "dense":
                    raise ConfigError(f"config.json: {where}mlp.kind must be dense, or mlp null")
                ff = _int(where + "mlp.", mlp, "ff")
            parsed.append(LilovikLayer(kind, mixer, ff))
        return cls(vocab=_int("", raw, "vocab"), width=_int("", raw, "width"), layers=tuple(parsed),
                   eps=_float("norm.", raw.get("norm"), "eps"),
                   logit_scale=_float("", raw, "logit_scale", default=1.0, positive=False))

    def to_dict(self):
        """A config.json that from_dict reads back to this object."""
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
                "logit_scale": self.logit_scale,
                "layers": [{"type": l.type, "mixer": l.mixer.to_dict(),
                            "mlp": None if l.ff is None else {"kind": "dense", "ff": l.ff}} for l in self.layers]}

    def to_spec(self):
        norm = NormSpec(self.width, self.eps, one_plus=True)
        blocks = []
        for layer in self.layers:
            m = layer.mixer
            if layer.type == ATTENTION:
                mixer = AttentionSpec(hidden=self.width, n_heads=m.heads, n_kv_heads=m.kv_heads, head_dim=m.dim, scale=m.scale,
                                      qk_norm_eps=self.eps, position=None, v_head_dim=m.vdim, exact_weights=True,
                                      softcap=m.softcap, norm_over="projection", bias=True,
                                      q_temperature=None if m.temp_coef is None else (m.temp_coef, m.temp_every),
                                      weights="sigmoid", slopes=m.slopes(), shift=True, mix=True)
            else:
                mixer = GatedAverageSpec(hidden=self.width, width=m.width)
            ffn = None if layer.ff is None else GatedMLPSpec(hidden=self.width, inter=layer.ff, activation="relu")
            blocks.append(SandwichBlockSpec(mixer_norm=norm, mixer=mixer, mixer_post_norm=norm, ffn_norm=norm if ffn else None,
                                            ffn=ffn, ffn_post_norm=norm if ffn else None))
        return ModelSpec(architecture=self.architecture, hidden=self.width, vocab=self.vocab, layers=tuple(blocks),
                         schedule=tuple(ScheduleEntry(l) for l in range(len(blocks))), final_norm=norm, tied_head=False,
                         max_positions=MAX_POSITIONS, frame="sinusoids",
                         frame_spec=SinusoidEmbeddingSpec(10000.0, self.logit_scale))
