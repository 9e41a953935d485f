"""Rotary position encoding: the table of angles (src/model.c:116-124).

A position encoding of the rotary family gives the attention mixer
  tables(n_positions, device) -> (cos, sin), float32 [n_positions, rotary_dim / 2]
  rotary_dim, interleaved
and the q/k preparation kernel applies them. The angles are made on the host
in float32 with abacus's own expression, pos * (1 / theta^(2i / rotary_dim)).
"""
import math

import numpy as np
import torch

from .base import POSITIONS


@POSITIONS.register("rotary")
class Rotary:
    def __init__(self, spec):
        if spec.pairing not in ("half", "interleaved"):
            raise ValueError(f"rotary pairing {spec.pairing!r} is neither half nor interleaved")
        if spec.rotary_dim < 2 or spec.rotary_dim % 2:
            raise ValueError(f"rotary_dim {spec.rotary_dim} must be even")
        scalings = (getattr(spec, "linear_factor", 1.0) != 1.0, bool(getattr(spec, "blend", None)), bool(getattr(spec, "bands", None)))
        if any(scalings) and not spec.exact_angles:
            raise ValueError("scaled frequencies are made with exact_angles")
        if scalings[2] and (scalings[1] or not spec.bands[3] > spec.bands[2]):
            raise ValueError("frequencies are scaled in bands or blended, not both, and the bands' high is above their low")
        self.spec = spec
        self.rotary_dim = spec.rotary_dim
        self.interleaved = spec.pairing == "interleaved"
        self._tables = {}

    def frequencies(self):
        """(the pairs' frequencies float64 [rotary_dim / 2], the factor on cosines and sines) with the spec's scaling."""
        s, dims = self.spec, self.rotary_dim
        i = np.arange(dims // 2, dtype=np.float64)
        freq = np.power(float(s.theta), -2.0 * i / dims) / float(getattr(s, "linear_factor", 1.0))
        blend, bands = getattr(s, "blend", None), getattr(s, "bands", None)
        if bands is not None:
            factor, original, low, high = (float(v) for v in bands)
            turns = original * freq / (2.0 * math.pi)  # a pair's turns over the original context
            share = (turns - low) / (high - low)
            between = (1.0 - share) * freq / factor + share * freq
            return np.where(turns > high, freq, np.where(turns < low, freq / factor, between)), 1.0
        if blend is None:
            return freq, 1.0
        factor, original, fast, slow = (float(v) for v in blend)

        def where(turns):  # the pair that makes `turns` turns over the original context
            return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(float(s.theta)))
        lo, hi = max(math.floor(where(fast)), 0), min(math.ceil(where(slow)), dims - 1)
        ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
        return freq / factor * ramp + freq * (1.0 - ramp), 0.1 * math.log(factor) + 1.0

    def tables(self, n_positions, device):
        key = str(device)
        have = self._tables.get(key)
        if have is None or have[0].shape[0] < n_positions:
            half = self.rotary_dim // 2
            if getattr(self.spec, "exact_angles", False):  # position * theta^(-2i / rotary_dim) in float64
                freq, amplitude = self.frequencies()
                angle = np.arange(n_positions, dtype=np.float64)[:, None] * freq[None, :]
                have = (torch.from_numpy((np.cos(angle) * amplitude).astype(np.float32)).to(device),
                        torch.from_numpy((np.sin(angle) * amplitude).astype(np.float32)).to(device))
                self._tables[key] = have
                return have
            i = np.arange(half, dtype=np.float32)
            inv = np.float32(1.0) / np.power(np.float32(self.spec.theta),
                                             (np.float32(2.0) * i) / np.float32(self.rotary_dim), dtype=np.float32)
            angle = (np.arange(n_positions, dtype=np.float32)[:, None] * inv[None, :]).astype(np.float32)
            have = (torch.from_numpy(np.cos(angle, dtype=np.float32)).to(device),
                    torch.from_numpy(np.sin(angle, dtype=np.float32)).to(device))
            self._tables[key] = have
        return have


class Sinusoids:
    """Fixed sinusoids per position: element 2i of a vector is sin(p * base^(-2i / size)), element 2i + 1 its cosine.

    tables(n_positions, device) -> (coarse, fine), float32 [.., ceil(size / 2), 2] (sine, cosine), made in float64: position
    256 a + b has the sum of the angles of coarse[a] and fine[b], so a million positions take 4,096 + 256 rows.
    """
    FINE = 256

    def __init__(self, size, base):
        self.size, self.base = size, float(base)
        self._tables = {}

    def tables(self, n_positions, device):
        key, rows = str(device), max(1, -(-n_positions // self.FINE))
        have = self._tables.get(key)
        if have is None or have[0].shape[0] < rows:
            i = np.arange((self.size + 1) // 2, dtype=np.float64)
            freq = np.power(self.base, -2.0 * i / self.size)

            def table(positions):
                angle = positions.astype(np.float64)[:, None] * freq[None, :]
                return torch.from_numpy(np.stack([np.sin(angle), np.cos(angle)], axis=-1).astype(np.float32)).to(device)
            have = (table(np.arange(rows) * self.FINE), table(np.arange(self.FINE)))
            self._tables[key] = have
        return have
