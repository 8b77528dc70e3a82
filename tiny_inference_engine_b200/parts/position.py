"""Rotary position encoding, rotate-half over the first `rotary_dim` dims of a head:
inv_freq[i] = 1 / theta^(2i / rotary_dim) in float32, angle = float(pos) * inv_freq[i]
(src/backend/rope.h:9-13, src/backend/cpu/cpu_backend.cpp:161-193). The table is computed
once on the host, as the reference does, so that angles are the same float32 products.

Options: `pairing` "halves" (dimension i with i + rotary_dim / 2; the default) or "neighbours" (2i with 2i + 1), and `angles`
"float32" (the products above; the default) or "float64" (a position's turns formed and reduced in double, so that far
positions lose nothing), for the kernels that take a `rotation()`."""
from __future__ import annotations

import numpy as np
import torch

from .. import ops
from ..errors import InvalidArgument
from .base import PositionEncoding, register_part


class RotaryEncoding(PositionEncoding):
    launches_only = True

    def __init__(self, spec, dtype, prefix: str = ""):
        self.theta = float(spec["theta"])
        self.head_dim = int(spec["head_dim"])
        self.rotary_dim = int(spec.params.get("rotary_dim", self.head_dim))
        if self.rotary_dim % 2 or not 0 < self.rotary_dim <= self.head_dim:
            raise InvalidArgument(f"rotary_dim {self.rotary_dim} must be even and at most head_dim {self.head_dim}")
        pairing, angles = spec.params.get("pairing", "halves"), spec.params.get("angles", "float32")
        if pairing not in ("halves", "neighbours") or angles not in ("float32", "float64"):
            raise InvalidArgument(f"a rotation pairs halves or neighbours with float32 or float64 angles, got {pairing!r}, {angles!r}")
        self.neighbours, self.double_angles = pairing == "neighbours", angles == "float64"
        i = np.arange(self.rotary_dim // 2, dtype=np.float32)
        expo = (np.float32(2.0) * i) / np.float32(self.rotary_dim)
        self.inv_freq_host = (np.float32(1.0) / np.power(np.float32(self.theta), expo, dtype=np.float32)).astype(np.float32)
        self._table = self._turns = None

    def fused_table(self):
        if self.neighbours or self.double_angles:
            return None                 # the fused kernel pairs halves and multiplies in float32
        return self._inverse_frequencies()

    def _inverse_frequencies(self):
        if self._table is None:
            self._table = torch.from_numpy(self.inv_freq_host).cuda()
        return self._table

    def rotation(self):
        return (self.turns_table() if self.double_angles else self._inverse_frequencies()), self.neighbours

    def turns_table(self):
        """float64 [rotary_dim / 2]: the turns a position makes, theta^(-2i/rotary_dim) / (2 pi). For kernels that form the
        angle in double precision, so that far positions lose nothing."""
        if self._turns is None:
            i = np.arange(self.rotary_dim // 2, dtype=np.float64)
            self._turns = torch.from_numpy(self.theta ** (-2.0 * i / self.rotary_dim) / (2.0 * np.pi)).cuda()
        return self._turns

    def apply(self, x, positions, heads, head_dim):
        table, neighbours = self.rotation()
        ops.rope(x, positions, table, heads, head_dim, neighbours)


class NoPositionEncoding(PositionEncoding):
    """Leaves q and k as they are."""

    launches_only = True
    is_identity = True

    def __init__(self, spec=None, dtype=None, prefix: str = ""):
        pass

    def apply(self, x, positions, heads, head_dim):
        return None


register_part("position", "rope", RotaryEncoding, replace=True)
register_part("position", "none", NoPositionEncoding, replace=True)
