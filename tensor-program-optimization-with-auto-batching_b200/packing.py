"""What the packed models of the designs without adapters share."""
from __future__ import annotations

import torch

from . import ops


def up(n, m):
    """``n`` rounded up to a multiple of ``m``."""
    return -(-n // m) * m


class PackedDesign:
    """Sizes every engine asks a model for, and zero-padded weights on the device: tiled for the tensor cores in bfloat16,
    as they are in float32."""

    name = ""
    dtypes = (torch.bfloat16, torch.float32)

    def __init__(self, cfg, vocab, width, n_layers, device, dtype):
        if dtype not in self.dtypes:
            raise ValueError(f"{self.name} runs in bfloat16 or float32, not {dtype}")
        self.cfg, self.dtype, self.device = dict(cfg), dtype, torch.device(device)
        self.V, self.L, self.width = vocab, n_layers, width
        self.H = up(width, 8)                          # pitch of residual and normalised rows
        self.tp_size, self.n_adapters = 1, 0           # (no adapters on these designs)

    def _mat(self, t, shape, dtype=None):
        """``t`` in the corner of a zero matrix of ``shape``, on the device."""
        out = torch.zeros(shape, dtype=dtype or self.dtype, device=self.device)
        out[tuple(slice(0, n) for n in t.shape)] = t.to(self.device).to(out.dtype)
        return out

    def _weight(self, t, shape):
        W = self._mat(t, shape)
        return ops.PackedWeight(W) if self.dtype == torch.bfloat16 else W

    def add_adapter(self, *_):
        raise ValueError(f"the {self.name} design has no adapters")
