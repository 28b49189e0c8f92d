"""Sinusoidal positions: a fixed vector of every position that is added to its embedded row,

    s(p)[2 i] = sin(p f_i),  s(p)[2 i + 1] = cos(p f_i),  f_i = base^(-2 i / width).

Frequencies are float64; the kernel takes a position's angle back into one turn in float64 and its sine and cosine in float32.
An embedding that can (``Embedding.join``) adds the vector in its own kernel."""

from __future__ import annotations

from typing import Dict, Optional

import torch

from .. import ops
from .base import POSITION_ENCODINGS, PositionEncoding, Runtime, StepContext


@POSITION_ENCODINGS.register("sinusoidal")
class SinusoidalPositions(PositionEncoding):
    def __init__(self, width: int, base: float = 10000.0):
        super().__init__(width=width, base=base)
        self.width, self.base = int(width), float(base)
        self.frequencies: Optional[torch.Tensor] = None

    def load(self, tensors: Dict[str, torch.Tensor], rt: Runtime) -> None:
        super().load(tensors, rt)
        pairs = torch.arange((self.width + 1) // 2, dtype=torch.float64)
        self.frequencies = torch.pow(torch.tensor(self.base, dtype=torch.float64), -2.0 * pairs / self.width).to(rt.device)

    def on_embeddings(self, residual: torch.Tensor, ctx: StepContext) -> None:
        ops.embed_sum(None, ctx.tokens, ctx.row_pos, ctx.row_slot, residual, frequencies=self.frequencies)
