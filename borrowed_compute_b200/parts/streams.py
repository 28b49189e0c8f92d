"""A residual stream of several copies a row (hyper-connections).

A row carries a bundle X [S, E] of float32 streams.  Around every sublayer stands a *connection* with three small tensors, ``in``
[S], ``out`` [S] and ``mix`` [S, S] (indexed [from, to]):

    u = sum_s in[s] X_s,    y = sublayer(norm(u)),    X_t <- sum_s mix[s, t] X_s + out[t] * scale * y

with ``scale`` a *channel scale* [E] (or none).  :class:`StreamBundle` is what the blocks of such a model are handed instead of one
residual tensor: ``enter`` gives a sublayer its normed input, ``leave`` takes its result, ``finish`` adds the streams up for the
model's last norm.  A result that leaves is kept until the next sublayer enters, so that one kernel (``csrc/hyper_streams.cu``)
does both and the bundle is read and written once a sublayer.
"""

from __future__ import annotations

from typing import Dict, Optional, Tuple

import torch

from .. import ops
from .base import CONNECTIONS, SCALES, Part, Runtime, TensorSpec
from .norm import RMSNorm


@CONNECTIONS.register("hyper")
class HyperConnection(Part):
    def __init__(self, streams: int):
        super().__init__(streams=streams)
        if not 1 <= int(streams) <= ops.HYPER_MAX_STREAMS:
            raise ValueError(f"{streams} streams are outside what the kernels take (1 to {ops.HYPER_MAX_STREAMS})")
        self.streams = int(streams)

    def tensors(self) -> Dict[str, TensorSpec]:
        S = self.streams
        return {"in": TensorSpec((S,), role="vector", init="ones"), "out": TensorSpec((S,), role="vector", init="ones"),
                "mix": TensorSpec((S, S), role="vector", init="identity")}

    def load(self, tensors: Dict[str, torch.Tensor], rt: Runtime) -> None:
        super().load(tensors, rt)
        self.w_in, self.w_out, self.w_mix = (tensors[n].contiguous() for n in ("in", "out", "mix"))


@SCALES.register("channel_scale")
class ChannelScale(Part):
    """One factor a channel on a sublayer's result; ``tensor`` is the name it carries after the part's prefix."""

    def __init__(self, width: int, tensor: str = "scale"):
        super().__init__(width=width, tensor=tensor)
        self.width, self.tensor = int(width), str(tensor)

    def tensors(self) -> Dict[str, TensorSpec]:
        return {self.tensor: TensorSpec((self.width,), role="vector", init="ones")}

    def load(self, tensors: Dict[str, torch.Tensor], rt: Runtime) -> None:
        super().load(tensors, rt)
        self.weight = tensors[self.tensor].contiguous()


class StreamBundle:
    """The streams of one step's rows.  ``y`` [rows, E] float32 is where the current sublayer adds its result."""

    def __init__(self, rows: int, streams: int, hidden_size: int, device: torch.device):
        self.x = torch.empty((rows, streams, hidden_size), dtype=torch.float32, device=device)
        self.y = torch.zeros((rows, hidden_size), dtype=torch.float32, device=device)
        self.pending: Optional[Tuple[HyperConnection, Optional[ChannelScale]]] = None

    def start(self, embedded: torch.Tensor, norm: Optional[RMSNorm]) -> None:
        """Every stream becomes the (normed) embedded rows."""
        ops.hyper_start(embedded, None if norm is None else norm.weight, self.x, 1.0 if norm is None else norm.eps)

    def _step(self, w_in: Optional[torch.Tensor], norm: RMSNorm, out: torch.Tensor, gather: Optional[torch.Tensor]) -> None:
        if self.pending is None:
            ops.hyper_step(self.x, None, None, None, None, w_in, norm.weight, out, norm.eps, gather)
        else:
            c, scale = self.pending
            ops.hyper_step(self.x, self.y, None if scale is None else scale.weight, c.w_mix, c.w_out, w_in, norm.weight, out, norm.eps, gather)

    def enter(self, connection: HyperConnection, norm: RMSNorm, out: torch.Tensor) -> torch.Tensor:
        """out = norm(sum_s in[s] X_s) in its type; returns the cleared buffer the sublayer adds its result into."""
        self._step(connection.w_in, norm, out, None)
        self.pending = None
        return self.y

    def leave(self, connection: HyperConnection, scale: Optional[ChannelScale]) -> None:
        """The sublayer's result lies in ``y``."""
        self.pending = (connection, scale)

    def finish(self, norm: RMSNorm, out: torch.Tensor, gather: Optional[torch.Tensor]) -> None:
        """out = norm(sum_s X_s) of the rows ``gather`` names (all if None)."""
        self._step(None, norm, out, gather)

    def total(self) -> torch.Tensor:
        """The sum of the streams as it stands after the last sublayer, for looking inside a step."""
        s = self.x.sum(dim=1)
        if self.pending is not None:
            c, scale = self.pending
            y = self.y if scale is None else self.y * scale.weight
            s = torch.einsum("rse,s->re", self.x, c.w_mix.sum(dim=1)) + c.w_out.sum() * y
        return s
