"""Token embedding and the output head (crates/bc-infer/src/model.rs:270-280, 361-370)."""

from __future__ import annotations

from typing import Any, Dict, Mapping, Optional

import torch

from .. import ops
from . import products
from .base import EMBEDDINGS, HEADS, CacheNeed, Embedding, Head, PositionEncoding, RunMemory, Runtime, StepContext, TensorSpec
from .sinusoidal import SinusoidalPositions


@EMBEDDINGS.register("token_embedding")
class TokenEmbedding(Embedding):
    """``scale`` multiplies every embedded row (1: as stored).

    ``bigram`` = {"buckets", "mul_prev", "mul_cur", "tensor"} adds a second embedding, named by a token and the one before it: row
    (before * mul_prev + token * mul_cur) mod buckets of a table of buckets + 1 rows, the last row for a sequence's first token.  The
    token before may have come in an earlier step, so token ids are kept page by page like keys and values are: they outlive a step,
    go back with a cut sequence, and are given back with it."""

    def __init__(self, vocab_size: int, hidden_size: int, tensor: str = "weight", scale: float = 1.0, bigram: Optional[Mapping[str, Any]] = None):
        super().__init__(vocab_size=vocab_size, hidden_size=hidden_size, tensor=tensor, scale=scale, bigram=bigram)
        self.vocab_size, self.hidden_size, self.tensor, self.scale = int(vocab_size), int(hidden_size), str(tensor), float(scale)
        self.bigram = None
        if bigram is not None:
            self.buckets, self.mul_prev, self.mul_cur = (int(bigram[k]) for k in ("buckets", "mul_prev", "mul_cur"))
            self.bigram = str(bigram.get("tensor", "bigram"))
            if self.buckets < 1 or not (0 <= self.mul_prev < 1 << 31 and 0 <= self.mul_cur < 1 << 31):
                raise ValueError(f"a bigram embedding wants at least one bucket and factors within 0 .. 2^31 - 1, got {dict(bigram)}")
        self.sinusoid: Optional[SinusoidalPositions] = None

    def tensors(self) -> Dict[str, TensorSpec]:
        out = {self.tensor: TensorSpec((self.vocab_size, self.hidden_size))}
        if self.bigram is not None:
            out[self.bigram] = TensorSpec((self.buckets + 1, self.hidden_size))
        return out

    def cache_need(self) -> Optional[CacheNeed]:
        return None if self.bigram is None else CacheNeed(((1, 1),), dtype=torch.int32)

    def join(self, position: PositionEncoding) -> bool:
        if type(position) is not SinusoidalPositions:
            return False
        self.sinusoid = position
        return True

    def load(self, tensors: Dict[str, torch.Tensor], rt: Runtime) -> None:
        super().load(tensors, rt)
        self.weight = tensors[self.tensor].contiguous()
        self.pairs = None if self.bigram is None else tensors[self.bigram].contiguous()

    def forward(self, ctx: StepContext, residual: torch.Tensor, mem: Optional[RunMemory] = None) -> None:
        if self.pairs is None and self.sinusoid is None:
            ops.embed(self.weight, ctx.tokens[: residual.shape[0]], residual, self.scale)
            return
        if self.pairs is not None and (mem is None or not mem.planes):
            raise RuntimeError("a bigram embedding was given no memory: the cache does not serve it")
        more = {} if self.pairs is None else {"pairs": self.pairs, "mul_prev": self.mul_prev, "mul_cur": self.mul_cur, "page_table": mem.page_table,
                                              "history": mem.planes[0]}
        ops.embed_sum(self.weight, ctx.tokens, ctx.row_pos, ctx.row_slot, residual, scale=self.scale,
                      frequencies=None if self.sinusoid is None else self.sinusoid.frequencies, **more)

    def table(self) -> Optional[torch.Tensor]:
        return self.weight


@HEADS.register("linear_head")
class LinearHead(Head):
    """Scores = x W^T in float32.  A tied head has no tensor of its own and multiplies by
    the embedding table (model.rs:200); a folder that still stores one is tolerated.
    ``scale`` multiplies the scores (1: as they are); ``softcap`` > 0 then bounds them: s <- softcap * tanh(s / softcap)."""

    def __init__(self, vocab_size: int, hidden_size: int, tied: bool = False, tensor: str = "weight", softcap: float = 0.0, scale: float = 1.0):
        super().__init__(vocab_size=vocab_size, hidden_size=hidden_size, tied=tied, tensor=tensor, softcap=softcap, scale=scale)
        self.vocab_size, self.hidden_size, self.tied, self.tensor = int(vocab_size), int(hidden_size), bool(tied), str(tensor)
        self.softcap, self.scale = float(softcap), float(scale)
        self.weight: Optional[torch.Tensor] = None

    def tensors(self) -> Dict[str, TensorSpec]:
        return {self.tensor: TensorSpec((self.vocab_size, self.hidden_size), optional=self.tied)}

    def load(self, tensors: Dict[str, torch.Tensor], rt: Runtime) -> None:
        super().load(tensors, rt)
        self.weight = None if self.tied else tensors[self.tensor].contiguous()

    def forward(self, x: torch.Tensor, out: torch.Tensor, tied: Optional[torch.Tensor]) -> None:
        w = tied if self.tied else self.weight
        if w is None:
            raise RuntimeError("a tied head needs the embedding's table")
        products.linear(x, w, out, products.EPI_STORE_F32, "head product")
        if self.scale != 1.0:
            ops.scale_scores(out, self.scale)
        if self.softcap > 0.0:
            ops.softcap(out, self.softcap)
