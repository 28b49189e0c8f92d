"""Differential grouped-query attention over the paged cache.

Every head holds two query maps of ``head_dim`` values, every kv head two key maps over one set of values:

    A_m = softmax over the visible positions of (q_m . k_m * scale), times v        m = 0, 1
    lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff          (four vectors of head_dim numbers, one lambda for the layer)
    z = A_0 - lambda A_1,    out = z / sqrt(mean(z^2) + eps) * (1 - diff)            (the mean over the head's values)

- q and k pass an RMS norm a head and map with one weight each of ``head_dim`` values, then the rotation of the first dimensions of
  every map (the position encoding's);
- a row at position i sees j <= i with i - j < window or j < keep_first (window 0: every j <= i);
- ``own_kv`` False: the mixer has no keys and values of its own and reads those of the run that its schedule entry names
  (``RunSpec.memory_of``), as that run cached them, with its own queries and mask.

The cache keeps 2 kv_heads key maps (those of a kv head side by side) and kv_heads values a position.  The fused projection keeps its
float accumulators; norms, rotation, scores, softmax, the difference and its norm are float; q, the cached k and v and the result
take the activation type.
"""

from __future__ import annotations

from typing import Any, Dict, Mapping, Optional

import torch

from .. import ops
from . import products
from .base import MIXERS, POSITION_ENCODINGS, CacheNeed, Mixer, RunMemory, Runtime, StepContext, TensorSpec

# Tests: "rows" (the one-warp-a-row kernel, the checked twin), "tiles" (mma.sync tiles) or "tc" (tcgen05) wherever the sizes allow it;
# None: the part chooses.
force: Optional[str] = None
force_splits = 0        # tests: share a row's pages out over this many blocks in steps of few rows (0: the part chooses)


@MIXERS.register("differential_attention")
class DifferentialAttention(Mixer):
    def __init__(self, hidden_size: int, heads: int, kv_heads: int, head_dim: int, value_dim: int, norm_eps: float, diff: float,
                 position: Mapping[str, Any], scale: Optional[float] = None, window: int = 0, keep_first: int = 0, own_kv: bool = True):
        super().__init__(hidden_size=hidden_size, heads=heads, kv_heads=kv_heads, head_dim=head_dim, value_dim=value_dim, norm_eps=norm_eps,
                         diff=diff, position=position, scale=scale, window=window, keep_first=keep_first, own_kv=own_kv)
        if heads % kv_heads:
            raise ValueError(f"{heads} heads are not a multiple of {kv_heads} kv heads")
        if not 0 < head_dim <= 256 or not 0 < value_dim <= 256:
            raise ValueError(f"a map of {head_dim} or values of {value_dim} are refused by the differential attention kernels (1 to 256)")
        self.hidden_size, self.heads, self.kv_heads = int(hidden_size), int(heads), int(kv_heads)
        self.head_dim, self.value_dim = int(head_dim), int(value_dim)
        self.norm_eps, self.diff = float(norm_eps), float(diff)
        self.window, self.keep_first, self.own_kv = int(window), int(keep_first) if window else 0, bool(own_kv)
        self.scale = float(scale) if scale is not None else 1.0 / float(head_dim) ** 0.5
        pos = dict(position)
        self.position = POSITION_ENCODINGS.get(pos.pop("kind"))(**pos)
        self.rotary_dims = int(getattr(self.position, "head_dim", 0))
        if self.rotary_dims > self.head_dim:
            raise ValueError(f"{self.rotary_dims} rotated dimensions do not fit a map of {self.head_dim}")

    def tensors(self) -> Dict[str, TensorSpec]:
        H, G, d, v, e = self.heads, self.kv_heads, self.head_dim, self.value_dim, self.hidden_size
        out = {"q": TensorSpec((2 * H * d, e)), "q.norm": TensorSpec((d,), role="vector", init="ones"), "o": TensorSpec((e, H * v))}
        out.update({n: TensorSpec((d,), role="vector") for n in ("lq1", "lk1", "lq2", "lk2")})
        if self.own_kv:
            out.update({"k": TensorSpec((2 * G * d, e)), "k.norm": TensorSpec((d,), role="vector", init="ones"), "v": TensorSpec((G * v, e))})
        return out

    def cache_need(self) -> Optional[CacheNeed]:
        return CacheNeed(((2 * self.kv_heads, self.head_dim), (self.kv_heads, self.value_dim)), self.window, keep_first=self.keep_first)

    def load(self, tensors: Dict[str, torch.Tensor], rt: Runtime) -> None:
        super().load(tensors, rt)
        self.w_in = torch.cat([tensors["q"], tensors["k"], tensors["v"]], dim=0).contiguous() if self.own_kv else tensors["q"].contiguous()
        self.w_o = tensors["o"].contiguous()
        self.q_norm = tensors["q.norm"].contiguous()
        self.k_norm = tensors["k.norm"].contiguous() if self.own_kv else None
        lq1, lk1, lq2, lk2 = (tensors[n].double() for n in ("lq1", "lk1", "lq2", "lk2"))
        self.lam = float(torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + self.diff)      # of the weights alone: once
        self.position.load({}, rt)

    def path(self, ctx: StepContext, dtype: torch.dtype) -> str:
        """Which kernel this step's rows take: prompts tcgen05 tiles where the widths are 64 or 128, other widths and steps of few rows a
        sequence mma.sync tiles, the 32-bit path and what no tile takes one warp a row."""
        H, G, D, DV = self.heads, self.kv_heads, self.head_dim, self.value_dim
        if force in (None, "tc") and not ctx.decode and ctx.max_new * (H // G) > 16 and ops.diff_attention_tc_accepts(H, G, D, DV, dtype):
            return "tc"
        return "tiles" if force != "rows" and ops.diff_tiles_accepts(H, G, D, DV, dtype) else "rows"

    def forward(self, x: torch.Tensor, residual: torch.Tensor, ctx: StepContext, mem: RunMemory) -> None:
        if len(mem.planes) != 2:
            raise RuntimeError("differential attention was given no cache: the cache does not serve this run")
        rows, H, G, D, DV = x.shape[0], self.heads, self.kv_heads, self.head_dim, self.value_dim
        proj = torch.empty((rows, self.w_in.shape[0]), dtype=torch.float32, device=x.device)
        products.linear(x, self.w_in, proj, products.EPI_STORE_F32, "qkv product" if self.own_kv else "query product")
        table = self.position.rotary()
        q = torch.empty((rows, H * 2 * D), dtype=x.dtype, device=x.device)
        ops.qkv_prepare_heads(proj, self.q_norm, self.k_norm, None if table is None else table.cos_sin, ctx.row_pos, ctx.row_slot, mem.page_table, q,
                              mem.k_pages if self.own_kv else None, mem.v_pages if self.own_kv else None, 2 * H, 2 * G if self.own_kv else 0, D, DV,
                              self.rotary_dims if table is not None else 0, 0 if table is None else table.pairing, self.norm_eps,
                              write_cache=mem.writes and self.own_kv, value_heads=G if self.own_kv else 0)
        att = torch.empty((rows, H * DV), dtype=x.dtype, device=x.device)
        numbers = dict(window=self.window, keep_first=self.keep_first, scale=self.scale, lam=self.lam, eps=self.norm_eps, factor=1.0 - self.diff)
        path = self.path(ctx, x.dtype)
        if path == "rows":
            ops.diff_rows(q, mem.k_pages, mem.v_pages, mem.page_table, ctx.row_pos, ctx.row_slot, att, H, G, D, DV, **numbers)
        elif path == "tc":
            ops.diff_attention_tc(q, mem.k_pages, mem.v_pages, mem.page_table, ctx.seq_rows, ctx.seq_slot, ctx.seq_start, att, ctx.seqs, ctx.max_new, H, G, D, DV,
                                  **numbers)
        else:
            splits = 1
            if ctx.decode:
                splits = force_splits or ops.diff_tiles_splits(ctx.seqs, G, ctx.max_total, self.window, self.keep_first)
            ops.diff_tiles(q, mem.k_pages, mem.v_pages, mem.page_table, ctx.seq_rows, ctx.seq_slot, ctx.seq_start, ctx.row_slot, att, ctx.seqs,
                           ctx.max_new, H, G, D, DV, splits=splits, **numbers)
        products.linear(att, self.w_o, residual, products.EPI_ADD_F32, "output product")
