"""The gated delta rule with a decay a key channel: a recurrent mixer with one float state [head_dim, value_dim] a head.

q, k (kv_heads x head_dim) and v (heads x value_dim) from h, each through a short causal convolution over time a channel and silu
(the convolution's last inputs are per-sequence state too); q and k to unit length a head, q over sqrt(head_dim); heads / kv_heads
neighbouring heads share one q and k.  With b = sigmoid(W_b h), one number a head, and a decay a head and key channel

    c = exp(-exp(A_log) softplus(W_a2 (W_a1 h) + dt_bias))

a token moves the state and reads it:

    S <- diag(c) S;    r = b (v - S^T k);    S <- S + k r^T;    o = S^T q

Each head's o over its root mean square times a weight of value_dim numbers the heads share, times sigmoid(W_g2 (W_g1 h)), then W_o.

One product gives all that is read from h and keeps its float accumulators; convolution, unit vectors, decays, the state and the
read-out are float.  The outer products W_a2 and W_g2 take the inner vectors as float too: on the 32-bit path as they are, on the
tensor cores as two bfloat16 terms side by side (exact to about 2^-17) against the matrix stored twice.
"""

from __future__ import annotations

from typing import Dict, Optional

import torch

from .. import ops
from . import products
from .base import MIXERS, Mixer, RunMemory, Runtime, StateNeed, StepContext, TensorSpec

split_steps = False      # tests: steps of single rows through the kernels of a prompt step


@MIXERS.register("channel_delta")
class ChannelDelta(Mixer):
    def __init__(self, hidden_size: int, heads: int, kv_heads: int, head_dim: int, value_dim: int, taps: int, decay_rank: int, gate_rank: int,
                 norm_eps: float):
        super().__init__(hidden_size=hidden_size, heads=heads, kv_heads=kv_heads, head_dim=head_dim, value_dim=value_dim, taps=taps,
                         decay_rank=decay_rank, gate_rank=gate_rank, norm_eps=norm_eps)
        if heads % kv_heads:
            raise ValueError(f"{heads} heads are not a multiple of {kv_heads} kv heads")
        if not 0 < int(head_dim) <= 256:
            raise ValueError(f"a head of {head_dim} key channels is outside what the recurrence kernel takes (1 to 256)")
        if not 1 <= int(taps) <= ops.SSD_MAX_TAPS:
            raise ValueError(f"a convolution of {taps} taps is outside what the kernel takes (1 to {ops.SSD_MAX_TAPS})")
        self.hidden_size, self.heads, self.kv_heads = int(hidden_size), int(heads), int(kv_heads)
        self.head_dim, self.value_dim, self.taps = int(head_dim), int(value_dim), int(taps)
        self.decay_rank, self.gate_rank, self.norm_eps = int(decay_rank), int(gate_rank), float(norm_eps)
        self.channels = 2 * self.kv_heads * self.head_dim + self.heads * self.value_dim
        # Columns of the fused projection, each run starting at a multiple of 4: [q | k | v], the two inner vectors, b.
        up4 = lambda n: -(-n // 4) * 4
        self.a_at = up4(self.channels)
        self.g_at = self.a_at + up4(self.decay_rank)
        self.b_at = self.g_at + up4(self.gate_rank)
        self.columns = self.b_at + up4(self.heads)

    def tensors(self) -> Dict[str, TensorSpec]:
        e, gd, hd, hp = self.hidden_size, self.kv_heads * self.head_dim, self.heads * self.head_dim, self.heads * self.value_dim
        return {
            "q": TensorSpec((gd, e)), "q.conv": TensorSpec((gd, self.taps), role="vector"),
            "k": TensorSpec((gd, e)), "k.conv": TensorSpec((gd, self.taps), role="vector"),
            "v": TensorSpec((hp, e)), "v.conv": TensorSpec((hp, self.taps), role="vector"),
            "b": TensorSpec((self.heads, e)), "A_log": TensorSpec((self.heads,), role="vector", init="zeros"),
            "norm": TensorSpec((self.value_dim,), role="vector", init="ones"),
            "a1": TensorSpec((self.decay_rank, e)), "a2": TensorSpec((hd, self.decay_rank)),
            "dt_bias": TensorSpec((hd,), role="vector", init="zeros"),
            "g1": TensorSpec((self.gate_rank, e)), "g2": TensorSpec((hp, self.gate_rank)), "o": TensorSpec((e, hp)),
        }

    def state_need(self) -> Optional[StateNeed]:
        return StateNeed((self.heads, self.value_dim, self.head_dim), torch.float32)      # value channel by value channel

    def more_state_needs(self) -> Dict[str, StateNeed]:
        # The convolution's last inputs; one row more than needed when taps is 1, so that the tensor is never empty.
        return {"conv": StateNeed((max(self.taps - 1, 1), self.channels), torch.float32)}

    def load(self, tensors: Dict[str, torch.Tensor], rt: Runtime) -> None:
        super().load(tensors, rt)
        w = torch.zeros((self.columns, self.hidden_size), dtype=rt.dtype, device=tensors["q"].device)
        w[:self.channels] = torch.cat([tensors[n] for n in ("q", "k", "v")], dim=0)
        for at, name in ((self.a_at, "a1"), (self.g_at, "g1"), (self.b_at, "b")):
            w[at:at + tensors[name].shape[0]] = tensors[name]
        self.w_in, self.w_o = w, tensors["o"].contiguous()
        self.conv_t = torch.cat([tensors[n] for n in ("q.conv", "k.conv", "v.conv")], dim=0).t().contiguous()      # [taps, channels]
        self.w_a2, self.w_g2 = tensors["a2"].contiguous(), tensors["g2"].contiguous()
        self.terms = 1 if rt.is_f32 else 2
        self.w_a2_terms, self.w_g2_terms = (m if self.terms == 1 else torch.cat([m, m], dim=1).contiguous() for m in (self.w_a2, self.w_g2))
        self.a_log, self.dt_bias, self.norm_weight = (tensors[n].contiguous() for n in ("A_log", "dt_bias", "norm"))

    def forward(self, x: torch.Tensor, residual: torch.Tensor, ctx: StepContext, mem: RunMemory) -> None:
        tail = mem.states.get("mixer.conv")
        if mem.state is None or tail is None:
            raise RuntimeError("the delta rule was given no state: the cache does not serve this run")
        rows, H, G, D, P, dev = x.shape[0], self.heads, self.kv_heads, self.head_dim, self.value_dim, x.device
        f32 = torch.float32
        proj = torch.empty((rows, self.columns), dtype=f32, device=dev)
        products.linear(x, self.w_in, proj, products.EPI_STORE_F32, "delta projections")
        qkv = torch.empty((rows, self.channels), dtype=f32, device=dev)
        ops.ssd_prepare(proj, 0, 0, self.conv_t, None, None, None, tail, ctx.seq_rows, ctx.seq_slot, qkv, None, ctx.seqs, ctx.max_new,
                        write_tail=mem.writes)
        y = torch.empty((rows, H * P), dtype=x.dtype, device=dev)
        if ctx.decode and not split_steps and ops.delta_channel_step_accepts(D, P, self.decay_rank, self.gate_rank):
            # One row a sequence: outer products, unit vectors, one step of the recurrence, norm and gate in one launch.
            ops.delta_channel_step(qkv, proj, self.b_at, self.a_at, self.g_at, self.w_a2, self.w_g2, self.a_log, self.dt_bias, self.norm_weight,
                                   mem.state, ctx.row_slot, y, H, G, D, P, self.norm_eps, write_state=mem.writes)
            products.linear(y, self.w_o, residual, products.EPI_ADD_F32, "output product")
            return
        xa = torch.empty((rows, self.terms * self.decay_rank), dtype=x.dtype, device=dev)
        xg = torch.empty((rows, self.terms * self.gate_rank), dtype=x.dtype, device=dev)
        ops.delta_split(proj, self.a_at, xa, self.g_at, xg, self.terms)
        z = torch.empty((rows, H * D), dtype=f32, device=dev)
        products.linear(xa, self.w_a2_terms, z, products.EPI_STORE_F32, "low-rank product")
        gate = torch.empty((rows, H * P), dtype=f32, device=dev)
        products.linear(xg, self.w_g2_terms, gate, products.EPI_STORE_F32, "low-rank product")
        scal = torch.empty((rows, H, 2), dtype=f32, device=dev)
        ops.delta_channel_prepare(qkv, z, proj, self.b_at, self.a_log, self.dt_bias, scal, H, G, D)
        o = torch.empty((rows, H * P), dtype=f32, device=dev)
        ops.delta_channel_scan(qkv, z, scal, mem.state, ctx.seq_rows, ctx.seq_slot, o, ctx.seqs, H, G, D, P, write_state=mem.writes)
        ops.gated_norm(o, gate, 0, self.norm_weight, y, H, self.norm_eps, gate_first=False, row_slot=ctx.row_slot, activation="sigmoid")
        products.linear(y, self.w_o, residual, products.EPI_ADD_F32, "output product")
