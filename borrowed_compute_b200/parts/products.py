"""The one place that decides which kernel multiplies matrices.

``linear(x, w, out, epilogue)`` computes ``x @ w.T`` with float accumulation.  On the
32-bit path it is the CUDA-core kernel (tensor cores would round operands to tf32).  For
bfloat16 it is the tcgen05 tensor-core kernel; the CUDA-core kernel on the same operands is
its checked twin and can be forced for a test with ``force_simt``.
"""

from __future__ import annotations

import torch

from .. import ops
from ..ops import EPI_ADD_F32, EPI_RELU2, EPI_SILU_F32, EPI_STORE, EPI_STORE_F32, EPI_SWIGLU, EPI_XIELU  # noqa: F401  (re-exported)

force_simt = False


def takes_tensor_cores(x: torch.Tensor, w: torch.Tensor) -> bool:
    """Whether ``linear`` multiplies these operands on the tensor cores."""
    return x.dtype == torch.bfloat16 and not force_simt and hasattr(ops, "gemm_tc") and ops.gemm_tc_accepts(x, w)


def linear(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, epilogue: int, what: str = "", glu=None, act=None, cols=None) -> None:
    """``what`` names the product for a profile of the step ("qkv", "head", ...).  ``glu`` = (limit, alpha): the bounded gate of
    the tensor-core product's gated epilogue (callers ask ``takes_tensor_cores`` first).  ``act`` = (a, b): the numbers of EPI_XIELU;
    ``cols``: how many of the first output columns EPI_SILU_F32 gates."""
    if ops.timeline is not None and what:
        ops.label = what
        try:
            linear(x, w, out, epilogue, glu=glu, act=act, cols=cols)
        finally:
            ops.label = ""
        return
    if takes_tensor_cores(x, w):
        ops.gemm_tc(x, w, out, epilogue, glu=glu, act=act, cols=cols)
    elif glu is not None:
        raise ops.KernelError("a bounded gate in the epilogue comes with the tensor-core product")
    else:
        ops.gemm_simt(x, w, out, epilogue, act=act, cols=cols)
