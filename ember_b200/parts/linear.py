"""A weight matrix [out, in] on the device and the product y = x . W^T with a fused epilogue.

The kernel is chosen by dtype and shape: the tcgen05 tensor-core kernel for bfloat16 weights
and activations whose sizes it takes, the fp32 SIMT kernel otherwise (always on the float32
path: that is the true 32-bit product).
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from .base import Runtime


class Linear:
    def __init__(self, weight: torch.Tensor, bias: Optional[torch.Tensor] = None):
        self.weight = weight            # [N, K], float32 or bfloat16, on the device
        self.bias = bias                # float32 [N] or None
        self.n, self.k = weight.shape
        if weight.is_cuda and weight.dtype == torch.bfloat16:
            # the small-M tensor-core product sums its K parts in a shared fp32 scratch of up to 128 x N: made
            # now, so that no step (least of all one inside a captured graph's lifetime) has to grow it
            ops.reserve_scratch(weight.device, 128 * self.n)

    @classmethod
    def from_host(cls, w: torch.Tensor, rt: Runtime, bias: Optional[torch.Tensor] = None) -> "Linear":
        dev = rt.to_device(w, rt.weight_dtype(w.dtype))
        b = rt.to_device(bias, torch.float32) if bias is not None else None
        return cls(dev, b)

    # A prompt portion's product with so few columns has too few tiles for the SMs; added into zeros, K is cut as well.
    NARROW = 512

    def store_f32(self, ctx, x: torch.Tensor, out: torch.Tensor, m: int) -> None:
        """out[:m] = the product in fp32, in whichever way fills the device: stored, or (narrow products of prompt portions on
        the tensor cores) added into zeros in parts of K."""
        if m > 128 and self.n <= self.NARROW and self.k >= 1024 and ops.gemm_tc_usable(x, self.weight, self.bias, ops.EPI_ADD_F32):
            ops.zero(out, m * self.n, stream=ctx.stream)
            self(ctx, x, out, m, ops.EPI_ADD_F32)
        else:
            self(ctx, x, out, m, ops.EPI_STORE_F32)

    def __call__(self, ctx, x: torch.Tensor, out: torch.Tensor, m: int, epilogue: int = ops.EPI_STORE) -> None:
        if m <= 0:
            return
        if ops.gemm_tc_usable(x, self.weight, self.bias, epilogue):
            ops.gemm_tc(x, self.weight, out, m, epilogue, err=ctx.err, stream=ctx.stream, bias=self.bias)
        else:
            ops.gemm_simt(x, self.weight, out, m, epilogue, bias=self.bias, stream=ctx.stream)
