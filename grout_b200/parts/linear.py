"""y = x W^T with W stored [out, in], the one linear layer every part uses.

It picks the product by the weight's precision and by the number of rows:

* 32-bit weight: the true 32-bit CUDA-core product (``gemm_f32``); bf16
  activations are widened first and the result narrowed, so a tensor that the
  checkpoint stores in 32-bit is used in 32-bit.
* bf16 weight, up to 64 rows (every decode step): the TMA-fed tcgen05 product
  with the weight rows on the 128-row side of the MMA (``gemm_tc_bf16`` with
  ``swap``), or, for ``products.decode = "skinny"``, the mma.sync weight-streaming
  kernel (``gemm_skinny_bf16``).
* bf16 weight, more rows (a prompt): ``products.prefill = "auto"`` takes the product
  on pairs of SMs (``gemm_tc2_bf16``, tcgen05.mma.cta_group::2) where it is at
  least as fast as the library's product, which is the fused gate|up product with
  its SiLU epilogue when its rounds of 256 x 256 tiles on the GPU's pairs of SMs
  are mostly full (``ops.gemm_tc2_pays`` has the measurements), and the library's
  product elsewhere, where the reference uses a library too (cuBLAS GemmEx,
  src/cublas.rs:287-307).  ``"pair"`` takes the pair product for everything it can
  store, ``"tc"`` the single-SM tcgen05 kernel in its other orientation,
  ``"library"`` the library throughout.  Measured at 2,048 rows (us, library /
  pair): qkv 46 / 47, o 35 / 48, gate|up 140 + 24 for SiLU / 149 fused, down 73 / 102
  (o and down are 80 tiles on 74 pairs of SMs: a second round for six tiles).
"""
from __future__ import annotations

from typing import Optional

import torch

from ..kernels import ops
from .base import ProductChoice


class Linear:
    def __init__(self, weight: torch.Tensor, products: Optional[ProductChoice] = None):
        """``products``: which kernels take the products (a part passes
        ``ctx.products``); None means the defaults."""
        products = products or ProductChoice()
        self.decode_kernel, self.prefill_kernel = products.decode, products.prefill
        if weight.dim() != 2:
            raise ValueError(f"a linear weight is [out, in], got {tuple(weight.shape)}")
        if weight.dtype not in (torch.float32, torch.bfloat16):
            raise ValueError(f"a linear weight is float32 or bfloat16, got {weight.dtype}")
        self.weight = weight.contiguous()
        self.out_features, self.in_features = weight.shape

    def kernel_modules(self):
        if self.weight.dtype == torch.float32:
            return ("gemm_f32", "elementwise")
        if self.in_features % 8:
            return ()                                  # only the library's product takes such a width
        mods = ("gemm_tc",) if "tc" in (self.decode_kernel, self.prefill_kernel) else ()
        if self.decode_kernel == "skinny":
            mods += ("gemm_skinny_bf16",)
        if self.prefill_kernel in ("auto", "pair"):
            mods += ("gemm_tc2",)
        return mods

    def __call__(self, x: torch.Tensor, out_dtype: Optional[torch.dtype] = None,
                 partial_ok: bool = False, into: Optional[torch.Tensor] = None) -> torch.Tensor:
        """``into``: a contiguous 32-bit tensor for the result ([``n_parts(M)``, M, N]; implies
        32-bit partial sums).  ``partial_ok``: the caller hands the result to a kernel that can add
        32-bit partial sums (a norm's residual add, the q/k preparation); a product
        with few rows and few tiles may then come back as [S, M, N] float32, its
        split-K reduction left to that kernel."""
        out_dtype = torch.float32 if into is not None else (out_dtype or x.dtype)
        partial_ok = partial_ok or into is not None
        w = self.weight
        if w.dtype == torch.float32:
            if into is not None:
                return ops.gemm_f32(ops.cast(x, torch.float32), w, into=into)
            y = ops.gemm_f32(ops.cast(x, torch.float32), w)
            return ops.cast(y, out_dtype)
        if x.dtype != torch.bfloat16:
            raise ops.KernelError("a bfloat16 weight takes bfloat16 activations")
        M = x.shape[0]
        if self.in_features % 8 == 0:
            if M <= ops.SKINNY_MAX_ROWS:
                if self.decode_kernel == "tc":
                    return ops.gemm_tc_bf16(x, w, out_dtype, swap=True, split_out=partial_ok, into=into)
                return ops.gemm_skinny_bf16(x, w, out_dtype, into=into)
            if self.prefill_kernel == "tc":
                return ops.gemm_tc_bf16(x, w, out_dtype, swap=False, into=into)
            if ops.gemm_tc2_takes(self.out_features, out_dtype) and (
                    self.prefill_kernel == "pair" or
                    (self.prefill_kernel == "auto" and
                     ops.gemm_tc2_pays(M, self.out_features, x.device, fused_silu=False))):
                return ops.gemm_tc2_bf16(x, w, out_dtype, into=into)
        return ops.library_mm(x, w, out_dtype, into=into)

    def n_parts(self, M: int) -> int:
        """How many 32-bit partial sums the product with M rows makes when it is asked to
        leave them (``partial_ok``): 1 where it leaves its finished sum."""
        w = self.weight
        if (w.dtype == torch.bfloat16 and self.in_features % 8 == 0 and M <= ops.SKINNY_MAX_ROWS
                and self.decode_kernel == "tc"):
            return max(1, ops.gemm_tc_parts(M, self.out_features, self.in_features, w.device))
        return 1

    def silu_mul(self, x: torch.Tensor, interleave: int, activation: str = "silu",
                 bias: Optional[torch.Tensor] = None) -> torch.Tensor:
        """act(gate + bg) * (up + bu) of a fused gate|up weight, ``activation`` "silu",
        "gelu_tanh" or "relu", ``bias`` the fused [bg | bu] in the rows' order or None.  ``interleave`` 0: gate rows first, then up rows; 8: groups of 8
        gate rows followed by their 8 up rows, which lets the tcgen05 kernels finish
        the product in their epilogue."""
        w = self.weight
        if activation != "silu" or bias is not None:
            return self._gated(x, interleave, activation, bias)
        if (interleave == 8 and w.dtype == torch.bfloat16 and x.shape[0] <= ops.SKINNY_MAX_ROWS
                and self.in_features % 8 == 0):
            if self.decode_kernel == "tc":
                return ops.gemm_tc_bf16(x, w, x.dtype, swap=True, silu_mul=True)
            return ops.gemm_skinny_bf16(x, w, x.dtype, silu_mul=True)
        if (interleave == 8 and w.dtype == torch.bfloat16 and x.dtype == torch.bfloat16
                and self.in_features % 8 == 0 and self.out_features % 32 == 0
                and (self.prefill_kernel == "pair" or
                     (self.prefill_kernel == "auto" and
                      ops.gemm_tc2_pays(x.shape[0], self.out_features, x.device, fused_silu=True)))):
            return ops.gemm_tc2_bf16(x, w, x.dtype, silu_mul=True)
        return ops.silu_mul(self(x), interleave)

    def _gated(self, x: torch.Tensor, interleave: int, activation: str,
               bias: Optional[torch.Tensor] = None) -> torch.Tensor:
        """The gate|up product with another activation than silu ("gelu_tanh", "relu") or
        with a ``bias`` (32-bit, in the fused rows' order, added to the 32-bit sums before
        the gate): the tcgen05 kernels have it as an epilogue (the mma.sync decode kernel
        has not), under the rules of ``silu_mul``; elsewhere the product and an
        elementwise kernel."""
        w = self.weight
        fusable = (interleave == 8 and w.dtype == torch.bfloat16 and x.dtype == torch.bfloat16
                   and self.in_features % 8 == 0)
        if fusable and x.shape[0] <= ops.SKINNY_MAX_ROWS and self.decode_kernel == "tc":
            return ops.gemm_tc_bf16(x, w, x.dtype, swap=True, silu_mul=True, gate_act=activation, bias=bias)
        if (fusable and x.shape[0] > ops.SKINNY_MAX_ROWS and self.out_features % 32 == 0
                and (self.prefill_kernel == "pair" or
                     (self.prefill_kernel == "auto" and
                      ops.gemm_tc2_pays(x.shape[0], self.out_features, x.device, fused_silu=True)))):
            return ops.gemm_tc2_bf16(x, w, x.dtype, silu_mul=True, gate_act=activation, bias=bias)
        if bias is not None:
            return ops.bias_gate_mul(self(x, out_dtype=torch.float32), bias, activation, x.dtype, interleave)
        y = self(x)
        if activation == "relu":
            return ops.relu_mul(y, interleave)
        return ops.gelu_tanh_mul(y, interleave) if activation == "gelu_tanh" else ops.silu_mul(y, interleave)

    def relu_squared(self, x: torch.Tensor) -> torch.Tensor:
        """max(x W^T, 0)^2.  Where the product's kernel has the epilogue (the tcgen05
        kernels), the square is taken on the 32-bit sums and rounded once; the pair
        product takes a prompt's rows under the rule of the fused gate|up product
        (``ops.gemm_tc2_pays``): fusing saves the same pass over the activations."""
        w = self.weight
        if w.dtype == torch.bfloat16 and x.dtype == torch.bfloat16 and self.in_features % 8 == 0:
            if x.shape[0] <= ops.SKINNY_MAX_ROWS:
                if self.decode_kernel == "tc":
                    return ops.gemm_tc_bf16(x, w, x.dtype, swap=True, relu_squared=True)
            elif self.prefill_kernel == "tc":
                return ops.gemm_tc_bf16(x, w, x.dtype, swap=False, relu_squared=True)
            elif ops.gemm_tc2_takes(self.out_features, x.dtype) and (
                    self.prefill_kernel == "pair" or
                    (self.prefill_kernel == "auto" and
                     ops.gemm_tc2_pays(x.shape[0], self.out_features, x.device, fused_silu=True))):
                return ops.gemm_tc2_bf16(x, w, x.dtype, relu_squared=True)
        return ops.relu_squared(self(x))
