"""A projection ``y = x · Wᵀ`` over one weight matrix ``[out, in]``, possibly several checkpoint matrices
stacked along ``out`` (the reference's ``Linear``, csrc/model/layers/linear.cpp:35-95, stacks q/k/v and
gate/up the same way and has no bias).

Which kernel multiplies is decided here, per call, from the engine dtype and the shape:

* float32: the FMA kernel (``gemm_generic``), true 32-bit, any shape;
* bfloat16: the tensor-core kernels of this package where they take the shape; otherwise the library
  product (cuBLAS through ``torch.mm``), which is what the reference uses for every projection
  (csrc/ops/projection.cu:32-44); shapes that are not a multiple of 8 go to ``gemm_generic``.
"""
from __future__ import annotations

from typing import List, Optional, Sequence

import torch

from .. import kernels
from .base import LazyNorm
from .spec import TensorSpec


def matmul_nt(x: torch.Tensor, weight: torch.Tensor, out_dtype: Optional[torch.dtype] = None) -> torch.Tensor:
    """``x[M, K] @ weight[N, K]^T`` → ``[M, N]`` in ``out_dtype`` (default: x's dtype)."""
    M, K = x.shape
    N = weight.shape[0]
    out_dtype = out_dtype or x.dtype
    out = torch.empty((M, N), dtype=out_dtype, device=x.device)
    if M == 0:
        return out
    if x.dtype == torch.float32:
        kernels.gemm_generic(x, weight, out)
        return out
    from . import gemm_dispatch
    gemm_dispatch.bf16_matmul_nt(x, weight, out)
    return out


def per_head_products(a: torch.Tensor, w: torch.Tensor, out: torch.Tensor) -> None:
    """``out[h] = a[h] @ w[h]^T`` for every head h, or for every one of several products of one size; ``a [H, T, K]`` and
    ``out [H, T, N]`` may be views of rows in which the heads lie side by side, ``w [H, N, K]`` is dense.  bfloat16 with
    sizes in multiples of 8: the library's strided batched product (as for the plain projections); else the FMA kernel,
    which is also the 32-bit path."""
    from . import gemm_dispatch  # noqa: F401  (sets the library products to 32-bit accumulation before the first one runs)
    H, T, K = a.shape
    N = w.shape[1]
    if (a.dtype == torch.bfloat16 and out.dtype == torch.bfloat16 and K % 8 == 0 and N % 8 == 0
            and a.stride(1) % 8 == 0 and a.stride(0) % 8 == 0 and out.stride(1) % 8 == 0 and out.stride(0) % 8 == 0 and T > 0):
        torch.bmm(a, w.transpose(1, 2), out=out)
        kernels.launch_count += 1
        return
    kernels.gemm_generic_batched(a, w, out)


def padded_rows(weight: torch.Tensor, multiple: int = 8) -> torch.Tensor:
    """``weight`` with rows of zeros up to a multiple of ``multiple``: the product then takes the tensor-core and library
    paths that other projections take (nothing reads the columns that the extra rows produce)."""
    rows = weight.shape[0]
    if rows % multiple == 0:
        return weight
    pad = torch.zeros((multiple - rows % multiple, weight.shape[1]), dtype=weight.dtype, device=weight.device)
    return torch.cat([weight, pad]).contiguous()


def dense_operand(x: torch.Tensor) -> torch.Tensor:
    """``x`` (a column range of wider rows) as a product's kernels take it: as it is when its rows start on 16-byte
    boundaries (or in 32 bits), else a copy."""
    if x.dtype == torch.bfloat16 and (x.stride(0) % 8 or x.data_ptr() % 16):
        return x.contiguous()
    return x


class Linear:
    """``pad``: the loaded weight gets rows of zeros up to a multiple of eight (see ``padded_rows``; the output then has as
    many more columns).  ``free_out``: places in ``names`` whose number of rows the checkpoint decides, ``free_in``: the
    width is (see ``TensorSpec.free_axes``); ``out_features`` and ``in_features`` hold the real sizes once loaded."""

    def __init__(self, names: Sequence[str], out_features: Sequence[int], in_features: int, dtype: torch.dtype, *,
                 pad: bool = False, free_out: Sequence[int] = (), free_in: bool = False) -> None:
        if len(names) != len(out_features):
            raise ValueError("one out_features per name")
        self.names = list(names)
        self.out_features = list(out_features)
        self.in_features = in_features
        self.dtype = dtype
        self.pad = pad
        self.free_out = tuple(free_out)
        self.free_in = free_in
        self.weight: Optional[torch.Tensor] = None
        self.warm_next: Optional[torch.Tensor] = None     # what the step reads right after this projection (a hint for the L2)

    def tensors(self) -> List[TensorSpec]:
        return [TensorSpec(n, (o, self.in_features), free_axes=((0,) if i in self.free_out else ()) + ((1,) if self.free_in else ()))
                for i, (n, o) in enumerate(zip(self.names, self.out_features))]

    def load(self, store) -> None:
        specs = self.tensors()
        if self.free_out:
            parts = [store.get(s) for s in specs]
            self.out_features = [p.shape[0] for p in parts]
            self.weight = torch.cat(parts).contiguous()
        else:
            self.weight = store.get(specs[0]) if len(specs) == 1 else store.get_stacked(specs)
        self.in_features = self.weight.shape[1]
        if self.weight.dtype != self.dtype:
            self.weight = self.weight.to(self.dtype)
        if self.pad:
            self.weight = padded_rows(self.weight)

    def workspace_bytes(self, tokens: int, silu_pair: bool = False) -> int:
        """Bytes of the projection's output for ``tokens`` rows (with ``silu_pair`` the stacked product may exist
        beside the gated one)."""
        width = 2 if self.dtype == torch.bfloat16 else 4
        n = sum(self.out_features)
        return tokens * (n + n // 2 if silu_pair else n) * width

    def tie(self, weight: torch.Tensor) -> None:
        """Use another tensor's storage as this projection's weight (a tied output head)."""
        if tuple(weight.shape) != (sum(self.out_features), self.in_features):
            raise ValueError(f"tied weight has shape {list(weight.shape)}")
        self.weight = weight

    def forward(self, x, out_dtype: Optional[torch.dtype] = None, silu_pair: bool = False) -> torch.Tensor:
        """``x`` is a tensor [M, K] or a :class:`LazyNorm`.  ``silu_pair``: the weight is gates then ups and the
        result is ``silu(gate) * up`` [M, N/2]; the value ``"gelu_tanh"`` makes the gate the tanh form of GELU."""
        if self.weight is None:
            raise RuntimeError(f"projection {self.names} used before its weights were loaded")
        fused = self._forward_skinny(x, out_dtype, silu_pair)
        if fused is not None:
            return fused
        if isinstance(x, LazyNorm):
            x = x.materialize()
        if silu_pair and x.dtype == torch.bfloat16 and x.shape[0] > 0:
            from . import gemm_dispatch
            gated = gemm_dispatch.bf16_gated_matmul_nt(x, self.weight, silu_pair)
            if gated is not None:
                return gated
        y = matmul_nt(x, self.weight, out_dtype if not silu_pair else None)
        if not silu_pair:
            return y
        act = torch.empty((y.shape[0], y.shape[1] // 2), dtype=y.dtype, device=y.device)
        kernels.silu_mul(y, act, gelu=silu_pair == "gelu_tanh")
        return act

    def _forward_skinny(self, x, out_dtype, silu_pair) -> Optional[torch.Tensor]:
        """The few-rows kernel with the norm in its prologue and/or the gate in its epilogue, when it takes
        the shape; None otherwise."""
        w = self.weight
        if w.dtype != torch.bfloat16 or not w.is_contiguous():
            return None
        lazy = isinstance(x, LazyNorm)
        M = x.shape[0]
        N, K = w.shape
        if M == 0 or M > 16:
            return None
        out_dtype = out_dtype or torch.bfloat16
        if silu_pair and out_dtype != torch.bfloat16:
            return None
        out_cols = N // 2 if silu_pair else N
        from . import gemm_dispatch
        choice = gemm_dispatch.few_rows_kernel(M, N, K)
        if choice == "library":
            return None           # the library product (and the activation kernel after it) in forward()
        if choice == "wstream":
            # long K: the weight-streaming kernel (no norm prologue; the gate is in its epilogue)
            rows = x.materialize() if lazy else x
            if (silu_pair is not True or rows.dtype != torch.bfloat16 or rows.stride(1) != 1 or rows.stride(0) % 8 or w.stride(0) % 8
                    or not kernels.gemm_wstream_supports(M, N, K)):
                return None
            out = torch.empty((M, out_cols), dtype=torch.bfloat16, device=w.device)
            kernels.gemm_wstream(rows, w, out, silu_pair=True)
            return out
        if lazy and x._rows is None:
            stream = x.stream
            rms = x.norm.fusable_rms()
            if (rms is not None and stream.plain and stream.residual.is_contiguous()
                    and K <= gemm_dispatch.FUSED_NORM_MAX_K and kernels.gemm_skinny_supports(M, N, K, True)
                    and (stream.pending is None or stream.pending.is_contiguous())):
                out = torch.empty((M, out_cols), dtype=out_dtype, device=w.device)
                has_delta = stream.pending is not None
                kernels.gemm_skinny(w, out, residual=stream.residual, pending=stream.pending, norm_weight=rms[0],
                                    eps=rms[1], residual_out=stream.spare() if has_delta else None, silu_pair=silu_pair,
                                    warm=self.warm_next)
                if has_delta:
                    stream.swap()
                return out
        rows = x.materialize() if lazy else x
        if rows.dtype != torch.bfloat16 or rows.stride(1) != 1 or not kernels.gemm_skinny_supports(M, N, K, False):
            return None
        out = torch.empty((M, out_cols), dtype=out_dtype, device=w.device)
        kernels.gemm_skinny(w, out, act=rows, silu_pair=silu_pair, warm=self.warm_next)
        return out
