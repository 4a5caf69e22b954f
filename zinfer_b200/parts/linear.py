"""The one place that picks a contraction kernel: out (+)= a @ w.T (+ bias).

The reference has one matmul driver for every weight matrix, with an `accumulate` flag that
folds the residual add into the store (src/model.zig:903-1026, 918-920).  Here the float32 path
always takes the CUDA-core FMA kernel (true 32-bit); the bfloat16 path takes a tensor-core
kernel when the shape allows one and the same FMA kernel otherwise.

`a` may be a `NormedRows`: rows of the residual stream whose RMSNorm is still to be applied.
A kernel that can normalise its input itself takes it as it is; for any other kernel the norm
runs first, once, however many contractions read it.

`out` may be a `ResidualSink`: the residual rows together with the norm that reads them next.
A kernel that can then writes, beside the sum, what that norm needs (the rows times the norm's
weight in bfloat16 and partial sums of their squares), and the contraction behind the norm
scales its own sums by the rows' 1/rms: the norm costs neither a launch nor a pass over the rows.
"""
from __future__ import annotations

from typing import Optional, Union

import torch

from .. import kernels


class NormedRows:
    """RMSNorm(x) * weight that is computed when somebody needs it as a tensor."""

    def __init__(self, x: torch.Tensor, weight: torch.Tensor, eps: float, dtype: torch.dtype,
                 scaled: Optional["kernels.NormEmit"] = None):
        self.x, self.weight, self.eps, self.dtype = x, weight, eps, dtype
        self.scaled = scaled          # what the kernel that summed x wrote for this norm, if it did
        self._tensor: Optional[torch.Tensor] = None

    @property
    def shape(self):
        return self.x.shape

    def tensor(self) -> torch.Tensor:
        if self._tensor is None:
            self._tensor = kernels.rmsnorm(self.x, self.weight, self.eps, self.dtype)
        return self._tensor

    def kernel_input(self) -> "kernels.NormInput":
        return kernels.NormInput(self.x, self.weight, self.eps)


class ResidualSink:
    """The float32 residual rows as the target of an accumulating contraction (`linear(...,
    out=sink, accumulate=True)`), with the weight of the RMSNorm that reads them next.  `emit`
    is set once a kernel has written that norm's inputs beside the sum; it stays None when the
    kernel that ran cannot, and the norm then works from the rows as ever."""

    def __init__(self, rows: torch.Tensor, norm_weight: torch.Tensor):
        self.rows, self.norm_weight = rows, norm_weight
        self.emit: Optional["kernels.NormEmit"] = None


class ScaledSink:
    """The float32 residual rows as the target of an accumulating contraction whose result is first multiplied
    by a learned number per column (a layer scale): rows[:, n] += scale[n] * (a @ w.T)[:, n].  A kernel that can
    applies the scale in its epilogue; otherwise the product goes to a buffer and `kernels.scale_add` sums it in."""

    def __init__(self, rows: torch.Tensor, scale: torch.Tensor):
        self.rows, self.scale = rows, scale


FUSION_GROUP = 16     # rows per part and group in the interleaved weight layouts of the fused kernels


def interleave_rows(parts, group: int = FUSION_GROUP) -> torch.Tensor:
    """Rows of equally shaped matrices (or vectors) regrouped as `group` rows of the first, the
    same `group` rows of the second, ...: a block of a fused kernel then finds all parts of its
    outputs in adjacent rows.  The row count must be a multiple of `group`."""
    n = parts[0].shape[0]
    if n % group or any(p.shape != parts[0].shape for p in parts):
        raise ValueError(f"cannot interleave {[tuple(p.shape) for p in parts]} in groups of {group}")
    stacked = torch.stack([p.reshape(n // group, group, *p.shape[1:]) for p in parts], dim=1)
    return stacked.reshape(len(parts) * n, *parts[0].shape[1:]).contiguous()


TILE_ROWS = 256       # weight rows of a tile of the persistent contractions


def pad_rows(w: torch.Tensor) -> torch.Tensor:
    """A bfloat16 matrix (or a vector per row) of at least two tiles of rows, given zero rows up to a whole number of tiles, which is what
    the persistent contractions of prompt steps take; the result then has that many more columns, all zero.  Smaller ones, and
    float32 matrices, are left as they are."""
    n = w.shape[0]
    if w.dtype != torch.bfloat16 or n < 2 * TILE_ROWS or n % TILE_ROWS == 0:
        return w
    return torch.cat([w, w.new_zeros((-n % TILE_ROWS, *w.shape[1:]))], dim=0).contiguous()


def as_tensor(a: Union[torch.Tensor, NormedRows]) -> torch.Tensor:
    return a.tensor() if isinstance(a, NormedRows) else a


def scaled_or_tensor(a: Union[torch.Tensor, NormedRows]):
    """For a kernel that takes a `kernels.ScaledInput`: that, if the rows came prepared and nobody
    has asked for the normalised tensor yet; else the tensor."""
    if isinstance(a, NormedRows) and a.scaled is not None and a._tensor is None and a.dtype == torch.bfloat16:
        return kernels.ScaledInput(a.scaled.xw, a.scaled.ssq, a.eps)
    return as_tensor(a)


# A block that applies the norm itself reads all M rows again, so fusing the norm pays only while
# few blocks do so (about one per SM) or the rows are very few; measured on the LFM2-1.2B shapes:
# fused 12.5 us against 14.5 us for the short convolution's in_proj (128 blocks, 8 rows), but
# 75 us against 50 us for the head (2048 blocks).  A whole step with every norm fused against the
# rule below: 0.673 against 0.680 ms at 4 rows, 0.723 against 0.714 ms at 8 rows.
NORM_FUSION_MAX_BLOCKS = 160
NORM_FUSION_ANY_BLOCKS_ROWS = 4


def fused_input(a: Union[torch.Tensor, NormedRows], w: torch.Tensor, need_fused_rows: bool = False,
                blocks: Optional[int] = None):
    """What a skinny kernel should be given for `a`, or None if it does not take it: the pending
    norm itself when the kernel can apply it and that is the faster way (`blocks` = thread blocks
    the kernel will run, default one per 16 weight rows), else the (materialised) bfloat16 tensor."""
    takes = kernels.gemm_skinny_fused_takes if need_fused_rows else kernels.gemm_skinny_takes
    if isinstance(a, NormedRows):
        if a.dtype != torch.bfloat16:
            return None
        if a._tensor is None:
            if a.scaled is not None:
                si = kernels.ScaledInput(a.scaled.xw, a.scaled.ssq, a.eps)
                if takes(si, w):
                    return si
            ki = a.kernel_input()
            n_blocks = blocks if blocks is not None else -(-w.shape[0] // 16)
            worth = n_blocks <= NORM_FUSION_MAX_BLOCKS or a.shape[0] <= NORM_FUSION_ANY_BLOCKS_ROWS
            if worth and takes(ki, w):
                return ki
            max_rows = kernels.gemm_skinny_fused_max_m() if need_fused_rows else kernels.gemm_skinny_max_m()
            if a.shape[0] > max_rows:
                return None             # too many rows for these kernels: the norm stays pending for another
        a = a.tensor()
    return a if takes(a, w) else None


def linear(a: Union[torch.Tensor, NormedRows], w: torch.Tensor,
           out: Union[torch.Tensor, ResidualSink, "ScaledSink", None] = None, out_dtype=None,
           accumulate: bool = False, bias: Optional[torch.Tensor] = None, act: Optional[str] = None) -> torch.Tensor:
    """a [M, K] and w [N, K] in the run dtype; result [M, N] in `out_dtype` (default: run dtype),
    or added into `out` when `accumulate`.  `act` names an activation (`kernels.ACTIVATIONS`) applied to the
    result; `out` may be a `ScaledSink`: the result is multiplied by its scale per column and added to its
    rows.  Both run in the contraction's epilogue where the kernel has one, else as kernels of their own."""
    if isinstance(out, ScaledSink) or act is not None:
        return _linear_with_epilogue(a, w, out, out_dtype, accumulate, bias, act)
    sink = None
    if isinstance(out, ResidualSink):
        sink, out = out, out.rows
    if w.dtype == torch.bfloat16:
        from . import linear_bf16
        y = linear_bf16.try_linear(a, w, out, out_dtype, accumulate, bias, sink)
        if y is not None:
            return y
    return kernels.gemm_simt(as_tensor(a), w, out=out, out_dtype=out_dtype, accumulate=accumulate, bias=bias)


FUSED_EPILOGUE_MAX_ROWS = 16      # above, the tcgen05 contractions are the faster ones and the epilogue runs as a kernel


def _linear_with_epilogue(a, w, out, out_dtype, accumulate, bias, act):
    scale = None
    if isinstance(out, ScaledSink):
        if not accumulate:
            raise ValueError("a scaled sink is summed into: accumulate must be set")
        scale, out = out.scale, out.rows
    if isinstance(out, ResidualSink):
        out = out.rows
    if w.dtype == torch.bfloat16 and (act is None or act == "relu_squared") and a.shape[0] <= FUSED_EPILOGUE_MAX_ROWS:
        x = fused_input(a, w)
        if x is not None:                # few rows: activation and scale in the weight-streaming kernel's epilogue
            return kernels.gemm_skinny(x, w, out=out, out_dtype=out_dtype, accumulate=accumulate, bias=bias,
                                       col_scale=scale, act=act)
    if w.dtype == torch.bfloat16 and (act is None or act == "relu_squared") and a.shape[0] > kernels.GEMM_TC_SWAPPED_MAX_M:
        t = as_tensor(a)
        if kernels.gemm_tc_fuses(t, w, out, accumulate, out_dtype):   # many rows: the persistent tcgen05 forms' epilogue
            return kernels.gemm_tc(t, w, out=out, out_dtype=out_dtype, accumulate=accumulate, bias=bias, col_scale=scale,
                                   act=act)
    if scale is None:
        if accumulate:
            raise ValueError("an activated product is not summed into rows without a scale")
        y = linear(a, w, out=out, out_dtype=out_dtype, bias=bias)
        return kernels.activation(y, act, out=y)
    y = linear(a, w, out_dtype=torch.float32, bias=bias)
    if act is not None:
        kernels.activation(y, act, out=y)
    return kernels.scale_add(y, scale, out)
