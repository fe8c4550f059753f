"""Parts of a parallel block x <- x + (mixer(c(norm1(x))) + ff(norm2(x))) over a 32-bit residual, where
c(h) = h + a short causal convolution of h over time:

  `ResidualNormConv`   one launch per block boundary: adds the previous block's output to the residual (into
                       a second buffer), norms it once for both readers, convolves the mixer's input with the
                       state row of each sequence (csrc/residual_conv.cu)
  `UngatedMLP`         act(W_up h) with the xIELU activation in the GEMM's epilogue; writes into a column
                       slice of the block's joint buffer
  `JointOutput`        W_o and W_down side by side as ONE matrix: both halves of the block meet in the fp32
                       accumulators of a single GEMM over the joint buffer [mixer heads | activations]"""
from __future__ import annotations

import math
from typing import Optional, Sequence, Tuple

import torch
import torch.nn as nn
import torch.nn.functional as F

from .. import _lib
from .dense_kernel import dense_supported, gemm_16bit
from .linear import ColumnParallelLinear, RowParallelLinear


def _ld(t: Optional[torch.Tensor]) -> int:
    return t.stride(0) if t is not None else 0


class ResidualNormConv(nn.Module):
    def __init__(self, width: int, eps: float, taps: int = 0):
        """taps: taps of the convolution, the current token's included (0: no convolution)."""
        super().__init__()
        f32 = dict(dtype=torch.float32)
        self.width, self.eps, self.taps = width, float(eps), int(taps)
        self.weight1 = nn.Parameter(torch.ones(width, **f32), requires_grad=False)
        self.weight2 = nn.Parameter(torch.ones(width, **f32), requires_grad=False)
        # [taps, width]: channels contiguous; the last row multiplies the current token
        self.conv_weight = nn.Parameter(torch.zeros(self.taps, width, **f32), requires_grad=False) if self.taps else None

    @property
    def state_width(self) -> int:
        return max(self.taps - 1, 0) * self.width

    def load_conv(self, w: torch.Tensor) -> None:
        """w [width, taps] as a checkpoint stores it."""
        self.conv_weight.data.copy_(w.float().t())

    def forward(self, x: torch.Tensor, x_out: torch.Tensor, a: Optional[torch.Tensor], fb,
                state: Optional[torch.Tensor], out_dtype: torch.dtype, second: bool = True
                ) -> Tuple[torch.Tensor, Optional[torch.Tensor]]:
        """x, x_out: fp32 [T, W], different buffers; x_out = x + a.  -> (c(norm1(x_out)), norm2(x_out))."""
        if not x.is_cuda:
            raise _lib.B200Error("ResidualNormConv: tensors must live on a CUDA device (no CPU path)")
        if x.dtype != torch.float32 or x_out.dtype != torch.float32 or x.stride(1) != 1 or x_out.stride(1) != 1:
            raise _lib.B200Error("ResidualNormConv: the residual must be fp32 with contiguous rows")
        if a is not None and (a.dtype != out_dtype or a.stride(1) != 1):
            raise _lib.B200Error("ResidualNormConv: the term must have the output dtype and contiguous rows")
        T, W = x.shape
        h = torch.empty((T, W), dtype=out_dtype, device=x.device)
        n2 = torch.empty((T, W), dtype=out_dtype, device=x.device) if second else None
        rc = _lib.load().b200_residual_norm_conv(
            x.data_ptr(), x.stride(0), _lib.ptr(a), _ld(a), None, 0, x_out.data_ptr(), x_out.stride(0),
            self.weight1.data_ptr(), self.weight2.data_ptr(), self.eps, _lib.ptr(self.conv_weight),
            max(self.taps, 1), _lib.ptr(state), _ld(state), fb.req_pool_indices.data_ptr(), fb.tok_pos.data_ptr(),
            fb.ext_start.data_ptr(), fb.ext_len.data_ptr(), h.data_ptr(), h.stride(0), _lib.ptr(n2), _ld(n2),
            int(fb.batch_size), max(fb.extend_seq_lens_cpu), W, _lib.dtype_code(out_dtype), _lib.current_stream())
        _lib.check(rc, "b200_residual_norm_conv")
        return h, n2


def _softplus(z: float) -> float:
    return z if z > 30.0 else math.log1p(math.exp(z))


class UngatedMLP(nn.Module):
    def __init__(self, width: int, ff: int, params_dtype: torch.dtype = torch.bfloat16):
        super().__init__()
        self.ff = ff
        self.up_proj = ColumnParallelLinear(width, ff, bias=False, params_dtype=params_dtype, tp_rank=0, tp_size=1)
        self.pos, self.neg = _softplus(0.0), 0.5 + _softplus(0.0)

    def load_act(self, p: float, q: float) -> None:
        """xIELU's two learned numbers: curvature softplus(p) above zero, 1/2 + softplus(q) below."""
        self.pos, self.neg = _softplus(p), 0.5 + _softplus(q)

    def forward(self, h: torch.Tensor, out: torch.Tensor) -> None:
        """xielu(W_up h) into `out` [T, ff], which may be a column slice."""
        w = self.up_proj.weight
        if dense_supported(h, w) and out.stride(0) % 8 == 0 and out.data_ptr() % 16 == 0:
            gemm_16bit(h, w, out=out, xielu=(self.pos, self.neg))
            return
        z = F.linear(h, w)
        rc = _lib.load().b200_xielu_rows(z.data_ptr(), z.stride(0), out.data_ptr(), out.stride(0), z.shape[0],
                                         z.shape[1], self.pos, self.neg, _lib.dtype_code(z.dtype),
                                         _lib.current_stream())
        _lib.check(rc, "b200_xielu_rows")


class JointOutput(nn.Module):
    """Parts of the input are padded to multiples of 8 columns (16-byte rows for the GEMM); the padding's
    weights and activations are zero."""

    def __init__(self, parts: Sequence[int], width: int, params_dtype: torch.dtype = torch.bfloat16):
        super().__init__()
        self.parts = [int(n) for n in parts]
        self.offsets, at = [], 0
        for n in self.parts:
            self.offsets.append(at)
            at += (n + 7) // 8 * 8
        self.columns, self.params_dtype = at, params_dtype
        self.proj = RowParallelLinear(at, width, bias=False, params_dtype=params_dtype, tp_rank=0, tp_size=1)
        self.padded = at != sum(self.parts)
        if self.padded:
            self.proj.weight.data.zero_()

    def load_part(self, i: int, w: torch.Tensor) -> None:
        if w.shape[1] != self.parts[i]:
            raise ValueError(f"output projection of {w.shape[1]} inputs for {self.parts[i]}")
        self.proj.weight.data[:, self.offsets[i]:self.offsets[i] + self.parts[i]].copy_(w)

    def buffer(self, tokens: int, device) -> torch.Tensor:
        make = torch.zeros if self.padded else torch.empty
        return make((tokens, self.columns), dtype=self.params_dtype, device=device)

    def view(self, buf: torch.Tensor, i: int) -> torch.Tensor:
        return buf[:, self.offsets[i]:self.offsets[i] + self.parts[i]]

    def forward(self, buf: torch.Tensor) -> torch.Tensor:
        out, _ = self.proj(buf)
        return out
