"""Differential attention (Ye et al., "Differential Transformer") over a token pool whose row holds
[keys of both maps | values] of all key/value heads.  Per token at position i with mixer input h:

    [q ; k ; v] = W h + b                          one fused GEMM; q: H heads x 2 maps x D, k: G x 2 x D, v: G x E
    q, k, v     = causal convolution per channel   (optional; the last taps-1 projections are sequence state)
    q, k        = rotated by position / factor on the first `rope_dims` coordinates of every map (half pairing)
    a_m(i)      = sum_j softmax_j(scale q_m(i) . k_m(j)) v(j)          both maps over the same values
    d           = a_1 - lam a_2;   out = d / rms(d) * (1 - diff)       per head, over the E coordinates
    lam         = exp(lq1 . lk1) - exp(lq2 . lk2) + diff               one number

i sees j <= i in its own chunk of `chunk` positions, a sliding `window`, or all before.  With `kv_source`
the layer has queries only and reads the pool rows that another layer wrote.

Three kernels share the definition (csrc/diff_attn.cu, csrc/diff_attn_extend.cu), both maps, the
difference and the norm inside each: prompt portions of at least `tensor_core_min_tokens` tokens take the
tcgen05 kernel when the step brings `tensor_core_min_total` tokens of them, decoded tokens and short portions
the split-key mma.sync kernel (both: 16-bit engine, sizes of `b200_diff_attn_mma_supported`), everything else
the CUDA-core kernel with fp32 queries.  All read the pool only, so a position's result does not depend on
how the prompt was cut or batched beyond rounding."""
from __future__ import annotations

from typing import Optional

import torch
import torch.nn as nn

from ... import _lib
from ..linear import ColumnParallelLinear
from .sink_attention import SinkAttention

_SMS = {}


def _sm_count(device) -> int:
    key = device.index or 0
    if key not in _SMS:
        _SMS[key] = torch.cuda.get_device_properties(device).multi_processor_count
    return _SMS[key]


class DifferentialAttention(nn.Module):
    # prompt portions of at least this many tokens go to the tcgen05 kernel (0 = never) when a step brings
    # `tensor_core_min_total` tokens in such portions: the split-key kernel reads the keys once per TOKEN, the
    # tcgen05 kernel costs about as much for one tile of rows as for many.  Tests lower the total
    tensor_core_min_tokens = 16
    tensor_core_min_total = 96
    use_mma = True               # the 16-bit kernel for the other tokens

    def __init__(self, width: int, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, layer_id: int,
                 eps: float, diff: float, chunk: Optional[int] = None, window: Optional[int] = None,
                 rope_base: float = 10000.0, rope_dims: int = 0, rope_factor: float = 1.0, conv_taps: int = 0,
                 kv_source: Optional[int] = None, bias: bool = True, params_dtype: torch.dtype = torch.bfloat16):
        super().__init__()
        if heads % kv_heads:
            raise ValueError("query heads must be a multiple of key/value heads")
        if chunk and window:
            raise ValueError("a layer sees chunks or a sliding window, not both")
        self.width, self.heads, self.kv_heads, self.dim, self.vdim = width, heads, kv_heads, dim, vdim
        self.scale, self.layer_id, self.eps, self.diff = float(scale), layer_id, float(eps), float(diff)
        self.chunk, self.window = int(chunk or 0), int(window or 0)
        self.rope_dims, self.taps, self.kv_source = int(rope_dims), int(conv_taps), kv_source
        self.params_dtype = params_dtype
        own = kv_source is None
        self.parts = {"q": heads * 2 * dim, "k": kv_heads * 2 * dim if own else 0, "v": kv_heads * vdim if own else 0}
        self.channels = sum(self.parts.values())
        self.in_proj = ColumnParallelLinear(width, self.channels, bias=bias, params_dtype=params_dtype, tp_rank=0,
                                            tp_size=1)
        f32 = dict(dtype=torch.float32)
        # [taps, channels]: channels contiguous; the last row multiplies the current token
        self.conv_weight = nn.Parameter(torch.zeros(self.taps, self.channels, **f32), requires_grad=False) if self.taps else None
        self.lambda_parts = nn.Parameter(torch.zeros(4, dim, **f32), requires_grad=False)     # lq1, lk1, lq2, lk2
        self.register_buffer("lam", torch.full((1,), self.diff, **f32), persistent=False)
        # frequencies in fp64, kept as a sum of two fp32 tables: position * frequency stays exact far out
        f = torch.tensor([float(rope_base) ** (-2.0 * i / self.rope_dims) / float(rope_factor)
                          for i in range(self.rope_dims // 2)], dtype=torch.float64)
        hi = f.to(torch.float32)
        self.register_buffer("freq_hi", hi, persistent=False)
        self.register_buffer("freq_lo", (f - hi.double()).to(torch.float32), persistent=False)

    # ---- sizes ---------------------------------------------------------------------------------------
    @property
    def row_width(self) -> int:
        """Pool row of one token: both key maps of all key/value heads, then their values."""
        return self.kv_heads * (2 * self.dim + self.vdim)

    @property
    def state_width(self) -> int:
        return max(self.taps - 1, 0) * self.channels

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    # ---- weights -------------------------------------------------------------------------------------
    def _offset(self, which: str) -> int:
        names = list(self.parts)
        return sum(self.parts[n] for n in names[:names.index(which)])

    def load_part(self, which: str, w: torch.Tensor, is_bias: bool = False) -> None:
        lo, n = self._offset(which), self.parts[which]
        if w.shape[0] != n:
            raise ValueError(f"projection {which!r}: {w.shape[0]} rows for {n}")
        (self.in_proj.bias if is_bias else self.in_proj.weight).data[lo:lo + n].copy_(w)

    def load_conv(self, which: str, w: torch.Tensor) -> None:
        """w [channels of the part, taps] as a checkpoint stores it."""
        lo, n = self._offset(which), self.parts[which]
        self.conv_weight.data[:, lo:lo + n].copy_(w.float().t())

    def load_lambda(self, i: int, w: torch.Tensor) -> None:
        self.lambda_parts.data[i].copy_(w.float())

    def update_lambda(self) -> None:
        """The second map's weight, once per load (fp64, stored fp32)."""
        p = self.lambda_parts.data.double()
        self.lam.copy_((torch.exp((p[0] * p[1]).sum()) - torch.exp((p[2] * p[3]).sum()) + self.diff).float().reshape(1))

    # ---- forward -------------------------------------------------------------------------------------
    def _mma_ok(self, h: torch.Tensor, pool: torch.Tensor) -> bool:
        return (self.use_mma and h.dtype in (torch.bfloat16, torch.float16) and self.row_width % 8 == 0
                and self.scale > 0 and pool.stride(0) % 8 == 0
                and bool(_lib.load().b200_diff_attn_mma_supported(self.dim, self.vdim)))

    def forward(self, h: torch.Tensor, fb, state: Optional[torch.Tensor], out: torch.Tensor) -> None:
        """out: [T, heads * vdim] (may be a column slice), receives the heads before the output projection."""
        if not h.is_cuda:
            raise _lib.B200Error("DifferentialAttention: tensors must live on a CUDA device (no CPU path)")
        T, dev = h.shape[0], h.device
        H, G, D, E = self.heads, self.kv_heads, self.dim, self.vdim
        pool = fb.token_to_kv_pool.get_kv_buffer(self.layer_id)
        if pool.dtype != h.dtype or pool.shape[1] != self.row_width:
            raise _lib.B200Error("DifferentialAttention: the token pool does not fit this layer")
        y, _ = self.in_proj(h)
        lib, st, code = _lib.load(), _lib.current_stream(), _lib.dtype_code(h.dtype)
        mma = self._mma_ok(h, pool)
        plan = None
        if mma and self.tensor_core_min_tokens > 0 and out.stride(0) % 8 == 0 and out.data_ptr() % 16 == 0:
            if sum(n for n in fb.extend_seq_lens_cpu if n >= self.tensor_core_min_tokens) >= self.tensor_core_min_total:
                plan = SinkAttention._plan(fb, self.tensor_core_min_tokens)
        q16 = torch.empty((T, H * 2 * D), dtype=h.dtype, device=dev) if mma else None
        q32 = None if mma else torch.empty((T, H * 2 * D), dtype=torch.float32, device=dev)
        own = self.kv_source is None
        k_off, v_off = 0, G * 2 * D
        rc = lib.b200_conv_rot_write(
            y.data_ptr(), y.stride(0), _lib.ptr(self.conv_weight), max(self.taps, 1), _lib.ptr(state),
            state.stride(0) if state is not None else 0, fb.req_pool_indices.data_ptr(), fb.tok_pos.data_ptr(),
            fb.ext_start.data_ptr(), fb.ext_len.data_ptr(), self.freq_hi.data_ptr(), self.freq_lo.data_ptr(),
            self.rope_dims, fb.out_cache_loc.data_ptr(), pool.data_ptr(), pool.stride(0), k_off, v_off,
            _lib.ptr(q32), H * 2 * D, _lib.ptr(q16), H * 2 * D, 2 * H, 2 * G if own else 0, D,
            G * E if own else 0, int(fb.batch_size), max(fb.extend_seq_lens_cpu), code, st)
        _lib.check(rc, "b200_conv_rot_write")
        r2t, mult = fb.req_to_token_pool.req_to_token, 1.0 - self.diff
        rows = T if plan is None else plan["n_rest"]
        if plan is not None:
            rc = lib.b200_diff_attn_extend(
                q16.data_ptr(), q16.stride(0), pool.data_ptr(), pool.stride(0), k_off, v_off, out.data_ptr(),
                out.stride(0), r2t.data_ptr(), r2t.stride(0), plan["req"].data_ptr(), plan["prefix"].data_ptr(),
                plan["ext"].data_ptr(), plan["start"].data_ptr(), plan["bs"], plan["max_ext"], H, G, D, E,
                self.scale, self.window, self.chunk, self.lam.data_ptr(), mult, self.eps, code, st)
            _lib.check(rc, "b200_diff_attn_extend")
        if not rows:
            return
        some = _lib.ptr(plan["rest"]) if plan is not None else None
        limit = self.chunk or self.window
        max_keys = min(fb.max_seq_len, limit) if limit else fb.max_seq_len
        if mma:
            ns = int(lib.b200_diff_attn_mma_splits(rows, H, G, max_keys, _sm_count(dev)))
            part = torch.empty((rows * H * 2 * ns, E + 1), dtype=torch.float32, device=dev) if ns > 1 else None
            po = part.data_ptr() if part is not None else None
            rc = lib.b200_diff_attn_mma(
                q16.data_ptr(), q16.stride(0), pool.data_ptr(), pool.stride(0), k_off, v_off, r2t.data_ptr(),
                r2t.stride(0), fb.req_pool_indices.data_ptr(), fb.tok_pos.data_ptr(), fb.tok_b.data_ptr(), some,
                self.lam.data_ptr(), mult, self.eps, self.scale, self.window, self.chunk, out.data_ptr(),
                out.stride(0), rows, H, G, D, E, ns, po, po + rows * H * 2 * ns * E * 4 if po else None, code, st)
            _lib.check(rc, "b200_diff_attn_mma")
        else:
            rc = lib.b200_diff_attn(
                q32.data_ptr(), q32.stride(0), pool.data_ptr(), pool.stride(0), k_off, v_off, r2t.data_ptr(),
                r2t.stride(0), fb.req_pool_indices.data_ptr(), fb.tok_pos.data_ptr(), fb.tok_b.data_ptr(), some,
                self.lam.data_ptr(), mult, self.eps, self.scale, self.window, self.chunk, out.data_ptr(),
                out.stride(0), rows, H, G, D, E, max_keys, code, st)
            _lib.check(rc, "b200_diff_attn")
