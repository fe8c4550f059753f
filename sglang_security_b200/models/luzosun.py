"""Luzosun: decoder-only model of parallel blocks over a 32-bit residual stream,

    x = embed[token] * embedding_scale
    per layer:  x <- x + (mixer(c(norm1(x))) + ff(norm2(x)))     both norms of the same x,
                c(h) = h + causal convolution of h over time
    logits = head(norm_f(x))

The mixer is differential attention with short convolutions on its projections, rotated queries and keys and
chunked visibility; a layer may read the keys and values an earlier layer cached.  The feed-forward is an
ungated MLP with the xIELU activation, or absent.  Positions and angles, norms, convolutions and their state,
attention scores and sums and the residual are fp32; the matrix products run in the model dtype.  Built from
the shared layers ResidualNormConv, DifferentialAttention, UngatedMLP and JointOutput: per layer one launch
for residual sum + norms + convolution, one GEMM for q, k, v, one launch for convolution + rotation + cache
write, the attention, one GEMM with the activation in its epilogue, and one GEMM for both output matrices."""
from __future__ import annotations

import re
from typing import Iterable, Optional, Tuple

import torch
import torch.nn as nn

from ..configs.luzosun import LuzosunConfig, LuzosunLayerSpec
from ..layers.attention.differential_attention import DifferentialAttention
from ..layers.linear import ColumnParallelLinear
from ..layers.residual_conv import JointOutput, ResidualNormConv, UngatedMLP
from ..layers.residual_norm import ResidualRMSNorm
from ..layers.scalar_norm import residual_combine
from .registry import CacheSpec, register_model

_LAMBDA = ("lq1", "lk1", "lq2", "lk2")


class LuzosunLayer(nn.Module):
    def __init__(self, cfg: LuzosunConfig, spec: LuzosunLayerSpec, layer_id: int, params_dtype):
        super().__init__()
        self.layer_id, self.params_dtype = layer_id, params_dtype
        m, W = spec.mixer, cfg.width
        self.norms = ResidualNormConv(W, cfg.eps, cfg.canon_taps)
        self.mix = DifferentialAttention(W, m.heads, m.kv_heads, m.dim, m.vdim, m.scale, layer_id, cfg.eps, m.diff,
                                         chunk=m.chunk, rope_base=m.rope_base, rope_dims=m.rope_dims,
                                         rope_factor=m.rope_factor, conv_taps=m.conv, kv_source=m.kv_from,
                                         params_dtype=params_dtype)
        self.mlp = UngatedMLP(W, spec.mlp.ff, params_dtype) if spec.mlp else None
        self.out = JointOutput([self.mix.out_width] + ([spec.mlp.ff] if spec.mlp else []), W, params_dtype)

    @property
    def state_width(self) -> int:
        """Carry of a sequence: the last inputs of the block's convolution, then of the projections'."""
        return self.norms.state_width + self.mix.state_width

    def forward(self, x: torch.Tensor, x_out: torch.Tensor, a: Optional[torch.Tensor], fb) -> torch.Tensor:
        """x: fp32 residual before the previous block's output `a` is added; x_out receives the sum.
        -> this block's output, to be added by the next."""
        row = fb.state_pool.get(self.layer_id)
        cut = self.norms.state_width
        s_in = row[:, :cut] if row is not None and cut else None
        s_mix = row[:, cut:] if row is not None and self.mix.state_width else None
        h, n2 = self.norms(x, x_out, a, fb, s_in, self.params_dtype, second=self.mlp is not None)
        buf = self.out.buffer(x.shape[0], x.device)
        self.mix(h, fb, s_mix, self.out.view(buf, 0))
        if self.mlp is not None:
            self.mlp(n2, self.out.view(buf, 1))
        return self.out(buf)


@register_model("Luzosun")
class LuzosunForCausalLM(nn.Module):
    def __init__(self, config: LuzosunConfig, params_dtype: torch.dtype = torch.bfloat16):
        super().__init__()
        self.config, self.params_dtype = config, params_dtype
        self.embed = nn.Parameter(torch.empty(config.vocab, config.width, dtype=params_dtype), requires_grad=False)
        self.layers = nn.ModuleList(LuzosunLayer(config, s, i, params_dtype) for i, s in enumerate(config.layers))
        self.final_norm = ResidualRMSNorm(config.width, config.eps)
        self.head = ColumnParallelLinear(config.width, config.vocab, bias=False, params_dtype=params_dtype,
                                         tp_rank=0, tp_size=1)

    # ---- what the runner allocates -------------------------------------------------------------
    def cache_spec(self) -> CacheSpec:
        spec = CacheSpec(kind="rows")
        for i, layer in enumerate(self.layers):
            if layer.mix.kv_source is None:
                spec.row_dims[i] = layer.mix.row_width
            else:
                spec.source_of[i] = layer.mix.kv_source
            if layer.state_width:
                spec.state_widths[i] = layer.state_width
        return spec

    # ---- forward -------------------------------------------------------------------------------
    def forward(self, input_ids: torch.Tensor, forward_batch) -> torch.Tensor:
        x = self.embed[input_ids].float()
        if self.config.embedding_scale != 1.0:
            x.mul_(self.config.embedding_scale)
        spare = torch.empty_like(x)
        hook = forward_batch.extra.get("layer_hook") if forward_batch.extra else None
        a = None
        for layer in self.layers:
            a = layer(x, spare, a, forward_batch)
            x, spare = spare, x
            if hook is not None:
                hook(layer.layer_id, x + a.float())
        if a is not None:
            residual_combine(x, a=a)
        return x

    def compute_logits(self, hidden_rows: torch.Tensor) -> torch.Tensor:
        """-> fp32 [rows, vocab]: the product accumulates and is stored in fp32."""
        h = self.final_norm(hidden_rows.contiguous(), self.params_dtype)
        if h.dtype == torch.float32:
            return torch.mm(h, self.head.weight.t())
        return torch.mm(h, self.head.weight.t(), out_dtype=torch.float32)

    # ---- weights -------------------------------------------------------------------------------
    def load_weights(self, weights: Iterable[Tuple[str, torch.Tensor]]) -> None:
        seen = set()
        top = {"embed": lambda w: self.embed.data.copy_(w),
               "head": lambda w: self.head.weight_loader(self.head.weight, w),
               "final.norm": lambda w: self.final_norm.weight.data.copy_(w.float())}
        for name, w in weights:
            seen.add(name)
            if name in top:
                top[name](w)
                continue
            m = re.match(r"^l(\d+)\.(.+)$", name)
            if not m or int(m.group(1)) >= len(self.layers):
                raise ValueError(f"unexpected tensor {name!r}")
            self._load_layer_tensor(self.layers[int(m.group(1))], m.group(2), w)
        missing = self.expected_tensor_names() - seen
        if missing:
            raise ValueError(f"checkpoint lacks {len(missing)} tensors, e.g. {sorted(missing)[:4]}")
        for layer in self.layers:
            layer.mix.update_lambda()

    def _load_layer_tensor(self, layer: LuzosunLayer, key: str, w: torch.Tensor) -> None:
        mix, k = layer.mix, key[4:]
        parts = [n for n, size in mix.parts.items() if size]
        if key == "norm1":
            layer.norms.weight1.data.copy_(w.float())
        elif key == "norm2":
            layer.norms.weight2.data.copy_(w.float())
        elif key == "canon1" and layer.norms.taps:
            layer.norms.load_conv(w)
        elif key.startswith("mix."):
            if k == "o":
                layer.out.load_part(0, w)
            elif k in _LAMBDA:
                mix.load_lambda(_LAMBDA.index(k), w)
            elif k in parts:
                mix.load_part(k, w)
            elif k.endswith(".b") and k[:-2] in parts:
                mix.load_part(k[:-2], w, is_bias=True)
            elif k.endswith(".conv") and k[:-5] in parts and mix.taps:
                mix.load_conv(k[:-5], w)
            else:
                raise ValueError(f"unexpected tensor l{layer.layer_id}.{key}")
        elif key.startswith("mlp.") and layer.mlp is not None:
            if k == "up":
                layer.mlp.up_proj.weight_loader(layer.mlp.up_proj.weight, w)
            elif k == "down":
                layer.out.load_part(1, w)
            elif k == "act":
                p, q = w.float().cpu().reshape(-1).tolist()
                layer.mlp.load_act(p, q)
            else:
                raise ValueError(f"unexpected tensor l{layer.layer_id}.{key}")
        else:
            raise ValueError(f"unexpected tensor l{layer.layer_id}.{key}")

    def expected_tensor_names(self):
        names = {"embed", "head", "final.norm"}
        for i, layer in enumerate(self.layers):
            p, mix = f"l{i}.", layer.mix
            names.add(p + "norm1")
            if layer.norms.taps:
                names.add(p + "canon1")
            names |= {p + "mix." + k for k in ("o",) + _LAMBDA}
            for n, size in mix.parts.items():
                if size:
                    names |= {p + f"mix.{n}", p + f"mix.{n}.b"}
                    if mix.taps:
                        names.add(p + f"mix.{n}.conv")
            if layer.mlp is not None:
                names |= {p + "norm2", p + "mlp.up", p + "mlp.down", p + "mlp.act"}
        return names
