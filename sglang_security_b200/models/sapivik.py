"""Sapivik: decoder-only model over a 32-bit residual stream with an RMS norm on both sides of every sublayer,
in which a range of layers is repeated, each pass with the weights of the first:

    x = embed[token]
    per layer run:  x += m * post_1(mixer(pre_1(x)))
                    x += m * post_2(ff(pre_2(x)))              (layers with a feed-forward)
    ahead of every pass of the loop but the first:  x += embed[token]
    logits = head(norm_f(x))

A layer's mixer is a matrix memory gated channel by channel ("hgrn2") or grouped-query
attention whose values are the projected keys, with unit-norm rotated queries and keys, capped scores and an
element-wise output gate ("attention").  The feed-forward is a clamped gated MLP or a mixture of silu-gated
experts, some of which return their input, with a gated shared expert.  Norms, gates and memories, angles,
attention scores and weights, routers and the residual are fp32; the matrix products run in the model dtype.
Built from the shared layers AddNormed / ResidualRMSNorm, ChannelForgetMixer, SinkAttention, GatedMLP,
GroupedSoftmaxRouter / FusedExperts.

A layer run (pass) has its own pool rows or state, named by its place in the order of runs.  ONE launch per
sublayer boundary sums the sublayer's terms (expert rows with their weights, identity experts, the gated shared
expert), norms the sum, adds it to the residual, adds the embedding row where a pass begins, and emits the next
sublayer's pre-norm."""
from __future__ import annotations

import re
from typing import Iterable, Optional, Tuple

import torch
import torch.nn as nn

from ..configs.sapivik import ClampedSpec, IdentityExpertsSpec, SapivikConfig, SapivikLayerSpec
from ..layers.attention.sink_attention import SinkAttention
from ..layers.gated_mlp import GatedMLP
from ..layers.linear import ColumnParallelLinear
from ..layers.moe.fused_moe import FusedExperts, GroupedSoftmaxRouter
from ..layers.recurrent.linear_recurrence import ChannelForgetMixer
from ..layers.residual_norm import AddNormed, ResidualRMSNorm
from .registry import CacheSpec, register_model


class SapivikExperts(nn.Module):
    def __init__(self, width: int, spec: IdentityExpertsSpec, params_dtype):
        super().__init__()
        self.router = GroupedSoftmaxRouter(width, spec.experts, spec.top, identity=spec.identity, renormalize=False,
                                           scale=spec.scale, shared_gate=spec.shared_ff > 0)
        self.experts = FusedExperts(width, spec.ff, spec.experts, "silu", params_dtype)
        self.shared = GatedMLP(width, spec.shared_ff, "silu", params_dtype) if spec.shared_ff else None

    def forward(self, h: torch.Tensor) -> dict:
        """-> the terms of the sublayer's output, summed by AddNormed in fp32."""
        ids, wts, gate = self.router.route(h)
        terms = dict(rows=self.experts(h, ids), top=ids.shape[1], row_weights=wts)
        if self.router.identity:
            terms.update(row_ids=ids, experts=self.experts.experts, same=h)
        if self.shared is not None:
            terms.update(b=self.shared(h), b_gate=gate)
        return terms


class SapivikLayer(nn.Module):
    def __init__(self, cfg: SapivikConfig, spec: SapivikLayerSpec, layer_id: int, params_dtype):
        super().__init__()
        self.layer_id, self.type, self.params_dtype = layer_id, spec.type, params_dtype
        m, W = spec.mixer, cfg.width
        if spec.type == "hgrn2":
            self.mix = ChannelForgetMixer(W, m.heads, m.dim, m.vdim, layer_id, cfg.eps, params_dtype)
        else:
            self.mix = SinkAttention(W, m.heads, m.kv_heads, m.dim, m.dim, m.scale, layer_id, cfg.eps,
                                     rope_base=m.rope_base, rope_dims=m.rope_dims, qk_norm="unit", sink=False,
                                     bias=False, params_dtype=params_dtype, softcap=m.softcap, tied_values=True,
                                     out_gate=True)
        self.norm1 = ResidualRMSNorm(W, cfg.eps)          # used by the first layer run only: every other
        self.norm1b = AddNormed(W, cfg.eps, cfg.residual_mult)     # pre-norm is emitted by the launch before it
        self.dense = self.moe = self.norm2 = self.norm2b = None
        if isinstance(spec.mlp, ClampedSpec):
            self.dense = GatedMLP(W, spec.mlp.ff, "clamped", params_dtype, limit=spec.mlp.limit)
        elif spec.mlp is not None:
            self.moe = SapivikExperts(W, spec.mlp, params_dtype)
        if spec.mlp is not None:
            self.norm2 = ResidualRMSNorm(W, cfg.eps)
            self.norm2b = AddNormed(W, cfg.eps, cfg.residual_mult)

    def forward(self, x: torch.Tensor, h: torch.Tensor, fb, cache_id: int, next_weight: Optional[torch.Tensor],
                inject: Optional[Tuple[torch.Tensor, torch.Tensor]]) -> Optional[torch.Tensor]:
        """x: the fp32 residual [T, width], updated in place; h = norm_1(x) in the model dtype.  -> the next
        run's norm_1(x) (None after the last), x having received the rows of `inject` ahead of it."""
        dt = self.params_dtype
        last = dict(out_dtype=dt if next_weight is not None else None, next_weight=next_weight, inject=inject)
        y = self.mix(h, fb, cache_id=cache_id)
        if self.norm2 is None:
            return self.norm1b(x, a=y, **last)
        h2 = self.norm1b(x, a=y, out_dtype=dt, next_weight=self.norm2.weight)
        if self.dense is not None:
            return self.norm2b(x, a=self.dense(h2), **last)
        return self.norm2b(x, **self.moe(h2), **last)


@register_model("Sapivik")
class SapivikForCausalLM(nn.Module):
    def __init__(self, config: SapivikConfig, params_dtype: torch.dtype = torch.bfloat16):
        super().__init__()
        self.config, self.params_dtype = config, params_dtype
        self.runs = config.layer_runs()
        self.embed = nn.Parameter(torch.empty(config.vocab, config.width, dtype=params_dtype), requires_grad=False)
        self.layers = nn.ModuleList(SapivikLayer(config, s, i, params_dtype) for i, s in enumerate(config.layers))
        self.final_norm = ResidualRMSNorm(config.width, config.eps)
        self.head = ColumnParallelLinear(config.width, config.vocab, bias=False, params_dtype=params_dtype,
                                         tp_rank=0, tp_size=1)

    # ---- what the runner allocates -------------------------------------------------------------
    def cache_spec(self) -> CacheSpec:
        spec = CacheSpec(kind="rows")
        for run, (i, _) in enumerate(self.runs):
            mix = self.layers[i].mix
            if self.layers[i].type == "attention":
                spec.row_dims[run] = mix.row_width
            else:
                spec.state_widths[run] = mix.state_width()
        return spec

    # ---- forward -------------------------------------------------------------------------------
    def forward(self, input_ids: torch.Tensor, forward_batch) -> torch.Tensor:
        x = self.embed[input_ids].float()
        hook = forward_batch.extra.get("layer_hook") if forward_batch.extra else None
        h = self.layers[self.runs[0][0]].norm1(x, self.params_dtype) if self.runs else None
        for run, (i, _) in enumerate(self.runs):
            nxt, inject = None, None
            if run + 1 < len(self.runs):
                after, starts_pass = self.runs[run + 1]
                nxt = self.layers[after].norm1.weight
                inject = (self.embed, input_ids) if starts_pass else None
            h = self.layers[i](x, h, forward_batch, run, nxt, inject)
            if hook is not None:
                hook(i, x if inject is None else x - self.embed[input_ids].float())
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

    def _load_layer_tensor(self, layer: SapivikLayer, key: str, w: torch.Tensor) -> None:
        bad = ValueError(f"unexpected tensor l{layer.layer_id}.{key}")
        norms = {"norm1": layer.norm1, "norm1b": layer.norm1b, "norm2": layer.norm2, "norm2b": layer.norm2b}
        if key in norms:
            if norms[key] is not None:               # without a feed-forward there is nothing to norm
                norms[key].weight.data.copy_(w.float())
        elif key.startswith("mlp."):
            self._load_mlp_tensor(layer, key[4:], w, bad)
        elif key.startswith("mix."):
            k, mix = key[4:], layer.mix
            if k == "o":
                mix.o_proj.weight_loader(mix.o_proj.weight, w)
            elif layer.type == "attention" and k in ("q", "k", "g"):
                mix.load_part(k, w)
            elif layer.type == "hgrn2" and k in ("q", "f", "v"):
                mix.load_part(k, w)
            elif layer.type == "hgrn2" and k == "f.b":
                mix.f_bias.data.copy_(w.float().reshape(-1))
            elif layer.type == "hgrn2" and k == "lower":
                mix.f_lower.data.copy_(w.float().reshape(-1))
            elif layer.type == "hgrn2" and k == "norm":
                mix.norm_weight.data.copy_(w.float().repeat(mix.heads))
            else:
                raise bad
        else:
            raise bad

    def _load_mlp_tensor(self, layer: SapivikLayer, k: str, w: torch.Tensor, bad: Exception) -> None:
        if layer.dense is not None:
            mlp = layer.dense
        elif layer.moe is not None and k == "shared.sg" and layer.moe.shared is not None:
            layer.moe.router.shared_gate.data.copy_(w.float().reshape(-1))
            return
        elif layer.moe is not None and k.startswith("shared.") and layer.moe.shared is not None:
            mlp, k = layer.moe.shared, k[7:]
        elif layer.moe is not None:
            m = re.match(r"^e(\d+)\.(gate|up|down)$", k)
            ex = layer.moe.experts
            if k == "router":
                layer.moe.router.weight.data.copy_(w.float())
            elif k == "correction":
                layer.moe.router.correction.data.copy_(w.float().reshape(-1))
            elif m and int(m.group(1)) < ex.experts:
                e, lo = int(m.group(1)), 0 if m.group(2) == "gate" else ex.ff
                (ex.w_down.data[e] if m.group(2) == "down" else ex.w_gate_up.data[e, lo:lo + ex.ff]).copy_(w)
            else:
                raise bad
            return
        else:
            raise bad
        if k in ("gate", "up"):
            mlp.gate_up_proj.weight_loader(mlp.gate_up_proj.weight, w, 0 if k == "gate" else 1)
        elif k == "down":
            mlp.down_proj.weight_loader(mlp.down_proj.weight, w)
        else:
            raise bad

    def expected_tensor_names(self):
        names = {"embed", "head", "final.norm"}
        for i, L in enumerate(self.config.layers):
            p = f"l{i}."
            names |= {p + "norm1", p + "norm1b"}
            keys = ("q", "f", "f.b", "lower", "v", "norm", "o") if L.type == "hgrn2" else ("q", "k", "g", "o")
            names |= {p + "mix." + k for k in keys}
            if L.mlp is not None:
                names |= {p + "norm2", p + "norm2b"}
            if isinstance(L.mlp, ClampedSpec):
                names |= {p + "mlp." + k for k in ("gate", "up", "down")}
            elif L.mlp is not None:
                names |= {p + "mlp.router", p + "mlp.correction"}
                names |= {p + f"mlp.e{e}." + k for e in range(L.mlp.experts) for k in ("gate", "up", "down")}
                if L.mlp.shared_ff:
                    names |= {p + "mlp.shared." + k for k in ("gate", "up", "down", "sg")}
        return names
