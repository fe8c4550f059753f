"""Plain, slow restatement of the Sapivik design in float64 on the CPU: one function per mechanism, loops
over tokens, heads and experts, dense scores.  Shares no code with the package."""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """Every row of the last dimension over its root mean square, eps under the root."""
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z / (1.0 + torch.exp(-z))


def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-z))


def forget_gate(z: torch.Tensor, bias: torch.Tensor, lower: torch.Tensor) -> torch.Tensor:
    """Between `lower` (pre-activation far below zero) and 1."""
    return lower + (1.0 - lower) * sigmoid(z + bias)


def gated_memory(q: torch.Tensor, f: torch.Tensor, v: torch.Tensor,
                 start: Optional[torch.Tensor] = None):
    """q, f [T, heads, dim], v [T, heads, vdim] -> (outputs [T, heads, vdim], memory [heads, dim, vdim]).
    A channel keeps the share f of what it holds and takes the share 1 - f of the token's value."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype) if start is None else start.clone()
    out = []
    for t in range(T):
        S = f[t][:, :, None] * S + (1.0 - f[t])[:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hd,hde->he", q[t], S))
    return torch.stack(out), S


def rotate_neighbours(x: torch.Tensor, positions: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x [T, heads, dim]: coordinates (2i, 2i+1), i < dims / 2, turned by position * base^(-2i/dims)."""
    if not dims:
        return x
    y = x.clone()
    for i in range(dims // 2):
        a = positions.to(x.dtype)[:, None] * float(base) ** (-2.0 * i / dims)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i] = u * torch.cos(a) - v * torch.sin(a)
        y[..., 2 * i + 1] = v * torch.cos(a) + u * torch.sin(a)
    return y


def soft_cap(s: torch.Tensor, cap: Optional[float]) -> torch.Tensor:
    return cap * torch.tanh(s / cap) if cap else s


def causal_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float,
                     cap: Optional[float]) -> torch.Tensor:
    """q [T, heads, dim], k [T, kv_heads, dim], v [T, kv_heads, vdim] -> [T, heads, vdim]."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    seen = torch.tril(torch.ones(T, T, dtype=torch.bool))
    out = []
    for h in range(H):
        s = soft_cap(q[:, h] @ k[:, h // per].T * scale, cap)
        s = s.masked_fill(~seen, -math.inf)
        w = torch.exp(s - s.max(-1, keepdim=True).values)
        out.append((w / w.sum(-1, keepdim=True)) @ v[:, h // per])
    return torch.stack(out, 1)


def memory_mixer(W: Dict[str, torch.Tensor], p: str, m: dict, h: torch.Tensor, eps: float) -> torch.Tensor:
    T, H, D, E = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = silu(h @ W[p + "q"].T).view(T, H, D)
    f = forget_gate(h @ W[p + "f"].T, W[p + "f.b"], W[p + "lower"]).view(T, H, D)
    o, _ = gated_memory(q, f, (h @ W[p + "v"].T).view(T, H, E))
    o = unit_rms(o, eps) * W[p + "norm"]
    return o.reshape(T, H * E) @ W[p + "o"].T


def attention_mixer(W: Dict[str, torch.Tensor], p: str, m: dict, h: torch.Tensor, eps: float) -> torch.Tensor:
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = (h @ W[p + "q"].T).view(T, H, D)
    raw = (h @ W[p + "k"].T).view(T, G, D)
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    at = torch.arange(T)
    q = unit_rms(rotate_neighbours(q, at, rot["dims"], rot["base"]), eps)
    k = unit_rms(rotate_neighbours(raw, at, rot["dims"], rot["base"]), eps)
    o = causal_attention(q, k, raw, m["scale"], m.get("softcap")).reshape(T, H * D)
    return (o * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def clamped_ff(W: Dict[str, torch.Tensor], p: str, limit: float, h: torch.Tensor) -> torch.Tensor:
    g = (h @ W[p + "gate"].T).clamp(max=limit)
    u = (h @ W[p + "up"].T).clamp(-limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ W[p + "down"].T


def silu_ff(W: Dict[str, torch.Tensor], p: str, h: torch.Tensor) -> torch.Tensor:
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def route(z: torch.Tensor, correction: torch.Tensor, top: int, scale: float):
    """Router logits of one token -> (chosen experts, their weights)."""
    s = torch.exp(z - z.max())
    s = s / s.sum()
    ids = torch.argsort(s + correction, descending=True, stable=True)[:top]
    return ids.tolist(), (s[ids] * scale).tolist()


def expert_ff(W: Dict[str, torch.Tensor], p: str, mlp: dict, h: torch.Tensor) -> torch.Tensor:
    r = mlp["router"]
    z = h @ W[p + "router"].T
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(*route(z[t], W[p + "correction"], r["top"], r.get("scale", 1.0))):
            y = h[t] if e >= r["experts"] else silu_ff(W, f"{p}e{e}.", h[t:t + 1])[0]
            out[t] += w * y
    if mlp.get("shared"):
        out += sigmoid(h @ W[p + "shared.sg"].T) * silu_ff(W, p + "shared.", h)
    return out


def layer_order(n: int, loop: Optional[dict]) -> List[tuple]:
    """-> [(layer, whether the embedding output is added ahead of it)] in the order they run."""
    if not loop:
        return [(i, False) for i in range(n)]
    body = list(range(loop["start"], loop["stop"]))
    runs = [(i, False) for i in range(loop["start"])]
    for turn in range(loop["times"]):
        runs += [(i, turn > 0 and i == body[0]) for i in body]
    return runs + [(i, False) for i in range(loop["stop"], n)]


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens, layers_out: Optional[list] = None) -> torch.Tensor:
    W = {k: v.double() for k, v in weights.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    first = W["embed"][torch.as_tensor(tokens, dtype=torch.int64)]
    x = first.clone()
    for i, inject in layer_order(len(cfg["layers"]), cfg.get("loop")):
        L, p = cfg["layers"][i], f"l{i}."
        if inject:
            x = x + first
        mixer = memory_mixer if L["type"] == "hgrn2" else attention_mixer
        y = mixer(W, p + "mix.", L["mixer"], unit_rms(x, eps) * W[p + "norm1"], eps)
        x = x + mult * unit_rms(y, eps) * W[p + "norm1b"]
        if L.get("mlp"):
            h = unit_rms(x, eps) * W[p + "norm2"]
            if L["mlp"]["kind"] == "dense":
                y = clamped_ff(W, p + "mlp.", L["mlp"]["limit"], h)
            else:
                y = expert_ff(W, p + "mlp.", L["mlp"], h)
            x = x + mult * unit_rms(y, eps) * W[p + "norm2b"]
        if layers_out is not None:
            layers_out.append(x.clone())
    return (unit_rms(x, eps) * W["final.norm"]) @ W["head"].T
