"""Plain, slow restatement of the Luzosun design in float64: one function per mechanism, dense masks,
no caches and no batches.  It shares no code with the package; the tests compare the engine with it.

Notation: x residual [T, W]; a layer is  x <- x + (mixer(c(n1(x))) + ff(n2(x)))  with the two norms
of the same x and c(h) = h + conv(h).  `W` below is a dict name -> float64 tensor, `cfg` the parsed
config.json."""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def rms_div(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return rms_div(x, eps) * w


def causal_conv(u, w):
    """u [T, C], w [C, taps] (last column multiplies the current token), zeros before the start."""
    T, C = u.shape
    taps = w.shape[1]
    y = torch.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                y[t] += w[:, j] * u[s]
    return y


def rotate_halves(x, pos, dims, base, factor):
    """x [T, N, D]: coordinates i and i + dims/2 of every row turn by pos * base^(-2i/dims) / factor."""
    if not dims:
        return x
    half = dims // 2
    out = x.clone()
    for i in range(half):
        a = pos.to(F64) * (base ** (-2.0 * i / dims) / factor)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * c - v * s
        out[..., i + half] = v * c + u * s
    return out


def visible(T, chunk):
    """[T, T] bool: key j is seen from i when it is not later and lies in the same chunk of positions."""
    i = torch.arange(T)
    ok = i[None, :] <= i[:, None]
    if chunk:
        ok &= (i[None, :] // chunk) == (i[:, None] // chunk)
    return ok


def softmax_map(q, k, v, scale, mask):
    """One map: q [T, D], k [T, D], v [T, E]."""
    s = (q @ k.T) * scale
    s = s.masked_fill(~mask, -math.inf)
    return torch.softmax(s, -1) @ v


def mix_lambda(W, p, diff):
    return math.exp(float((W[p + "lq1"] * W[p + "lk1"]).sum())) - \
        math.exp(float((W[p + "lq2"] * W[p + "lk2"]).sum())) + diff


def combine_maps(a1, a2, lam, diff, eps):
    return rms_div(a1 - lam * a2, eps) * (1.0 - diff)


def project(h, W, name):
    return h @ W[name].T + W[name + ".b"]


def keys_values(h, W, p, m):
    """-> rotated keys [T, G * 2, D] (map 1 and map 2 of head 0, of head 1, ...) and values [T, G, E]."""
    T, G, D, E = h.shape[0], m.get("kv_heads", m["heads"]), m["dim"], m["vdim"]
    k, v = project(h, W, p + "k"), project(h, W, p + "v")
    if p + "k.conv" in W:
        k, v = causal_conv(k, W[p + "k.conv"]), causal_conv(v, W[p + "v.conv"])
    return rotated(k.view(T, G * 2, D), m), v.view(T, G, E)


def rotated(x, m):
    rot = m.get("rot") or {}
    return rotate_halves(x, torch.arange(x.shape[0]), rot.get("dims", 0), rot.get("base", 1e4),
                         (rot.get("scaling") or {}).get("factor", 1.0))


def attention(h, W, p, m, eps, kv):
    """kv: (keys, values) of the layer whose cache is read."""
    T, H, G, D, E = h.shape[0], m["heads"], m.get("kv_heads", m["heads"]), m["dim"], m["vdim"]
    q = project(h, W, p + "q")
    if p + "q.conv" in W:
        q = causal_conv(q, W[p + "q.conv"])
    q = rotated(q.view(T, H * 2, D), m)
    k, v = kv
    mask = visible(T, (m.get("mask") or {}).get("size", 0))
    lam = mix_lambda(W, p, m["diff"])
    out = torch.zeros(T, H, E, dtype=F64)
    for hh in range(H):
        g = hh // (H // G)
        a = [softmax_map(q[:, 2 * hh + i], k[:, 2 * g + i], v[:, g], m["scale"], mask) for i in (0, 1)]
        out[:, hh] = combine_maps(a[0], a[1], lam, m["diff"], eps)
    return out.reshape(T, H * E) @ W[p + "o"].T


def softplus(z):
    return math.log1p(math.exp(z)) if z < 30 else z


def xielu(z, p, q):
    pos = softplus(p) * z * z + 0.5 * z
    zn = torch.clamp(z, max=0.0)
    neg = (0.5 + softplus(q)) * (torch.expm1(zn) - zn) + 0.5 * z
    return torch.where(z > 0, pos, neg)


def feed_forward(h, W, p):
    a = W[p + "act"]
    return xielu(h @ W[p + "up"].T, float(a[0]), float(a[1])) @ W[p + "down"].T


def forward(cfg, weights, tokens, layers_out=None):
    """-> logits [T, vocab], float64."""
    W = {k: v.to(F64) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.tensor(list(tokens))] * (cfg.get("embedding") or {}).get("scale", 1.0)
    kvs = {}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        h = rms_norm(x, W[p + "norm1"], eps)
        if p + "canon1" in W:
            h = h + causal_conv(h, W[p + "canon1"])
        src = m.get("kv_from")
        if src is None:
            kvs[i] = keys_values(h, W, p + "mix.", m)
        y = attention(h, W, p + "mix.", m, eps, kvs[i if src is None else src])
        if L.get("mlp"):
            y = y + feed_forward(rms_norm(x, W[p + "norm2"], eps), W, p + "mlp.")
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms_norm(x, W["final.norm"], eps) @ W["head"].T
