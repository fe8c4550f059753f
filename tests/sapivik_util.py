"""Helpers of the Sapivik tests: small random configurations and weights as a model folder, and hand-made
batches (dozetar_util) with what the attention layer reads besides the kernels' tables."""
from __future__ import annotations

from types import SimpleNamespace
from typing import Dict, Optional, Sequence

import torch

from desirax_util import Driver, rel_err, rel_errs, write_model  # noqa: F401  (shared test plumbing)
from dozetar_util import HandBatch, cut  # noqa: F401


def mem(heads=3, dim=12, vdim=20):
    return "hgrn2", {"heads": heads, "dim": dim, "vdim": vdim}


def att(heads=4, kv_heads=2, dim=20, rot_dims=8, base=900.0, cap: Optional[float] = 12.0, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": float(scale or dim ** -0.5)}
    if cap:
        m["softcap"] = cap
    if rot_dims:
        m["rot"] = {"base": base, "dims": rot_dims}
    return "attention", m


def dense(ff=36, limit=1.5):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts=5, identity=3, top=3, scale=1.6, ff=20, shared_ff: Optional[int] = 28):
    f = {"kind": "moe", "router": {"experts": experts, "identity": identity, "top": top, "scale": scale},
         "expert": {"ff": ff}}
    if shared_ff:
        f["shared"] = {"ff": shared_ff}
    return f


def config(layers: Sequence[tuple], loop: Optional[tuple] = None, vocab=83, width=40, eps=1e-4, mult=0.45) -> dict:
    c = {"architecture": "Sapivik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
         "layers": [{"type": kind, "mixer": m, "mlp": f} for (kind, m), f in layers]}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def random_weights(cfg: dict, seed: int = 0) -> Dict[str, torch.Tensor]:
    """bf16 tensors (so that a bf16 and a fp32 engine load the same values)."""
    g = torch.Generator().manual_seed(seed)
    W, bf = cfg["width"], torch.bfloat16

    def lin(o, i, gain=1.0):
        return (torch.randn(o, i, generator=g) * gain / i ** 0.5).to(bf)

    def vec(n, mean=1.0, sd=0.2):
        return (mean + sd * torch.randn(n, generator=g)).to(bf)

    w = {"embed": torch.randn(cfg["vocab"], W, generator=g).to(bf), "head": lin(cfg["vocab"], W, 3.0),
         "final.norm": vec(W)}
    for i, L in enumerate(cfg["layers"]):
        p, m, q = f"l{i}.", L["mixer"], f"l{i}.mix."
        w[p + "norm1"], w[p + "norm1b"] = vec(W), vec(W)
        H, D = m["heads"], m["dim"]
        if L["type"] == "hgrn2":
            E = m["vdim"]
            w[q + "q"], w[q + "f"], w[q + "v"] = lin(H * D, W, 2.0), lin(H * D, W, 1.5), lin(H * E, W)
            w[q + "f.b"] = vec(H * D, 1.5, 1.5)
            w[q + "lower"] = (torch.rand(H * D, generator=g) * 0.9 * (torch.rand(H * D, generator=g) > 0.2)).to(bf)
            w[q + "norm"], w[q + "o"] = vec(E), lin(W, H * E)
        else:
            G = m["kv_heads"]
            w[q + "q"], w[q + "k"], w[q + "g"] = lin(H * D, W), lin(G * D, W), lin(H * D, W, 1.5)
            w[q + "o"] = lin(W, H * D)
        f = L["mlp"]
        if not f:
            continue
        w[p + "norm2"], w[p + "norm2b"] = vec(W), vec(W)

        def ff(q, n):
            w[q + "gate"], w[q + "up"], w[q + "down"] = lin(n, W, 1.5), lin(n, W, 1.5), lin(W, n)

        if f["kind"] == "dense":
            ff(p + "mlp.", f["ff"])
        else:
            r = f["router"]
            total = r["experts"] + r["identity"]
            for e in range(r["experts"]):
                ff(p + f"mlp.e{e}.", f["expert"]["ff"])
            w[p + "mlp.router"] = lin(total, W, 2.0)
            w[p + "mlp.correction"] = vec(total, 0.0, 0.1)
            if f.get("shared"):
                ff(p + "mlp.shared.", f["shared"]["ff"])
                w[p + "mlp.shared.sg"] = lin(1, W, 1.5)
    return w


class LayerBatch:
    """One token pool over a HandBatch, and the ForwardBatch-like object an attention layer reads."""

    def __init__(self, slots: int, context: int, row_width: int, dtype, page=16, seed=0, stale=3.0):
        self.hb = HandBatch(slots, context, page=page, seed=seed)
        self.pool = torch.full((self.hb.pool_rows, row_width), stale, dtype=dtype, device="cuda")

    def step(self, entries):
        pre = [self.hb.lens[r] for r, _ in entries]
        fb = self.hb.step(entries)
        ext = [n for _, n in entries]
        fb.extend_prefix_lens_cpu, fb.extend_seq_lens_cpu = pre, ext
        fb.positions, fb.max_seq_len, fb.extra = fb.tok_pos.long(), max(p + e for p, e in zip(pre, ext)), {}
        fb.req_to_token_pool = SimpleNamespace(req_to_token=fb.req_to_token)
        fb.token_to_kv_pool = SimpleNamespace(get_kv_buffer=lambda i: self.pool)
        return fb
