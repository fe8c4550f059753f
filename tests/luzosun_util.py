"""Helpers of the Luzosun tests: small random configurations and weights as a model folder, and the
hand-made batches of dozetar_util for driving single kernels."""
from __future__ import annotations

from typing import Dict, Optional, Sequence

import torch

from desirax_util import Driver, rel_err, rel_errs, write_model  # noqa: F401  (shared test plumbing)
from dozetar_util import HandBatch, cut  # noqa: F401


def diff(heads=4, kv_heads=2, dim=12, vdim=20, chunk: Optional[int] = 40, conv=4, rot_dims=8, base=1000.0,
         factor: Optional[float] = 2.5, lam=0.4, scale=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "diff": lam,
         "scale": float(scale if scale is not None else dim ** -0.5)}
    if chunk:
        m["mask"] = {"size": chunk}
    if conv:
        m["conv"] = conv
    if rot_dims:
        m["rot"] = {"base": base, "dims": rot_dims}
        if factor:
            m["rot"]["scaling"] = {"factor": factor}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def dense(ff=56):
    return {"kind": "dense", "ff": ff}


def config(layers: Sequence[tuple], vocab=89, width=40, eps=1e-5, emb=3.0, taps=3) -> dict:
    return {"architecture": "Luzosun", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "embedding": {"scale": emb}, "canon": {"taps": taps},
            "layers": [{"type": "attention", "mixer": m, "mlp": f} for m, f in layers]}


def random_weights(cfg: dict, seed: int = 0) -> Dict[str, torch.Tensor]:
    """bf16 tensors (so that a bf16 and a fp32 engine load the same values)."""
    g = torch.Generator().manual_seed(seed)
    W, bf = cfg["width"], torch.bfloat16

    def lin(o, i, gain=1.0):
        return (torch.randn(o, i, generator=g) * gain / i ** 0.5).to(bf)

    def vec(n, mean=1.0, sd=0.2):
        return (mean + sd * torch.randn(n, generator=g)).to(bf)

    w = {"embed": (torch.randn(cfg["vocab"], W, generator=g) / cfg["embedding"]["scale"]).to(bf),
         "head": lin(cfg["vocab"], W, 3.0), "final.norm": vec(W)}
    for i, L in enumerate(cfg["layers"]):
        p, m, q = f"l{i}.", L["mixer"], f"l{i}.mix."
        H, G, D, E, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m.get("conv")
        w[p + "norm1"] = vec(W)
        if cfg["canon"]["taps"]:
            w[p + "canon1"] = (torch.randn(W, cfg["canon"]["taps"], generator=g) * 0.4).to(bf)
        parts = {"q": H * 2 * D} if m.get("kv_from") is not None else {"q": H * 2 * D, "k": G * 2 * D, "v": G * E}
        for n, rows in parts.items():
            w[q + n], w[q + n + ".b"] = lin(rows, W, 1.5), vec(rows, 0.0, 0.3)
            if taps:
                w[q + n + ".conv"] = (torch.randn(rows, taps, generator=g) * 0.6).to(bf)
        for n in ("lq1", "lk1", "lq2", "lk2"):
            w[q + n] = vec(D, 0.0, 0.3)
        w[q + "o"] = lin(W, H * E)
        if L["mlp"]:
            w[p + "norm2"], ff = vec(W), L["mlp"]["ff"]
            w[p + "mlp.up"], w[p + "mlp.down"], w[p + "mlp.act"] = lin(ff, W, 1.5), lin(W, ff), vec(2, 0.0, 0.8)
    return w
