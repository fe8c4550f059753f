"""Sapivik's mechanisms one at a time on the GPU kernels, each against its plain restatement: the
channel-gated memory (portions, slots, odd sizes), the tied attention on all of its kernels (a key that stands
out at every border), the residual launch with all of its terms, the router with identity experts."""
import pytest
import torch

import sapivik_plain as P
import sapivik_util as U

pytestmark = pytest.mark.gpu
DEV = "cuda"


def _err(got, want):
    return float((got.double().cpu() - want).abs().max() / want.abs().max().clamp_min(1e-9))


# ---- memory with a forget gate per channel -------------------------------------------------------------
def _batch(hb, entries):
    fb = hb.step(entries)
    fb.extend_seq_lens_cpu = [n for _, n in entries]
    return fb


def _run_memory(H, D, E, lens, cuts, dtype, seed=0, gate_gain=2.0, gate_mean=1.0, chunk_min=32):
    """`lens` sequences fed together in portions `cuts[i]`; -> (outputs per sequence, oracle per sequence)."""
    from sglang_security_b200.layers.recurrent.linear_recurrence import channel_recurrence, state_width

    g = torch.Generator().manual_seed(seed)
    hb = U.HandBatch(len(lens), max(lens) + 1)
    state = torch.full((len(lens), state_width(H, D, E, False)), 7.0, device=DEV)      # stale values everywhere
    bias = torch.randn(H * D, generator=g) + gate_mean
    lower = torch.rand(H * D, generator=g) * 0.9 * (torch.rand(H * D, generator=g) > 0.3)
    data = [(torch.randn(n, H * D, generator=g).to(dtype), (torch.randn(n, H * D, generator=g) * gate_gain).to(dtype),
             torch.randn(n, H * E, generator=g).to(dtype)) for n in lens]
    got, at, todo = [[] for _ in lens], [0] * len(lens), [list(c) for c in cuts]
    while any(todo):
        entries = [(i, todo[i].pop(0)) for i in range(len(lens)) if todo[i]]
        fb = _batch(hb, entries)
        part = torch.cat([torch.cat([d[at[i]:at[i] + n] for d in data[i]], 1) for i, n in entries]).to(DEV)
        out = channel_recurrence(part[:, :H * D], part[:, H * D:2 * H * D], part[:, 2 * H * D:], bias.to(DEV),
                                 lower.to(DEV), H, D, E, state, fb, chunk_min=chunk_min)
        o = 0
        for i, n in entries:
            got[i].append(out[o:o + n].cpu())
            at[i] += n
            o += n
    want = []
    for (q, z, v), n in zip(data, lens):
        f = P.forget_gate(z.double(), bias.double(), lower.double()).view(n, H, D)
        want.append(P.gated_memory(P.silu(q.double()).view(n, H, D), f, v.double().view(n, H, E))[0].reshape(n, H * E))
    return [torch.cat(x) for x in got], want


@pytest.mark.parametrize("H,D,E", [(2, 16, 16), (3, 24, 20), (1, 40, 72), (2, 72, 9), (4, 1, 1), (1, 130, 33), (2, 64, 128),
                                   (1, 128, 96)])
def test_memory_portions_against_token_by_token(H, D, E):
    lens = [137, 5, 161]
    cuts = [U.cut(137, [2, 50, 1, 16]), [5], U.cut(161, [133, 1, 1, 2])]
    got, want = _run_memory(H, D, E, lens, cuts, torch.float32)
    one, _ = _run_memory(H, D, E, lens, [[1] * n for n in lens], torch.float32)
    whole, _ = _run_memory(H, D, E, lens, [[n] for n in lens], torch.float32)
    for a, b, c, w in zip(got, one, whole, want):
        assert _err(a, w) <= 5e-6 and _err(b, w) <= 5e-6 and _err(c, w) <= 5e-6
    # the token-by-token kernel alone: the same sums in the same order however the sequence is cut
    walk, _ = _run_memory(H, D, E, lens, cuts, torch.float32, chunk_min=0)
    assert all(torch.equal(a, b) for a, b in zip(walk, one))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16, torch.float16])
@pytest.mark.parametrize("H,D,E", [(2, 5, 6), (1, 33, 31), (3, 64, 16), (2, 100, 40), (1, 128, 130), (5, 32, 64), (2, 8, 3)])
def test_memory_chunks_of_any_length(dtype, H, D, E):
    """Portions around the 16-token chunk, each continued: every place of a chunk is a portion's first and last."""
    lens = [150, 97, 64]
    cuts = [[1, 2, 15, 16, 17, 33, 31, 35], [48, 1, 47, 1], [18, 14, 16, 2, 14]]
    got, want = _run_memory(H, D, E, lens, cuts, dtype, seed=2, chunk_min=2)
    for a, w in zip(got, want):
        assert _err(a, w) <= 5e-6


@pytest.mark.parametrize("mean,gain", [(9.0, 1.0), (-9.0, 1.0), (0.0, 30.0), (0.0, 0.1)])
def test_memory_gates_near_their_ends(mean, gain):
    """Gates that hardly forget (the written share is tiny and must keep its leading digits), that forget all but
    the lower bound, that saturate either way, and that stay in the middle."""
    got, want = _run_memory(2, 24, 16, [300], [[150, 2, 148]], torch.float32, seed=3, gate_mean=mean, gate_gain=gain)
    assert _err(got[0], want[0]) <= 1e-5


def test_memory_16_bit_rows_and_long_decoding():
    got, want = _run_memory(2, 32, 48, [420], [[20] + [1] * 400], torch.bfloat16, seed=5)
    assert _err(got[0], want[0]) <= 1e-5
    got, want = _run_memory(2, 64, 64, [700], [[690] + [1] * 10], torch.bfloat16, seed=6, gate_mean=5.0)
    assert _err(got[0], want[0]) <= 1e-5


def test_memory_cta_sizes_share_one_state_layout():
    H, D, E, B = 8, 64, 128, 24
    got, want = _run_memory(H, D, E, [75] * B, [[72] + [1] * 3 for _ in range(B)], torch.float32, seed=9)
    for a, b in zip(got, want):
        assert _err(a, b) <= 5e-6
    one, _ = _run_memory(H, D, E, [75], [[72, 1, 1, 1]], torch.float32, seed=9)
    assert _err(one[0], want[0]) <= 5e-6


def test_memory_of_a_reused_slot_is_ignored():
    from sglang_security_b200.layers.recurrent.linear_recurrence import channel_recurrence, state_width

    H, D, E = 2, 16, 8
    for n in (9, 90):
        hb = U.HandBatch(1, 128)
        state, outs = torch.zeros((1, state_width(H, D, E, False)), device=DEV), []
        for _ in range(2):
            g = torch.Generator().manual_seed(7)
            q, z, v = (torch.randn(n, k, generator=g).to(DEV) for k in (H * D, H * D, H * E))
            outs.append(channel_recurrence(q, z, v, None, None, H, D, E, state, _batch(hb, [(0, n)])))
            hb.release(0)                     # the next sequence in this row starts at position 0
        assert torch.equal(outs[0], outs[1]) and state.abs().max() > 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_memory_mixer_with_its_norm(dtype):
    from sglang_security_b200.layers.recurrent.linear_recurrence import ChannelForgetMixer

    from types import SimpleNamespace
    cfg = U.config([(U.mem(3, 12, 20), None)])
    w = U.random_weights(cfg, 4)
    mix = ChannelForgetMixer(40, 3, 12, 20, 0, 1e-4, dtype).to(DEV)
    for k in "qfv":
        mix.load_part(k, w[f"l0.mix.{k}"])
    mix.f_bias.data.copy_(w["l0.mix.f.b"])
    mix.f_lower.data.copy_(w["l0.mix.lower"])
    mix.norm_weight.data.copy_(w["l0.mix.norm"].float().repeat(3))
    mix.o_proj.weight.data.copy_(w["l0.mix.o"])
    h = torch.randn(50, 40, generator=torch.Generator().manual_seed(5)).to(dtype)
    hb = U.HandBatch(2, 64)
    states = {9: torch.zeros((2, mix.state_width()), device=DEV)}
    got = []
    for lo, hi in ((0, 33), (33, 34), (34, 50)):
        fb = _batch(hb, [(1, hi - lo)])
        fb.state_pool = SimpleNamespace(get=lambda i: states[i])
        got.append(mix(h[lo:hi].to(DEV), fb, cache_id=9))
    want = P.memory_mixer({k: t.double() for k, t in w.items()}, "l0.mix.", cfg["layers"][0]["mixer"], h.double(), 1e-4)
    assert _err(torch.cat(got), want) <= (2e-5 if dtype == torch.float32 else 3e-2)


# ---- attention whose values are its keys -----------------------------------------------------------------
PATHS = {"core32": torch.float32, "core16": torch.bfloat16, "split": torch.bfloat16, "prompt": torch.bfloat16}


def _layer(monkeypatch, path, W, m, w, eps=1e-4):
    """The attention layer pinned to one kernel: CUDA cores in 32 or 16 bits, the split-key kernel, or the
    tensor-core prompt kernel for every portion."""
    from sglang_security_b200.layers.attention.sink_attention import SinkAttention

    monkeypatch.setattr(SinkAttention, "tensor_core_min_tokens", 1 if path == "prompt" else 0)
    monkeypatch.setattr(SinkAttention, "split_decode", path == "split")
    rot = m.get("rot") or {"base": 1.0, "dims": 0}
    att = SinkAttention(W, m["heads"], m["kv_heads"], m["dim"], m["dim"], m["scale"], 0, eps, rope_base=rot["base"],
                        rope_dims=rot["dims"], qk_norm="unit", sink=False, bias=False, params_dtype=PATHS[path],
                        softcap=m.get("softcap") or 0.0, tied_values=True, out_gate=True).to(DEV)
    for k in "qkg":
        att.load_part(k, w[k].to(DEV))
    att.o_proj.weight.data.copy_(w["o"])
    return att


def _att_weights(W, m, seed):
    g = torch.Generator().manual_seed(seed)
    lin = lambda o, i: (torch.randn(o, i, generator=g) / i ** 0.5).bfloat16()
    n, k = m["heads"] * m["dim"], m["kv_heads"] * m["dim"]
    return {"q": lin(n, W), "k": lin(k, W), "g": lin(n, W), "o": lin(W, n)}


def _feed(att, h, cuts, dtype, page=16, seed=0):
    lb = U.LayerBatch(2, h.shape[0] + page, att.row_width, dtype, page=page, seed=seed)
    lb.hb.step([(1, 3)])                                # another request owns the first page handed out
    outs, at = [], 0
    for n in cuts:
        outs.append(att(h[at:at + n].to(dtype).to(DEV), lb.step([(0, n)])).cpu())
        at += n
    return torch.cat(outs)


TOL = {"core32": 2e-5, "core16": 2e-2, "split": 2e-2, "prompt": 2e-2}


@pytest.mark.parametrize("path,H,G,D,rot,cap,scale", [
    ("core32", 4, 2, 20, 8, 12.0, 0.9), ("core32", 3, 1, 10, 10, None, 0.3), ("core32", 2, 2, 7, 0, 3.0, 1.0),
    ("core32", 10, 1, 34, 2, 50.0, 2.0), ("core16", 6, 2, 48, 16, 20.0, 0.5), ("core16", 5, 5, 12, 12, None, 0.4),
    ("split", 4, 2, 64, 16, 30.0, 0.3), ("split", 8, 1, 128, 128, 9.0, 0.2), ("split", 12, 1, 64, 0, None, 0.2),
    ("prompt", 4, 2, 64, 16, 30.0, 0.3), ("prompt", 8, 1, 128, 64, 50.0, 0.1), ("prompt", 3, 3, 64, 32, 2.0, 0.5),
    ("prompt", 6, 2, 128, 0, 60.0, 1.0), ("prompt", 16, 2, 64, 64, None, 0.15), ("prompt", 2, 1, 64, 8, 200.0, 0.75), ("prompt", 4, 1, 128, 16, 5.0, 0.03)])
def test_tied_attention_prompts_portions_decoding(monkeypatch, path, H, G, D, rot, cap, scale):
    T, W = 210, 48
    _, m = U.att(H, G, D, rot, 700.0, cap, scale)
    w = _att_weights(W, m, 11)
    dtype = PATHS[path]
    h = torch.randn(T, W, generator=torch.Generator().manual_seed(12)).to(dtype)
    want = P.attention_mixer({k: t.double() for k, t in w.items()}, "", m, h.double(), 1e-4)
    att = _layer(monkeypatch, path, W, m, w)
    for cuts in ([T], U.cut(T, [2, 31, 1, 1, 70]), [150] + [1] * 60):
        assert _err(_feed(att, h, cuts, dtype), want) <= TOL[path], cuts[:3]


@pytest.mark.parametrize("path", list(PATHS))
@pytest.mark.parametrize("decode", [False, True])
def test_a_key_that_stands_out(monkeypatch, path, decode):
    """Queries and keys are the inputs themselves; one key points where the query points and its VALUE (the same
    projection, before the norm) is 60 times as long: seen, it decides the output.  Placed at the first token, at
    page, tile and part borders, hundreds of tokens back, right before the query and right after it."""
    T, D, H, query = 420, 64, 2, 400
    _, m = U.att(H, 1, D, 0, 1.0, 40.0, 0.5)
    eye = torch.eye(D)
    w = {"q": eye.repeat(H, 1).bfloat16(), "k": eye.bfloat16(), "g": torch.zeros(H * D, D).bfloat16(),
         "o": torch.cat([eye, eye * 0], 1).bfloat16()}
    base = torch.randn(T, D, generator=torch.Generator().manual_seed(21)).to(PATHS[path])
    att = _layer(monkeypatch, path, D, m, w)
    Wd = {k: t.double() for k, t in w.items()}
    for key in (0, 1, 15, 16, 47, 48, 63, 64, 127, 128, 319, 320, 399, 401, 410):
        h = base.clone()
        h[key] = (h[query].double() * 60.0).to(h.dtype)
        cuts = [390] + [1] * 30 if decode else ([T] if key % 2 else [130, 290])
        got = _feed(att, h, cuts, PATHS[path])[query]
        want = P.attention_mixer(Wd, "", m, h.double(), 1e-4)[query]
        assert _err(got, want) <= TOL[path], key
        assert (got.abs().max() > 20 * base[query].abs().max() / 2) == (key < query), key


def test_unit_norm_hides_the_length_of_a_key_from_the_scores_only():
    """Scaling one token's key projection leaves the weights alone and scales its value."""
    _, m = U.att(1, 1, 6, 4, 50.0, None, 1.0)
    g = torch.Generator().manual_seed(3)
    raw = torch.randn(9, 1, 6, generator=g).double()
    q = P.unit_rms(torch.randn(9, 1, 6, generator=g).double(), 1e-12)
    long = raw.clone()
    long[4] *= 100.0
    a = P.causal_attention(q, P.unit_rms(raw, 1e-12), raw, 1.0, None)
    b = P.causal_attention(q, P.unit_rms(long, 1e-12), raw, 1.0, None)
    assert torch.allclose(a, b) and not torch.allclose(a, P.causal_attention(q, P.unit_rms(long, 1e-12), long, 1.0, None))


def test_preparation_far_from_the_start(monkeypatch):
    """Rotation and unit norm of queries and keys, and the untouched values, at positions beyond 70000."""
    from sglang_security_b200 import _lib

    n, first, H, G = 5, 70000, 3, 2
    for D, dims, dtype in ((10, 6, torch.float32), (64, 16, torch.bfloat16), (128, 128, torch.bfloat16),
                           (64, 0, torch.float16), (256, 64, torch.bfloat16)):
        g = torch.Generator().manual_seed(41)
        y = torch.randn(n, (H + G) * D, generator=g).to(dtype)
        pos = torch.arange(first, first + n, dtype=torch.int32)
        loc = torch.tensor([9, 3, 4, 0, 7], dtype=torch.int64, device=DEV)
        pool = torch.zeros((12, 2 * G * D), device=DEV, dtype=dtype)
        f = torch.tensor([3e5 ** (-2.0 * i / max(dims, 1)) for i in range(dims // 2)], dtype=torch.float64)
        hi = f.float()
        yd, hid, lod, posd = y.to(DEV), hi.to(DEV), (f - hi.double()).float().to(DEV), pos.to(DEV)
        q32 = torch.empty((n, H * D), device=DEV)
        q16 = torch.empty((n, H * D), device=DEV, dtype=dtype)
        k = yd[:, H * D:]
        rc = _lib.load().b200_qk_norm_rope_write(
            yd.data_ptr(), yd.stride(0), k.data_ptr(), k.stride(0), k.data_ptr(), k.stride(0), None, None, D, D, 1e-3,
            hid.data_ptr() if dims else None, lod.data_ptr() if dims else None, dims, posd.data_ptr(), loc.data_ptr(),
            pool.data_ptr(), pool.stride(0), 0, G * D, q32.data_ptr(), q32.stride(0), q16.data_ptr(), q16.stride(0), n, H,
            G, D, D, _lib.dtype_code(dtype), 0)
        _lib.check(rc, "prep")
        unit = lambda x, heads: P.unit_rms(P.rotate_neighbours(x.double().view(n, heads, D), pos, dims, 3e5), 1e-3)
        tol = 3e-6 if dtype == torch.float32 else 8e-3
        assert _err(q32, unit(y[:, :H * D], H).reshape(n, -1)) <= 3e-6
        assert _err(q16, unit(y[:, :H * D], H).reshape(n, -1)) <= tol
        assert _err(pool[loc][:, :G * D], unit(y[:, H * D:], G).reshape(n, -1)) <= tol
        assert torch.equal(pool[loc][:, G * D:].cpu(), y[:, H * D:])


# ---- the residual launch with all of its terms ---------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16, torch.float16])
@pytest.mark.parametrize("width", [8, 40, 333, 1030, 2048, 3000, 8200])
def test_residual_launch_terms(dtype, width):
    from sglang_security_b200.layers.residual_norm import AddNormed

    g = torch.Generator().manual_seed(1)
    T, top, E, eps = 5, 3, 4, 1e-3
    r = lambda *s: torch.randn(*s, generator=g)
    x, b, same, table = r(T, width), r(T, width).to(dtype), r(T, width).to(dtype), r(9, width).to(dtype)
    rows, wts, gate = r(T * top, width).to(dtype), r(T, top).abs(), torch.rand(T, generator=g)
    ids = torch.tensor([[0, 5, 3], [4, 6, 5], [1, 2, 0], [3, 4, 2], [6, 0, 1]], dtype=torch.int32)
    rows.view(T, top, width)[ids >= E] = float("nan")              # rows of identity experts are never written
    tok = torch.tensor([8, 0, 3, 3, 1])
    mod = AddNormed(width, eps, mult=0.3).to(DEV)
    mod.weight.data.copy_(1 + 0.3 * r(width))
    nw = 1 + 0.3 * r(width)
    w = mod.weight.double().cpu()
    terms = rows.double().view(T, top, width).clone()
    terms[ids >= E] = 0.0
    own = (ids >= E).double() * wts.double()
    y = gate.double()[:, None] * b.double() + (wts.double()[..., None] * terms).sum(1) + own.sum(1, keepdim=True) * same.double()
    d = lambda t: t.to(DEV)
    for inject in (False, True):
        want = x.double() + 0.3 * P.unit_rms(y, eps) * w + (table[tok].double() if inject else 0.0)
        xs = d(x.clone())
        h = mod(xs, b=d(b), b_gate=d(gate), rows=d(rows), top=top, row_weights=d(wts), row_ids=d(ids), experts=E,
                same=d(same), out_dtype=dtype, next_weight=d(nw), inject=(d(table), d(tok)) if inject else None)
        assert _err(xs, want) <= 3e-6
        assert _err(h, P.unit_rms(want, eps) * nw.double()) <= (3e-6 if dtype == torch.float32 else 8e-3)


# ---- router, identity experts, shared expert -----------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("E,ident,top,scale,T,push", [(5, 3, 3, 1.6, 40, 0.0), (3, 1, 4, 0.7, 9, 0.0), (4, 0, 1, 1.0, 150, 0.0),
                                                      (6, 6, 5, 2.5, 33, 0.3), (2, 5, 3, 1.0, 17, 9.0),
                                                      (7, 2, 2, 3.0, 64, -9.0), (40, 9, 8, 1.0, 20, 0.0), (1, 1, 1, 1.0, 3, 0.0)])
def test_router_with_identity_experts_and_gated_shared_expert(dtype, E, ident, top, scale, T, push):
    """push: a correction on the identity experts, so that they are chosen now and then, always, or never."""
    from sglang_security_b200.configs.sapivik import IdentityExpertsSpec
    from sglang_security_b200.layers.residual_norm import AddNormed
    from sglang_security_b200.models.sapivik import SapivikExperts

    W = 40
    mlp = U.moe(E, ident, top, scale, 24, 16 if E != 4 else None)
    w = U.random_weights(U.config([(U.mem(), mlp)], width=W), 6)
    w = {k[7:]: t for k, t in w.items() if k.startswith("l0.mlp.")}
    w["correction"][E:] += push
    ex = SapivikExperts(W, IdentityExpertsSpec(E, ident, top, scale, 24, 16 if E != 4 else 0), dtype).to(DEV)
    ex.router.weight.data.copy_(w["router"])
    ex.router.correction.data.copy_(w["correction"])
    for e in range(E):
        ex.experts.load_expert(e, w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"])
    if ex.shared is not None:
        ex.shared.load(w["shared.gate"].to(DEV), w["shared.up"].to(DEV), w["shared.down"].to(DEV))
        ex.router.shared_gate.data.copy_(w["shared.sg"][0])
    h = torch.randn(T, W, generator=torch.Generator().manual_seed(8)).to(dtype)
    Wd = {k: t.double() for k, t in w.items()}
    terms = ex(h.to(DEV))
    ids, wts, _ = ex.router.route(h.to(DEV))
    for t in range(T):
        oid, owt = P.route(h[t].double() @ Wd["router"].T, Wd["correction"], top, scale)
        assert sorted(ids[t].tolist()) == sorted(oid)
        assert dict(zip(ids[t].tolist(), wts[t].tolist())) == pytest.approx(dict(zip(oid, owt)), rel=1e-4, abs=1e-6)
    chosen = (ids >= E).float().mean().item()
    if push > 1 and top <= ident:
        assert chosen == 1.0                                        # every choice returns the input
    if push < -1:
        assert chosen == 0.0
    mod = AddNormed(W, 1e-6).to(DEV)
    x = torch.zeros(T, W, device=DEV)
    mod(x, **terms)
    want = P.unit_rms(P.expert_ff(Wd, "", mlp, h.double()), 1e-6)
    assert _err(x, want) <= (1e-5 if dtype == torch.float32 else 3e-2)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("limit", [0.4, 7.0])
def test_clamped_feed_forward(dtype, limit):
    from sglang_security_b200.layers.gated_mlp import GatedMLP

    cfg = U.config([(U.mem(), U.dense(48, limit))])
    w = {k[7:]: t for k, t in U.random_weights(cfg, 2).items() if k.startswith("l0.mlp.")}
    mlp = GatedMLP(40, 48, "clamped", dtype, limit=limit).to(DEV)
    mlp.load(*(w[k].to(DEV) for k in ("gate", "up", "down")))
    h = torch.randn(30, 40, generator=torch.Generator().manual_seed(9)).to(dtype)
    want = P.clamped_ff({k: t.double() for k, t in w.items()}, "", limit, h.double())
    assert _err(mlp(h.to(DEV)), want) <= (1e-5 if dtype == torch.float32 else 2e-2)
