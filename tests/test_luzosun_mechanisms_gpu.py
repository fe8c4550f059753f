"""Luzosun mechanisms one by one on the GPU against the plain float64 restatement: residual sum + two norms +
input convolution, projection convolution + rotation + cache write (both with carried inputs, portions down to
one token, stale and reused state rows), differential attention on its three kernels (chunks, windows, edges
with a key that stands out), the xIELU activation in rows and in the GEMM epilogue, the joint output matrix."""
import pytest
import torch

import luzosun_plain as P
import luzosun_util as U
from sglang_security_b200 import _lib

pytestmark = pytest.mark.gpu
DEV = "cuda"
F64 = torch.float64


def _gen(seed):
    return torch.Generator().manual_seed(seed)


def _walk(hb, seqs, sizes, run):
    """Feeds the sequences {row: [T, C] tensor} in unequal portions; run(fb, entries, at) -> rows per token."""
    got, at, step = {r: [] for r in seqs}, {r: 0 for r in seqs}, 0
    while any(at[r] < len(seqs[r]) for r in seqs):
        entries = [(r, min(sizes[(step + r) % len(sizes)], len(seqs[r]) - at[r])) for r in seqs if at[r] < len(seqs[r])]
        fb = hb.step(entries)
        fb.extend_seq_lens_cpu = [n for _, n in entries]
        y, o = run(fb, entries, at), 0
        for r, n in entries:
            got[r].append([t[o:o + n].double().cpu() for t in y])
            o += n
            at[r] += n
        step += 1
    return {r: [torch.cat(ts) for ts in zip(*got[r])] for r in seqs}


# ---- residual sum, two norms, input convolution ---------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width, taps", [(40, 3), (300, 4), (27, 2), (1030, 7), (64, 0), (36, 1), (8, 12)])
@pytest.mark.parametrize("sizes", [[1, 3, 2, 1, 40, 5, 17], [16, 33, 2]])
def test_residual_norms_and_input_convolution(dtype, width, taps, sizes):
    from sglang_security_b200.layers.residual_conv import ResidualNormConv

    g, eps = _gen(1), 1e-3
    m = ResidualNormConv(width, eps, taps).to(DEV)
    w1, w2 = 1 + 0.3 * torch.randn(width, generator=g), 1 + 0.3 * torch.randn(width, generator=g)
    cw = 0.6 * torch.randn(width, taps, generator=g)
    m.weight1.data.copy_(w1)
    m.weight2.data.copy_(w2)
    if taps:
        m.load_conv(cw)
    lens = {0: 120, 1: 61, 2: 9}
    xs = {r: torch.randn(n, width, generator=g) for r, n in lens.items()}
    aa = {r: torch.randn(n, width, generator=g).to(dtype) for r, n in lens.items()}
    state = torch.full((3, max(m.state_width, 1) + 8), 7.0, device=DEV)          # stale values everywhere
    hb = U.HandBatch(3, 160)

    def run(fb, entries, at):
        x, a = (torch.cat([s[r][at[r]:at[r] + n] for r, n in entries]).to(DEV) for s in (xs, aa))
        x_out = torch.full_like(x, 5.0)
        h, n2 = m(x, x_out, a, fb, state[:, 4:] if m.state_width else None, dtype)
        return x_out, h, n2

    def want(x):
        h = P.rms_norm(x, w1.double(), eps)
        return h + P.causal_conv(h, cw.double()) if taps else h

    got = _walk(hb, xs, sizes, run)
    tol = 2e-5 if dtype == torch.float32 else 8e-3                               # relative: rounded to 16 bits
    for r in xs:
        x = xs[r].double() + aa[r].double()
        assert (got[r][0] - x).abs().max() < 1e-6
        for y, ref in ((got[r][1], want(x)), (got[r][2], P.rms_norm(x, w2.double(), eps))):
            assert ((y - ref).abs() / (1 + ref.abs())).max() < tol, r
    hb.release(1)                                    # a reused row: the new sequence starts from zeros
    xs, aa = {1: torch.randn(20, width, generator=g)}, {1: torch.zeros(20, width, dtype=dtype)}
    got = _walk(hb, xs, [1, 2, 17], run)
    ref = want(xs[1].double())
    assert ((got[1][1] - ref).abs() / (1 + ref.abs())).max() < tol


# ---- projection convolution, rotation, cache write -------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,E,rot,taps,own", [(4, 2, 12, 20, 8, 3, True), (3, 1, 7, 5, 6, 2, True), (2, 2, 16, 8, 0, 4, True),
                                                  (6, 2, 32, 64, 32, 4, True), (2, 1, 8, 6, 8, 0, True), (4, 2, 12, 20, 8, 3, False),
                                                  (1, 1, 4, 4, 2, 9, True), (2, 1, 8, 12, 4, 1, True)])
def test_projection_convolution_rotation_and_cache(dtype, H, G, D, E, rot, taps, own):
    g, base, factor, far = _gen(2), 5000.0, 1.7, 40000
    C = H * 2 * D + (G * 2 * D + G * E if own else 0)
    cw = 0.6 * torch.randn(C, taps, generator=g)
    lens = {0: 90, 1: 21, 2: 5}
    ys = {r: torch.randn(n, C, generator=g).to(dtype) for r, n in lens.items()}
    f = torch.tensor([base ** (-2.0 * i / rot) / factor for i in range(rot // 2)], dtype=F64)
    hi = f.float()
    lo, cwt = (f - hi.double()).float().to(DEV), cw.t().contiguous().to(DEV)
    hi = hi.to(DEV)
    state = torch.full((3, max(taps - 1, 0) * C + 4), 7.0, device=DEV)
    hb = U.HandBatch(3, far + 160)
    # row 2 continues a sequence that is already long: what it carries is set by hand
    before = torch.randn(max(taps - 1, 1), C, generator=g)
    hb.lens[2] = far
    if taps > 1:
        state[2, :(taps - 1) * C] = before[:taps - 1].reshape(-1).to(DEV)
    pool = torch.full((hb.pool_rows, G * (2 * D + E) + 4), 3.0, dtype=dtype, device=DEV)
    lib, code = _lib.load(), _lib.dtype_code(dtype)
    pos_of = {0: 0, 1: 0, 2: far}

    def run(fb, entries, at):
        y = torch.cat([ys[r][at[r]:at[r] + n] for r, n in entries]).to(DEV)
        T = y.shape[0]
        q32 = torch.empty((T, H * 2 * D), device=DEV)
        q16 = torch.empty((T, H * 2 * D), dtype=dtype, device=DEV)
        rc = lib.b200_conv_rot_write(
            y.data_ptr(), y.stride(0), cwt.data_ptr() if taps else None, max(taps, 1), state.data_ptr(), state.stride(0),
            fb.req_pool_indices.data_ptr(), fb.tok_pos.data_ptr(), fb.ext_start.data_ptr(), fb.ext_len.data_ptr(),
            hi.data_ptr(), lo.data_ptr(), rot, fb.out_cache_loc.data_ptr(), pool.data_ptr(), pool.stride(0), 4, 4 + G * 2 * D,
            q32.data_ptr(), q32.stride(0), q16.data_ptr(), q16.stride(0), 2 * H, 2 * G if own else 0, D, G * E if own else 0,
            len(entries), max(n for _, n in entries), code, 0)
        _lib.check(rc, "b200_conv_rot_write")
        torch.cuda.synchronize()
        return q32, q16, pool[fb.out_cache_loc]

    got = _walk(hb, ys, [1, 3, 2, 1, 37, 5], run)
    for r, y in ys.items():
        u = y.double()
        if r == 2 and taps > 1:
            u = torch.cat([before[:taps - 1].double(), u])
        z = P.causal_conv(u, cw.double())[-len(y):] if taps else u
        pos = pos_of[r] + torch.arange(len(y))
        maps = P.rotate_halves(z[:, :(2 * H + (2 * G if own else 0)) * D].reshape(len(y), -1, D), pos, rot, base, factor).reshape(len(y), -1)
        q, k, v = maps[:, :2 * H * D], maps[:, 2 * H * D:], z[:, maps.shape[1]:]
        assert (got[r][0] - q).abs().max() < 3e-5, r
        tol = 3e-5 if dtype == torch.float32 else 1e-2
        assert ((got[r][1] - q).abs() / (1 + q.abs())).max() < tol
        row = got[r][2]
        if own:
            assert ((row[:, 4:4 + G * 2 * D] - k).abs() / (1 + k.abs())).max() < tol
            assert ((row[:, 4 + G * 2 * D:] - v).abs() / (1 + v.abs())).max() < tol
            assert (row[:, :4] == 3).all()
        else:
            assert (row == 3).all()                  # a layer without keys of its own leaves the rows alone


# ---- differential attention ------------------------------------------------------------------------
def _attend(q, k, v, lam, mult, scale, cuts, dtype, kernel, window=0, chunk=0, page=16, seed=0, eps=1e-5, splits=None):
    """One sequence, q [T, H, 2, D], k [T, G, 2, D], v [T, G, E], in portions `cuts` through one kernel
    ("core", "mma" or "extend"); the pool rows of the sequence are written by hand on shuffled pages."""
    T, H, _, D = q.shape
    G, E = v.shape[1], v.shape[2]
    hb = U.HandBatch(2, T + page, page=page, seed=seed)
    hb.step([(1, 3)])                                   # another request owns the first pages handed out
    pool = torch.full((hb.pool_rows, G * (2 * D + E)), 3.0, dtype=dtype, device=DEV)
    pool[0] = 0
    lib, code, lam_d = _lib.load(), _lib.dtype_code(dtype), torch.tensor([lam], device=DEV)
    outs, at, tail = [], 0, 8                           # the result is a column slice of wider rows
    for n in cuts:
        fb = hb.step([(0, n)])
        pool[fb.out_cache_loc] = torch.cat([k[at:at + n].reshape(n, -1), v[at:at + n].reshape(n, -1)], 1).to(dtype).to(DEV)
        qq = q[at:at + n].reshape(n, -1).to(torch.float32 if kernel == "core" else dtype).to(DEV)
        buf = torch.full((n, H * E + tail), 9.0, dtype=dtype, device=DEV)
        out = buf[:, :H * E]
        base = (qq.data_ptr(), qq.stride(0), pool.data_ptr(), pool.stride(0), 0, G * 2 * D)
        table = (fb.req_to_token.data_ptr(), fb.req_to_token.stride(0), fb.req_pool_indices.data_ptr())
        if kernel == "extend":
            i32 = [torch.tensor([x], dtype=torch.int32, device=DEV) for x in (at, n, 0)]
            rc = lib.b200_diff_attn_extend(*base, out.data_ptr(), out.stride(0), *table, *(t.data_ptr() for t in i32), 1, n,
                                           H, G, D, E, scale, window, chunk, lam_d.data_ptr(), mult, eps, code, 0)
        else:
            args = (*base, *table, fb.tok_pos.data_ptr(), fb.tok_b.data_ptr(), None, lam_d.data_ptr(), mult, eps, scale,
                    window, chunk, out.data_ptr(), out.stride(0), n, H, G, D, E)
            if kernel == "core":
                rc = lib.b200_diff_attn(*args, at + n if seed % 2 == 0 else 0, code, 0)
            else:
                ns = splits or lib.b200_diff_attn_mma_splits(n, H, G, at + n, 148)
                po = torch.empty(n * H * 2 * ns * E, device=DEV)
                pl = torch.empty(n * H * 2 * ns, device=DEV)
                rc = lib.b200_diff_attn_mma(*args, ns, po.data_ptr(), pl.data_ptr(), code, 0)
        _lib.check(rc, kernel)
        torch.cuda.synchronize()
        assert lib.b200_diff_attn_extend_error() == 0
        assert (buf[:, H * E:] == 9).all()
        outs.append(out.double().cpu())
        at += n
    return torch.cat(outs).view(T, H, E)


def _plain(q, k, v, lam, mult, scale, window=0, chunk=0, eps=1e-5):
    T, H, _, D = q.shape
    G, E = v.shape[1], v.shape[2]
    mask = P.visible(T, chunk)
    if window:
        i = torch.arange(T)
        mask &= i[None, :] > i[:, None] - window
    out = torch.zeros(T, H, E, dtype=F64)
    for h in range(H):
        g = h // (H // G)
        a = [P.softmax_map(q[:, h, m], k[:, g, m], v[:, g], scale, mask) for m in (0, 1)]
        out[:, h] = P.combine_maps(a[0], a[1], lam, 1.0 - mult, eps)
    return out


def _qkv(T, H, G, D, E, seed, dtype):
    g = _gen(seed)
    r = lambda *s: torch.randn(*s, generator=g).to(dtype).double()
    return r(T, H, 2, D), r(T, G, 2, D), r(T, G, E)


def _err(got, want):
    return float((got - want).abs().max() / want.abs().max())


TOL = {torch.float32: 3e-5, torch.bfloat16: 3e-2}


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,E,window,chunk", [(4, 2, 12, 20, 0, 40), (3, 1, 7, 5, 0, 1), (2, 2, 16, 130, 9, 0),
                                                  (6, 2, 32, 64, 0, 0), (1, 1, 8, 8, 1, 0), (10, 2, 5, 33, 0, 150),
                                                  (5, 1, 64, 100, 0, 33)])
def test_differential_attention_on_cuda_cores(dtype, H, G, D, E, window, chunk):
    T = 150
    q, k, v = _qkv(T, H, G, D, E, 11, dtype)
    want = _plain(q, k, v, 0.7, 0.6, D ** -0.5, window, chunk)
    for i, cuts in enumerate(([T], U.cut(T, [2, 31, 1, 1, 17]), [100] + [1] * 50)):
        got = _attend(q, k, v, 0.7, 0.6, D ** -0.5, cuts, dtype, "core", window, chunk, seed=i)
        assert _err(got, want) <= TOL[dtype], cuts[:3]


SIZES = [(8, 2, 32, 64), (8, 1, 64, 128), (2, 2, 32, 128), (12, 1, 64, 64), (3, 1, 128, 128), (6, 2, 64, 128), (1, 1, 32, 64)]


@pytest.mark.parametrize("H,G,D,E", SIZES)
@pytest.mark.parametrize("window,chunk", [(0, 0), (0, 100), (50, 0), (0, 64), (0, 7)])
def test_differential_attention_on_the_split_kernel(H, G, D, E, window, chunk):
    """Decoded tokens and short portions (mma.sync); several split counts, also more than there are keys for."""
    T = 330
    q, k, v = _qkv(T, H, G, D, E, 12, torch.bfloat16)
    want = _plain(q, k, v, 0.7, 0.6, D ** -0.5, window, chunk)
    for cuts, ns in (([T], 1), ([200, 1, 2, 127], 3), ([300] + [1] * 30, None)):
        got = _attend(q, k, v, 0.7, 0.6, D ** -0.5, cuts, torch.bfloat16, "mma", window, chunk, splits=ns)
        assert _err(got, want) <= TOL[torch.bfloat16], (cuts[:3], ns)


@pytest.mark.parametrize("H,G,D,E", SIZES)
@pytest.mark.parametrize("window,chunk", [(0, 0), (0, 100), (50, 0), (0, 64), (0, 7), (0, 333)])
def test_differential_attention_on_the_prompt_kernel(H, G, D, E, window, chunk):
    """Prompt portions on tcgen05: tiles that start in the middle of a chunk, portions that end mid-tile."""
    T = 450
    q, k, v = _qkv(T, H, G, D, E, 13, torch.bfloat16)
    want = _plain(q, k, v, 0.7, 0.6, D ** -0.5, window, chunk)
    for cuts in ([T], [200, 130, 1, 119], [63, 64, 65, 258]):
        got = _attend(q, k, v, 0.7, 0.6, D ** -0.5, cuts, torch.bfloat16, "extend", window, chunk)
        assert _err(got, want) <= TOL[torch.bfloat16], cuts


@pytest.mark.parametrize("kernel", ["core", "mma", "extend"])
def test_large_scores_need_the_running_maximum(kernel):
    """Scores that grow along the sequence by far more than the rescale threshold."""
    T, H, G, D, E = 400, 2, 1, 32, 64
    q, k, v = _qkv(T, H, G, D, E, 14, torch.bfloat16)
    k = (k * torch.linspace(0.2, 12.0, T, dtype=F64)[:, None, None, None]).bfloat16().double()
    want = _plain(q, k, v, 0.5, 0.6, 0.5)
    got = _attend(q, k, v, 0.5, 0.6, 0.5, [T], torch.bfloat16, kernel)
    assert _err(got, want) <= 4e-2


@pytest.mark.parametrize("kernel", ["core", "mma", "extend"])
@pytest.mark.parametrize("which", [0, 1])
@pytest.mark.parametrize("decode", [False, True])
def test_chunk_and_window_edges_with_a_key_that_stands_out(kernel, which, decode):
    """One map's key gets a score far above the rest and a value no other key has: whether it is seen decides
    the direction of the output.  Chunks of 100 over positions 0 .. 400, query 399 / 300: the first key of
    the chunk, the one before it, page and tile borders, the very first token, the query itself."""
    T, H, G, D, E = 400, 2, 1, 32, 64
    base = _qkv(T, H, G, D, E, 15, torch.bfloat16)
    cases = [(399, 0, 100, 300, True), (399, 0, 100, 299, False), (399, 0, 100, 0, False), (399, 0, 100, 383, True),
             (399, 0, 100, 399, True), (300, 0, 100, 300, True), (300, 0, 100, 299, False), (299, 0, 100, 200, True),
             (299, 0, 100, 199, False), (399, 37, 0, 363, True), (399, 37, 0, 362, False), (399, 0, 0, 0, True),
             (399, 0, 0, 64, True), (128, 0, 64, 128, True), (128, 0, 64, 127, False), (127, 0, 64, 64, True)]
    for query, window, chunk, key, seen in cases:
        q, k, v = (t.clone() for t in base)
        k *= 0.1
        k[key, 0, which] = q[query, 0, which] / q[query, 0, which].norm() * 40.0
        v[key, 0] = 0.0
        v[key, 0, 5] = 200.0
        k, v = k.bfloat16().double(), v.bfloat16().double()
        cuts = [query - 2, 1, 1, 1] + ([T - query - 1] if query + 1 < T else []) if decode else [T]
        got = _attend(q, k, v, 0.8, 0.6, 1.0, cuts, torch.bfloat16, kernel, window, chunk)[query, 0]
        want = _plain(q, k, v, 0.8, 0.6, 1.0, window, chunk)[query, 0]
        assert _err(got, want) <= 4e-2, (query, key)
        # the value's direction dominates the normed output exactly when the key is seen
        dominant = int(got.abs().argmax()) == 5 and got.abs()[5] > 0.95 * got.norm()
        assert dominant == seen, (query, window, chunk, key)
        first = query // chunk * chunk if chunk else (max(0, query - window + 1) if window else 0)
        if seen and query - first > 10:              # among many keys the maps enter with opposite signs
            assert (got[5] > 0) == (which == 0)


def test_second_map_enters_with_its_weight():
    T, H, G, D, E = 60, 2, 1, 16, 24
    q, k, v = _qkv(T, H, G, D, E, 16, torch.float32)
    for lam in (0.0, 1.0, -0.5):
        want = _plain(q, k, v, lam, 0.25, 0.3)
        assert _err(_attend(q, k, v, lam, 0.25, 0.3, [T], torch.float32, "core"), want) <= TOL[torch.float32]
    # equal maps with weight one cancel: eps alone keeps the result finite
    q[:, :, 1], k[:, :, 1] = q[:, :, 0], k[:, :, 0]
    got = _attend(q, k, v, 1.0, 0.25, 0.3, [T], torch.float32, "core")
    assert torch.isfinite(got).all() and got.abs().max() < 1e-2


def test_token_list_restricts_a_launch():
    """Rows that another kernel serves are left alone."""
    T, H, G, D, E = 40, 2, 1, 32, 64
    q, k, v = _qkv(T, H, G, D, E, 17, torch.bfloat16)
    want = _plain(q, k, v, 0.7, 0.6, 0.2)
    hb = U.HandBatch(1, 64)
    fb = hb.step([(0, T)])
    pool = torch.zeros((hb.pool_rows, G * (2 * D + E)), dtype=torch.bfloat16, device=DEV)
    pool[fb.out_cache_loc] = torch.cat([k.reshape(T, -1), v.reshape(T, -1)], 1).bfloat16().to(DEV)
    some = torch.tensor([3, 17, 39], dtype=torch.int32, device=DEV)
    lam, lib = torch.tensor([0.7], device=DEV), _lib.load()
    for kernel in ("core", "mma"):
        qq = q.reshape(T, -1).to(torch.float32 if kernel == "core" else torch.bfloat16).to(DEV)
        out = torch.full((T, H * E), 9.0, dtype=torch.bfloat16, device=DEV)
        args = (qq.data_ptr(), qq.stride(0), pool.data_ptr(), pool.stride(0), 0, G * 2 * D, fb.req_to_token.data_ptr(),
                fb.req_to_token.stride(0), fb.req_pool_indices.data_ptr(), fb.tok_pos.data_ptr(), fb.tok_b.data_ptr(),
                some.data_ptr(), lam.data_ptr(), 0.6, 1e-5, 0.2, 0, 0, out.data_ptr(), out.stride(0), 3, H, G, D, E)
        if kernel == "core":
            _lib.check(lib.b200_diff_attn(*args, T, 0, 0), kernel)
        else:
            po, pl = torch.empty(3 * H * 2 * 2 * E, device=DEV), torch.empty(3 * H * 2 * 2, device=DEV)
            _lib.check(lib.b200_diff_attn_mma(*args, 2, po.data_ptr(), pl.data_ptr(), 0, 0), kernel)
        got = out.double().cpu().view(T, H, E)
        assert _err(got[[3, 17, 39]], want[[3, 17, 39]]) <= 3e-2
        rest = [i for i in range(T) if i not in (3, 17, 39)]
        assert (got[rest] == 9).all()


# ---- activation and joint output -------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_activation_rows(dtype):
    from sglang_security_b200.layers.residual_conv import UngatedMLP

    z = torch.cat([3 * torch.randn(5, 333, generator=_gen(21)), torch.logspace(-7, 1, 333).repeat(2, 1),
                   -torch.logspace(-7, 1.5, 333).repeat(2, 1)]).to(dtype)
    m = UngatedMLP(8, 8)
    m.load_act(0.9, -1.3)
    wide = torch.full((z.shape[0], 400), 9.0, dtype=dtype, device=DEV)
    out = wide[:, 11:344]
    zd = z.to(DEV)
    _lib.check(_lib.load().b200_xielu_rows(zd.data_ptr(), zd.stride(0), out.data_ptr(), out.stride(0), z.shape[0], 333,
                                           m.pos, m.neg, _lib.dtype_code(dtype), 0), "xielu")
    want = P.xielu(z.double(), 0.9, -1.3)
    assert ((out.double().cpu() - want).abs() / (want.abs() + 0.1 * z.double().abs() + 1e-9)).max() < (2e-5 if dtype == torch.float32 else 6e-3)
    assert (wide[:, :11] == 9).all() and (wide[:, 344:] == 9).all()


@pytest.mark.parametrize("tokens, width, ff", [(1, 64, 96), (33, 256, 520), (300, 128, 4096), (2000, 256, 2048), (7, 36, 50)])
def test_activation_in_the_projection(tokens, width, ff):
    """The GEMM epilogue (any tile and split count) and, where rows are not 16-byte multiples, the row kernel."""
    from sglang_security_b200.layers.residual_conv import JointOutput, UngatedMLP

    g = _gen(22)
    m = UngatedMLP(width, ff).to(DEV)
    m.load_act(-0.4, 0.6)
    h = torch.randn(tokens, width, generator=g).bfloat16()
    w = (torch.randn(ff, width, generator=g) * 1.5 / width ** 0.5).bfloat16()
    m.up_proj.weight.data.copy_(w)
    joint = JointOutput([20, ff], 24, torch.bfloat16).to(DEV)
    wo, wd = (torch.randn(24, n, generator=g) / n ** 0.5 for n in (20, ff))
    joint.load_part(0, wo.bfloat16())
    joint.load_part(1, wd.bfloat16())
    buf = joint.buffer(tokens, DEV)
    left = torch.randn(tokens, 20, generator=g).bfloat16()
    joint.view(buf, 0).copy_(left)
    m(h.to(DEV), joint.view(buf, 1))
    want = P.xielu(h.double() @ w.double().T, -0.4, 0.6)
    got = joint.view(buf, 1).double().cpu()
    assert ((got - want).abs() / (1 + want.abs())).max() < 2e-2
    assert torch.equal(joint.view(buf, 0).cpu(), left)
    y = left.double() @ wo.bfloat16().double().T + got @ wd.bfloat16().double().T
    assert ((joint(buf).double().cpu() - y).abs() / (1 + y.abs())).max() < 1e-2


def test_the_activation_near_zero_keeps_its_relative_accuracy():
    """e^z - 1 - z cancels near zero: the epilogue's series must hold there."""
    from sglang_security_b200.layers.dense_kernel import gemm_16bit

    z = -torch.logspace(-4, 1, 512)
    x = torch.zeros(512, 64, dtype=torch.bfloat16)
    x[:, 0] = z.bfloat16()
    w = torch.zeros(8, 64, dtype=torch.bfloat16)
    w[:, 0] = 1.0
    got = gemm_16bit(x.to(DEV), w.to(DEV), xielu=(0.7, 3.0))[:, 0].double().cpu()
    zz = z.bfloat16().double()
    want = 3.0 * (torch.expm1(zz) - zz) + 0.5 * zz
    assert ((got - want).abs() / (want.abs() + zz.abs() * 1e-2)).max() < 6e-3
