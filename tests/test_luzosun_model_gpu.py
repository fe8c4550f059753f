"""Luzosun through the engine (loader, ModelRunner, pools, scheduler) against the plain restatement: whole
prompts, per-layer residuals, token-by-token decoding, portions down to two tokens, unequal requests in one
batch with pages and request slots freed and used again, chunk edges made visible by a peaked softmax, layers
that share another's keys and values, long decoding, and greedy generation through Engine.generate."""
import pytest
import torch

import luzosun_plain as P
import luzosun_util as U
from sglang_security_b200.layers.attention.differential_attention import DifferentialAttention

pytestmark = pytest.mark.gpu

CONFIGS = {
    # shared keys and values with another chunk, head count, weight and tap count than their owner's
    "a": lambda: U.config([(U.diff(), U.dense()), (U.diff(kv_from=0, heads=6, chunk=24, lam=0.7, conv=2), U.dense(24)),
                           (U.diff(heads=2, kv_heads=2, dim=16, vdim=8, chunk=33, rot_dims=16, factor=None), None),
                           (U.diff(kv_from=0, chunk=None, scale=0.5, rot_dims=8, lam=0.2), U.dense(40))]),
    # sizes that are multiples of nothing, 3 : 1 grouping, unpadded and padded joint matrices
    "b": lambda: U.config([(U.diff(heads=3, kv_heads=1, dim=7, vdim=5, chunk=19, conv=3, rot_dims=6, base=70.0), U.dense(21)),
                           (U.diff(heads=3, kv_heads=3, dim=5, vdim=9, chunk=64, conv=5, rot_dims=2), U.dense(30))],
                          vocab=131, width=27, eps=1e-3, taps=2),
    # ones: one head, chunks of one position, one tap, no taps, no rotation, no feed-forward, embedding scale 1
    "c": lambda: U.config([(U.diff(heads=1, kv_heads=1, dim=4, vdim=4, chunk=1, conv=1, rot_dims=4), None),
                           (U.diff(heads=2, kv_heads=1, dim=8, vdim=6, chunk=None, conv=0, rot_dims=0), None),
                           (U.diff(heads=1, kv_heads=1, dim=2, vdim=3, chunk=50, conv=6, rot_dims=2, factor=1.0, lam=0.0), U.dense(1))],
                          vocab=33, width=24, emb=1.0, taps=1),
    # no input convolution; long taps
    "e": lambda: U.config([(U.diff(conv=9), U.dense()), (U.diff(kv_from=0, conv=3), None)], taps=0),
    # sizes of the tensor-core kernels (map / value size 32 / 64, 64 / 128, 64 / 64, 128 / 128), 4 : 1, 1 : 1, 3 : 1
    "d": lambda: U.config([(U.diff(heads=4, kv_heads=1, dim=32, vdim=64, chunk=70, rot_dims=16), U.dense(64)),
                           (U.diff(heads=2, kv_heads=2, dim=64, vdim=128, chunk=None, rot_dims=64), None),
                           (U.diff(kv_from=0, heads=8, kv_heads=1, dim=32, vdim=64, chunk=128, rot_dims=16), U.dense(48)),
                           (U.diff(heads=3, kv_heads=1, dim=64, vdim=64, chunk=96, rot_dims=32), None),
                           (U.diff(heads=2, kv_heads=1, dim=128, vdim=128, chunk=100, rot_dims=128), U.dense(64))],
                          vocab=101, width=64),
    "g": lambda: U.config([(U.diff(chunk=90), None)], vocab=61, width=48, taps=5),
}


def _model(tmp_path, name, seed=0, sharp=0.0):
    cfg = CONFIGS[name]()
    if sharp:        # a peaked softmax: one key more or less in sight moves the logits a lot
        for L in cfg["layers"]:
            L["mixer"]["scale"] *= sharp
    w = U.random_weights(cfg, seed)
    return cfg, w, U.write_model(str(tmp_path / name), cfg, w)


def _tokens(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


# 16 bits: the norm of the maps' difference carries the rounding of every stored activation to the logits (90th
# percentile, see rel_err); a fault of the cache or the state is of order one
TOL = {torch.float32: 1e-4, torch.bfloat16: 0.12}
SHARP = {torch.float32: 5.0, torch.bfloat16: 2.0}
TOL_SHARP = {torch.float32: 5e-4, torch.bfloat16: 0.25}


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_matches_plain_model(tmp_path, name, dtype):
    cfg, w, folder = _model(tmp_path, name)
    toks = _tokens(cfg, 200, 1)
    want = P.forward(cfg, w, toks)
    d = U.Driver(folder, dtype)
    d.step([("r", toks)], end=["r"])
    assert U.rel_err(d.result("r"), want, dtype) <= TOL[dtype]


@pytest.mark.parametrize("name", ["a", "b", "c", "e"])
def test_layer_outputs_match_plain_model_fp32(tmp_path, name):
    from sglang_security_b200.managers.schedule_batch import Req, StepItem

    cfg, w, folder = _model(tmp_path, name)
    toks = _tokens(cfg, 50, 2)
    want = []
    P.forward(cfg, w, toks, layers_out=want)
    d = U.Driver(folder, torch.float32)
    req = Req(rid="x", input_ids=list(toks))
    d.runner.admit(req)
    got = []
    d.sched.run_step([StepItem(req, list(toks), want=[0])], layer_hook=lambda i, x: got.append(x.double().cpu().clone()))
    assert len(got) == len(want)
    for g, t in zip(got, want):
        assert (g - t).abs().max() <= 2e-5 * t.abs().max()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", ["a", "b", "c", "d", "e"])
def test_prefill_then_token_by_token(tmp_path, name, dtype):
    cfg, w, folder = _model(tmp_path, name, sharp=SHARP[dtype])
    toks = _tokens(cfg, 150, 3)
    want = P.forward(cfg, w, toks)
    d = U.Driver(folder, dtype)
    d.step([("r", toks[:60])])
    for t in toks[60:]:
        d.step([("r", [t])])
    assert U.rel_err(d.result("r"), want, dtype) <= TOL_SHARP[dtype]
    d2 = U.Driver(folder, dtype)                 # from the very first token on, one at a time
    for t in toks[:45]:
        d2.step([("s", [t])])
    assert U.rel_err(d2.result("s"), want[:45], dtype) <= TOL_SHARP[dtype]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("sizes", [[2], [3, 64, 2, 17, 1], [64, 5]])
@pytest.mark.parametrize("name", ["a", "d"])
def test_portions_of_a_prompt(tmp_path, name, dtype, sizes):
    cfg, w, folder = _model(tmp_path, name, sharp=SHARP[dtype])
    toks = _tokens(cfg, 150, 4)
    want = P.forward(cfg, w, toks)
    d = U.Driver(folder, dtype)
    at = 0
    for n in U.cut(len(toks), sizes):
        d.step([("r", toks[at:at + n])])
        at += n
    assert U.rel_err(d.result("r"), want, dtype) <= TOL_SHARP[dtype]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", ["a", "b", "d", "g"])
def test_unequal_requests_in_one_batch_with_slots_and_pages_reused(tmp_path, name, dtype):
    cfg, w, folder = _model(tmp_path, name)
    lens = {"p": 150, "q": 37, "r": 90, "s": 1, "t": 64, "u": 129, "v": 20}
    toks = {k: _tokens(cfg, n, 10 + i) for i, (k, n) in enumerate(lens.items())}
    want = {k: P.forward(cfg, w, t) for k, t in toks.items()}
    d = U.Driver(folder, dtype, max_tokens=512, max_requests=3)      # fewer slots and pages than requests need
    at = {k: 0 for k in lens}
    waiting, live, sizes, step = list(lens), [], [33, 1, 2, 64, 1, 7], 0
    while waiting or live:
        while waiting and len(live) < 3 and sum(-(-lens[k] // 64) for k in live + [waiting[0]]) <= 8:
            live.append(waiting.pop(0))
        portions, ended = [], []
        for j, k in enumerate(live):
            n = min(sizes[(step + j) % len(sizes)], lens[k] - at[k])
            portions.append((k, toks[k][at[k]:at[k] + n]))
            at[k] += n
            if at[k] == lens[k]:
                ended.append(k)
        d.step(portions, end=ended)
        live = [k for k in live if k not in ended]
        step += 1
    for k in lens:
        assert U.rel_err(d.result(k), want[k], dtype) <= TOL[dtype], k
    assert d.runner.free_token_slots() == d.runner.max_total_tokens


def test_batch_does_not_change_a_request_fp32(tmp_path):
    cfg, w, folder = _model(tmp_path, "a")
    a, b = _tokens(cfg, 80, 20), _tokens(cfg, 45, 21)
    alone = U.Driver(folder, torch.float32)
    alone.step([("a", a)], end=["a"])
    both = U.Driver(folder, torch.float32)
    both.step([("b", b[:30]), ("a", a[:50])])
    both.step([("a", a[50:]), ("b", b[30:31])])
    assert (alone.result("a") - both.result("a")).abs().max() <= 1e-4


@pytest.mark.parametrize("sharp", [0.0, 2.0])
def test_long_portions_on_the_prompt_kernel_beside_decoded_tokens(tmp_path, monkeypatch, sharp):
    """Portions of 16 tokens and more take the tcgen05 kernel, shorter ones and decoded tokens the split-key
    kernel, in the same step; every cut must give the whole prompt's logits, as the CUDA-core kernel does."""
    monkeypatch.setattr(DifferentialAttention, "tensor_core_min_total", 0)
    cfg, w, folder = _model(tmp_path, "d", sharp=sharp)
    a, b = _tokens(cfg, 300, 40), _tokens(cfg, 170, 41)
    want_a, want_b = P.forward(cfg, w, a), P.forward(cfg, w, b)
    tol = (TOL_SHARP if sharp else TOL)[torch.bfloat16]
    d = U.Driver(folder, torch.bfloat16)
    d.step([("a", a)], end=["a"])
    assert U.rel_err(d.result("a"), want_a, torch.bfloat16) <= tol
    d = U.Driver(folder, torch.bfloat16)
    d.step([("a", a[:130]), ("b", b[:5])])
    d.step([("a", a[130:131]), ("b", b[5:150])])
    d.step([("a", a[131:290]), ("b", b[150:151])])
    d.step([("a", a[290:]), ("b", b[151:])])
    err_a, err_b = U.rel_err(d.result("a"), want_a, torch.bfloat16), U.rel_err(d.result("b"), want_b, torch.bfloat16)
    assert err_a <= tol and err_b <= tol
    monkeypatch.setattr(DifferentialAttention, "use_mma", False)     # the CUDA-core kernel alone agrees
    d = U.Driver(folder, torch.bfloat16)
    d.step([("a", a)], end=["a"])
    core = U.rel_err(d.result("a"), want_a, torch.bfloat16)
    assert core <= tol and err_a <= 2.0 * core + 0.02                # the divided step is as close to the oracle


def test_a_key_across_a_chunk_edge_does_not_reach_the_logits(tmp_path):
    """Token streams that differ in the tokens of an earlier chunk only (and not within reach of the
    convolutions) give the same logits in a one-layer model; a change inside the chunk does not."""
    cfg, w, folder = _model(tmp_path, "g", sharp=6.0)               # one layer, chunks of 90
    a = _tokens(cfg, 179, 50)
    b = list(a)
    b[30] = (b[30] + 1) % cfg["vocab"]
    c = list(a)
    c[92] = (c[92] + 1) % cfg["vocab"]
    res = []
    for toks in (a, b, c):
        d = U.Driver(folder, torch.float32)
        d.step([("r", toks[:120])])
        d.step([("r", toks[120:])])
        res.append(d.result("r")[110:])
    assert torch.equal(res[0], res[1])
    assert (res[0] - res[2]).abs().max() > 1e-3


def test_long_decoding(tmp_path):
    cfg, w, folder = _model(tmp_path, "a")
    toks = _tokens(cfg, 430, 5)
    want = P.forward(cfg, w, toks)
    d = U.Driver(folder, torch.float32)
    d.step([("r", toks[:30])])
    for t in toks[30:]:
        d.step([("r", [t])])
    assert U.rel_err(d.result("r"), want) <= 1e-4


def test_long_decoding_16_bit_split_keys(tmp_path):
    """Hundreds of keys per decoded token: the split-key kernel with several parts per row."""
    cfg, w, folder = _model(tmp_path, "d")
    toks = _tokens(cfg, 900, 6)
    want = P.forward(cfg, w, toks)
    d = U.Driver(folder, torch.bfloat16)
    d.step([("r", toks[:840])])
    for t in toks[840:]:
        d.step([("r", [t])])
    assert U.rel_err(d.result("r"), want, torch.bfloat16) <= TOL[torch.bfloat16]
    assert U.rel_err(d.result("r")[840:], want[840:], torch.bfloat16) <= TOL[torch.bfloat16]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_greedy_generation_through_the_engine(tmp_path, dtype):
    from sglang_security_b200.entrypoints.engine import Engine
    from sglang_security_b200.managers.schedule_batch import SamplingParams

    cfg, w, folder = _model(tmp_path, "a")
    prompts = [_tokens(cfg, n, 30 + i) for i, n in enumerate([70, 9, 130, 33, 2])]     # more requests than slots
    eng = Engine(folder, dtype, max_total_tokens=1024, max_running_requests=3, chunked_prefill_size=48)
    outs = eng.generate(prompts, SamplingParams(max_new_tokens=12))
    assert eng.runner.free_token_slots() == eng.runner.max_total_tokens
    for i, (p, o) in enumerate(zip(prompts, outs)):
        assert len(o) == 12
        if dtype == torch.float32:
            # teacher-forced: every generated token is (within rounding) the oracle's best token there
            logits, slack = P.forward(cfg, w, p + o[:-1])[len(p) - 1:], 1e-3
        else:
            # 16 bits: held to the same engine fed the same tokens as one prompt (the scheduler's cuts, slots
            # and pages must not matter); the fp32 run holds the engine to the oracle
            d = U.Driver(folder, dtype)
            d.step([(f"r{i}", p + o[:-1])], end=[f"r{i}"])
            logits, slack = d.result(f"r{i}").double()[len(p) - 1:], 0.1
        best = logits.max(-1).values
        took = logits[torch.arange(len(o)), torch.tensor(o)]
        assert ((best - took) <= slack * logits.std(-1)).all()
