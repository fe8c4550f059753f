"""Sapivik through the engine (loader, ModelRunner, pools, scheduler) against the plain restatement: whole
prompts, per-run residuals, token-by-token decoding, portions down to two tokens, unequal requests in one batch
with pages and request slots freed and used again, passes of a loop with caches and states of their own, a far
key that stands out, long decoding, and greedy generation through Engine.generate."""
import pytest
import torch

import sapivik_plain as P
import sapivik_util as U
from sglang_security_b200.layers.attention.sink_attention import SinkAttention

pytestmark = pytest.mark.gpu

CONFIGS = {
    # every mixer and feed-forward; the loop starts after and stops before the ends
    "a": lambda: U.config([(U.mem(), U.dense()), (U.att(), U.moe()), (U.mem(2, 16, 8), U.moe(4, 1, 2, 0.8, 16, None)),
                           (U.att(6, 3, 12, 12, 60.0, 5.0, 0.6), U.dense(24, 0.5)), (U.mem(1, 30, 10), None)], loop=(1, 4, 2)),
    # sizes that are multiples of nothing, the loop at the very front, an attention layer without feed-forward
    "b": lambda: U.config([(U.att(3, 1, 7, 6, 70.0, 9.0, 0.7), None), (U.mem(3, 5, 9), U.dense(21, 2.5)),
                           (U.att(5, 5, 9, 2, 30.0, None, 0.4), U.moe(3, 2, 4, 2.2, 13, 11))],
                          loop=(0, 2, 3), vocab=131, width=27, eps=1e-3, mult=0.8),
    # ones: one head, one channel, one expert, top 1, no loop, no rotation, multiplier 1
    "c": lambda: U.config([(U.mem(1, 1, 1), U.moe(1, 0, 1, 1.0, 1, 1)), (U.att(1, 1, 4, 0, 1.0, 1.0, 1.0), U.dense(1, 1.0)),
                           (U.att(2, 1, 2, 2, 10.0, None, 1.0), U.moe(1, 1, 1, 1.0, 3, None)), (U.mem(1, 1, 7), None)],
                          vocab=33, width=24, mult=1.0),
    # sizes of the tensor-core kernels, 4 : 1, 2 : 1 and 1 : 1, caps that do and do not reach the scores; the loop
    # stops at the last layer
    "d": lambda: U.config([(U.mem(2, 64, 64), U.moe(6, 2, 3, 1.5, 32, 48)), (U.att(4, 1, 64, 16, 500.0, 30.0, 0.2), U.dense(72, 3.0)),
                           (U.att(2, 2, 128, 64, 9000.0, 4.0, 0.1), U.moe(5, 1, 2, 1.0, 40, 24)),
                           (U.att(4, 2, 64, 0, 1.0, None, 0.125), U.dense(64))],
                          loop=(1, 4, 2), vocab=101, width=64),
    # a single layer that runs four times; attention only / memory only
    "e": lambda: U.config([(U.att(), U.dense())], loop=(0, 1, 4), vocab=61, width=48),
    "f": lambda: U.config([(U.mem(4, 40, 24), U.dense()), (U.mem(1, 130, 33), U.moe())], loop=(1, 2, 3), vocab=61, width=36),
}


def _model(tmp_path, name, seed=0, sharp=0.0):
    cfg = CONFIGS[name]()
    if sharp:        # a peaked softmax: one key more or less in sight moves the logits a lot
        for L in cfg["layers"]:
            if L["type"] == "attention":
                L["mixer"]["scale"] *= sharp
                L["mixer"].pop("softcap", None)
    w = U.random_weights(cfg, seed)
    return cfg, w, U.write_model(str(tmp_path / name), cfg, w)


def _tokens(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


TOL = {torch.float32: 1e-4, torch.bfloat16: 0.08}
SHARP = {torch.float32: 5.0, torch.bfloat16: 2.0}
TOL_SHARP = {torch.float32: 5e-4, torch.bfloat16: 0.15}


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_matches_plain_model(tmp_path, name, dtype):
    cfg, w, folder = _model(tmp_path, name)
    toks = _tokens(cfg, 200, 1)
    want = P.forward(cfg, w, toks)
    d = U.Driver(folder, dtype)
    d.step([("r", toks)], end=["r"])
    assert U.rel_err(d.result("r"), want, dtype) <= TOL[dtype]


@pytest.mark.parametrize("name", list(CONFIGS))
def test_residual_after_every_layer_run_fp32(tmp_path, name):
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
@pytest.mark.parametrize("name", list(CONFIGS))
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
@pytest.mark.parametrize("name", ["a", "b", "d", "e", "f"])
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
            if step % 5 == 4 and j == 1:
                continue                                             # left out of a step, goes on later
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
    assert U.rel_err(both.result("a"), alone.result("a")) <= 2e-5


@pytest.mark.parametrize("sharp", [0.0, 2.0])
def test_long_portions_on_the_prompt_kernel_beside_decoded_tokens(tmp_path, monkeypatch, sharp):
    """Portions of 128 tokens and more take the tcgen05 kernel, shorter ones and decoded tokens the split-key
    kernel, in the same step; every cut must give the whole prompt's logits, as the CUDA-core kernel does."""
    cfg, w, folder = _model(tmp_path, "d", sharp=sharp)
    a, b = _tokens(cfg, 430, 40), _tokens(cfg, 290, 41)
    want_a, want_b = P.forward(cfg, w, a), P.forward(cfg, w, b)
    tol = (TOL_SHARP if sharp else TOL)[torch.bfloat16]
    d = U.Driver(folder, torch.bfloat16)
    d.step([("a", a)], end=["a"])
    assert U.rel_err(d.result("a"), want_a, torch.bfloat16) <= tol
    d = U.Driver(folder, torch.bfloat16)
    d.step([("a", a[:150]), ("b", b[:5])])
    d.step([("a", a[150:151]), ("b", b[5:170])])
    d.step([("b", b[170:171]), ("a", a[151:400])])
    d.step([("a", a[400:]), ("b", b[171:])])
    err_a, err_b = U.rel_err(d.result("a"), want_a, torch.bfloat16), U.rel_err(d.result("b"), want_b, torch.bfloat16)
    assert err_a <= tol and err_b <= tol
    monkeypatch.setattr(SinkAttention, "tensor_core_min_tokens", 0)  # the CUDA-core kernel alone agrees
    monkeypatch.setattr(SinkAttention, "split_decode", False)
    d = U.Driver(folder, torch.bfloat16)
    d.step([("a", a)], end=["a"])
    core = U.rel_err(d.result("a"), want_a, torch.bfloat16)
    assert core <= tol and err_a <= 2.0 * core + 0.02                # the divided step is as close to the oracle


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", ["e", "d"])
def test_a_far_key_that_stands_out(tmp_path, name, dtype):
    """One attention layer's query projection is its key projection with the input coordinates reversed and one
    token's embedding is another's reversed, so the query of the one points at the key of the other: whether that
    far key is seen decides the logits.  First token, page borders, hundreds of tokens back; in every pass."""
    cfg = CONFIGS[name]()
    layer = 0 if name == "e" else 1
    m = cfg["layers"][layer]["mixer"]
    m["scale"], m["kv_heads"], cfg["residual_mult"] = 12.0 / m["dim"], m["heads"], 1.0
    m.pop("softcap", None)
    m.pop("rot", None)
    w = U.random_weights(cfg, 3)
    w[f"l{layer}.norm1"].fill_(1.0)
    w[f"l{layer}.mix.q"] = w[f"l{layer}.mix.k"].flip(1)
    w["embed"][5] = w["embed"][4].flip(0)
    folder = U.write_model(str(tmp_path / "m"), cfg, w)
    toks = [t if t not in (4, 5) else 6 for t in _tokens(cfg, 330, 7)]
    toks[320] = 4
    plain = P.forward(cfg, w, toks)[320]
    for at in (0, 63, 64, 127, 128, 200, 319):
        seq = list(toks)
        seq[at] = 5
        want = P.forward(cfg, w, seq)
        if name == "e":                          # elsewhere other layers stand between the two embeddings
            assert U.rel_errs(want[320:321], plain[None]).item() > 0.3
        for cuts in ([330], [310] + [1] * 20):
            d, o = U.Driver(folder, dtype), 0
            for n in cuts:
                d.step([("r", seq[o:o + n])])
                o += n
            assert U.rel_errs(d.result("r")[320:321], want[320:321]).item() <= TOL_SHARP[dtype], at


def test_passes_keep_caches_and_states_of_their_own(tmp_path):
    """A loop of n passes is not the model run once, nor passes that share one cache: token by token, a shared
    cache or state would hold the last pass' rows."""
    for name in ("e", "f"):
        cfg, w, folder = _model(tmp_path, name, sharp=3.0)
        toks = _tokens(cfg, 60, 9)
        want = P.forward(cfg, w, toks)
        once = P.forward({**cfg, "loop": {**cfg["loop"], "times": 1}}, w, toks)
        assert U.rel_err(once, want) > 0.1
        d = U.Driver(folder, torch.float32)
        for t in toks:
            d.step([("r", [t])])
        assert U.rel_err(d.result("r"), want) <= 5e-4
        runs = len(d.runner.model.runs)
        spec = d.runner.model.cache_spec()
        assert runs == len(spec.row_dims) + len(spec.state_widths)


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
