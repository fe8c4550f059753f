"""Sapivik on the host: configuration read-out and rejections, the order of layer runs, registry, tensor names
and fused layouts, and self-checks of the plain restatement on hand-made cases."""
import math

import pytest
import torch

import sapivik_plain as P
import sapivik_util as U
from sglang_security_b200.configs.model_config import ModelConfig
from sglang_security_b200.configs.sapivik import (ChannelMemorySpec, ClampedSpec, IdentityExpertsSpec,
                                                  TiedAttentionSpec, sapivik_config)
from sglang_security_b200.models.registry import resolve_model_cls, supported_architectures


def _cfg():
    return U.config([(U.mem(), U.dense()), (U.att(), U.moe()), (U.mem(2, 7, 5), None),
                     (U.att(3, 3, 6, rot_dims=0, cap=None), U.moe(4, 0, 1, 1.0, 8, None))], loop=(1, 3, 2))


def test_configuration_reads_every_size_from_the_file():
    c = sapivik_config(_cfg())
    assert (c.vocab, c.width, c.eps, c.residual_mult, c.num_layers, c.loop) == (83, 40, 1e-4, 0.45, 4, (1, 3, 2))
    assert c.layers[0].mixer == ChannelMemorySpec(3, 12, 20)
    assert c.layers[1].mixer == TiedAttentionSpec(4, 2, 20, 20 ** -0.5, 12.0, 900.0, 8)
    assert (c.layers[3].mixer.softcap, c.layers[3].mixer.rope_dims) == (0.0, 0)
    assert c.layers[0].mlp == ClampedSpec(36, 1.5) and c.layers[2].mlp is None
    assert c.layers[1].mlp == IdentityExpertsSpec(5, 3, 3, 1.6, 20, 28)
    assert c.layers[3].mlp == IdentityExpertsSpec(4, 0, 1, 1.0, 8, 0)


@pytest.mark.parametrize("loop, runs", [
    (None, [0, 1, 2, 3]), ((1, 3, 1), [0, 1, 2, 3]), ((1, 3, 3), [0, 1, 2, 1, 2, 1, 2, 3]), ((0, 2, 2), [0, 1, 0, 1, 2, 3]),
    ((2, 4, 2), [0, 1, 2, 3, 2, 3]), ((0, 4, 2), [0, 1, 2, 3, 0, 1, 2, 3]), ((2, 3, 4), [0, 1, 2, 2, 2, 2, 3]),
])
def test_order_of_layer_runs(loop, runs):
    cfg = _cfg()
    cfg.pop("loop")
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    got = sapivik_config(cfg).layer_runs()
    assert [i for i, _ in got] == runs and got == P.layer_order(4, cfg.get("loop"))
    # the embedding output is added ahead of every pass but the first, and nowhere else
    assert sum(a for _, a in got) == (loop[2] - 1 if loop else 0)
    assert all(i == loop[0] for i, a in got if a)


@pytest.mark.parametrize("edit, text", [
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "cannot share"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=24), "values are the keys"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "rotated"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=22), "rotated"),
    (lambda c: c["layers"][0].update(type="mamba2"), "unknown mixer"),
    (lambda c: c["layers"][0]["mixer"].update(heads=0), "heads"),
    (lambda c: c["layers"][0]["mlp"].update(kind="glu"), "unknown feed-forward"),
    (lambda c: c["layers"][0]["mlp"].update(limit=0.0), "positive"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=9), "top 9"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(identity=-1), "top"),
    (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c["loop"].update(start=4), "loop"),
    (lambda c: c["loop"].update(times=0), "loop"),
])
def test_inconsistent_configurations_are_rejected(edit, text):
    c = _cfg()
    edit(c)
    with pytest.raises(ValueError, match=text):
        sapivik_config(c)


def test_registry_tensor_names_and_layouts(tmp_path):
    assert "Sapivik" in supported_architectures()
    cfg = _cfg()
    w = U.random_weights(cfg)
    mc = ModelConfig(U.write_model(str(tmp_path / "m"), cfg, w))
    model = resolve_model_cls(mc.architecture)(mc.hf_config, params_dtype=torch.float32)
    assert model.expected_tensor_names() == set(w)
    model.load_weights(w.items())
    eq = lambda a, b: torch.equal(a.float(), b.float())
    mix = model.layers[0].mix
    assert eq(mix.qfv_proj.weight, torch.cat([w["l0.mix.q"], w["l0.mix.f"], w["l0.mix.v"]]))
    assert eq(mix.norm_weight, w["l0.mix.norm"].repeat(3)) and eq(mix.f_lower, w["l0.mix.lower"])
    mix = model.layers[1].mix
    assert eq(mix.qkv_proj.weight, torch.cat([w["l1.mix.q"], w["l1.mix.k"], w["l1.mix.g"]]))
    assert mix.row_width == 2 * 2 * 20 and mix.q_norm_weight is None and mix.sink is None
    assert mix.score_bound == pytest.approx(12.0 * math.tanh(20 ** 0.5 / 12.0))
    ex = model.layers[1].moe
    assert eq(ex.experts.w_gate_up[4], torch.cat([w["l1.mlp.e4.gate"], w["l1.mlp.e4.up"]]))
    assert ex.router.weight.shape == (8, 40) and eq(ex.router.shared_gate, w["l1.mlp.shared.sg"][0])
    spec = model.cache_spec()                    # runs 0 1 2 1 2 3: every pass has rows / a state of its own
    assert set(spec.row_dims) == {1, 3, 5} and set(spec.state_widths) == {0, 2, 4}
    assert spec.row_dims[1] == spec.row_dims[3] == 80 and spec.state_widths[2] == spec.state_widths[4]
    with pytest.raises(ValueError, match="lacks"):
        model.load_weights((k, v) for k, v in w.items() if k != "l0.mix.lower")
    for name in ("l0.mix.k", "l1.mix.v", "l1.mlp.e5.gate", "l3.mlp.shared.up", "l2.mlp.gate", "l9.norm1", "pos"):
        with pytest.raises(ValueError, match="unexpected"):
            model.load_weights([(name, w["head"])])
    with pytest.raises(ValueError, match="rows"):
        model.load_weights([("l1.mix.k", w["l1.mix.q"])])


def test_plain_memory_on_a_hand_made_case():
    """A channel that forgets nothing writes nothing; one that forgets everything holds the last value."""
    v = torch.tensor([[[2.0, -1.0]], [[4.0, 3.0]], [[8.0, 5.0]]], dtype=torch.float64)
    f = torch.tensor([[[1.0, 0.0, 0.5]]] * 3, dtype=torch.float64)
    _, S = P.gated_memory(torch.ones(3, 1, 3, dtype=torch.float64), f, v)
    assert S[0, 0].tolist() == [0.0, 0.0] and S[0, 1].tolist() == [8.0, 5.0]
    assert S[0, 2].tolist() == [0.25 * 1.0 + 0.5 * 2.0 + 4.0, 0.25 * -0.5 + 0.5 * 1.5 + 2.5]
    z = torch.tensor([-40.0, 0.0, 40.0], dtype=torch.float64)
    assert torch.allclose(P.forget_gate(z, torch.zeros(3), torch.full((3,), 0.25)), torch.tensor([0.25, 0.625, 1.0]).double())


def test_plain_router_and_activation_on_hand_made_cases():
    z = torch.log(torch.tensor([4.0, 3.0, 2.0, 1.0], dtype=torch.float64))
    ids, wts = P.route(z, torch.tensor([0.0, 0.0, 0.0, 1.0]).double(), 2, 3.0)
    assert ids == [3, 0] and wts == pytest.approx([0.3, 1.2])       # chosen by s + correction, weighted by s alone
    W = {"gate": torch.tensor([[1.0]]), "up": torch.tensor([[10.0]]), "down": torch.tensor([[1.0]])}
    W = {k: t.double() for k, t in W.items()}
    want = 2.0 / (1.0 + math.exp(-3.404)) * 3.0
    assert P.clamped_ff(W, "", 2.0, torch.tensor([[5.0]]).double()).item() == pytest.approx(want)
    want = -5.0 / (1.0 + math.exp(8.51)) * -1.0                     # the gate is clamped from above only
    assert P.clamped_ff(W, "", 2.0, torch.tensor([[-5.0]]).double()).item() == pytest.approx(want)


def test_plain_rotation_keeps_norms_and_distances():
    g = torch.Generator().manual_seed(1)
    x = torch.randn(1, 1, 10, generator=g).double().expand(50, 1, 10)
    y = P.rotate_neighbours(x, torch.arange(50), 6, 30.0)
    assert torch.allclose(y.norm(dim=-1), x.norm(dim=-1)) and torch.equal(y[..., 6:], x[..., 6:])
    dots = (y[:-7, 0] * y[7:, 0]).sum(-1)                           # depends on the distance only
    assert torch.allclose(dots, dots[:1].expand_as(dots))
    assert torch.allclose(P.unit_rms(y, 1e-3), P.rotate_neighbours(P.unit_rms(x, 1e-3), torch.arange(50), 6, 30.0))
