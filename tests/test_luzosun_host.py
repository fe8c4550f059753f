"""Luzosun on the host: configuration read-out and rejections, registry, tensor names and fused layouts, and
self-checks of the plain restatement (what a position sees, the two maps' weight, the activation)."""
import math

import pytest
import torch

import luzosun_plain as P
import luzosun_util as U
from sglang_security_b200.configs.luzosun import DifferentialSpec, UngatedSpec, luzosun_config
from sglang_security_b200.configs.model_config import ModelConfig
from sglang_security_b200.models.registry import resolve_model_cls, supported_architectures


def _cfg():
    return U.config([(U.diff(), U.dense()), (U.diff(kv_from=0, heads=6, chunk=16, lam=0.7, conv=2), None),
                     (U.diff(heads=3, kv_heads=3, dim=7, vdim=5, chunk=None, conv=0, rot_dims=0), U.dense(24))])


def test_configuration_reads_every_size_from_the_file():
    c = luzosun_config(_cfg())
    assert (c.vocab, c.width, c.eps, c.embedding_scale, c.canon_taps, c.num_layers) == (89, 40, 1e-5, 3.0, 3, 3)
    a, b, d = (L.mixer for L in c.layers)
    assert isinstance(a, DifferentialSpec)
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.chunk, a.conv, a.diff, a.kv_from) == (4, 2, 12, 20, 40, 4, 0.4, None)
    assert (a.rope_dims, a.rope_base, a.rope_factor, a.scale) == (8, 1000.0, 2.5, 12 ** -0.5)
    assert (b.heads, b.chunk, b.diff, b.conv, b.kv_from) == (6, 16, 0.7, 2, 0)
    assert (d.chunk, d.conv, d.rope_dims, d.rope_factor) == (None, 0, 0, 1.0)
    assert c.layers[0].mlp == UngatedSpec(56) and c.layers[1].mlp is None and c.layers[2].mlp == UngatedSpec(24)


def test_taps_follow_the_tensors():
    c = luzosun_config(_cfg())
    c.resolve_shapes({"l0.canon1": (40, 5), "l1.canon1": (40, 5), "l2.canon1": (40, 5), "l0.mix.q.conv": (96, 6)})
    assert c.canon_taps == 5 and c.layers[0].mixer.conv == 6 and c.layers[1].mixer.conv == 2


@pytest.mark.parametrize("edit, text", [
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "cannot share"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rotated"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=14), "rotated"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(scaling={"factor": 0.0}), "positive"),
    (lambda c: c["layers"][1]["mixer"].update(kv_from=1), "earlier layer"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=1), "earlier layer"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=24), "differ"),
    (lambda c: c["layers"][0].update(type="mamba2"), "unknown mixer"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "unknown feed-forward"),
])
def test_inconsistent_configurations_are_rejected(edit, text):
    c = _cfg()
    edit(c)
    with pytest.raises(ValueError, match=text):
        luzosun_config(c)


def test_registry_and_tensor_names(tmp_path):
    assert "Luzosun" in supported_architectures()
    cfg = _cfg()
    w = U.random_weights(cfg)
    mc = ModelConfig(U.write_model(str(tmp_path / "m"), cfg, w))
    assert mc.architecture == "Luzosun"
    mc.hf_config.resolve_shapes({k: tuple(v.shape) for k, v in w.items()})
    model = resolve_model_cls("Luzosun")(mc.hf_config, params_dtype=torch.bfloat16)
    assert model.expected_tensor_names() == set(w)
    model.load_weights(w.items())
    spec = model.cache_spec()
    assert spec.row_dims == {0: 2 * (2 * 12 + 20), 2: 3 * (2 * 7 + 5)} and spec.source_of == {1: 0}
    c0 = 4 * 24 + 2 * 24 + 2 * 20
    assert spec.state_widths == {0: 2 * 40 + 3 * c0, 1: 2 * 40 + 1 * 6 * 24, 2: 2 * 40}
    a, b = model.layers[0], model.layers[1]
    # fused [q ; k ; v], the convolutions stacked channel-contiguous, both output matrices side by side
    assert torch.equal(a.mix.in_proj.weight[96:144], w["l0.mix.k"]) and torch.equal(a.mix.in_proj.bias[144:], w["l0.mix.v.b"])
    assert torch.equal(a.mix.conv_weight[3, :96], w["l0.mix.q.conv"][:, 3].float())
    assert torch.equal(a.norms.conv_weight[0], w["l0.canon1"][:, 0].float())
    assert torch.equal(a.out.proj.weight[:, :80], w["l0.mix.o"]) and torch.equal(a.out.proj.weight[:, 80:], w["l0.mlp.down"])
    assert b.mlp is None and b.out.columns == 120 and b.mix.parts == {"q": 144, "k": 0, "v": 0}
    # 3 x 5 value columns are padded to 16 with zero weights
    c = model.layers[2].out
    assert c.offsets == [0, 16] and c.columns == 40 and c.padded and not c.proj.weight[:, 15].any()
    assert abs(float(a.mix.lam) - P.mix_lambda({k: v.double() for k, v in w.items()}, "l0.mix.", 0.4)) < 1e-6
    with pytest.raises(ValueError, match="lacks"):
        model.load_weights((k, v) for k, v in w.items() if k != "l1.mix.lq2")
    for extra in ("l1.mix.k", "l1.mlp.up", "l2.mix.q.conv", "l0.mix.zz", "l7.norm1"):
        with pytest.raises(ValueError, match="unexpected"):
            model.load_weights(list(w.items()) + [(extra, w["l0.mix.q"])])


def test_what_a_position_sees():
    m = P.visible(10, 4)
    assert [int(x) for x in m[3].nonzero()] == [0, 1, 2, 3] and [int(x) for x in m[4].nonzero()] == [4]
    assert [int(x) for x in m[7].nonzero()] == [4, 5, 6, 7] and [int(x) for x in m[9].nonzero()] == [8, 9]
    assert [int(x) for x in P.visible(5, 0)[4].nonzero()] == [0, 1, 2, 3, 4]
    assert P.visible(6, 1).sum() == 6


def test_second_map_weight_and_difference():
    W = {"lq1": torch.tensor([1.0, 2.0]), "lk1": torch.tensor([0.5, 0.25]), "lq2": torch.tensor([1.0, -1.0]),
         "lk2": torch.tensor([0.0, 1.0])}
    assert abs(P.mix_lambda(W, "", 0.3) - (math.e - math.exp(-1.0) + 0.3)) < 1e-6
    a1, a2 = torch.tensor([[3.0, 1.0]], dtype=torch.float64), torch.tensor([[1.0, 1.0]], dtype=torch.float64)
    o = P.combine_maps(a1, a2, 1.0, 0.25, 0.0)                  # difference (2, 0): rms sqrt(2)
    assert torch.allclose(o, torch.tensor([[2 / math.sqrt(2.0) * 0.75, 0.0]], dtype=torch.float64))


def test_activation_by_hand():
    z = torch.tensor([2.0, 0.0, -1.0], dtype=torch.float64)
    y = P.xielu(z, 0.0, 1.0)
    assert abs(float(y[0]) - (math.log(2.0) * 4 + 1.0)) < 1e-12 and float(y[1]) == 0.0
    assert abs(float(y[2]) - ((0.5 + math.log1p(math.e)) * math.exp(-1.0) - 0.5)) < 1e-12


def test_convolution_and_rotation_by_hand():
    u = torch.tensor([[1.0], [2.0], [4.0]], dtype=torch.float64)
    y = P.causal_conv(u, torch.tensor([[10.0, 1.0]], dtype=torch.float64))
    assert y.flatten().tolist() == [1.0, 12.0, 24.0]
    x = torch.zeros(3, 1, 6, dtype=torch.float64)
    x[:, 0, 0] = 1.0
    r = P.rotate_halves(x, torch.arange(3), 4, 100.0, 2.0)      # pair (0, 2) turns by p / 2
    assert abs(float(r[2, 0, 0]) - math.cos(1.0)) < 1e-12 and abs(float(r[2, 0, 2]) - math.sin(1.0)) < 1e-12
    assert not r[:, 0, 4:].any()
