"""Segorax without a GPU: the reader of its config.json and its messages, the layout of parts, the declared tensors against
the names a checkpoint uses, the rotation's frequencies, and the plain implementation's mechanisms against hand-made cases."""
import copy
import math

import numpy as np
import pytest

import plain_segorax as ps
import segorax_util as su
from mimirmind_b200.config.model_config import ConfigError
from mimirmind_b200.registry import get_architecture, is_supported_architecture
from mimirmind_b200.weights.store import expected_tensors


def parse(cfg):
    return get_architecture("Segorax").parse_config(cfg, "config.json")


def spec_of(cfg):
    return get_architecture("Segorax").build_spec(parse(cfg))


def test_every_size_and_constant_comes_from_the_file():
    assert is_supported_architecture("Segorax")
    cfg, spec = parse(su.CONFIGS["A"]), spec_of(su.CONFIGS["A"])
    assert (cfg.vocab, cfg.width, cfg.norm_eps, cfg.residual_mult, cfg.embedding_scale, cfg.logit_scale) == (103, 72, 1e-5, 0.6, 3.0, 0.7)
    assert [layer.mixer.kind for layer in spec.layers] == ["latent_attention"] * 4 and all(layer.block["mult"] == 0.6 for layer in spec.layers)
    far, low = spec.layers[0].mixer, spec.layers[1].mixer
    assert (far["heads"], far["key_dim"], far["rot_dim"], far["value_dim"], far["rank"], far["scale"], far["q_rank"], far["sink"]) == \
        (3, 12, 8, 20, 32, 0.4, 0, None)
    assert far["rotary"] == {"dims": 8, "base": 700.0, "layout": "pairs", "scaling": {"factor": 4.0, "original": 64.0, "fast": 16.0, "slow": 1.0}}
    assert (low["q_rank"], low["q"], low["q_down"], low["q_norm"], low["sink"], low["eps"]) == (24, "mix.uq", "mix.dq", "mix.dq.norm", "mix.sink", 1e-5)
    assert low["rotary"]["scaling"] is None and low["g"] is None
    f = spec.layers[0].feed_forward
    assert (f["ff"], f["experts"], f["top"], f["groups"], f["keep"], f["group_score"], f["scoring"], f["gated"], f["activation"]) == \
        (40, 9, 2, 3, 1, "top2_sum", "sigmoid", False, "gelu_erf")
    assert f["shared"]["ff"] == 24 and f["shared_gate"] == "mlp.shared.sg" and f["correction"] == "mlp.correction"
    assert (spec.layers[1].feed_forward.kind, spec.layers[1].feed_forward["activation"]) == ("swiglu", "gelu_tanh")
    assert spec.layers[2].feed_forward.kind == "none"
    last = spec.layers[3].feed_forward
    assert (last["groups"], last["keep"], last["shared"], last["shared_gate"]) == (1, 1, None, None)
    assert spec.final_norm["gain"] == 0.7 and spec.embedding["scale"] == 3.0 and spec.head["tied_to"] is None


def test_what_may_be_absent():
    cfg, spec = parse(su.CONFIGS["C"]), spec_of(su.CONFIGS["C"])
    assert (cfg.residual_mult, cfg.embedding_scale, cfg.logit_scale) == (1.0, 1.0, 1.0)
    assert spec.final_norm["gain"] == 1.0 and spec.layers[1].feed_forward["groups"] == 1


@pytest.mark.parametrize("name", sorted(su.CONFIGS))
def test_declared_tensors_are_the_checkpoints(name):
    exp, have = expected_tensors(spec_of(su.CONFIGS[name])), su.tensor_shapes(su.CONFIGS[name])
    assert {k for k, v in exp.items() if not v.optional} == set(have)
    for k, shape in have.items():
        assert tuple(exp[k].shape) == tuple(shape), k


@pytest.mark.parametrize("edit,message", [
    (lambda c: c.pop("vocab"), "vocab"),
    (lambda c: c["norm"].pop("eps"), "norm.eps"),
    (lambda c: c["layers"][0].update(type="attention"), "'attention' is not one of"),
    (lambda c: c["layers"][1]["mixer"].pop("q_rank"), "layers[1].mixer.q_rank"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "layers[0].mixer.scale"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=10), "at most rot_dim"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), "layers[0].mixer.rot.scaling.slow"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0), "must be positive"),
    (lambda c: c["layers"][0]["mlp"].update(kind="gated"), "'gated' is not one of"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4), "equal groups"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=4), "cannot be chosen"),
    (lambda c: c.update(layers=[]), "non-empty list"),
])
def test_messages_name_the_key(edit, message):
    cfg = copy.deepcopy(su.CONFIGS["A"])
    edit(cfg)
    with pytest.raises(ConfigError) as e:
        parse(cfg)
    assert message in str(e.value)


@pytest.mark.parametrize("base,dims,scaling", [(10000.0, 64, None), (700.0, 8, (4.0, 64, 16.0, 1.0)), (5000.0, 40, (6.0, 1500, 24.0, 2.0)),
                                               (20.0, 2, (3.0, 40, 1.5, 1.4)), (300.0, 12, (2.5, 200, 8.0, 2.0)), (50.0, 10, (4.0, 10, 32.0, 4.0))])
def test_the_rotations_frequencies(base, dims, scaling):
    """The product's frequencies equal the plain ones; every interpolated frequency lies between the original and the divided one,
    the fastest pairs keep theirs and the slowest are divided in full; the factor on cos and sin grows with the stretch."""
    from mimirmind_b200.parts.rope import exact_frequencies
    sc = dict(zip(("factor", "original", "fast", "slow"), scaling)) if scaling else None
    f, factor = exact_frequencies(base, dims, sc)
    want, want_factor = ps.rotation(dims, base, sc)
    assert np.abs(f.numpy() / want - 1.0).max() < 1e-12 and factor == want_factor
    plain, _ = ps.rotation(dims, base)
    if sc is None:
        assert factor == 1.0 and np.array_equal(want, plain)
    else:
        assert (want <= plain * (1 + 1e-12)).all() and (want >= plain / sc["factor"] * (1 - 1e-12)).all()
        assert factor == pytest.approx(1.0 + 0.1 * math.log(sc["factor"]))


def test_interpolation_by_hand():
    """dims 16, base 256: frequencies 2^-i; original 1024 / (2 pi t) and the pair numbers worked out by hand."""
    sc = {"factor": 4.0, "original": 2.0 * math.pi * 1024.0, "fast": 256.0, "slow": 16.0}
    # number(t) = 16 ln(1024 / t) / (2 ln 256) = log2(1024 / t): fast 2, slow 6
    f, factor = ps.rotation(16, 256.0, sc)
    base = 2.0 ** -np.arange(8)
    ramp = np.array([0, 0, 0, 0.25, 0.5, 0.75, 1, 1])
    assert np.allclose(f, base * (1 - ramp) + base / 4 * ramp, rtol=1e-12) and factor == 0.1 * math.log(4.0) + 1.0


def test_plain_rotation_turns_neighbours_and_keeps_lengths():
    x = np.zeros((2, 1, 6))
    x[:, 0, 2] = 1.0
    y = ps.rotate_pairs(x, [0, 3], 4, 100.0)
    assert np.allclose(y[0], x[0])
    assert np.allclose(y[1, 0], [0, 0, math.cos(3 * 100 ** -0.5), math.sin(3 * 100 ** -0.5), 0, 0])


def test_plain_choice_by_hand():
    """Scores 0.5 everywhere: the correction alone decides, and the weights stay 0.5.  Groups (0,1), (2,3), (4,5) with choice
    scores (9, -8), (3, 2), (1, -0.5) around 0.5: by the sum of two the second group wins, by the best one the first would."""
    h, w = np.zeros((1, 4)), np.ones((6, 4))
    corr = np.array([9.0, -8.0, 3.0, 2.0, 1.0, -0.5])
    idx, wts = ps.router_choice(h, w, corr, 2, (3, 1))
    assert idx.tolist() == [[2, 3]] and np.allclose(wts, 0.5)
    assert ps.router_choice(h, w, corr, 2, None)[0].tolist() == [[0, 2]]
    # negative choice scores: an expert of a kept group comes before any of a dropped one, whatever its sign
    idx, _ = ps.router_choice(h, w, np.array([-1.0, -2.0, -9.0, -1.2, -3.0, -3.0]), 2, (3, 1))
    assert idx.tolist() == [[0, 1]]


def test_plain_sink_and_activations():
    q = np.zeros((2, 1, 3))
    v = np.array([[[1.0]], [[3.0]]])
    o = ps.softmax_attention(q, q, v, 1.0, np.array([0.0]))
    assert np.allclose(o[:, 0, 0], [0.5, 4.0 / 3.0])                # a sink of 0 counts as one more key of score 0
    assert np.allclose(ps.softmax_attention(q, q, v, 1.0)[:, 0, 0], [1.0, 2.0])
    assert ps.gelu_erf(np.array([1.0]))[0] == pytest.approx(0.8413447460685429)
    assert ps.gelu_tanh(np.array([1.0]))[0] == pytest.approx(0.8411919906082768)


def test_the_final_norm_carries_the_logit_scale():
    """The norm part multiplies its weight by the gain once, in fp32, and then has no native form under another constant."""
    import torch
    from mimirmind_b200.config.spec import PartSpec
    from mimirmind_b200.parts.base import Runtime, WeightView
    from mimirmind_b200.parts.norm import RMSNorm
    w = torch.tensor([1.0, 2.0, 3.0]).to(torch.bfloat16)
    part = RMSNorm(PartSpec("rmsnorm", {"width": 3, "eps": 1e-6, "weight": "n", "gain": 0.3}), WeightView({"n": w}), Runtime(torch.bfloat16, torch.device("cpu")))
    assert torch.equal(part.weight, w.float() * 0.3) and part.native() is None
    assert RMSNorm(PartSpec("rmsnorm", {"width": 3, "eps": 1e-6, "weight": "n"}), WeightView({"n": w}), Runtime(torch.bfloat16, torch.device("cpu"))).native() is not None
