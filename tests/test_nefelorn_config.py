"""Nefelorn without a GPU: the reader of its config.json and its messages, the layout of parts, the declared tensors against
the names a checkpoint uses, what the cache keeps for readers with masks of their own, and the plain implementation's mechanisms
against hand-made cases."""
import copy
import math

import numpy as np
import pytest

import nefelorn_util as nu
import plain_nefelorn as pn
from mimirmind_b200.cache.manager import CacheManager, GroupSpec
from mimirmind_b200.cache.pages import INVALID_PAGE
from mimirmind_b200.config.model_config import ConfigError
from mimirmind_b200.registry import get_architecture, is_supported_architecture
from mimirmind_b200.weights.store import expected_tensors


def parse(cfg):
    return get_architecture("Nefelorn").parse_config(cfg, "config.json")


def spec_of(cfg):
    return get_architecture("Nefelorn").build_spec(parse(cfg))


def test_every_size_and_constant_comes_from_the_file():
    assert is_supported_architecture("Nefelorn")
    cfg, spec = parse(nu.CONFIGS["A"]), spec_of(nu.CONFIGS["A"])
    assert (cfg.vocab, cfg.width, cfg.norm_eps, cfg.embedding_scale, cfg.logit_softcap) == (101, 72, 1e-5, 3.0, 8.0)
    assert all(layer.mixer.kind == "masked_attention" and layer.block.kind == "sandwich_norm" for layer in spec.layers)
    far, near, reader = (spec.layers[i].mixer for i in (0, 1, 2))
    assert (far["heads"], far["kv_heads"], far["key_dim"], far["value_dim"], far["scale"], far["eps"]) == (6, 2, 24, 16, 0.25, 1e-5)
    assert (far["window"], far["chunk"], far["keep"], far["unit_qk"], far["q_norm"], far["k_norm"], far["g"]) == \
        (0, 37, 0, False, "mix.q.norm", "mix.k.norm", "mix.g")
    assert far["rotary"] == {"dims": 24, "base": 700.0, "scaling": {"factor": 4.0, "original": 64.0, "fast": 16.0, "slow": 1.0}}
    assert (near["window"], near["chunk"], near["keep"], near["unit_qk"], near["q_norm"], near["k_norm"], near["g"]) == (29, 0, 5, True, None, None, None)
    assert near["rotary"] == {"dims": 8, "base": 900.0, "scaling": None} and spec.layers[3].mixer["keep"] == 0
    assert (reader["k"], reader["v"], reader["k_norm"], reader["q_norm"], reader["chunk"]) == (None, None, None, "mix.q.norm", 90)
    assert [e.cache_from for e in spec.schedule] == [None, None, 0, None, 0]
    f = spec.layers[0].feed_forward
    assert (f["ff"], f["experts"], f["top"], f["scoring"], f["renorm"], f["weight_scale"], f["activation"]) == (40, 9, 3, "sigmoid", True, 1.7, "silu")
    assert (spec.layers[1].feed_forward.kind, spec.layers[1].feed_forward["activation"], spec.layers[1].feed_forward["ff"]) == ("dense_mlp", "gelu_erf", 88)
    assert spec.layers[2].feed_forward.kind == "none" and "ffn_post_norm" not in spec.layers[2].extras
    assert spec.head["softcap"] == 8.0 and spec.embedding["scale"] == 3.0 and spec.head["tied_to"] is None


def test_what_may_be_absent():
    cfg, spec = parse(nu.CONFIGS["C"]), spec_of(nu.CONFIGS["C"])
    assert (cfg.embedding_scale, cfg.logit_softcap) == (1.0, 0.0) and spec.layers[0].feed_forward["weight_scale"] == 1.0
    assert spec.layers[3].mixer["rotary"]["scaling"] is None
    bare = copy.deepcopy(nu.CONFIGS["A"])
    for layer in bare["layers"]:
        layer["mixer"].pop("mask"), layer["mixer"].pop("rot")
    mixers = [layer.mixer for layer in spec_of(bare).layers]
    assert all((m["window"], m["chunk"], m["keep"], m["rotary"]) == (0, 0, 0, None) for m in mixers)


@pytest.mark.parametrize("name", sorted(nu.CONFIGS))
def test_declared_tensors_are_the_checkpoints(name):
    exp, have = expected_tensors(spec_of(nu.CONFIGS[name])), nu.tensor_shapes(nu.CONFIGS[name])
    assert {k for k, v in exp.items() if not v.optional} == set(have)
    for k, shape in have.items():
        assert tuple(exp[k].shape) == tuple(shape), k


@pytest.mark.parametrize("edit,message", [
    (lambda c: c.pop("vocab"), "vocab"),
    (lambda c: c["norm"].pop("eps"), "norm.eps"),
    (lambda c: c["layers"][0].update(type="retention"), "'retention' is not one of"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "layers[1].mixer.scale"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "not a multiple"),
    (lambda c: c["layers"][0]["mixer"]["mask"].pop("size"), "layers[0].mixer.mask.size"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=26), "at most dim"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), "layers[0].mixer.rot.scaling.slow"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0), "must be positive"),
    (lambda c: c["layers"][0]["mlp"].update(kind="gated"), "'gated' is not one of"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=10), "of 9 experts"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=2), "does not name an earlier layer"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=2), "without keys and values of its own"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=1), "have other sizes"),
    (lambda c: c.update(logit_softcap=-1.0), "must not be negative"),
    (lambda c: c.update(layers=[]), "non-empty list"),
])
def test_messages_name_the_key(edit, message):
    cfg = copy.deepcopy(nu.CONFIGS["A"])
    edit(cfg)
    with pytest.raises(ConfigError) as e:
        parse(cfg)
    assert message in str(e.value)


# ---- what the cache keeps -----------------------------------------------------------------------------------------------------
def visible(mask, pos, j):
    window, chunk, keep = mask
    if not window and not chunk:
        return True
    return j < keep or ((not window or pos - j < window) and (not chunk or pos // chunk == j // chunk))


@pytest.mark.parametrize("masks", [[(0, 13, 0)], [(0, 4, 0)], [(9, 0, 3)], [(9, 0, 6)], [(0, 13, 0), (0, 30, 0)], [(7, 0, 0), (0, 20, 0)],
                                   [(7, 0, 5), (12, 0, 0)], [(6, 10, 2)], [(0, 0, 0), (5, 0, 0)]])
def test_pages_go_when_no_reader_can_see_them_and_not_before(masks):
    """Against the masks token by token: after every commit a page is held exactly while some later query of some reader sees a
    token of it (or it is still being filled)."""
    ps = 4
    bounded = all(w or c for w, c, _k in masks)
    m = CacheManager([GroupSpec("g", (0,), 1, 8, 0, (), tuple(masks))], page_size=ps, pages_per_group=64, max_requests=1)
    m.add_request("a")
    n = 0
    for step in [3, 1, 1, 5, 2, 9, 1, 1, 1, 1, 7, 16, 2, 1, 1, 3]:
        assert m.reserve("a", n + step)
        n += step
        m.commit("a", n)
        m.check()
        table = m.table("a", "g")
        for b, page in enumerate(table):
            seen = any(visible(mask, pos, j) for mask in masks for pos in range(n, n + 40) for j in range(b * ps, min(n, (b + 1) * ps)))
            assert (page != INVALID_PAGE) == (seen or b * ps + ps > n or not bounded), (n, b)
    m.release("a")
    assert m.free_pages("g") == 64


def test_a_prompt_longer_than_the_pool_of_runs():
    """A group that every reader looks at through runs needs pages for the stretch in view only: the scheduler takes the prompt."""
    from mimirmind_b200.engine.scheduler import Request, Scheduler, SchedulerConfig
    m = CacheManager([GroupSpec("g", (0,), 1, 8, 0, (), ((0, 16, 0), (12, 0, 3)))], page_size=4, pages_per_group=10, max_requests=1)
    s = Scheduler(SchedulerConfig(16, 1, 0, 1000), m)
    r = Request("r", list(range(100)), max_new=20)
    assert s.add(r)
    while s.has_work():
        plan = s.schedule()
        s.commit(plan, {e.request.id: 7 for e in plan if e.samples})
        m.check()
    assert r.finish_reason == "length" and len(r.generated) == 20 and m.allocators["g"].reuses > 0


# ---- the plain implementation by hand -----------------------------------------------------------------------------------------
def test_plain_masks():
    c = pn.chunk_mask(7, 3)
    assert c.astype(int).tolist() == [[1, 0, 0, 0, 0, 0, 0], [1, 1, 0, 0, 0, 0, 0], [1, 1, 1, 0, 0, 0, 0], [0, 0, 0, 1, 0, 0, 0],
                                      [0, 0, 0, 1, 1, 0, 0], [0, 0, 0, 1, 1, 1, 0], [0, 0, 0, 0, 0, 0, 1]]
    w = pn.window_mask(6, 2, 1)
    assert w.astype(int).tolist() == [[1, 0, 0, 0, 0, 0], [1, 1, 0, 0, 0, 0], [1, 1, 1, 0, 0, 0], [1, 0, 1, 1, 0, 0], [1, 0, 0, 1, 1, 0], [1, 0, 0, 0, 1, 1]]


def test_plain_norms_and_cap():
    w = {"n": np.array([2.0, 1.0]), "n.b": np.array([0.5, 0.0]), "n.alpha": np.array(0.5)}
    assert np.allclose(pn.squash(np.array([[1.0, -100.0]]), w, "n"), [[2.0 * math.tanh(0.5) + 0.5, -1.0]])
    assert np.allclose(pn.unit_rms(np.array([[3.0, 4.0]]), 0.0), np.array([[3.0, 4.0]]) / math.sqrt(12.5))
    assert pn.soft_cap(np.array([3.0]), 2.0)[0] == pytest.approx(2.0 * math.tanh(1.5)) and pn.soft_cap(np.array([3.0]), None)[0] == 3.0
    assert pn.gelu_erf(np.array([1.0]))[0] == pytest.approx(0.8413447460685429)


def test_plain_rotation_pairs_halves_and_keeps_the_rest():
    x = np.zeros((2, 1, 7))
    x[:, 0, 1], x[:, 0, 6] = 1.0, 5.0
    y = pn.rotate_halves(x, [0, 3], {"dims": 4, "base": 100.0})
    assert np.allclose(y[0], x[0])
    assert np.allclose(y[1, 0], [0, math.cos(3 * 100 ** -0.5), 0, math.sin(3 * 100 ** -0.5), 0, 0, 5.0])


def test_plain_interpolation_by_hand():
    """dims 16, base 256: frequencies 2^-i; the pair numbers of 256 and 16 turns over 1024 * 2 pi positions are 2 and 6."""
    f, factor = pn.rotation(16, 256.0, {"factor": 4.0, "original": 2.0 * math.pi * 1024.0, "fast": 256.0, "slow": 16.0})
    base, ramp = 2.0 ** -np.arange(8), np.array([0, 0, 0, 0.25, 0.5, 0.75, 1, 1])
    assert np.allclose(f, base * (1 - ramp) + base / 4 * ramp, rtol=1e-12) and factor == 0.1 * math.log(4.0) + 1.0


def test_plain_router_by_hand():
    """Logits 0, ln 3, -ln 3: scores 1/2, 3/4, 1/4; the best two over their sum, times the factor."""
    h, w = np.array([[1.0]]), np.array([[0.0], [math.log(3.0)], [-math.log(3.0)]])
    idx, wts = pn.router_choice(h, w, 2, 2.5)
    assert idx.tolist() == [[1, 0]] and np.allclose(wts, [[1.5, 1.0]])


def test_plain_gate_multiplies_heads():
    """One head, value 1: the output is the gate's logistic."""
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 1, "scale": 1.0, "mask": {"size": 4}, "rot": {"dims": 0, "base": 1.0}}
    w = {"q": np.eye(2), "k": np.eye(2), "v": np.array([[1.0, 0.0]]), "o": np.eye(1), "g": np.array([[0.0, 2.0]]), "q.norm": np.ones(2), "k.norm": np.ones(2)}
    out, _k, _v = pn.chunked_attention(np.array([[1.0, 0.5], [1.0, -1.0]]), w, "", m, 1e-6, [0, 1])
    assert np.allclose(out[:, 0], pn.sigmoid(np.array([1.0, -2.0])))
