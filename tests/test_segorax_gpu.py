"""Segorax on the GPU against the plain implementation (tests/plain_segorax.py): each mechanism alone, then whole models under
every way of cutting, decoding from the first token, slots and pages used again, generation through the engine's own entry
point, the replay program and the command line."""
import numpy as np
import pytest
import torch

import plain_segorax as ps
import replay_util as ru
import segorax_util as su
from conftest import random_tokens

pytestmark = pytest.mark.gpu

DEV = "cuda"
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
# relative root-mean-square error of a logits row against float64
ROW_TOL = {"float32": 5e-5, "bfloat16": 5e-2}


def rel_rms(got, want):
    d = np.asarray(got, dtype=np.float64) - want
    return np.sqrt((d * d).mean(axis=-1)) / max(np.sqrt((want * want).mean()), 1e-9)


def dev(a, dtype=torch.float32):
    return torch.from_numpy(np.ascontiguousarray(a)).to(DEV).to(dtype)


def bf16_round(a):
    return torch.from_numpy(np.asarray(a, dtype=np.float32)).to(torch.bfloat16).float().numpy().astype(np.float64)


def i32(a):
    return torch.tensor(a, dtype=torch.int32, device=DEV)


# ---- one mixer in a pool of pages -----------------------------------------------------------------------------------
class Ctx:
    """What a mixer reads of a step's context: requests given as (first token, tokens, held tokens after the step, table row)."""

    def __init__(self, reqs, page_size, rt):
        self.q_len, self.kv_len = [n for n, _kv in reqs], [kv for _n, kv in reqs]
        self.q_start = np.concatenate([[0], np.cumsum(self.q_len)[:-1]]).tolist()
        self.n_tokens, self.n_requests = sum(self.q_len), len(reqs)
        self.positions = i32(sum([list(range(kv - n, kv)) for n, kv in reqs], []))
        self.token_req = i32(sum([[r] * n for r, (n, _kv) in enumerate(reqs)], []))
        self.max_q_len, self.max_kv_len, self.page_size, self.runtime = max(self.q_len), max(self.kv_len), page_size, rt
        self.plans, self.derived, self.plain_only, self.dump = {}, {}, False, None


class MixerAlone:
    """A latent attention part over a pool of shuffled pages whose unwritten rows are NaN; every request keeps its own pages."""

    def __init__(self, cfg_layer, width, eps, w, dtype, page_size, lengths, seed=0):
        from mimirmind_b200.models.segorax import build_spec
        from mimirmind_b200.config.segorax_config import parse_segorax_config
        from mimirmind_b200.parts.base import Runtime, WeightView
        from mimirmind_b200.registry import MIXERS
        cfg = {"architecture": "Segorax", "vocab": 8, "width": width, "norm": {"eps": eps}, "layers": [dict(cfg_layer, mlp=None)]}
        spec = build_spec(parse_segorax_config(cfg)).layers[0].mixer
        self.rt = Runtime(DT[dtype], torch.device(DEV))
        self.part = MIXERS.get(spec.kind)(spec, WeightView({k: dev(v, DT[dtype]) for k, v in w.items()}), self.rt)
        self.page_size, m = page_size, cfg_layer["mixer"]
        rng = np.random.RandomState(seed)
        need = [-(-n // page_size) for n in lengths]
        perm = rng.permutation(sum(need) + 5)
        self.width_pages = max(need)
        self.tables, at = [], 0
        for k in need:
            self.tables.append(perm[at:at + k].tolist() + [-1] * (self.width_pages - k))
            at += k
        self.pool = torch.full((sum(need) + 5, 1, page_size, m["kv_rank"] + m["rot_dim"]), float("nan"), dtype=DT[dtype], device=DEV)

    def step(self, xs, which, starts):
        """xs: rows per request of the batch; which: their requests; starts: how many tokens each held before."""
        from mimirmind_b200.parts.base import LayerCache
        ctx = Ctx([(len(x), s + len(x)) for x, s in zip(xs, starts)], self.page_size, self.rt)
        cache = LayerCache(arrays={"latent": self.pool}, block_table=i32([self.tables[r] for r in which]), page_size=self.page_size)
        out = self.part.forward(dev(np.concatenate(xs), self.rt.dtype), ctx, cache).float().cpu().numpy()
        return [out[s:s + n] for s, n in zip(ctx.q_start, ctx.q_len)]


def mixer_weights(layer, width, rng, dtype, gain=1.0):
    shapes = {k[len("l0."):]: v for k, v in su.tensor_shapes({"width": width, "vocab": 8, "layers": [dict(layer, mlp=None)]}).items() if k.startswith("l0.mix")}
    w = {}
    for k, shape in shapes.items():
        w[k] = 1.0 + 0.1 * rng.randn(*shape) if k.endswith("norm") else (1.0 + rng.randn(*shape) if k.endswith("sink") else gain * rng.randn(*shape) / np.sqrt(shape[1]))
    return {k: bf16_round(v) if dtype == "bfloat16" else np.asarray(v, dtype=np.float32).astype(np.float64) for k, v in w.items()}


def plain_mixer(x, w, layer, eps):
    low = layer["type"] == "latent_attention"
    return ps.latent_attention(x, w, "mix.", layer["mixer"], eps, list(range(len(x))), low, low)


@pytest.fixture(params=["tensor-memory", "absorbed", "fp32-arithmetic"])
def route(request, monkeypatch):
    """Long portions over keys and values made in full (sizes that kernel takes), always the absorbed form on the tensor cores, or
    the fp32-arithmetic kernel only."""
    from mimirmind_b200.kernels import attention
    monkeypatch.setattr(attention, "USE_LATENT_EXPANDED", request.param == "tensor-memory")
    monkeypatch.setattr(attention, "USE_LATENT_MMA", request.param != "fp32-arithmetic")
    yield request.param
    from mimirmind_b200.kernels import ops
    ops.check_tcgen05_errors(torch.device(DEV))


MIXERS_ALONE = {
    "low, sizes of tiles": su.low(4, 64, 64, 128, 96, 128, 0.09, 10000.0, None),
    "low, narrow": su.low(6, 24, 8, 40, 40, 48, 0.3, 100.0, None),
    "low, one head": su.low(1, 64, 32, 72, 64, 80, 0.12, 500.0, None),
    "low, many heads": su.low(40, 16, 16, 24, 72, 32, 0.25, 3000.0, None),
    "low, odd sizes": su.low(3, 9, 6, 5, 21, 19, 0.4, 40.0, None),
    "low, a wide latent": su.low(3, 96, 64, 104, 128, 512, 0.08, 50000.0, None),
    "far, sizes of tiles": su.far(3, 128, 64, 64, 192, 0.07, 10000.0, (8.0, 96, 32.0, 1.0), None),
    "far, narrow": su.far(5, 16, 16, 8, 64, 0.3, 300.0, (4.0, 100, 8.0, 1.0), None),
    "far, wide": su.far(2, 160, 32, 136, 64, 0.07, 7000.0, (3.0, 300, 20.0, 2.0), None),
    "far, four pieces": su.far(3, 136, 64, 120, 96, 0.07, 7000.0, (3.0, 300, 20.0, 2.0), None),
    "far, two rotated pieces": su.far(5, 8, 72, 56, 40, 0.12, 900.0, (6.0, 150, 30.0, 1.0), None),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(MIXERS_ALONE))
def test_latent_attention_alone(name, dtype, route):
    """One mixer, three requests: a long prompt whole, then portions of several sizes beside single tokens of others, over pages
    of their own in a pool full of NaN."""
    if dtype == "float32" and route != "tensor-memory":
        pytest.skip("the 32-bit mode has one route")
    layer, width, eps = MIXERS_ALONE[name], 96, 1e-5
    rng = np.random.RandomState(len(name))
    w = mixer_weights(layer, width, rng, dtype)
    lengths = [300, 170, 401]
    xs = [rng.randn(n, width) for n in lengths]
    if dtype == "bfloat16":
        xs = [bf16_round(x) for x in xs]
    want = [plain_mixer(x, w, layer, eps) for x in xs]
    scale = max(np.abs(v).max() for v in want)
    tol = (3e-5 if dtype == "float32" else 3e-2) * scale
    for page in (16, 8):
        m = MixerAlone(layer, width, eps, w, dtype, page, lengths, seed=page)
        held = [0, 0, 0]
        for batch in ([(0, 300)], [(1, 90), (2, 129)], [(2, 2), (1, 1)], [(1, 77), (2, 1)], [(1, 1), (2, 65)], [(2, 3), (1, 1)], [(2, 200)], [(2, 1)]):
            got = m.step([xs[r][held[r]:held[r] + n] for r, n in batch], [r for r, _ in batch], [held[r] for r, _ in batch])
            for (r, n), g in zip(batch, got):
                assert not np.isnan(g).any(), (page, r, held[r], n)
                err = np.abs(g - want[r][held[r]:held[r] + n]).max()
                assert err <= tol, (page, r, held[r], n, err, tol)
                held[r] += n
        assert held == lengths


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["low", "far"])
def test_one_key_that_stands_out(kind, dtype, route):
    """One token's shared key part answers one query direction far above the rest (through the rotation, whatever the distance):
    the asker's result is that token's value.  Spots at the sequence's start, at page borders and tile borders, and hundreds of
    tokens back; asked in a portion, in a portion of two tokens and alone; and the token just behind the asker stays unseen."""
    if dtype == "float32" and route != "tensor-memory":
        pytest.skip("the 32-bit mode has one route")
    H, dk, dr, dv, r, T, width, page = 2, 16, 16, 16, 32, 620, 64, 16
    layer = su.low(H, dk, dr, dv, 48, r, 1.0, 1e9, None) if kind == "low" else su.far(H, dk, dr, dv, r, 1.0, 1e9, (1.0, 64, 32.0, 1.0), None)
    rng = np.random.RandomState(7)
    w = mixer_weights(layer, width, rng, dtype, 0.3)
    # numbers 14, 15 of the rotated part turn by 1e9^(-14/16) a position: not measurably over this sequence
    q_name = "mix.uq" if kind == "low" else "mix.q"
    w["mix.dkv"][r:] = 0.0
    w["mix.dkv"][r + 15, 0] = 1.0                                   # the shared key part is x[0]
    w[q_name][:] = 0.0
    if kind == "low":
        w["mix.dq"][:] = 0.0
        w["mix.dq"][0, 1], w["mix.dq"][1, 2] = 1.0, 1.0             # x[1] asks, x[2] is a constant that keeps the latent's norm
        w["mix.dq.norm"][:] = 1.0
        w["mix.sink"][:] = -3.0
        for h in range(H):
            w[q_name][h * (dk + dr) + dk + 15, 0] = 8.0
    else:
        for h in range(H):
            w[q_name][h * (dk + dr) + dk + 15, 1] = 8.0
    if dtype == "bfloat16":
        w = {k: bf16_round(v) for k, v in w.items()}
    for spot in (0, 1, 15, 16, 31, 63, 64, 127, 128, 300, 511):
        x = 0.5 * rng.randn(T, width)
        x[:, 0], x[:, 1], x[:, 2] = 0.0, 0.0, 1.0
        x[spot, 0] = 12.0
        askers = sorted({min(T - 1, spot + d) for d in (0, 1, 2, 33, 130)} | {T - 1})
        x[askers, 1] = 4.0
        if spot in askers:
            x[spot, 1] = 4.0
        if dtype == "bfloat16":
            x = bf16_round(x)
        want = plain_mixer(x, w, layer, 1e-6)
        latent = ps.rms_norm((x @ w["mix.dkv"].T)[:, :r], w["mix.dkv.norm"], 1e-6)
        pinned = (latent[spot] @ w["mix.uv"].T) @ w["mix.o"].T
        tol = (1e-4 if dtype == "float32" else 3e-2) * np.abs(want).max()
        for a in askers:
            assert np.abs(want[a] - pinned).max() <= 1e-3 * np.abs(pinned).max()       # the set-up does what it says
        m = MixerAlone(layer, width, 1e-6, w, dtype, page, [T, T], seed=spot)
        whole = m.step([x], [0], [0])[0]
        assert np.abs(whole - want).max() <= tol, spot
        held = 0
        for a in askers:                                       # up to the asker in a portion, it in a portion of two or alone
            pair = (a % 2 == 0) and a - 1 > held
            head = a - (1 if pair else 0)
            if head > held:
                g = m.step([x[held:head]], [1], [held])[0]
                assert np.abs(g - want[held:head]).max() <= tol, (spot, a)
            g = m.step([x[head:a + 1]], [1], [head])[0]
            assert np.abs(g - want[head:a + 1]).max() <= tol and np.abs(g[-1] - pinned).max() <= tol, (spot, a, pair)
            held = a + 1
        if spot > 0:                                           # the token before the spot does not see it
            assert np.abs(whole[spot - 1] - want[spot - 1]).max() <= tol and np.abs(want[spot - 1] - pinned).max() > 10 * tol


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_sink_takes_its_share(dtype, route):
    """A sink that drowns a head, one that vanishes and one that weighs as much as a key of score 0, over a portion, a portion of two
    tokens and single tokens (whose keys are shared out over several blocks: the sink counts once)."""
    if dtype == "float32" and route != "tensor-memory":
        pytest.skip("the 32-bit mode has one route")
    layer, width = su.low(3, 16, 16, 32, 32, 64, 0.2, 100.0, None), 96
    rng = np.random.RandomState(5)
    w = mixer_weights(layer, width, rng, dtype, 0.7)
    w["mix.sink"] = np.array([60.0, -60.0, 0.0])
    w["mix.o"] = np.eye(width)
    T = 420
    x = rng.randn(T, width)
    x = bf16_round(x) if dtype == "bfloat16" else x
    want = plain_mixer(x, w, layer, 1e-6)
    none = ps.latent_attention(x, w, "mix.", layer["mixer"], 1e-6, list(range(T)), True, False)
    tol = (2e-5 if dtype == "float32" else 3e-2) * np.abs(none).max()
    m = MixerAlone(layer, width, 1e-6, w, dtype, 16, [T], seed=1)
    got = np.concatenate([m.step([x[a:b]], [0], [a])[0] for a, b in ((0, 3), (3, 4), (4, 200), (200, 202), (202, 203), (203, 419), (419, 420))])
    assert np.abs(got - want).max() <= tol
    assert np.abs(got[:, :32]).max() < 1e-6 and np.abs(got[:, 32:64] - none[:, 32:64]).max() <= tol
    assert np.abs(want[:, 64:] - none[:, 64:])[:40].max() > 3 * tol


@pytest.mark.parametrize("scaling", [None, (4.0, 64, 16.0, 1.0), (40.0, 4096, 32.0, 1.0)])
def test_rotation_of_neighbours_far_out(scaling):
    """Positions up to 500,000 turn as exactly as near ones; with interpolation both cos and sin carry the factor; numbers beyond
    ``rot_dims`` pass.  The latent's norm and the pages they land in."""
    from mimirmind_b200.kernels import ops
    from mimirmind_b200.parts.latent_attention import split_frequencies
    from mimirmind_b200.parts.rope import exact_frequencies
    rng = np.random.RandomState(11)
    H, dk, dr, r, rot, page, base, eps = 3, 5, 14, 22, 12, 8, 10000.0, 1e-5
    sc = dict(zip(("factor", "original", "fast", "slow"), scaling)) if scaling else None
    positions = np.array([0, 1, 7, 8, 4095, 100000, 500001])
    n = len(positions)
    c_rows, q_rows, wn = rng.randn(n, 4 + r + dr), rng.randn(n, H * (dk + dr)), 1.0 + 0.1 * rng.randn(r)
    hi, lo = split_frequencies(base, rot, DEV, sc)
    table = ops.rope_half_table(i32(positions.tolist()), hi, lo, exact_frequencies(base, rot, sc)[1])
    q_plain, q_full = torch.zeros((n, H * dk), device=DEV), torch.zeros((n, H * (r + dr)), device=DEV)
    pages = torch.zeros((n, 1, page, r + dr), device=DEV)
    slots = i32([t * page + t % page for t in range(n)])
    ops.latent_prep(dev(c_rows), 0, 4, dev(wn), eps, table, rot, q_plain, q_full, pages, slots, page, H, dk, dr, r, q_rows=dev(q_rows), pairs=True)
    q = q_rows.astype(np.float32).astype(np.float64).reshape(n, H, dk + dr)
    c = c_rows.astype(np.float32).astype(np.float64)[:, 4:]
    assert np.array_equal(q_plain.cpu().numpy().reshape(n, H, dk), q[..., :dk].astype(np.float32))
    turned = ps.rotate_pairs(q[..., dk:], positions, rot, base, sc)
    assert np.abs(q_full.cpu().numpy().reshape(n, H, r + dr)[..., r:] - turned).max() <= 4e-6
    key = ps.rotate_pairs(c[:, r:], positions, rot, base, sc)
    lat = ps.rms_norm(c[:, :r], wn.astype(np.float32), eps)
    for t in range(n):
        row = pages[t, 0, t % page].cpu().numpy()
        assert np.abs(row[:r] - lat[t]).max() <= 4e-6 and np.abs(row[r:] - key[t]).max() <= 4e-6
    assert int((pages.abs().sum(dim=-1) > 0).sum()) == n


# ---- experts ----------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("E,top,groups", [(9, 2, (3, 1)), (12, 4, (4, 2)), (8, 8, None), (6, 1, (6, 2)), (32, 8, (8, 3)), (160, 6, (8, 4)), (5, 3, None), (72, 5, (36, 30))])
@pytest.mark.parametrize("D", [40, 51])
def test_the_routers_choice(E, top, groups, D):
    """Corrections of both signs that reorder the experts and make choice scores negative; the weights are the plain scores."""
    from mimirmind_b200.kernels import ops
    rng = np.random.RandomState(E)
    for n in (3, 2100):
        x, w, corr = rng.randn(n, D).astype(np.float32), (rng.randn(E + 1, D) * 0.4).astype(np.float32), (rng.randn(E) - 0.5).astype(np.float32)
        count, keep = groups or (1, 1)
        idx, wts, gate = ops.moe_router(dev(x), dev(w), top, count, keep, scoring="sigmoid", correction=dev(corr), group_score="top2_sum", gate=True)
        z = x.astype(np.float64) @ w.T.astype(np.float64)
        want, s = ps.router_choice(x.astype(np.float64), w[:E].astype(np.float64), corr.astype(np.float64), top, groups)
        same = (np.sort(idx.cpu().numpy(), 1) == np.sort(want, 1)).all(1)
        assert same.mean() >= 0.999                                     # float64 against fp32: near ties of thousands of rows
        assert np.abs(np.sort(wts.cpu().numpy(), 1) - np.sort(s, 1))[same].max() <= 2e-6
        assert np.abs(gate.cpu().numpy() - ps.sigmoid(z[:, E])).max() <= 2e-6
        plain_idx, plain_w = ops.moe_router(dev(x), dev(w[:E]), top, count, keep, scoring="sigmoid")    # without correction and gate: best-expert groups
        assert (ps.sigmoid(z[:, :E])[np.arange(n)[:, None], plain_idx.cpu().numpy()] - plain_w.cpu().numpy()).__abs__().max() <= 2e-6


def test_groups_count_by_their_two_best():
    """The first group has the best expert, the second the best two: one rule takes the one, the other rule the other."""
    from mimirmind_b200.kernels import ops
    x, w = torch.ones((2, 4), device=DEV), torch.zeros((6, 4), device=DEV)
    corr = dev(np.array([9.0, -8.0, 3.0, 2.0, 1.0, -0.5]))
    pick = lambda rule: sorted(ops.moe_router(x, w, 2, 3, 1, scoring="sigmoid", correction=corr, group_score=rule)[0][0].tolist())
    assert pick("top2_sum") == [2, 3] and pick("max") == [0, 1]
    # every choice score negative: minus infinity, not zero, keeps the dropped groups out
    idx, wts = ops.moe_router(x, w, 2, 3, 1, scoring="sigmoid", correction=dev(np.array([-1.0, -2.0, -9.0, -1.2, -3.0, -3.0])), group_score="top2_sum")
    assert sorted(idx[1].tolist()) == [0, 1] and np.allclose(wts.cpu().numpy(), 0.5)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n,d,ff,E,top,groups,shared", [(70, 64, 40, 9, 2, (3, 1), 24), (1, 50, 9, 4, 3, (4, 3), 7), (8, 256, 96, 16, 4, (4, 2), 64), (300, 128, 64, 8, 3, None, None),
                                                        (16, 320, 128, 6, 2, None, 33), (17, 320, 128, 6, 2, (3, 2), 128), (2100, 96, 32, 6, 2, (2, 1), 48), (600, 72, 136, 5, 4, None, 16)])
def test_experts_of_two_matrices_against_the_plain_ones(n, d, ff, E, top, groups, shared, dtype):
    """Every product route (a decode step's tiles, a portion's, a prompt's grouped products, 32-bit), whole and in pieces."""
    from mimirmind_b200.config.spec import PartSpec
    from mimirmind_b200.kernels import ops
    from mimirmind_b200.parts.base import Runtime, WeightView
    from mimirmind_b200.parts.moe import RoutedExperts
    rng = np.random.RandomState(n + d)
    w = {"mlp.router": rng.randn(E, d) * 4.0 / np.sqrt(d), "mlp.correction": rng.randn(E) * 0.7}
    for e in range(E):
        w.update({f"mlp.e{e}.up": rng.randn(ff, d) * 1.5 / np.sqrt(d), f"mlp.e{e}.down": rng.randn(d, ff) / np.sqrt(ff)})
    mlp = {"router": {"top": top}}
    if groups:
        mlp["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    shared_spec = None
    if shared:
        w.update({"mlp.shared.up": rng.randn(shared, d) * 1.5 / np.sqrt(d), "mlp.shared.down": rng.randn(d, shared) / np.sqrt(shared), "mlp.shared.sg": rng.randn(1, d) * 2.0 / np.sqrt(d)})
        mlp["shared"] = {"ff": shared}
        shared_spec = PartSpec("dense_mlp", {"hidden": d, "ff": shared, "activation": "gelu_erf", "up": "mlp.shared.up", "down": "mlp.shared.down"})
    w = {k: bf16_round(v) for k, v in w.items()}
    x = bf16_round(rng.randn(n, d))
    spec = PartSpec("routed_experts", {"hidden": d, "ff": ff, "experts": E, "top": top, "groups": (groups or (1, 1))[0], "keep": (groups or (1, 1))[1], "gated": False,
                                       "router": "mlp.router", "expert": "mlp.e{}", "scoring": "sigmoid", "correction": "mlp.correction", "group_score": "top2_sum",
                                       "activation": "gelu_erf", "shared": shared_spec, "shared_gate": "mlp.shared.sg" if shared else None})
    rt = Runtime(DT[dtype], torch.device(DEV))
    ctx = Ctx([(n, n)], 16, rt)
    part = RoutedExperts(spec, WeightView({k: dev(v, DT[dtype]) for k, v in w.items()}), rt)
    want = ps.experts_feed_forward(x, w, "mlp.", mlp)
    got = part.forward(dev(x, DT[dtype]), ctx).float().cpu().numpy()
    b = part.forward_split(dev(x, DT[dtype]), ctx)
    place = torch.arange(n * top, device=DEV) if b.place is None else b.place.long()
    y = (b.rows.float()[place].reshape(n, top, d) * b.weights[:, :, None]).sum(1)
    if shared:
        y = y + b.gate[:, None] * b.other.float()
    for g in (got, y.cpu().numpy()):
        err = np.abs(g - want).max(axis=-1) / np.abs(want).max()
        if dtype == "float32":
            assert err.max() <= 2e-5
        else:
            assert np.median(err) <= 2e-2 and (err > 5e-2).mean() <= 0.02
    ops.check_tcgen05_errors(torch.device(DEV))


# ---- dense feed-forward, norms and the small passes ---------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n,d,ff", [(1, 256, 96), (8, 320, 480), (9, 64, 48), (33, 512, 640), (64, 320, 96), (65, 96, 80), (256, 256, 136), (500, 320, 264), (70, 50, 21), (5, 72, 33)])
def test_the_gated_feed_forward_with_the_tanh_form_of_gelu(n, d, ff, dtype):
    """Every route: weight-streaming products of up to 8 and up to 64 rows, the pass of its own, the tcgen05 product, 32-bit."""
    from mimirmind_b200.config.spec import PartSpec
    from mimirmind_b200.kernels import ops
    from mimirmind_b200.parts.base import Runtime, WeightView
    from mimirmind_b200.parts.mlp import SwiGLU
    rng = np.random.RandomState(n * d)
    w = {"mlp.gate": bf16_round(rng.randn(ff, d) * 2.0 / np.sqrt(d)), "mlp.up": bf16_round(rng.randn(ff, d) / np.sqrt(d)), "mlp.down": bf16_round(rng.randn(d, ff) / np.sqrt(ff))}
    x = bf16_round(rng.randn(n, d))
    rt = Runtime(DT[dtype], torch.device(DEV))
    spec = PartSpec("swiglu", {"hidden": d, "intermediate": ff, "activation": "gelu_tanh", "gate": "mlp.gate", "up": "mlp.up", "down": "mlp.down"})
    part = SwiGLU(spec, WeightView({k: dev(v, DT[dtype]) for k, v in w.items()}), rt)
    assert part.native() is None and not part.fuses(n)
    got = part.forward(dev(x, DT[dtype]), Ctx([(n, n)], 16, rt)).float().cpu().numpy()
    want = ps.dense(x, w, "mlp.")
    assert np.abs(got - want).max() <= (2e-5 if dtype == "float32" else 2e-2) * np.abs(want).max()
    ops.check_tcgen05_errors(torch.device(DEV))


@pytest.mark.parametrize("n,d,ff", [(1, 256, 64), (8, 512, 96), (20, 96, 48), (64, 64, 128), (300, 4096, 256), (40, 50, 21)])
def test_the_exact_gelu_on_every_route(n, d, ff):
    from mimirmind_b200.config.spec import PartSpec
    from mimirmind_b200.parts.base import Runtime, WeightView
    from mimirmind_b200.parts.mlp import DenseMLP
    rng = np.random.RandomState(ff)
    w = {"up": bf16_round(rng.randn(ff, d) * 2.0 / np.sqrt(d)), "down": bf16_round(rng.randn(d, ff) / np.sqrt(ff))}
    x = bf16_round(rng.randn(n, d))
    want = ps.gelu_erf(x @ w["up"].T) @ w["down"].T
    for dtype in ("float32", "bfloat16"):
        rt = Runtime(DT[dtype], torch.device(DEV))
        part = DenseMLP(PartSpec("dense_mlp", {"hidden": d, "ff": ff, "activation": "gelu_erf", "up": "up", "down": "down"}),
                        WeightView({k: dev(v, DT[dtype]) for k, v in w.items()}), rt)
        got = part.forward(dev(x, DT[dtype]), Ctx([(n, n)], 16, rt)).float().cpu().numpy()
        assert np.abs(got - want).max() <= (2e-5 if dtype == "float32" else 2e-2) * np.abs(want).max(), dtype


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n,d", [(5, 64), (33, 54), (2, 4096), (3, 1160), (1, 13000)])
def test_the_norm_on_a_sublayers_output(n, d, dtype):
    """One branch, two of which one is gated per token, and rows of chosen experts in the order of the choice or by place; a branch
    so small that eps matters."""
    from mimirmind_b200.kernels import ops
    rng = np.random.RandomState(d)
    x, w, top = rng.randn(n, d), 1.0 + 0.1 * rng.randn(d), 3
    f32 = lambda t: t.astype(np.float32).astype(np.float64)
    act = (lambda t: bf16_round(t)) if dtype == "bfloat16" else f32
    a, b, rows = act(rng.randn(n, d)), act(rng.randn(n, d)), rng.randn(n * top, d)
    gate, wts, place = rng.rand(n), rng.rand(n, top), rng.permutation(n * top)
    x32, w32 = f32(x), f32(w)
    cases = [("one", a, dict(), a), ("tiny", act(1e-3 * a), dict(), act(1e-3 * a)),
             ("two", a, dict(b=dev(b, DT[dtype]), gate=dev(gate), ca=0.8, cb=1.1), 0.8 * a + 1.1 * f32(gate)[:, None] * b),
             ("two, no gate", a, dict(b=dev(b, DT[dtype])), a + b)]
    for where in (None, place):
        for row_dtype in ((torch.float32,) if dtype == "float32" else (torch.float32, torch.bfloat16)):
            r = bf16_round(rows) if row_dtype == torch.bfloat16 else f32(rows)
            if where is None and row_dtype == torch.bfloat16:
                continue
            y = (r[np.arange(n * top) if where is None else where].reshape(n, top, d) * f32(wts)[:, :, None]).sum(1)
            cases.append(("rows", (r, row_dtype), dict(wts=dev(wts), place=None if where is None else i32(where.tolist()), b=dev(b, DT[dtype]), gate=dev(gate)), y + f32(gate)[:, None] * b))
            if row_dtype == DT[dtype]:
                cases.append(("rows alone", (r, row_dtype), dict(wts=dev(wts), place=None if where is None else i32(where.tolist())), y))
    for what, branch, kw, y in cases:
        res = dev(x)
        t = dev(branch[0], branch[1]) if isinstance(branch, tuple) else dev(branch, DT[dtype])
        out = torch.empty((n, d), dtype=DT[dtype], device=DEV)
        ops.output_norm(res, t, dev(w), 1e-5, 0.37, out=out, **kw)
        want = x32 + 0.37 * ps.rms_norm(y, w32, 1e-5)
        assert np.abs(res.cpu().numpy() - want).max() <= 2e-6 * np.abs(want).max() + 1e-6, what
        assert torch.equal(out, res.to(DT[dtype])), what


def test_a_gated_sum_and_interleaved_activations():
    from mimirmind_b200.kernels import ops
    rng = np.random.RandomState(2)
    a, b, g = rng.randn(7, 33), rng.randn(7, 33), rng.rand(7)
    got = ops.scaled_sum2(dev(a), dev(b), 0.5, 2.0, dev(g)).cpu().numpy()
    assert np.abs(got - (0.5 * a + 2.0 * g[:, None] * b)).max() <= 1e-5
    gate, up = rng.randn(5, 24), rng.randn(5, 24)
    both = np.stack([gate.reshape(5, 3, 8), up.reshape(5, 3, 8)], 2).reshape(5, 48)
    want = ps.gelu_tanh(gate) * up
    assert np.abs(ops.glu_rows(dev(both), torch.float32, "gelu_tanh", interleave=8).cpu().numpy() - want).max() <= 1e-5
    assert np.abs(ops.glu_rows(dev(np.concatenate([gate, up], 1)), torch.float32, "gelu_tanh").cpu().numpy() - want).max() <= 1e-5


# ---- whole models -------------------------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def models(tmp_path_factory):
    cache = {}

    def get(name, dtype="float32"):
        """The 16-bit runs get the model with every expert chosen: one expert taken for another on a near tie of rounded scores
        changes a row by far more than rounding does, which says nothing about the kernels.  The choice among experts is held to
        the plain implementation by the 32-bit runs and by the experts' own tests."""
        key = (name, dtype == "bfloat16")
        if key not in cache:
            cfg = su.every_expert_chosen(su.CONFIGS[name]) if key[1] else su.CONFIGS[name]
            folder = su.write_model(str(tmp_path_factory.mktemp(f"segorax_{name}")), cfg, seed=len(cache) + 17)
            cache[key] = (folder,) + ps.load_folder(folder)
        return cache[key]

    return get


def check_rows(trace, outputs, reqs, ref, dtype, what):
    got = ru.collect(trace, outputs)
    for rid, toks in reqs.items():
        err = rel_rms(np.stack([got[(rid, p)] for p in range(len(toks))]), ref[rid])
        over = int((err > ROW_TOL[dtype]).sum())
        assert over == 0 and not np.isnan(err).any(), (
            f"{what} {dtype} request {rid}: {over} of {len(toks)} rows above the bound, median {np.median(err):.3g}, worst {err.max():.3g} at "
            f"position {int(err.argmax())}, first above: {int(np.argmax(err > ROW_TOL[dtype]))}")
    return got


@pytest.mark.parametrize("name", sorted(su.CONFIGS))
def test_every_layer_against_the_plain_stream(name, models):
    """The residual stream after every layer of a short prompt, in float32."""
    from mimirmind_b200.engine.loader import load_model
    from mimirmind_b200.engine.runner import ModelRunner, StepEntry

    class Keep:
        def __init__(self):
            self.rows = {}

        def write(self, block, stage, rows):
            if stage == "l_out":
                self.rows[block] = rows.detach().float().cpu().numpy().copy()

    folder, cfg, w = models(name)
    toks = random_tokens(cfg["vocab"], 29, 3)
    streams = []
    ps.forward(cfg, w, toks, collect=streams)
    model, _ = load_model(folder, "float32")
    runner = ModelRunner(model, page_size=16, num_pages=8, max_requests=2)
    keep = Keep()
    runner.stage_dump = keep
    runner.add_request("s")
    runner.step([StepEntry("s", toks, [28])])
    assert sorted(keep.rows) == list(range(len(cfg["layers"])))
    for i, want in enumerate(streams):
        assert np.abs(keep.rows[i] - want).max() <= 3e-5 * np.abs(want).max(), f"layer {i}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,page_size", [("A", 16), ("B", 16), ("C", 8), ("A", 32), ("D", 16)])
def test_every_way_of_cutting_matches_the_plain_implementation(name, page_size, dtype, models):
    folder, cfg, w = models(name, dtype)
    reqs = {f"{name}{i}": random_tokens(cfg["vocab"], n, 100 * i + n) for i, n in enumerate(su.LENGTHS[name])}
    ref = {rid: ps.forward(cfg, w, t) for rid, t in reqs.items()}
    results = {}
    t = ru.Trace()
    for rid, toks in reqs.items():
        ru.whole(t, rid, toks)
    out, _ = ru.run_in_process(folder, dtype, t, t.max_live_tokens(), page_size)
    results["whole"] = check_rows(t, out, reqs, ref, dtype, "whole")
    t = ru.Trace()
    for rid, toks in reqs.items():
        ru.tail_one_by_one(t, rid, toks, 80)
    out, _ = ru.run_in_process(folder, dtype, t, t.max_live_tokens(), page_size)
    results["tail"] = check_rows(t, out, reqs, ref, dtype, "tail one by one")
    t = ru.Trace()
    for i, (rid, toks) in enumerate(reqs.items()):
        ru.chunks(t, rid, toks, [[17, 7, 5, 3, 2], [2, 64, 3, 31], [33, 2, 2, 65, 128], [2]][i % 4])
    out, _ = ru.run_in_process(folder, dtype, t, t.max_live_tokens(), page_size)
    results["chunks"] = check_rows(t, out, reqs, ref, dtype, "portions")
    t = ru.Trace()
    twice = dict(reqs)
    twice.update({rid + "x": toks for rid, toks in reqs.items()})
    ru.mixed(t, twice, seed=len(name) + page_size)
    out, runner = ru.run_in_process(folder, dtype, t, t.max_live_tokens(), page_size)
    ref2 = dict(ref)
    ref2.update({rid + "x": ref[rid] for rid in reqs})
    results["mixed"] = check_rows(t, out, twice, ref2, dtype, "mixed")
    assert runner.manager.reuses() > 0, "the pool was large enough that no page was used again"
    for g in runner.manager.groups:
        assert runner.manager.free_pages(g) == runner.manager.total_pages(g)
    if dtype == "float32":
        # the 32-bit kernels sum in an order fixed by position: cutting changes nothing at all
        for mode in ("tail", "chunks", "mixed"):
            for key, row in results["whole"].items():
                assert np.array_equal(results[mode][key], row), f"{mode}: {key} differs from the whole run"


@pytest.mark.parametrize("name,dtype", [("A", "float32"), ("C", "float32"), ("D", "bfloat16")])
def test_decoding_from_the_first_token(name, dtype, models):
    folder, cfg, w = models(name, dtype)
    toks = random_tokens(cfg["vocab"], 260, 5)
    t = ru.Trace()
    ru.chunks(t, "d", toks, [1])
    out, _ = ru.run_in_process(folder, dtype, t, t.max_live_tokens())
    check_rows(t, out, {"d": toks}, {"d": ps.forward(cfg, w, toks)}, dtype, "decode from the first token")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_pages_and_slots_used_again_start_clean(dtype, models):
    """Two slots and just enough pages, five requests one after the other and in pairs: none sees what another left."""
    from mimirmind_b200.engine.loader import load_model
    from mimirmind_b200.engine.runner import ModelRunner, StepEntry
    folder, cfg, w = models("B", dtype)
    model, _ = load_model(folder, dtype)
    runner = ModelRunner(model, page_size=16, num_pages=13, max_requests=2)
    reqs = [random_tokens(cfg["vocab"], n, n) for n in (80, 3, 110, 31, 140)]
    ref = [ps.forward(cfg, w, t) for t in reqs]
    assert runner.add_request(0) and runner.add_request(1) and not runner.add_request(2)
    got0 = runner.step([StepEntry(0, reqs[0][:70], [69]), StepEntry(1, reqs[1], [2])]).cpu().numpy()
    runner.release(1)
    assert runner.add_request(2)
    got1 = runner.step([StepEntry(2, reqs[2][:7], [6]), StepEntry(0, reqs[0][70:], [9])]).cpu().numpy()
    runner.release(0)
    assert runner.add_request(3)
    got2 = runner.step([StepEntry(3, reqs[3], [30]), StepEntry(2, reqs[2][7:], [102])]).cpu().numpy()
    runner.release(2), runner.release(3)
    assert runner.add_request(4)
    got3 = runner.step([StepEntry(4, reqs[4], [0, 139])]).cpu().numpy()
    for got, want in ((got0[0], ref[0][69]), (got0[1], ref[1][2]), (got1[0], ref[2][6]), (got1[1], ref[0][79]), (got2[0], ref[3][30]),
                      (got2[1], ref[2][109]), (got3[0], ref[4][0]), (got3[1], ref[4][139])):
        assert rel_rms(got, want) <= ROW_TOL[dtype]


@pytest.mark.parametrize("name,dtype", [("A", "float32"), ("B", "bfloat16")])
def test_greedy_generation_through_the_engine(name, dtype, models):
    """Engine.generate (scheduler, prompt portions, captured decode steps) picks the plain implementation's tokens."""
    from mimirmind_b200 import Engine
    folder, cfg, w = models(name, dtype)
    prompts = [random_tokens(cfg["vocab"], n, 40 + n) for n in (5, 17, 33, 90)]
    eng = Engine.from_folder(folder, dtype=dtype, page_size=16, cache_tokens=1024, max_context=512, token_budget=80, max_active=4)
    res = eng.generate(prompts, max_new_tokens=24)
    exact = 0
    for p, r in zip(prompts, res):
        assert r.stats.generated_tokens == 24 and r.stats.finish_reason == "length"
        rows = ps.forward(cfg, w, list(p) + list(r.tokens))[len(p) - 1:-1]
        for i, tok in enumerate(r.tokens):
            best = int(np.argmax(rows[i]))
            exact += tok == best
            if dtype == "float32":
                assert rows[i][tok] >= rows[i][best] - 1e-4, f"token {i}: engine chose {tok}, plain {best}"
    assert exact >= (96 if dtype == "float32" else 80)
    assert eng.runner.manager.free_pages() == eng.runner.manager.total_pages()
    again = eng.generate(prompts, max_new_tokens=24)          # slots and pages used again
    if dtype == "float32":
        assert [r.tokens for r in again] == [r.tokens for r in res]


def test_the_replay_program_on_this_design(models, tmp_path):
    folder, cfg, w = models("C")
    reqs = {f"r{i}": random_tokens(cfg["vocab"], n, 11 + i) for i, n in enumerate([3, 90, 41, 150])}
    ref = {rid: ps.forward(cfg, w, t) for rid, t in reqs.items()}
    t = ru.Trace()
    ru.mixed(t, reqs, seed=3)
    t.step([("last", [1, 2, 3], [])], end=["last"])
    out = ru.run_program(folder, "float32", t, t.max_live_tokens(), str(tmp_path / "out"), cfg["vocab"])
    check_rows(t, out, reqs, ref, "float32", "program")


def test_the_command_line_generates_with_this_design(models, tmp_path):
    """bin/mimirmind: smoke generates from a test model (its greedy tokens are the plain implementation's); random-weights
    mode writes a folder of this design from its config.json, and smoke generates from that too."""
    import json
    import os
    import subprocess
    import sys
    from conftest import ROOT
    folder, cfg, w = models("A")
    exe = [sys.executable, os.path.join(ROOT, "bin", "mimirmind")]
    conf = {"defaultModel": "m", "models": [{"id": "m", "path": folder}], "runtime": {"dtype": "float32", "maxContextTokens": 256, "cacheTokens": 512}}
    (tmp_path / "config.json").write_text(json.dumps(conf))
    out = subprocess.run(exe + ["smoke", "--config", str(tmp_path / "config.json"), "--prompt", "5 17 3 99", "--max-new", "6"],
                         capture_output=True, text=True, timeout=300)
    assert out.returncode == 0, out.stderr
    lines = out.stdout.strip().splitlines()
    got = [int(t) for t in lines[0].split()]
    assert len(got) == 6 and lines[1] == "generated 6"
    toks = [5, 17, 3, 99]
    for tok in got:
        row = ps.forward(cfg, w, toks)[-1]
        assert row[tok] >= row.max() - 1e-4
        toks.append(tok)
    (tmp_path / "mc.json").write_text(json.dumps(su.CONFIGS["B"]))
    rw = subprocess.run(exe + ["random-weights", "--model-config", str(tmp_path / "mc.json"), "--seed", "9", "--out", str(tmp_path / "rw"),
                               "--dtype", "bfloat16"], capture_output=True, text=True, timeout=300)
    assert rw.returncode == 0, rw.stderr
    conf["models"][0]["path"] = str(tmp_path / "rw")
    conf["runtime"]["dtype"] = "bfloat16"
    (tmp_path / "config2.json").write_text(json.dumps(conf))
    out = subprocess.run(exe + ["smoke", "--config", str(tmp_path / "config2.json"), "--prompt", "1 2 3", "--max-new", "4"],
                         capture_output=True, text=True, timeout=300)
    assert out.returncode == 0, out.stderr
    assert out.stdout.strip().splitlines()[1] == "generated 4"
