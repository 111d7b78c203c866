"""Nefelorn on the GPU against the plain implementation (tests/plain_nefelorn.py): each mechanism alone, then whole models under
every way of cutting, decoding from the first token, slots and pages used again, generation through the engine's own entry
point, the replay program and the command line."""
import numpy as np
import pytest
import torch

import nefelorn_util as nu
import plain_nefelorn as pn
import replay_util as ru
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


def f32(a):
    return np.asarray(a, dtype=np.float32).astype(np.float64)


def bf16_round(a):
    return torch.from_numpy(np.asarray(a, dtype=np.float32)).to(torch.bfloat16).float().numpy().astype(np.float64)


def rounded(a, dtype):
    return bf16_round(a) if dtype == "bfloat16" else f32(a)


def i32(a):
    return torch.tensor(a, dtype=torch.int32, device=DEV)


# ---- one mixer in a pool of pages -----------------------------------------------------------------------------------
class Ctx:
    """What a mixer reads of a step's context: requests given as (tokens, held tokens after the step)."""

    def __init__(self, reqs, page_size, rt):
        self.q_len, self.kv_len = [n for n, _kv in reqs], [kv for _n, kv in reqs]
        self.q_start = np.concatenate([[0], np.cumsum(self.q_len)[:-1]]).tolist()
        self.n_tokens, self.n_requests = sum(self.q_len), len(reqs)
        self.positions = i32(sum([list(range(kv - n, kv)) for n, kv in reqs], []))
        self.token_req = i32(sum([[r] * n for r, (n, _kv) in enumerate(reqs)], []))
        self.max_q_len, self.max_kv_len, self.page_size, self.runtime = max(self.q_len), max(self.kv_len), page_size, rt
        self.plans, self.derived, self.plain_only, self.dump = {}, {}, False, None


class MixerAlone:
    """A masked attention part over pools of shuffled pages whose unwritten rows are NaN, or huge where whole pages are fetched (the
    kernels on tensor memory multiply what follows the last token in its page by zero weights: a pool holds finite numbers only);
    every request keeps its own pages, or with ``forget`` gives back those that its mask no longer reaches, as the cache manager does."""

    def __init__(self, layer, width, eps, w, dtype, page_size, lengths, seed=0, forget=False):
        from mimirmind_b200.config.nefelorn_config import parse_nefelorn_config
        from mimirmind_b200.models.nefelorn import build_spec
        from mimirmind_b200.parts.base import Runtime, WeightView
        from mimirmind_b200.registry import MIXERS
        cfg = {"architecture": "Nefelorn", "vocab": 8, "width": width, "norm": {"eps": eps}, "layers": [dict(layer, mlp=None)]}
        spec = build_spec(parse_nefelorn_config(cfg)).layers[0].mixer
        self.rt = Runtime(DT[dtype], torch.device(DEV))
        self.part = MIXERS.get(spec.kind)(spec, WeightView({k: dev(v, DT[dtype]) for k, v in w.items()}), self.rt)
        self.page_size, m = page_size, layer["mixer"]
        rng = np.random.RandomState(seed)
        need = [-(-n // page_size) for n in lengths]
        perm = rng.permutation(sum(need) + 5)
        self.width_pages = max(need)
        self.tables, at = [], 0
        for k in need:
            self.tables.append(perm[at:at + k].tolist() + [-1] * (self.width_pages - k))
            at += k
        from mimirmind_b200.kernels import attention
        self.junk = 3e4 if attention.USE_SINK_TCGEN05 and attention.USE_SINK_MMA and dtype == "bfloat16" else float("nan")
        self.pools = {a: torch.full((sum(need) + 5, m["kv_heads"], page_size, size), self.junk, dtype=DT[dtype], device=DEV)
                      for a, size in (("k", m["dim"]), ("v", m["vdim"]))}
        self.mask, self.forget = m["mask"], forget
        self.chunked = layer["type"] == "attention"

    def step(self, xs, which, starts):
        """xs: rows per request of the batch; which: their requests; starts: how many tokens each held before."""
        from mimirmind_b200.parts.base import LayerCache
        ctx = Ctx([(len(x), s + len(x)) for x, s in zip(xs, starts)], self.page_size, self.rt)
        cache = LayerCache(arrays=self.pools, block_table=i32([self.tables[r] for r in which]), page_size=self.page_size)
        out = self.part.forward(dev(np.concatenate(xs), self.rt.dtype), ctx, cache).float().cpu().numpy()
        if self.forget:
            for r, kv in zip(which, ctx.kv_len):
                size, keep = self.mask["size"], self.mask.get("keep_first", 0)
                dead = kv // size * size if self.chunked else max(0, kv + 1 - size)
                for b in range(-(-keep // self.page_size), dead // self.page_size):
                    if self.tables[r][b] >= 0:
                        for pool in self.pools.values():
                            pool[self.tables[r][b]] = self.junk
                        self.tables[r][b] = -1
        return [out[s:s + n] for s, n in zip(ctx.q_start, ctx.q_len)]


def mixer_weights(layer, width, rng, dtype, gain=1.0):
    shapes = {k[len("l0."):]: v for k, v in nu.tensor_shapes({"width": width, "vocab": 8, "layers": [dict(layer, mlp=None)]}).items() if k.startswith("l0.mix")}
    w = {k: 1.0 + 0.1 * rng.randn(*s) if k.endswith("norm") else (3.0 if k.endswith(".g") else gain) * rng.randn(*s) / np.sqrt(s[1]) for k, s in shapes.items()}
    return {k: rounded(v, dtype) for k, v in w.items()}


def plain_mixer(x, w, layer, eps):
    f = pn.chunked_attention if layer["type"] == "attention" else pn.window_attention
    return f(x, w, "mix.", layer["mixer"], eps, list(range(len(x))))[0]


@pytest.fixture(params=["tensor-memory", "mma.sync", "fp32-arithmetic"])
def route(request, monkeypatch):
    """The tcgen05 and TMA kernels (sizes they take), always the mma.sync ones, or the fp32-arithmetic kernel only."""
    from mimirmind_b200.kernels import attention
    monkeypatch.setattr(attention, "USE_SINK_TCGEN05", request.param == "tensor-memory")
    monkeypatch.setattr(attention, "USE_SINK_TMA_DECODE", request.param == "tensor-memory")
    monkeypatch.setattr(attention, "USE_SINK_MMA", request.param != "fp32-arithmetic")
    yield request.param
    from mimirmind_b200.kernels import ops
    ops.check_tcgen05_errors(torch.device(DEV))


YARN = (4.0, 100, 8.0, 1.0)
MIXERS_ALONE = {
    "runs, 128": nu.runs(4, 2, 128, 128, 0.09, 150, (128, 10000.0, YARN), None),
    "runs, 64": nu.runs(8, 2, 64, 64, 0.12, 64, (64, 3000.0, YARN), None),
    "runs, unequal": nu.runs(6, 3, 96, 32, 0.1, 129, (32, 500.0), None),
    "runs, one token": nu.runs(2, 1, 64, 64, 0.1, 1, (64, 500.0), None),
    "runs, seven": nu.runs(2, 2, 64, 128, 0.1, 7, (48, 500.0), None),
    "runs, longer than anything": nu.runs(2, 1, 128, 128, 0.1, 5000, (128, 500.0), None),
    "runs, odd sizes": nu.runs(3, 1, 9, 5, 0.4, 50, (6, 40.0, YARN), None),
    "window, 128": nu.near(4, 2, 128, 128, 0.05, 150, 4, (64, 10000.0), None),
    "window, 64": nu.near(6, 2, 64, 64, 0.1, 64, 70, (64, 3000.0), None),
    "window, many kept": nu.near(2, 1, 64, 64, 0.1, 33, 200, (32, 3000.0), None),
    "window, unequal": nu.near(6, 2, 32, 96, 0.15, 100, 17, (16, 500.0), None),
    "window, one token": nu.near(2, 1, 128, 128, 0.05, 1, 1, (64, 500.0), None),
    "window, nothing kept": nu.near(2, 2, 64, 32, 0.1, 90, 0, (64, 500.0), None),
    "window, kept meets it": nu.near(2, 2, 64, 64, 0.1, 128, 128, (64, 500.0), None),
    "window, odd sizes": nu.near(4, 2, 11, 13, 0.3, 21, 6, (10, 40.0), None),
    "window, wide heads": nu.near(40, 8, 256, 128, 0.04, 90, 3, (128, 900.0), None),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(MIXERS_ALONE))
def test_masked_attention_alone(name, dtype, route):
    """One mixer, three requests: a long prompt whole, then portions of several sizes beside single tokens of others, over pages
    of their own in pools full of junk, to which the pages return that the mask has left behind."""
    if dtype == "float32" and route != "tensor-memory":
        pytest.skip("the 32-bit mode has one route")
    layer, width, eps = MIXERS_ALONE[name], 96, 1e-5
    rng = np.random.RandomState(len(name))
    w = mixer_weights(layer, width, rng, dtype)
    lengths = [300, 170, 401]
    xs = [rounded(rng.randn(n, width), dtype) for n in lengths]
    want = [plain_mixer(x, w, layer, eps) for x in xs]
    scale = max(np.abs(v).max() for v in want)
    tol = (3e-5 if dtype == "float32" else 3e-2) * scale
    for page in (16, 8):
        m = MixerAlone(layer, width, eps, w, dtype, page, lengths, seed=page, forget=True)
        held = [0, 0, 0]
        for batch in ([(0, 300)], [(1, 90), (2, 129)], [(2, 2), (1, 1)], [(1, 77), (2, 1)], [(1, 1), (2, 65)], [(2, 3), (1, 1)], [(2, 200)], [(2, 1)]):
            got = m.step([xs[r][held[r]:held[r] + n] for r, n in batch], [r for r, _ in batch], [held[r] for r, _ in batch])
            for (r, n), g in zip(batch, got):
                assert not np.isnan(g).any(), (page, r, held[r], n)
                err = np.abs(g - want[r][held[r]:held[r] + n]).max()
                assert err <= tol, (page, r, held[r], n, err, tol)
                held[r] += n
        assert held == lengths


def one_key_layer(kind, size, keep, head):
    """Heads whose last number neither turns nor mixes: a planted key can stand out by it at any distance."""
    return nu.runs(2, 1, head, head, 2.0, size, (head // 2, 50.0, YARN), None) if kind == "runs" else nu.near(2, 1, head, head, 2.0, size, keep, (head // 2, 50.0), None)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind,size,keep,head", [("runs", 100, 0, 64), ("runs", 64, 0, 32), ("window", 100, 5, 64), ("window", 96, 21, 32), ("window", 33, 0, 128)])
def test_one_key_just_inside_and_just_outside(kind, size, keep, head, dtype, route):
    """One token's key answers the asking queries far above the rest.  Askers just inside and just outside the window or run, at page
    and tile borders and far away, in whole prompts, portions of two tokens and alone: a visible spot pins the result to its value, an
    invisible one leaves no trace; the kept first tokens are seen from anywhere."""
    if dtype == "float32" and route != "tensor-memory":
        pytest.skip("the 32-bit mode has one route")
    layer, width, T, eps = one_key_layer(kind, size, keep, head), 64, 420, 1e-6
    rng = np.random.RandomState(size)
    w = mixer_weights(layer, width, rng, dtype, 0.3)
    w["mix.k"][head - 1], w["mix.q"][:] = 0.0, 0.0
    w["mix.k"][:, 0] = 0.0
    w["mix.k"][head - 1, 0] = 1.0                                   # x[0] is the key that stands out
    for h in range(2):
        w["mix.q"][h * head + head - 1, 1] = 1.0                    # x[1] asks
    if kind == "runs":
        w["mix.q.norm"][:], w["mix.k.norm"][:], w["mix.g"][:] = 1.0, 1.0, 0.5
    w = {k: rounded(v, dtype) for k, v in w.items()}
    mask = pn.chunk_mask(T, size) if kind == "runs" else pn.window_mask(T, size, keep)
    seen = {True: 0, False: 0}
    for spot in sorted({0, 1, keep - 1, keep, 15, 16, 63, 64, size - 1, size, 127, 128, 200, 2 * size + 3}):
        if not 0 <= spot < T - 2:
            continue
        x = 0.5 * rng.randn(T, width)
        x[:, 0] = 0.0
        x[spot, 0] = 60.0
        edge = (spot // size + 1) * size if kind == "runs" else spot + size
        x[:, 1] = 4.0                                               # every token asks
        x = rounded(x, dtype)
        want = plain_mixer(x, w, layer, eps)
        v = x[spot] @ w["mix.v"].T
        tol = (1e-4 if dtype == "float32" else 3e-2) * np.abs(want).max()
        m = MixerAlone(layer, width, eps, w, dtype, 16, [T, T], seed=spot, forget=True)
        whole = m.step([x], [0], [0])[0]
        assert np.abs(whole - want).max() <= tol, spot
        held, askers = 0, sorted({a for a in (spot, spot + 1, edge - 1, edge, edge + 1, spot + 130, T - 1) if spot <= a < T})
        for a in askers:
            gate = pn.sigmoid(x[a] @ w["mix.g"].T) if kind == "runs" else np.ones(2)
            pinned = np.concatenate([gate[h] * v for h in range(2)]) @ w["mix.o"].T
            close = np.abs(want[a] - pinned).max() <= 0.05 * np.abs(pinned).max()
            assert close == bool(mask[a, spot]), (spot, a)            # the set-up does what it says
            seen[bool(mask[a, spot])] += 1
            pair = (a % 2 == 0) and a - 1 > held
            head_to = a - (1 if pair else 0)
            if head_to > held:
                g = m.step([x[held:head_to]], [1], [held])[0]
                assert np.abs(g - want[held:head_to]).max() <= tol, (spot, a)
            if a >= held:
                g = m.step([x[max(held, head_to):a + 1]], [1], [max(held, head_to)])[0]
                assert np.abs(g - want[max(held, head_to):a + 1]).max() <= tol, (spot, a, pair)
            held = a + 1
    assert min(seen.values()) >= 10


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_readers_own_mask_over_anothers_keys(dtype, route):
    """Two masks over one pool: the owner's runs, and a reader whose runs are longer or shorter, with queries and gates of its own."""
    if dtype == "float32" and route != "tensor-memory":
        pytest.skip("the 32-bit mode has one route")
    from mimirmind_b200.config.nefelorn_config import parse_nefelorn_config
    from mimirmind_b200.models.nefelorn import build_spec
    from mimirmind_b200.parts.base import LayerCache, WeightView
    from mimirmind_b200.registry import MIXERS
    width, T, eps = 64, 330, 1e-5
    owner = nu.runs(4, 2, 64, 64, 0.12, 48, (64, 700.0, YARN), None)
    rng = np.random.RandomState(3)
    w = mixer_weights(owner, width, rng, dtype)
    x, y = rounded(rng.randn(T, width), dtype), rounded(rng.randn(T, width), dtype)
    _o, k, v = pn.chunked_attention(x, w, "mix.", owner["mixer"], eps, list(range(T)))
    for size in (20, 48, 170):
        reader = nu.runs(4, 2, 64, 64, 0.2, size, (64, 700.0, YARN), None, kv_from=0)
        wr = mixer_weights(reader, width, rng, dtype)
        assert set(wr) == {"mix.q", "mix.o", "mix.g", "mix.q.norm"}
        cfg = {"architecture": "Nefelorn", "vocab": 8, "width": width, "norm": {"eps": eps}, "layers": [owner, reader]}
        spec = build_spec(parse_nefelorn_config(cfg)).layers[1].mixer
        m = MixerAlone(owner, width, eps, w, dtype, 16, [T])
        part = MIXERS.get(spec.kind)(spec, WeightView({n: dev(t, DT[dtype]) for n, t in wr.items()}), m.rt)
        want = pn.chunked_attention(y, wr, "mix.", reader["mixer"], eps, list(range(T)), shared=(k, v))[0]
        held = 0
        for n in (100, 1, 2, 17, 64, 1, 1, 144):
            m.step([x[held:held + n]], [0], [held])
            ctx = Ctx([(n, held + n)], 16, m.rt)
            cache = LayerCache(arrays=m.pools, block_table=i32([m.tables[0]]), page_size=16, writes=False)
            got = part.forward(dev(y[held:held + n], m.rt.dtype), ctx, cache).float().cpu().numpy()
            assert np.abs(got - want[held:held + n]).max() <= (3e-5 if dtype == "float32" else 3e-2) * np.abs(want).max(), (size, held, n)
            held += n
        with pytest.raises(RuntimeError, match="reads another"):
            part.forward(dev(y[:2], m.rt.dtype), Ctx([(2, 2)], 16, m.rt), LayerCache(arrays=m.pools, block_table=i32([m.tables[0]]), page_size=16))


# ---- norms and rotation of queries and keys -----------------------------------------------------------------------------------
@pytest.mark.parametrize("H,G,dk,dv,rot", [(4, 2, 64, 32, 64), (6, 3, 96, 64, 32), (3, 1, 9, 5, 6), (40, 8, 256, 128, 128), (24, 8, 128, 16, 96), (16, 4, 128, 128, 128), (64, 8, 256, 8, 32), (2, 2, 24, 12, 24), (7, 7, 16, 3, 2), (5, 1, 40, 8, 0)])
@pytest.mark.parametrize("scaling", [None, (8.0, 512, 32.0, 1.0)])
def test_norms_and_rotation_far_out(H, G, dk, dv, rot, scaling):
    """Positions up to 500,000 turn as exactly as near ones; the norm over the whole projection, the unit norm after the rotation and
    neither; rows in fp32 and bfloat16; queries alone; keys and values in the pages of their tokens and nowhere else."""
    from mimirmind_b200.kernels import ops
    from mimirmind_b200.parts.latent_attention import split_frequencies
    from mimirmind_b200.parts.rope import exact_frequencies
    rng = np.random.RandomState(H * dk + rot)
    page, base, eps = 8, 10000.0, 1e-4
    sc = dict(zip(("factor", "original", "fast", "slow"), scaling)) if scaling else None
    positions = np.array([0, 1, 7, 8, 4095, 100000, 500001])
    n = len(positions)
    spec = {"dims": rot, "base": base, "scaling": sc}
    table = None
    if rot:
        hi, lo = split_frequencies(base, rot, DEV, sc)
        table = ops.rope_half_table(i32(positions.tolist()), hi, lo, exact_frequencies(base, rot, sc)[1])
    wide = (H + G) * dk + G * dv + H
    for row_dtype in (torch.float32, torch.bfloat16):
        act = torch.bfloat16 if row_dtype == torch.bfloat16 else torch.float32
        rows = bf16_round(rng.randn(n, wide)) if act == torch.bfloat16 else f32(rng.randn(n, wide))
        rows[1] *= 0.01                                                  # eps counts
        if act == torch.bfloat16:
            rows = bf16_round(rows)
        wq, wk = f32(1.0 + 0.3 * rng.randn(H * dk)), f32(1.0 + 0.3 * rng.randn(G * dk))
        for whole, unit in ((True, False), (False, True), (True, True), (False, False)):
            q, k = rows[:, :H * dk], rows[:, H * dk:(H + G) * dk]
            if whole:
                q, k = pn.unit_rms(q, eps) * wq, pn.unit_rms(k, eps) * wk
            q, k = pn.rotate_halves(pn.heads(q, H), positions, spec), pn.rotate_halves(pn.heads(k, G), positions, spec)
            if unit:
                q, k = pn.unit_rms(q, eps), pn.unit_rms(k, eps)
            tol = 1e-5 if act == torch.float32 else 1e-2
            pools = [torch.zeros((n, G, page, d), dtype=act, device=DEV) for d in (dk, dv)]
            slots = i32([t * page + t % page for t in range(n - 1)] + [-1])      # the last token has no place to go
            for own in (True, False):
                q_out = torch.zeros((n, H * dk), dtype=act, device=DEV)
                ops.qk_prep(dev(rows, row_dtype), 0, H * dk, (H + G) * dk, dev(wq) if whole else None, dev(wk) if whole else None, eps, table, rot, unit, q_out,
                            pools[0] if own else None, pools[1] if own else None, slots if own else None, page, H, G, dk, dv)
                got = q_out.float().cpu().numpy().reshape(n, H, dk)
                assert np.abs(got - q).max() <= tol * np.abs(q).max(), (whole, unit, own)
            for pool, want in ((pools[0], k), (pools[1], rows[:, (H + G) * dk:(H + G) * dk + G * dv].reshape(n, G, dv))):
                for t in range(n - 1):
                    assert np.abs(pool[t, :, t % page].float().cpu().numpy() - want[t]).max() <= tol * np.abs(want).max(), (whole, unit, t)
                    pool[t, :, t % page] = 0
                assert not pool.any()


# ---- the norm without statistics ------------------------------------------------------------------------------------------------
def tanh_norm_numbers(rng, d):
    w, b, alpha = f32(1.0 + 0.3 * rng.randn(d)), f32(0.4 * rng.randn(d)), float(np.float32(0.3 + rng.rand()))
    return (dev(w), dev(b), alpha), lambda x: np.tanh(alpha * x) * w + b


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n,d", [(5, 64), (33, 54), (2, 4096), (700, 260), (1, 13001), (9, 3)])
def test_the_norms_around_a_sum(n, d, dtype):
    """A branch normed and added, the sum normed; the same with the branch in pieces, in order and by place; a plain pending sum; rows
    picked out."""
    from mimirmind_b200.kernels import ops
    rng = np.random.RandomState(d)
    x, top = f32(2.0 * rng.randn(n, d)), 3
    post, plain_post = tanh_norm_numbers(rng, d)
    then, plain_then = tanh_norm_numbers(rng, d)
    a, wts, place = rounded(3.0 * rng.randn(n, d), dtype), f32(rng.rand(n, top)), rng.permutation(n * top)
    cases = [("whole", a, dict(), a)]
    for row_dtype in ("float32",) if dtype == "float32" else ("float32", "bfloat16"):
        rows = rounded(2.0 * rng.randn(n * top, d), row_dtype)
        for where in (None, place):
            y = (rows[np.arange(n * top) if where is None else where].reshape(n, top, d) * wts[:, :, None]).sum(1)
            cases.append((row_dtype, (rows, row_dtype), dict(wts=dev(wts), place=None if where is None else i32(where.tolist())), y))
    for what, branch, kw, y in cases:
        t = dev(branch[0], DT[branch[1]]) if isinstance(branch, tuple) else dev(branch, DT[dtype])
        for first in (True, False):
            want = x + (plain_post(y) if first else y)
            for second in (True, False):
                res = dev(x)
                out = torch.empty((n, d), dtype=DT[dtype], device=DEV) if second else None
                got = ops.tanh_norm_chain(res, t, post if first else None, then if second else None, out, **kw)
                assert np.abs(res.cpu().numpy() - want).max() <= 3e-6 * np.abs(want).max(), (what, first, second)
                if second:
                    ref = plain_then(res.double().cpu().numpy())
                    assert np.abs(got.float().cpu().numpy() - ref).max() <= (3e-6 if dtype == "float32" else 8e-3) * np.abs(ref).max(), (what, first)
    rows = rng.randint(0, n, size=max(1, n // 2))
    out = torch.empty((len(rows), d), dtype=DT[dtype], device=DEV)
    got = ops.tanh_norm_chain(dev(x), None, None, then, out, rows=i32(rows.tolist())).float().cpu().numpy()
    assert np.abs(got - plain_then(x[rows])).max() <= (3e-6 if dtype == "float32" else 8e-3) * np.abs(x).max()


@pytest.mark.parametrize("m", [1, 2, 7, 8, 9, 16, 17, 33, 64])
@pytest.mark.parametrize("n,k", [(256, 512), (4096, 1024), (48, 256), (1040, 288)])
def test_norms_in_the_epilogue_of_a_product(m, n, k):
    from mimirmind_b200.kernels import ops
    rng = np.random.RandomState(m + n)
    x, w, res = bf16_round(rng.randn(m, k)), bf16_round(2.0 * rng.randn(n, k) / np.sqrt(k)), f32(rng.randn(m, n))
    post, plain_post = tanh_norm_numbers(rng, n)
    then, plain_then = tanh_norm_numbers(rng, n)
    want = res + plain_post(x @ w.T)
    for second in (then, None):
        r = dev(res)
        out = ops.gemv_bf16_tanh(dev(x, torch.bfloat16), dev(w, torch.bfloat16), r, post, second)
        assert np.abs(r.cpu().numpy() - want).max() <= 2e-5 * np.abs(want).max()
        if second is None:
            assert out is None
        else:
            ref = plain_then(r.double().cpu().numpy())
            assert np.abs(out.float().cpu().numpy() - ref).max() <= 8e-3 * np.abs(ref).max()
    ops.check_tcgen05_errors(torch.device(DEV))


def test_the_cap_on_logits():
    from mimirmind_b200.kernels import ops
    x = np.concatenate([np.linspace(-90.0, 90.0, 301), [1e-6, -1e-6, 1e4]]).astype(np.float32)
    for cap in (7.0, 30.0):
        got = ops.soft_cap(dev(x).reshape(1, -1), cap).cpu().numpy()[0]
        assert np.abs(got - pn.soft_cap(x.astype(np.float64), cap)).max() <= 2e-6 * cap


# ---- experts ----------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("E,top,scale", [(9, 2, 1.7), (8, 8, 0.5), (6, 1, 2.0), (160, 6, 1.0), (5, 3, 2.5), (33, 32, 1.3)])
@pytest.mark.parametrize("D", [40, 51])
def test_the_routers_weights(E, top, scale, D):
    """Logistic scores over their sum, times the factor; without renorming the scores as they are, times the factor."""
    from mimirmind_b200.kernels import ops
    rng = np.random.RandomState(E)
    for n in (3, 2100):
        x, w = rng.randn(n, D).astype(np.float32), (rng.randn(E, D) * 0.5).astype(np.float32)
        idx, wts = ops.moe_router(dev(x), dev(w), top, 1, 1, scoring="sigmoid", renorm=True, scale=scale)
        want, s = pn.router_choice(x.astype(np.float64), w.astype(np.float64), top, scale)
        same = (np.sort(idx.cpu().numpy(), 1) == np.sort(want, 1)).all(1)
        assert same.mean() >= 0.999                                     # float64 against fp32: near ties of thousands of rows
        assert np.abs(np.sort(wts.cpu().numpy(), 1) - np.sort(s, 1))[same].max() <= 3e-6 * scale
        idx2, raw = ops.moe_router(dev(x), dev(w), top, 1, 1, scoring="sigmoid", scale=scale)
        z = pn.sigmoid(x.astype(np.float64) @ w.T.astype(np.float64))
        assert torch.equal(idx, idx2) and np.abs(raw.cpu().numpy() - scale * np.take_along_axis(z, idx.cpu().numpy().astype(np.int64), 1)).max() <= 3e-6 * scale
        soft = ops.moe_router(dev(x), dev(w), top, 1, 1)[1]
        assert np.abs(soft.sum(1).cpu().numpy() - 1.0).max() <= 1e-5    # the softmax's weights still add up to one
    tiny = ops.moe_router(torch.ones((2, 4), device=DEV), torch.full((3, 4), -40.0, device=DEV), 2, 1, 1, scoring="sigmoid", renorm=True, scale=2.0)[1]
    assert np.isfinite(tiny.cpu().numpy()).all()                        # scores that vanish: the sum is never zero


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n,d,ff,E,top", [(70, 64, 40, 9, 2), (1, 50, 9, 4, 3), (8, 256, 96, 16, 4), (300, 128, 64, 8, 4), (2100, 96, 32, 6, 2)])
def test_experts_against_the_plain_ones(n, d, ff, E, top, dtype):
    """Every product route (a decode step's tiles, a portion's, a prompt's grouped products, 32-bit), whole and in pieces."""
    from mimirmind_b200.config.spec import PartSpec
    from mimirmind_b200.kernels import ops
    from mimirmind_b200.parts.base import Runtime, WeightView
    from mimirmind_b200.parts.moe import RoutedExperts
    rng = np.random.RandomState(n + d)
    w = {"mlp.router": rng.randn(E, d) * 4.0 / np.sqrt(d)}
    for e in range(E):
        w.update({f"mlp.e{e}.{name}": rng.randn(*s) * 1.5 / np.sqrt(s[1]) for name, s in (("gate", (ff, d)), ("up", (ff, d)), ("down", (d, ff)))})
    w, x = {k: bf16_round(v) for k, v in w.items()}, bf16_round(rng.randn(n, d))
    mlp = nu.moe(ff, E, top, 1.9)
    spec = PartSpec("routed_experts", {"hidden": d, "ff": ff, "experts": E, "top": top, "router": "mlp.router", "expert": "mlp.e{}", "scoring": "sigmoid",
                                       "renorm": True, "weight_scale": 1.9})
    rt = Runtime(DT[dtype], torch.device(DEV))
    ctx = Ctx([(n, n)], 16, rt)
    part = RoutedExperts(spec, WeightView({k: dev(v, DT[dtype]) for k, v in w.items()}), rt)
    assert part.splits_weighed()
    want = pn.experts_feed_forward(x, w, "mlp.", mlp)
    got = part.forward(dev(x, DT[dtype]), ctx).float().cpu().numpy()
    b = part.forward_split(dev(x, DT[dtype]), ctx)
    place = torch.arange(n * top, device=DEV) if b.place is None else b.place.long()
    y = (b.rows.float()[place].reshape(n, top, d) * b.weights[:, :, None]).sum(1)
    for g in (got, y.cpu().numpy()):
        err = np.abs(g - want).max(axis=-1) / np.abs(want).max()
        if dtype == "float32":
            assert err.max() <= 2e-5
        else:
            assert np.median(err) <= 2e-2 and (err > 5e-2).mean() <= 0.02
    ops.check_tcgen05_errors(torch.device(DEV))


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
            cfg = nu.every_expert_chosen(nu.CONFIGS[name]) if key[1] else nu.CONFIGS[name]
            folder = nu.write_model(str(tmp_path_factory.mktemp(f"nefelorn_{name}")), cfg, seed=len(cache) + 17)
            cache[key] = (folder,) + pn.load_folder(folder)
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


@pytest.mark.parametrize("name", sorted(nu.CONFIGS))
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
    pn.forward(cfg, w, toks, collect=streams)
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
@pytest.mark.parametrize("name,page_size", [("A", 16), ("B", 16), ("C", 8), ("A", 32), ("B", 64), ("D", 16)])
def test_every_way_of_cutting_matches_the_plain_implementation(name, page_size, dtype, models):
    folder, cfg, w = models(name, dtype)
    reqs = {f"{name}{i}": random_tokens(cfg["vocab"], n, 100 * i + n) for i, n in enumerate(nu.LENGTHS[name])}
    ref = {rid: pn.forward(cfg, w, t) for rid, t in reqs.items()}
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


@pytest.mark.parametrize("name,dtype", [("A", "float32"), ("B", "bfloat16"), ("C", "float32"), ("D", "bfloat16")])
def test_decoding_from_the_first_token(name, dtype, models):
    folder, cfg, w = models(name, dtype)
    toks = random_tokens(cfg["vocab"], 330, 5)
    t = ru.Trace()
    ru.chunks(t, "d", toks, [1])
    out, _ = ru.run_in_process(folder, dtype, t, t.max_live_tokens())
    check_rows(t, out, {"d": toks}, {"d": pn.forward(cfg, w, toks)}, dtype, "decode from the first token")


def test_a_pool_that_holds_only_what_the_masks_reach(models):
    """Far fewer pages than the sequence has tokens: runs, windows and kept tokens of every group fit, and a shared group keeps what
    its widest reader looks at."""
    from mimirmind_b200.engine.loader import load_model
    from mimirmind_b200.engine.runner import ModelRunner, StepEntry
    folder, cfg, w = models("A")
    model, _ = load_model(folder, "float32")
    groups = model.cache_groups()
    assert {m for g in groups for m in g.masks} == {(0, 37, 0), (0, 90, 0), (0, 21, 0), (29, 0, 5), (50, 0, 0)} and len(groups) == 3
    shared = next(g for g in groups if len(g.masks) == 3)
    assert shared.entries == (0,)
    runner = ModelRunner(model, page_size=8, num_pages={g.name: 14 if g is shared else 9 for g in groups}, max_requests=1)
    toks = random_tokens(cfg["vocab"], 300, 8)
    ref = pn.forward(cfg, w, toks)
    assert runner.add_request("r")
    at = 0
    for n in [13, 1, 1, 2, 9, 1, 16] * 7:
        n = min(n, len(toks) - at)
        if n == 0:
            break
        got = runner.step([StepEntry("r", toks[at:at + n], list(range(n)))]).cpu().numpy()
        assert rel_rms(got, ref[at:at + n]).max() <= ROW_TOL["float32"], at
        at += n
    assert at == len(toks) and runner.manager.reuses() > 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_pages_and_slots_used_again_start_clean(dtype, models):
    """Two slots and just enough pages, five requests one after the other and in pairs: none sees what another left."""
    from mimirmind_b200.engine.loader import load_model
    from mimirmind_b200.engine.runner import ModelRunner, StepEntry
    folder, cfg, w = models("B", dtype)
    model, _ = load_model(folder, dtype)
    runner = ModelRunner(model, page_size=16, num_pages=13, max_requests=2)
    reqs = [random_tokens(cfg["vocab"], n, n) for n in (80, 3, 110, 31, 140)]
    ref = [pn.forward(cfg, w, t) for t in reqs]
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
    """Engine.generate (scheduler, prompt portions, captured decode steps) picks the plain implementation's tokens, over the edges of
    windows and runs."""
    from mimirmind_b200 import Engine
    folder, cfg, w = models(name, dtype)
    prompts = [random_tokens(cfg["vocab"], n, 40 + n) for n in (5, 17, 33, 130)]
    eng = Engine.from_folder(folder, dtype=dtype, page_size=16, cache_tokens=1024, max_context=512, token_budget=80, max_active=4)
    res = eng.generate(prompts, max_new_tokens=40)
    exact = 0
    for p, r in zip(prompts, res):
        assert r.stats.generated_tokens == 40 and r.stats.finish_reason == "length"
        rows = pn.forward(cfg, w, list(p) + list(r.tokens))[len(p) - 1:-1]
        for i, tok in enumerate(r.tokens):
            best = int(np.argmax(rows[i]))
            exact += tok == best
            if dtype == "float32":
                assert rows[i][tok] >= rows[i][best] - 1e-4, f"token {i}: engine chose {tok}, plain {best}"
    assert exact >= (160 if dtype == "float32" else 130)
    assert eng.runner.manager.free_pages() == eng.runner.manager.total_pages()
    again = eng.generate(prompts, max_new_tokens=40)          # slots and pages used again
    if dtype == "float32":
        assert [r.tokens for r in again] == [r.tokens for r in res]


def test_the_replay_program_on_this_design(models, tmp_path):
    folder, cfg, w = models("C")
    reqs = {f"r{i}": random_tokens(cfg["vocab"], n, 11 + i) for i, n in enumerate([3, 90, 41, 150])}
    ref = {rid: pn.forward(cfg, w, t) for rid, t in reqs.items()}
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
        row = pn.forward(cfg, w, toks)[-1]
        assert row[tok] >= row.max() - 1e-4
        toks.append(tok)
    (tmp_path / "mc.json").write_text(json.dumps(nu.CONFIGS["B"]))
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
