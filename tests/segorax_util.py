"""Small Segorax configurations and weights for the tests.  The tensor list is derived here from the configuration (the
names a checkpoint of the design uses), independently of the package's own list."""
import copy
import json
import os

import numpy as np


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, groups=None, shared=None):
    router = {"experts": experts, "top": top}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    out = {"kind": "moe", "expert": {"ff": ff}, "router": router}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def low(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base, mlp):
    """Queries through a latent, a sink."""
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
                      "rot": {"base": base, "dims": rot_dim}}}


def far(heads, dim, rot_dim, vdim, kv_rank, scale, base, scaling, mlp):
    """Direct queries, an interpolated rotation."""
    return {"type": "latent_attention_2", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
                      "rot": {"base": base, "dims": rot_dim, "scaling": dict(zip(("factor", "original", "fast", "slow"), scaling))}}}


def config(vocab, width, eps, mult, emb_scale, logit_scale, layers):
    out = {"architecture": "Segorax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    for key, v in (("residual_mult", mult), ("logit_scale", logit_scale), ("embedding", None if emb_scale is None else {"scale": emb_scale})):
        if v is not None:
            out[key] = v
    return out


CONFIGS = {
    # both kinds in turn, the interpolated one first; a layer without a feed-forward; groups of three of which one is kept, no groups,
    # with and without a shared expert; a logit scale that is no power of two
    "A": config(103, 72, 1e-5, 0.6, 3.0, 0.7, [
        far(3, 12, 8, 20, 32, 0.4, 700.0, (4.0, 64, 16.0, 1.0), moe(40, 9, 2, (3, 1), 24)),
        low(5, 16, 4, 8, 24, 16, 0.35, 50.0, dense(88)),
        low(2, 8, 16, 24, 56, 48, 0.3, 10000.0, None),
        far(4, 24, 12, 16, 40, 0.25, 300.0, (2.5, 200, 8.0, 2.0), moe(16, 5, 3)),
    ]),
    # sizes that the tensor-core kernels take, in several of their forms (one, two and three 64-wide pieces of a key, values of 64 and
    # 128), prompt-sized expert products, every group kept
    "B": config(333, 320, 1e-6, 1.0, 10.0, 0.5, [
        low(6, 64, 64, 128, 160, 128, 0.1, 20000.0, moe(128, 8, 2, (4, 2), 192)),
        far(4, 128, 32, 64, 192, 0.08, 1000.0, (16.0, 128, 32.0, 1.0), moe(64, 12, 4, (2, 2), 64)),
        low(9, 40, 24, 96, 96, 64, 0.15, 100000.0, dense(480)),
    ]),
    # sizes that fit no tile: odd width, head and latent sizes, one head, one expert per group, every expert chosen, nothing of
    # what may be absent; the interpolation's borders cross (fast and slow so close that the ramp is a step)
    "C": config(61, 50, 1e-6, None, None, None, [
        low(1, 7, 6, 9, 13, 11, 0.5, 30.0, moe(9, 4, 3, (4, 3), 7)),
        far(7, 5, 2, 3, 10, 0.6, 20.0, (3.0, 40, 1.5, 1.4), moe(33, 3, 3, None, 5)),
        low(3, 10, 10, 6, 17, 24, 0.4, 500.0, dense(21)),
    ]),
    # wider: forty heads (more than a tile's rows), a latent of 256, many small experts in groups of four, eight chosen
    "D": config(700, 512, 1e-5, 0.25, 12.0, 2.0, [
        low(40, 32, 16, 32, 200, 256, 0.15, 5000.0, moe(48, 32, 8, (8, 3), 96)),
        far(12, 96, 64, 112, 144, 0.09, 40000.0, (40.0, 512, 32.0, 1.0), dense(640)),
    ]),
}
LENGTHS = {"A": [1, 9, 77, 310], "B": [2, 70, 290, 450], "C": [3, 33, 160], "D": [4, 130, 360]}


def every_expert_chosen(cfg):
    """The same model with ``top = experts`` and every group kept: the choice cannot flip on a near tie, and the weights move
    smoothly with the scores."""
    out = copy.deepcopy(cfg)
    for layer in out["layers"]:
        if layer["mlp"] is not None and layer["mlp"]["kind"] == "moe":
            r = layer["mlp"]["router"]
            r["top"] = r["experts"]
            if "groups" in r:
                r["groups"]["keep"] = r["groups"]["count"]
    return out


def tensor_shapes(cfg):
    d, v = cfg["width"], cfg["vocab"]
    out = {"embed": (v, d), "head": (v, d), "final.norm": (d,)}
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer["mlp"]
        H, dk, dr, dv, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        out[p + "norm1"] = (d,)
        if layer["type"] == "latent_attention":
            rq = m["q_rank"]
            out.update({p + "mix.dq": (rq, d), p + "mix.dq.norm": (rq,), p + "mix.uq": (H * (dk + dr), rq), p + "mix.sink": (H,)})
        else:
            out[p + "mix.q"] = (H * (dk + dr), d)
        out.update({p + "mix.dkv": (r + dr, d), p + "mix.dkv.norm": (r,), p + "mix.uk": (H * dk, r), p + "mix.uv": (H * dv, r), p + "mix.o": (d, H * dv)})
        if f is None:
            continue
        out[p + "norm2"] = (d,)
        if f["kind"] == "dense":
            out.update({p + "mlp.gate": (f["ff"], d), p + "mlp.up": (f["ff"], d), p + "mlp.down": (d, f["ff"])})
            continue
        E, ff = f["router"]["experts"], f["expert"]["ff"]
        out.update({p + "mlp.router": (E, d), p + "mlp.correction": (E,)})
        for e in range(E):
            out.update({p + f"mlp.e{e}.up": (ff, d), p + f"mlp.e{e}.down": (d, ff)})
        if f.get("shared"):
            ff = f["shared"]["ff"]
            out.update({p + "mlp.shared.up": (ff, d), p + "mlp.shared.down": (d, ff), p + "mlp.shared.sg": (1, d)})
    return out


def random_weights(cfg, seed, gain=1.0):
    """Weights large enough that every mechanism moves the logits: matrices ~ N(0, gain / sqrt(in)), norm weights ~ 1 + 0.1 N,
    sinks ~ 1 + N, corrections ~ 0.7 N (choice scores of both signs, far from the order of the scores), routers spread wide."""
    rng = np.random.RandomState(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".")[-1]
        if leaf in ("norm", "norm1", "norm2"):
            w = 1.0 + 0.1 * rng.randn(*shape)
        elif leaf == "sink":
            w = 1.0 + rng.randn(*shape)
        elif leaf == "correction":
            w = 0.7 * rng.randn(*shape)
        elif leaf in ("router", "sg"):
            w = rng.randn(*shape) * 3.0 / np.sqrt(shape[1])
        elif name == "embed":
            w = rng.randn(*shape) / cfg.get("embedding", {}).get("scale", 1.0)
        else:
            w = rng.randn(*shape) * gain / np.sqrt(shape[1])
        out[name] = w.astype(np.float32)
    return out


def write_model(folder, cfg, seed, gain=1.0, overrides=None):
    """config.json + model.safetensors (bfloat16) in ``folder``."""
    import torch
    from mimirmind_b200.weights.safetensors_io import write_safetensors
    w = random_weights(cfg, seed, gain)
    w.update(overrides or {})
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), {k: torch.from_numpy(np.asarray(v)).to(torch.bfloat16) for k, v in w.items()})
    return folder
