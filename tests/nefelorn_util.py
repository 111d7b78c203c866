"""Small Nefelorn configurations and weights for the tests.  The tensor list is derived here from the configuration (the
names a checkpoint of the design uses), independently of the package's own list."""
import copy
import json
import os

import numpy as np


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, scale=None):
    router = {"experts": experts, "top": top}
    if scale is not None:
        router["scale"] = scale
    return {"kind": "moe", "expert": {"ff": ff}, "router": router}


def _rot(dims, base, scaling=None):
    out = {"base": base, "dims": dims}
    if scaling:
        out["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return out


def runs(heads, kv_heads, dim, vdim, scale, size, rot, mlp, kv_from=None):
    """Chunks, norms over the whole projection, a gate per head; perhaps another layer's keys and values."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size}, "rot": _rot(*rot)}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def near(heads, kv_heads, dim, vdim, scale, size, keep, rot, mlp):
    """A window beside the first tokens, unit queries and keys after the rotation."""
    mask = {"size": size}
    if keep is not None:
        mask["keep_first"] = keep
    return {"type": "attention_2", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": mask, "rot": _rot(*rot)}}


def config(vocab, width, eps, emb_scale, cap, layers):
    out = {"architecture": "Nefelorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if emb_scale is not None:
        out["embedding"] = {"scale": emb_scale}
    if cap is not None:
        out["logit_softcap"] = cap
    return out


CONFIGS = {
    # both kinds with every feed-forward; a reader whose runs are longer than the owner's, and one whose runs are shorter; windows and
    # runs that end inside pages; two interpolated rotations and a plain one
    "A": config(101, 72, 1e-5, 3.0, 8.0, [
        runs(6, 2, 24, 16, 0.25, 37, (24, 700.0, (4.0, 64, 16.0, 1.0)), moe(40, 9, 3, 1.7)),
        near(3, 3, 16, 24, 0.3, 29, 5, (8, 900.0), dense(88)),
        runs(6, 2, 24, 16, 0.35, 90, (24, 700.0, (4.0, 64, 16.0, 1.0)), None, kv_from=0),
        near(8, 2, 12, 8, 0.4, 50, None, (12, 60.0), moe(24, 4, 1, 0.5)),
        runs(6, 2, 24, 16, 0.2, 21, (24, 700.0, (4.0, 64, 16.0, 1.0)), dense(56), kv_from=0),
    ]),
    # sizes that the tensor-core kernels take: equal key and value sizes of 64 and 128 (tensor memory and TMA), unequal ones (mma.sync),
    # prompt-sized expert products, streaming products with the norms in their epilogues; kept tokens beyond a page
    "B": config(330, 256, 1e-6, 9.0, 5.0, [
        near(8, 2, 128, 128, 0.05, 160, 20, (64, 10000.0), dense(512)),
        runs(4, 4, 64, 64, 0.15, 144, (64, 50000.0, (16.0, 128, 32.0, 1.0)), moe(128, 8, 2, 2.0)),
        runs(4, 4, 64, 64, 0.1, 200, (64, 50000.0, (16.0, 128, 32.0, 1.0)), moe(64, 12, 5, 1.3), kv_from=1),
        near(6, 2, 96, 32, 0.07, 70, 3, (96, 3000.0), moe(96, 6, 2, 2.5)),
        near(2, 1, 64, 64, 0.08, 133, 140, (32, 3000.0), dense(192)),
    ]),
    # sizes that fit no tile: odd width, vocabulary, head and value sizes, one head; nothing of what may be absent; a window of one
    # token, runs of one token, no kept tokens, every expert chosen; the interpolation's borders cross
    "C": config(59, 50, 1e-6, None, None, [
        near(1, 1, 10, 7, 0.6, 1, 2, (6, 30.0), moe(9, 4, 4)),
        runs(7, 7, 6, 3, 0.5, 13, (2, 20.0, (3.0, 40, 1.5, 1.4)), dense(21)),
        near(4, 2, 9, 5, 0.5, 17, 0, (4, 50.0), dense(33)),
        runs(3, 1, 5, 11, 0.7, 1, (4, 90.0), moe(7, 3, 2, 3.0)),
    ]),
    # wide heads in numbers that fill more than one turn of a block, long windows and runs
    "D": config(500, 384, 1e-6, 12.0, 11.0, [
        runs(36, 4, 256, 32, 0.06, 250, (128, 5000.0), dense(640)),
        near(40, 8, 224, 128, 0.06, 190, 33, (224, 40000.0), moe(48, 32, 8, 2.0)),
    ]),
}
LENGTHS = {"A": [1, 9, 77, 310], "B": [2, 70, 290, 450], "C": [3, 33, 160], "D": [4, 130, 360]}


def every_expert_chosen(cfg):
    """The same model with ``top = experts``: the choice cannot flip on a near tie, and the weights move smoothly with the scores."""
    out = copy.deepcopy(cfg)
    for layer in out["layers"]:
        if layer["mlp"] is not None and layer["mlp"]["kind"] == "moe":
            layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
    return out


def tensor_shapes(cfg):
    d, v = cfg["width"], cfg["vocab"]
    out = {"embed": (v, d), "head": (v, d)}

    def norm(name):
        out.update({name: (d,), name + ".b": (d,), name + ".alpha": ()})

    norm("final.norm")
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer["mlp"]
        H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        norm(p + "norm1"), norm(p + "norm1b")
        out.update({p + "mix.q": (H * dk, d), p + "mix.o": (d, H * dv)})
        own, whole = m.get("kv_from") is None, layer["type"] == "attention"
        if own:
            out.update({p + "mix.k": (G * dk, d), p + "mix.v": (G * dv, d)})
        if whole:
            out.update({p + "mix.q.norm": (H * dk,), p + "mix.g": (H, d)})
            if own:
                out[p + "mix.k.norm"] = (G * dk,)
        if f is None:
            continue
        norm(p + "norm2"), norm(p + "norm2b")
        if f["kind"] == "dense":
            out.update({p + "mlp.up": (f["ff"], d), p + "mlp.down": (d, f["ff"])})
            continue
        out[p + "mlp.router"] = (f["router"]["experts"], d)
        ff = f["expert"]["ff"]
        for e in range(f["router"]["experts"]):
            out.update({p + f"mlp.e{e}.gate": (ff, d), p + f"mlp.e{e}.up": (ff, d), p + f"mlp.e{e}.down": (d, ff)})
    return out


def random_weights(cfg, seed, gain=1.0):
    """Weights large enough that every mechanism moves the logits: matrices ~ N(0, gain / sqrt(in)), norm weights ~ 1 + 0.1 N, offsets
    ~ 0.2 N, slopes between 0.4 and 1.2, gates and routers spread wide."""
    rng = np.random.RandomState(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".")[-1]
        if leaf in ("norm", "norm1", "norm1b", "norm2", "norm2b"):
            w = 1.0 + 0.1 * rng.randn(*shape)
        elif leaf == "b":
            w = 0.2 * rng.randn(*shape)
        elif leaf == "alpha":
            w = np.asarray(0.4 + 0.8 * rng.rand())
        elif leaf in ("router", "g"):
            w = rng.randn(*shape) * 3.0 / np.sqrt(shape[1])
        elif name == "head":                     # logits that the cap bends
            w = 6.0 * rng.randn(*shape) / np.sqrt(shape[1])
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
