"""Nefelorn: a decoder of chunked and windowed attention between norms without statistics, laid out from parts.

A layer: ``x += norm1b(mixer(norm1(x)))``, ``x += norm2b(ffn(norm2(x)))``; every norm is ``w tanh(alpha x) + b`` with one slope per
tensor.  Mixers, by the layer's ``type``:

* ``attention``: grouped heads; queries and keys normed over their whole projection, then rotated (interpolated by YaRN where the
  configuration says so); a query sees its own run of tokens only; a logistic gate per head.  A layer may use an earlier layer's
  cached keys and values (``kv_from``): it is then a schedule entry that reads that entry's cache, with its own queries and mask.
* ``attention_2``: grouped heads; queries and keys rotated, then divided by their root mean square per head; a sliding window beside
  the first tokens of the sequence.

Feed-forward: two matrices around the exact gelu, or routed experts with logistic scores that are renormed over the chosen ones
and multiplied by a factor.  The embedding is scaled, the logits are bent into ``(-cap, cap)``.  Tensor names: ``embed``,
``l<i>.norm1|norm1b|norm2|norm2b`` (each with ``.alpha`` and ``.b``), ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.

This module only *describes* the model; it holds no arithmetic.
"""
from __future__ import annotations

from ..config.nefelorn_config import ARCHITECTURE, DenseFeedForward, NefelornConfig, parse_nefelorn_config
from ..config.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from ..registry import register_architecture


def build_spec(cfg: NefelornConfig) -> ModelSpec:
    d, eps = cfg.width, cfg.norm_eps

    def norm(name: str) -> PartSpec:
        return PartSpec("tanh_norm", {"width": d, "weight": name, "offset": name + ".b", "alpha": name + ".alpha"}, category="norm")

    layers, schedule = [], []
    for i, layer in enumerate(cfg.layers):
        m = layer.mixer
        rotary = None
        if m.rot_dims:
            rotary = {"dims": m.rot_dims, "base": m.rot_base, "scaling": m.rot_scaling.as_dict() if m.rot_scaling else None}
        chunked, own = layer.type == "attention", m.kv_from is None
        mixer = PartSpec("masked_attention", {
            "hidden": d, "heads": m.heads, "kv_heads": m.kv_heads, "key_dim": m.dim, "value_dim": m.vdim, "scale": m.scale, "eps": eps,
            "window": m.window, "chunk": m.chunk, "keep": m.keep, "rotary": rotary, "unit_qk": not chunked,
            "q_norm": "mix.q.norm" if chunked else None, "k_norm": "mix.k.norm" if chunked and own else None,
            "q": "mix.q", "k": "mix.k" if own else None, "v": "mix.v" if own else None, "g": "mix.g" if chunked else None, "o": "mix.o"})
        extras = {"mixer_post_norm": norm("norm1b")}
        f = layer.mlp
        if f is None:
            ffn, ffn_norm = PartSpec("none", {}), PartSpec("none", {})
            extras["unused"] = PartSpec("unused_sublayer", {"tensors": [
                (n + suffix, shape) for n in ("norm2", "norm2b") for suffix, shape in (("", (d,)), (".b", (d,)), (".alpha", ()))]},
                category="connection")
        else:
            ffn_norm = norm("norm2")
            extras["ffn_post_norm"] = norm("norm2b")
            if isinstance(f, DenseFeedForward):
                ffn = PartSpec("dense_mlp", {"hidden": d, "ff": f.ff, "activation": "gelu_erf", "up": "mlp.up", "down": "mlp.down"})
            else:
                ffn = PartSpec("routed_experts", {
                    "hidden": d, "ff": f.ff, "experts": f.experts, "top": f.top, "groups": 1, "keep": 1, "router": "mlp.router",
                    "expert": "mlp.e{}", "scoring": "sigmoid", "renorm": True, "weight_scale": f.scale, "weight_on": "output",
                    "activation": "silu"})
        layers.append(LayerSpec(prefix=f"l{i}.", block=PartSpec("sandwich_norm", {}), mixer=mixer, feed_forward=ffn,
                                mixer_norm=norm("norm1"), ffn_norm=ffn_norm, extras=extras))
        schedule.append(ScheduleEntry(i, m.kv_from))
    return ModelSpec(
        architecture=cfg.architecture, hidden_size=d, vocab_size=cfg.vocab, max_positions=cfg.max_positions,
        embedding=PartSpec("token_embedding", {"vocab": cfg.vocab, "width": d, "scale": cfg.embedding_scale, "weight": "embed"}),
        layers=tuple(layers), schedule=tuple(schedule), final_norm=norm("final.norm"),
        head=PartSpec("lm_head", {"vocab": cfg.vocab, "width": d, "weight": "head", "tied_to": None, "softcap": cfg.logit_softcap}),
        eos_token_ids=cfg.eos_token_ids)


register_architecture(ARCHITECTURE, parse_nefelorn_config, build_spec)
