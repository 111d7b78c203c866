"""Segorax: a decoder of latent attention whose sublayers are normed on their output only, laid out from parts.

A layer: ``x <- x + m norm1(mixer(x))``, ``x <- x + m norm2(ffn(x))`` with one multiplier ``m`` for the model; the sublayers read
the stream itself.  Mixers, by the layer's ``type`` (both cache one normed latent and one rotated key part per token, and both
rotate neighbouring numbers):

* ``latent_attention``: queries through a normed latent of their own, a learned sink per head in the softmax;
* ``latent_attention_2``: queries straight from the stream, a rotation interpolated by YaRN, no sink.

Feed-forward: a dense gated one (tanh form of gelu), or routed experts of two matrices (exact gelu) with logistic scores,
a correction per expert for the choice, a choice limited to the groups whose two best experts score highest, weights as they
are, and a shared expert behind a gate per token.  The embedding and the logits are scaled (the latter by the final norm's
weight).  Tensor names: ``embed``, ``l<i>.norm1|norm2``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.

This module only *describes* the model; it holds no arithmetic.
"""
from __future__ import annotations

from ..config.segorax_config import ARCHITECTURE, DenseFeedForward, SegoraxConfig, parse_segorax_config
from ..config.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from ..registry import register_architecture


def build_spec(cfg: SegoraxConfig) -> ModelSpec:
    d, eps = cfg.width, cfg.norm_eps

    def norm(name: str, gain: float = 1.0) -> PartSpec:
        return PartSpec("rmsnorm", {"width": d, "eps": eps, "weight": name, "gain": gain}, category="norm")

    layers = []
    for i, layer in enumerate(cfg.layers):
        m = layer.mixer
        rotary = None
        if m.rot_dims:
            rotary = {"dims": m.rot_dims, "base": m.rot_base, "layout": "pairs", "scaling": m.rot_scaling.as_dict() if m.rot_scaling else None}
        names = {"q_down": "mix.dq", "q_norm": "mix.dq.norm", "q": "mix.uq"} if m.q_rank else {"q": "mix.q"}
        mixer = PartSpec("latent_attention", {
            "hidden": d, "heads": m.heads, "key_dim": m.dim, "rot_dim": m.rot_dim, "value_dim": m.vdim, "rank": m.kv_rank, "q_rank": m.q_rank,
            "scale": m.scale, "eps": eps, "rotary": rotary, "down": "mix.dkv", "down_norm": "mix.dkv.norm", "up_k": "mix.uk", "up_v": "mix.uv",
            "g": None, "sink": "mix.sink" if m.sink else None, "o": "mix.o", **names})
        extras, ffn_norm = {}, norm("norm2")
        f = layer.mlp
        if f is None:
            ffn, ffn_norm = PartSpec("none", {}), PartSpec("none", {})
            extras["unused"] = PartSpec("unused_sublayer", {"tensors": [("norm2", (d,))]}, category="connection")
        elif isinstance(f, DenseFeedForward):
            ffn = PartSpec("swiglu", {"hidden": d, "intermediate": f.ff, "activation": "gelu_tanh", "gate": "mlp.gate", "up": "mlp.up", "down": "mlp.down"})
        else:
            shared = None
            if f.shared_ff is not None:
                shared = PartSpec("dense_mlp", {"hidden": d, "ff": f.shared_ff, "activation": "gelu_erf", "up": "mlp.shared.up", "down": "mlp.shared.down"})
            ffn = PartSpec("routed_experts", {
                "hidden": d, "ff": f.ff, "experts": f.experts, "top": f.top, "groups": f.groups, "keep": f.keep, "group_score": "top2_sum",
                "router": "mlp.router", "correction": "mlp.correction", "expert": "mlp.e{}", "gated": False, "scoring": "sigmoid",
                "weight_on": "output", "activation": "gelu_erf", "shared": shared, "shared_gate": "mlp.shared.sg" if shared is not None else None})
        layers.append(LayerSpec(prefix=f"l{i}.", block=PartSpec("output_norm", {"mult": cfg.residual_mult}), mixer=mixer, feed_forward=ffn,
                                mixer_norm=norm("norm1"), ffn_norm=ffn_norm, extras=extras))
    return ModelSpec(
        architecture=cfg.architecture, hidden_size=d, vocab_size=cfg.vocab, max_positions=cfg.max_positions,
        embedding=PartSpec("token_embedding", {"vocab": cfg.vocab, "width": d, "scale": cfg.embedding_scale, "weight": "embed"}),
        layers=tuple(layers), schedule=tuple(ScheduleEntry(i) for i in range(len(layers))),
        final_norm=norm("final.norm", cfg.logit_scale),
        head=PartSpec("lm_head", {"vocab": cfg.vocab, "width": d, "weight": "head", "tied_to": None}),
        eos_token_ids=cfg.eos_token_ids)


register_architecture(ARCHITECTURE, parse_segorax_config, build_spec)
