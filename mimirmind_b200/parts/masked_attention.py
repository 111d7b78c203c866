"""Softmax attention with grouped heads whose view of the past is a window, a run of tokens, or either beside the first tokens.

``q, k, v = h W^T`` with ``H`` query heads and ``G`` key/value heads (query head ``h`` reads key/value head ``h // (H/G)``), keys of
size ``key_dim`` and values of size ``value_dim``.  Options, each a parameter, in the order they act:

* ``q_norm`` / ``k_norm``: all numbers of the projection of q (of k) are divided by their common root mean square and multiplied by a
  weight per number;
* ``rotary``: ``{"dims", "base", "scaling"}``: the first ``dims`` numbers of every q and k head turn by position, number ``i`` paired
  with ``i + dims/2``; ``scaling`` holds YaRN's numbers (``rope.exact_frequencies``) or is None;
* ``unit_qk``: every q and k head is divided by its own root mean square;
* the mask: ``window`` (the last tokens, the query's included; 0: no limit), ``chunk`` (the query's own run of that many tokens,
  counted from position 0; 0: no runs), ``keep`` (the first tokens of the sequence, seen whatever the other two say);
* ``g``: a projection with one row per head; a head's result is multiplied by the logistic of its number.

Without ``k`` and ``v`` the part has no keys and values of its own: its schedule entry reads another entry's cache (keys as they
stand there, normed and rotated), with queries and mask of its own.

One product makes q, k, v and the gates as fp32 rows; norms, rotation and the cache write are one launch over them
(``csrc/attention_prep.cu``); the attention kernels of :mod:`..kernels.attention` take the mask and apply the gate to what they
write.  Keys and values are two per-token arrays of the paged cache.
"""
from __future__ import annotations

from typing import List, Optional

import torch

from ..config.spec import PartSpec, TensorSpec
from ..kernels import ops
from ..registry import MIXERS
from .base import CacheArray, ElementwiseSink, KVCacheSpec, LayerCache, Mixer, Runtime, StepContext, WeightView
from .latent_attention import split_frequencies
from .linear import linear, linear_into
from .rope import exact_frequencies


@MIXERS.register("masked_attention")
class MaskedAttention(Mixer):
    """spec params: hidden, heads, kv_heads, key_dim, value_dim, scale, eps, window, chunk, keep, rotary ({"dims", "base", "scaling"}
    or None), unit_qk (bool), and the tensor names q, k, v (k and v None: another entry's cache is read), o, q_norm, k_norm, g (each
    of these three may be None)."""

    @classmethod
    def tensor_specs(cls, spec: PartSpec, prefix: str) -> List[TensorSpec]:
        d, H, G, dk, dv = spec["hidden"], spec["heads"], spec["kv_heads"], spec["key_dim"], spec["value_dim"]
        rows = {"q": H * dk, "k": G * dk, "v": G * dv}
        out = [TensorSpec(prefix + spec[n], (r, d)) for n, r in rows.items() if spec.get(n)] + [TensorSpec(prefix + spec["o"], (d, H * dv))]
        for n, r in (("q_norm", H * dk), ("k_norm", G * dk)):
            if spec.get(n):
                out.append(TensorSpec(prefix + spec[n], (r,), role="norm"))
        if spec.get("g"):
            out.append(TensorSpec(prefix + spec["g"], (H, d)))
        return out

    def __init__(self, spec: PartSpec, weights: WeightView, rt: Runtime):
        super().__init__(spec, weights, rt)
        self.hidden, self.heads, self.kv_heads = int(spec["hidden"]), int(spec["heads"]), int(spec["kv_heads"])
        self.key_dim, self.value_dim = int(spec["key_dim"]), int(spec["value_dim"])
        if self.heads % self.kv_heads:
            raise ValueError("masked attention: heads must be a multiple of kv_heads")
        self.scale, self.eps = float(spec["scale"]), float(spec["eps"])
        self.window, self.chunk, self.keep = (int(spec.get(n, 0) or 0) for n in ("window", "chunk", "keep"))
        if not self.window and not self.chunk:
            self.keep = 0                                      # everything is seen anyway
        H, G, dk, dv = self.heads, self.kv_heads, self.key_dim, self.value_dim
        self.owns = bool(spec.get("k"))
        names = ["q"] + (["k", "v"] if self.owns else []) + (["g"] if spec.get("g") else [])
        ws = [weights.take(spec[n]) for n in names]
        if len({w.dtype for w in ws}) > 1:
            ws = [w.float() for w in ws]
        self.w_in = torch.cat(ws, dim=0).contiguous()          # [H dk (+ G dk + G dv) (+ H), hidden]
        del ws
        self.k_off, self.v_off = H * dk, H * dk + G * dk
        self.g_off = (self.v_off + G * dv if self.owns else H * dk) if spec.get("g") else None
        self.q_norm = weights.take(spec["q_norm"]).float().contiguous() if spec.get("q_norm") else None
        self.k_norm = weights.take(spec["k_norm"]).float().contiguous() if spec.get("k_norm") else None
        self.unit_qk = bool(spec.get("unit_qk", False))
        rot = spec.get("rotary")
        self.rot_dims, self.f_hi, self.f_lo, self.rot_key, self.rot_factor = 0, None, None, None, 1.0
        if rot and int(rot["dims"]):
            self.rot_dims, base, scaling = int(rot["dims"]), float(rot["base"]), rot.get("scaling")
            if self.rot_dims % 2 or self.rot_dims > dk:
                raise ValueError("masked attention: the rotated dimensions must be even and at most the key size")
            self.f_hi, self.f_lo = split_frequencies(base, self.rot_dims, rt.device, scaling)
            self.rot_factor = exact_frequencies(base, self.rot_dims, scaling)[1]
            self.rot_key = ("rope_half_exact", self.rot_dims, base) + (tuple(sorted(scaling.items())) if scaling else ())
        self.w_o = weights.take(spec["o"]).contiguous()

    def kv_cache_spec(self) -> Optional[KVCacheSpec]:
        return KVCacheSpec(self.kv_heads, self.key_dim, self.window, chunk=self.chunk, keep=self.keep,
                           arrays=(CacheArray("k", (self.kv_heads, self.key_dim)), CacheArray("v", (self.kv_heads, self.value_dim))))

    def fuses_elementwise(self, n_tokens: int) -> bool:
        return ops.gemv_tanh_supported(self.rt, self.w_o, n_tokens)

    def forward(self, x: torch.Tensor, ctx: StepContext, cache: LayerCache, sink: Optional[ElementwiseSink] = None):
        n = x.shape[0]
        H, G, dk, dv = self.heads, self.kv_heads, self.key_dim, self.value_dim
        if cache.writes != self.owns:
            raise RuntimeError("masked attention: an entry with keys of its own writes its cache, one without reads another entry's")
        a = linear(x, self.w_in, None, self.rt, out_dtype=torch.float32)
        rot = None
        if self.rot_dims:
            if self.rot_key not in ctx.derived:
                ctx.derived[self.rot_key] = ops.rope_half_table(ctx.positions, self.f_hi, self.f_lo, self.rot_factor)
            rot = ctx.derived[self.rot_key]
        k_pages = v_pages = slots = None
        if self.owns:
            k_pages, v_pages = cache.arrays["k"], cache.arrays["v"]
            skey = ("slots", cache.block_table.data_ptr(), cache.page_size)
            if skey not in ctx.derived:
                ctx.derived[skey] = ops.slot_mapping(ctx.positions, ctx.token_req, cache.block_table, cache.page_size)
            slots = ctx.derived[skey]
        q = torch.empty((n, H * dk), dtype=self.rt.dtype, device=a.device)
        ops.qk_prep(a, 0, self.k_off, self.v_off, self.q_norm, self.k_norm, self.eps, rot, self.rot_dims, self.unit_qk, q, k_pages, v_pages, slots,
                    cache.page_size, H, G, dk, dv)
        out = torch.empty((n, H * dv), dtype=self.rt.dtype, device=a.device)
        from ..kernels import attention as attn_kernels
        gate = a[:, self.g_off:self.g_off + H] if self.g_off is not None else None
        attn_kernels.paged_sink_attention(q, cache, out, ctx, H, G, dk, dv, self.window, self.scale, False, chunk=self.chunk, keep=self.keep, gate=gate)
        return linear_into(out, self.w_o, self.rt, sink)
