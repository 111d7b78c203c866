"""Mixture of experts with a softmax (or sigmoid) router and a choice that may be limited to the best runs of experts.

``s = softmax(h·W_routerᵀ)`` over all ``experts`` in fp32; the experts stand in ``groups`` equal runs of neighbours, a run is
scored by its best expert and only the ``keep`` best runs are eligible; the ``top`` eligible experts with the largest ``s``
are chosen and weighted by ``s / (sum of the chosen s + 1e-20)``.  Expert: ``W_down (silu(W_gate h) ⊙ W_up h)``, no biases.
The output is the weighted sum of the chosen experts' outputs.

Further options, each a parameter.  ``scoring`` ``sigmoid``: ``s = sigmoid(z)`` and the chosen experts are weighted by their
``s`` as it is, or with ``renorm`` by ``s`` over the chosen ones' sum.  ``weight_scale`` multiplies the weights.  ``weight_on`` ``input``: the weight multiplies the expert's input, the output is ``sum_e expert_e(w_e h)``
(both of an expert's first products are linear, so the weight is applied to their results in fp32).  ``activation``
``clamped`` with ``limit``: ``g = min(W_gate h, limit)``, ``u = clamp(W_up h, -limit, limit)``, ``y = g sigmoid(1.702 g) (u + 1)``.
``shared``: the PartSpec of a feed-forward that every token goes through beside its routed experts; the two results add up.
``shared_gate``: its result is multiplied by ``sigmoid(w h)``, one number per token.  ``correction``: a number per expert that is
added to its score for the choice only (of runs and of experts), the weights are the scores without it.  ``group_score``
``top2_sum``: a run is scored by the sum of its two best choice scores.  ``gated`` False: experts of two matrices,
``W_down act(W_up h)`` with a plain ``activation``.

The experts' matrices are stacked at load (``[E, 2F, D]`` gate and up rows, ``[E, D, F]``).  A step routes on the
device, puts the rows of every expert side by side, and runs two grouped products over them: for prompt-sized steps in
bfloat16 the tcgen05 product over row tiles laid out on the device (``csrc/gemm_tcgen05.cu``, SwiGLU in its epilogue),
otherwise the ``mma.sync`` or fp32 kernels of ``csrc/moe.cu``.  Nothing waits for the host, so a decode step with this
feed-forward can be captured.
"""
from __future__ import annotations

from typing import List

import torch

from ..config.spec import PartSpec, TensorSpec
from ..kernels import ops
from ..registry import FEED_FORWARDS
from .base import FeedForward, Runtime, SplitBranch, StepContext, WeightView
from .linear import linear


GROUPED_MIN_ROWS = 1024      # (token, choice) rows from which a step's expert products run on tensor memory


def ctx_plain(ctx) -> bool:
    return ctx is not None and getattr(ctx, "plain_only", False)


@FEED_FORWARDS.register("routed_experts")
class RoutedExperts(FeedForward):
    """spec params: hidden, ff, experts, top, groups, keep, router (tensor name), expert (a name pattern with ``{}`` for
    the expert's number, e.g. ``mlp.e{}``; its matrices are ``.gate`` (if gated), ``.up``, ``.down``), scoring (``softmax`` or
    ``sigmoid``), renorm (default: as the scoring has it), weight_scale (default 1), weight_on (``output`` or ``input``), gated (default True), activation (gated: ``silu``, ``clamped`` or ``gelu_tanh``;
    else one of a plain feed-forward's), limit, correction (tensor name or None), group_score (``max`` or ``top2_sum``), shared
    (PartSpec or None), shared_gate (tensor name or None)."""

    @classmethod
    def tensor_specs(cls, spec: PartSpec, prefix: str) -> List[TensorSpec]:
        d, f = spec["hidden"], spec["ff"]
        out = [TensorSpec(prefix + spec["router"], (spec["experts"], d), role="router")]
        if spec.get("correction"):
            out.append(TensorSpec(prefix + spec["correction"], (spec["experts"],), role="bias"))
        for e in range(spec["experts"]):
            stem = prefix + spec["expert"].format(e)
            if spec.get("gated", True):
                out.append(TensorSpec(stem + ".gate", (f, d)))
            out += [TensorSpec(stem + ".up", (f, d)), TensorSpec(stem + ".down", (d, f))]
        if spec.get("shared") is not None:
            if spec.get("shared_gate"):
                out.append(TensorSpec(prefix + spec["shared_gate"], (1, d)))
            out += FEED_FORWARDS.get(spec["shared"].kind).tensor_specs(spec["shared"], prefix)
        return out

    def __init__(self, spec: PartSpec, weights: WeightView, rt: Runtime):
        super().__init__(spec, weights, rt)
        self.hidden, self.ff = int(spec["hidden"]), int(spec["ff"])
        self.experts, self.top = int(spec["experts"]), int(spec["top"])
        self.groups, self.keep = int(spec.get("groups", 1)), int(spec.get("keep", 1))
        if self.experts % self.groups or not (0 < self.keep <= self.groups) or not (0 < self.top <= self.keep * (self.experts // self.groups)):
            raise ValueError("routed experts: the experts split into equal runs, 0 < keep <= runs, and top fits into the kept runs")
        self.scoring, self.weight_on = spec.get("scoring", "softmax"), spec.get("weight_on", "output")
        self.activation, self.limit = spec.get("activation", "silu"), float(spec.get("limit", 0.0) or 0.0)
        self.renorm = spec.get("renorm")
        self.weight_scale = float(spec.get("weight_scale", 1.0))
        self.gated, self.group_score = bool(spec.get("gated", True)), spec.get("group_score", "max")
        known = ops.GLU_ACTIVATIONS if self.gated else ops.ACTIVATIONS
        if (self.scoring not in ops.ROUTER_SCORINGS or self.weight_on not in ("output", "input") or self.activation not in known
                or self.group_score not in ops.GROUP_SCORES):
            raise ValueError("routed experts: scoring is 'softmax' or 'sigmoid', weight_on 'output' or 'input', group_score 'max' or "
                             f"'top2_sum', activation one of {', '.join(sorted(known))}")
        self.shared = FEED_FORWARDS.get(spec["shared"].kind)(spec["shared"], weights, rt) if spec.get("shared") is not None else None
        self.w_router = weights.take(spec["router"]).float().contiguous()        # the router runs in fp32
        self.correction = weights.take(spec["correction"]).float().contiguous() if spec.get("correction") else None
        self.shared_gated = self.shared is not None and bool(spec.get("shared_gate"))
        if self.shared_gated:      # one more row of the router's matrix
            self.w_router = torch.cat([self.w_router, weights.take(spec["shared_gate"]).float().reshape(1, -1)], dim=0).contiguous()
        stacked_in, stacked_out = [], []
        f, d = self.ff, self.hidden
        # bfloat16 with sizes the tensor-memory product takes: gate and up rows alternate in blocks of 8, so that a tile of
        # the product holds a gate value beside its up value and the activation is the product's epilogue
        self.tensor_memory = (rt.dtype == torch.bfloat16 and rt.matmul != "simt" and f % 8 == 0 and d % 8 == 0)
        self.interleaved = self.tensor_memory and self.gated
        for e in range(self.experts):
            stem = spec["expert"].format(e)
            gate, up = weights.take(stem + ".gate") if self.gated else None, weights.take(stem + ".up")
            if not self.gated:
                stacked_in.append(up)
            elif self.interleaved:
                stacked_in.append(torch.stack([gate.view(f // 8, 8, d), up.view(f // 8, 8, d)], dim=1).reshape(2 * f, d))
            else:
                stacked_in.append(torch.cat([gate, up], dim=0))
            stacked_out.append(weights.take(stem + ".down"))
        self.w_in = torch.stack(stacked_in).to(rt.dtype).contiguous()       # [E, 2F, D], or [E, F, D] without gates
        self.w_out = torch.stack(stacked_out).to(rt.dtype).contiguous()     # [E, D, F]
        del stacked_in, stacked_out

    def forward_branches(self, x: torch.Tensor, ctx: StepContext):
        """The feed-forward's result as a list of (tensor, factor) whose weighted sum it is: the routed experts and, if the
        layer has one that no token's own number gates, the shared expert."""
        if self.shared is None or self.shared_gated:
            return [(self.forward(x, ctx), 1.0)]
        return [(self._combined(x, ctx)[0], 1.0), (self.shared.forward(x, ctx), 1.0)]

    def forward(self, x: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        y, gate = self._combined(x, ctx)
        return y if self.shared is None else ops.scaled_sum2(y, self.shared.forward(x, ctx), 1.0, 1.0, gate)

    def splits_weighed(self) -> bool:
        """True if the result in pieces (``forward_split``) is the chosen rows with their weights and nothing else."""
        return self.shared is None and self.weight_on == "output"

    def forward_split(self, x: torch.Tensor, ctx: StepContext) -> SplitBranch:
        """The result in pieces: every token's chosen rows with their weights, and the shared expert's with its gate."""
        y, wts, place, gate = self._routed(x, ctx)
        if wts is None:
            y, place = ops.moe_combine(y, None, self.rt.dtype, place=place, top=self.top), None
        return SplitBranch(y, wts, place, self.shared.forward(x, ctx) if self.shared is not None else None, gate)

    def _combined(self, x: torch.Tensor, ctx: StepContext):
        y, wts, place, gate = self._routed(x, ctx)
        return ops.moe_combine(y, wts, self.rt.dtype, place=place, top=self.top), gate

    def _routed(self, x: torch.Tensor, ctx: StepContext):
        """(the chosen experts' output rows, their weights or None where they rode on the input, the rows' places or None, the
        shared expert's gate per token or None)."""
        n = x.shape[0]
        chosen = ops.moe_router(x, self.w_router, self.top, self.groups, self.keep, scoring=self.scoring, correction=self.correction,
                                group_score=self.group_score, gate=self.shared_gated, renorm=self.renorm, scale=self.weight_scale)
        idx, wts, gate = chosen if self.shared_gated else chosen + (None,)
        n_rows = n * self.top
        on_input = self.weight_on == "input"
        if self.tensor_memory and n_rows >= GROUPED_MIN_ROWS and not ctx_plain(ctx):
            # prompt-sized: the rows are copied into sorted order once, and both products run on tensor memory over tiles of
            # 128 rows of one expert; the outputs stay in sorted order and the weighted sum fetches them by place
            rows = ops.moe_sort(idx, self.experts, with_tiles=True)
            if on_input:        # the weight rides on the copy: expert(w h) with w h rounded to the rows' dtype
                sorted_x = ops.moe_gather_scaled(x, rows, wts)
            else:
                sorted_x = torch.empty((n_rows, self.hidden), dtype=x.dtype, device=x.device)
                ops.gather_rows(x, rows.row_token, sorted_x)
            hidden = ops.moe_gemm_grouped(sorted_x, self.w_in, rows, swiglu=self.gated, activation=self.activation, limit=self.limit,
                                          single=not self.gated)
            y = ops.moe_gemm_grouped(hidden, self.w_out, rows, swiglu=False)
            return y, (None if on_input else wts), rows.place, gate
        rows = ops.moe_sort(idx, self.experts)
        tc = self.rt.matmul != "simt"
        hidden = ops.moe_gemm(x, self.w_in, rows, n_rows, self.top, self.gated, self.rt.dtype, tensor_cores=tc, interleaved=self.interleaved,
                              activation=self.activation, limit=self.limit, row_scale=wts if on_input else None, single=not self.gated)
        y = ops.moe_gemm(hidden, self.w_out, rows, n_rows, self.top, False, torch.float32, tensor_cores=tc)
        return y, (None if on_input else wts), None, gate


@FEED_FORWARDS.register("gated_mlp")
class GatedMLP(FeedForward):
    """A two-matrix gated feed-forward with its activation as a parameter: ``y = W_down act(W_gate h, W_up h)``, no biases.
    ``activation`` ``silu``: ``silu(g) u``; ``clamped`` with ``limit``: ``g = min(g, limit)``, ``u = clamp(u, -limit, limit)``,
    ``g sigmoid(1.702 g) (u + 1)``.  The gate's and the up projection's rows are one product with an fp32 result, the
    activation a pass of its own.

    spec params: hidden, intermediate, activation, limit, gate, up, down (tensor names under the prefix)."""

    @classmethod
    def tensor_specs(cls, spec: PartSpec, prefix: str) -> List[TensorSpec]:
        d, f = spec["hidden"], spec["intermediate"]
        return [TensorSpec(prefix + spec["gate"], (f, d)), TensorSpec(prefix + spec["up"], (f, d)), TensorSpec(prefix + spec["down"], (d, f))]

    def __init__(self, spec: PartSpec, weights: WeightView, rt: Runtime):
        super().__init__(spec, weights, rt)
        self.hidden, self.intermediate = int(spec["hidden"]), int(spec["intermediate"])
        self.activation, self.limit = spec.get("activation", "silu"), float(spec.get("limit", 0.0) or 0.0)
        if self.activation not in ops.GLU_ACTIVATIONS:
            raise ValueError("gated mlp: activation is 'silu' or 'clamped'")
        gate, up = weights.take(spec["gate"]), weights.take(spec["up"])
        if gate.dtype != up.dtype:
            gate, up = gate.float(), up.float()
        self.w_gate_up = torch.cat([gate, up], dim=0).contiguous()          # [2F, D]
        del gate, up
        self.w_down = weights.take(spec["down"]).contiguous()               # [D, F]

    def forward(self, x: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        gu = linear(x, self.w_gate_up, None, self.rt, out_dtype=torch.float32)
        return linear(ops.glu_rows(gu, self.rt.dtype, self.activation, self.limit), self.w_down, None, self.rt)
