"""Gated feed-forward: ``y = (act(x·Wgᵀ) ⊙ x·Wuᵀ)·Wdᵀ`` with SiLU (or the tanh form of gelu) as the activation.

No biases (src/runtime/arch/Qwen2Backend.cpp:443-458); ``silu(g) = g / (1 + exp(−g))``
(src/compute/Activations.cpp:25-36).  Gate and up weights are concatenated at load so
that one product feeds the activation kernel.
"""
from __future__ import annotations

from typing import List, Optional

import torch

from ..config.spec import PartSpec, TensorSpec
from ..kernels import ops
from ..registry import FEED_FORWARDS
from .base import ElementwiseSink, FactoredRows, FeedForward, NativeDesc, ResidualSink, Runtime, StepContext, WeightView
from .linear import linear, linear_into


@FEED_FORWARDS.register("swiglu")
class SwiGLU(FeedForward):
    """spec params: hidden, intermediate, gate, up, down (tensor names under the prefix), activation (``silu``, the default, or
    ``gelu_tanh``)."""

    @classmethod
    def tensor_specs(cls, spec: PartSpec, prefix: str) -> List[TensorSpec]:
        d, f = spec["hidden"], spec["intermediate"]
        return [
            TensorSpec(prefix + spec["gate"], (f, d)),
            TensorSpec(prefix + spec["up"], (f, d)),
            TensorSpec(prefix + spec["down"], (d, f)),
        ]

    def __init__(self, spec: PartSpec, weights: WeightView, rt: Runtime):
        super().__init__(spec, weights, rt)
        self.hidden = int(spec["hidden"])
        self.intermediate = int(spec["intermediate"])
        self.activation = str(spec.get("activation", "silu"))
        if self.activation not in ("silu", "gelu_tanh"):
            raise ValueError("swiglu: activation is 'silu' or 'gelu_tanh'")
        gate = weights.take(spec["gate"])
        up = weights.take(spec["up"])
        if gate.dtype != up.dtype:
            gate, up = gate.float(), up.float()
        f, d = gate.shape
        # Interleave gate and up rows in blocks of 8 (rows 16j..16j+7 = gate[8j..], 16j+8..16j+15 = up[8j..]):
        # a tensor-core tile then holds a gate value and its up value together, so the activation can be
        # an epilogue of the product.  Plain concatenation when the width is not a multiple of 8.
        self.interleave = 8 if f % 8 == 0 else 0
        if self.interleave:
            self.w_gate_up = torch.stack([gate.view(f // 8, 8, d), up.view(f // 8, 8, d)], dim=1).reshape(2 * f, d).contiguous()
        else:
            self.w_gate_up = torch.cat([gate, up], dim=0).contiguous()  # [2F, d]
        del gate, up
        self.w_down = weights.take(spec["down"]).contiguous()       # [d, F]

    def native(self):
        if type(self) is not SwiGLU or self.activation != "silu":
            return None
        return NativeDesc("swiglu", {"hidden": self.hidden, "intermediate": self.intermediate, "interleave": self.interleave},
                          {"w_gate_up": self.w_gate_up, "w_down": self.w_down})

    def _tensor_cores(self) -> bool:
        return bool(self.interleave) and self.rt.dtype == torch.bfloat16 and self.w_gate_up.dtype == torch.bfloat16 \
            and self.w_down.dtype == torch.bfloat16 and self.rt.matmul != "simt"

    def fuses(self, n_tokens: int) -> bool:
        return self.activation == "silu" and self._small(n_tokens)

    def _small(self, n_tokens: int) -> bool:
        return (self._tensor_cores() and ops.small_batch_supported(n_tokens, 2 * self.intermediate, self.hidden)
                and ops.small_batch_supported(n_tokens, self.hidden, self.intermediate))

    def forward(self, x, ctx: StepContext, sink: Optional[ResidualSink] = None):
        m = x.shape[0]
        if self.activation != "silu":
            return linear(self._hidden(x), self.w_down, None, self.rt)
        if self.fuses(m):
            # a few tokens: two weight-streaming products; 1/rms and activation in the first one's epilogue,
            # residual add and the next norm in the second one's
            xin, scale = (x.xw, x.scale) if isinstance(x, FactoredRows) else (x, None)
            act = ops.gemv_bf16(xin, self.w_gate_up, None, xin.dtype, swiglu=True, scale=scale)
            if sink is None:
                return ops.gemv_bf16(act, self.w_down, None, xin.dtype)
            made = ops.gemv_bf16_residual(act, self.w_down, sink.residual, sink.norm_weight, sink.eps)
            return FactoredRows(*made) if made is not None else None
        if self._tensor_cores() and m >= ops.TCGEN05_SWIGLU_MIN_ROWS and ops.gemm_tcgen05_supported(m, 2 * self.intermediate, self.hidden):
            # prefill-sized: tcgen05 product with the activation as its epilogue (the [m, 2F] intermediate never exists)
            act = ops.gemm_tcgen05(x, self.w_gate_up, None, x.dtype, swiglu=True)
        else:
            gu = linear(x, self.w_gate_up, None, self.rt)
            act = torch.empty((m, self.intermediate), dtype=x.dtype, device=x.device)
            ops.silu_mul(gu, act, self.interleave)
        return linear(act, self.w_down, None, self.rt)


    def _hidden(self, x: torch.Tensor) -> torch.Tensor:
        """act(gate) * up for another activation than silu: in the epilogue of the weight-streaming products (a few tokens) or
        of the tcgen05 product (prompt-sized steps), otherwise an fp32 product and a pass over it."""
        m = x.shape[0]
        if self._small(m):
            return ops.gemv_bf16_glu(x, self.w_gate_up, self.activation)
        if self._tensor_cores() and m >= ops.TCGEN05_SWIGLU_MIN_ROWS and ops.gemm_tcgen05_supported(m, 2 * self.intermediate, self.hidden):
            return ops.gemm_tcgen05_glu(x, self.w_gate_up, self.activation)
        gu = linear(x, self.w_gate_up, None, self.rt, out_dtype=torch.float32)
        return ops.glu_rows(gu, self.rt.dtype, self.activation, interleave=self.interleave)


# From this model width on the up product of a prompt portion takes its bias and activation as the epilogue of this
# library's tcgen05 product; below it the library product and a separate pass are faster (measured, 2,048 tokens, whole
# step of 8 layers: width 4096 / ff 16384: 4.68 against 4.71 ms; width 2048 / ff 8192: 2.46 against 2.20 ms, where the
# step is bound by launching and the tensor maps of every call cost host time).
FUSED_UP_MIN_HIDDEN = 4096
# The exact gelu as a pass of its own takes longer (width 2048 / ff 8192: product 51 + pass 25 us against 67 us in one).
FUSED_UP_MIN_HIDDEN_OF = {"gelu_erf": 2048}


@FEED_FORWARDS.register("dense_mlp")
class DenseMLP(FeedForward):
    """Two-matrix feed-forward ``y = act(x·W_upᵀ + b_up)·W_downᵀ + b_down`` with the activation as a parameter
    (``relu2``: the square of relu; ``gelu_tanh``; ``silu``; ``relu``; ``gelu_erf``, the exact form).  Bias and activation are one fp32 pass over the
    hidden rows (``csrc/bias_act.cu``).

    spec params: hidden, ff, activation, bias (bool), up, down (weights; biases are the name + ``bias_suffix``)."""

    @classmethod
    def tensor_specs(cls, spec: PartSpec, prefix: str) -> List[TensorSpec]:
        d, f = spec["hidden"], spec["ff"]
        out = [TensorSpec(prefix + spec["up"], (f, d)), TensorSpec(prefix + spec["down"], (d, f))]
        if spec.get("bias", False):
            sfx = spec.get("bias_suffix", ".b")
            out += [TensorSpec(prefix + spec["up"] + sfx, (f,), role="bias"), TensorSpec(prefix + spec["down"] + sfx, (d,), role="bias")]
        return out

    def __init__(self, spec: PartSpec, weights: WeightView, rt: Runtime):
        super().__init__(spec, weights, rt)
        self.hidden, self.ff = int(spec["hidden"]), int(spec["ff"])
        self.activation = str(spec.get("activation", "relu2"))
        if self.activation not in ops.ACTIVATIONS:
            raise ValueError(f"dense_mlp: activation '{self.activation}' is not one of {', '.join(sorted(ops.ACTIVATIONS))}")
        self.w_up = weights.take(spec["up"]).contiguous()
        self.w_down = weights.take(spec["down"]).contiguous()
        self.b_up = self.b_down = None
        if spec.get("bias", False):
            sfx = spec.get("bias_suffix", ".b")
            self.b_up = weights.take(spec["up"] + sfx).contiguous()
            self.b_down = weights.take(spec["down"] + sfx).contiguous()

    def fuses_elementwise(self, n_tokens: int) -> bool:
        return self.b_down is None and ops.gemv_tanh_supported(self.rt, self.w_down, n_tokens)

    def forward(self, x: torch.Tensor, ctx: StepContext, sink: Optional[ElementwiseSink] = None):
        if sink is not None:
            return linear_into(self._hidden(x, ctx), self.w_down, self.rt, sink)
        return linear(self._hidden(x, ctx), self.w_down, self.b_down, self.rt)

    def _hidden(self, x: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        if (x.dtype == torch.bfloat16 and self.w_up.dtype == torch.bfloat16 and self.rt.matmul != "simt" and not ctx.plain_only
                and ops.small_batch_supported(x.shape[0], self.ff, self.hidden)):
            # a few tokens: bias and activation in the epilogue of the weight-streaming product
            return ops.gemv_bf16_act(x, self.w_up, self.b_up, self.activation)
        if (x.dtype == torch.bfloat16 and self.w_up.dtype == torch.bfloat16 and self.rt.matmul != "simt" and not ctx.plain_only
                and x.shape[0] >= ops.TCGEN05_SWIGLU_MIN_ROWS and self.hidden >= FUSED_UP_MIN_HIDDEN_OF.get(self.activation, FUSED_UP_MIN_HIDDEN)
                and ops.gemm_tcgen05_supported(x.shape[0], self.ff, self.hidden)):
            # prompt-sized and deep enough: the tcgen05 product with bias and activation as its epilogue (the hidden rows
            # never exist without their activation), as the gated feed-forward does with SwiGLU
            return ops.gemm_tcgen05_act(x, self.w_up, self.b_up, self.activation)
        hidden = linear(x, self.w_up, None, self.rt)
        return ops.bias_act(hidden, self.b_up, self.activation, hidden)


@FEED_FORWARDS.register("none")
class NoFeedForward(FeedForward):
    """Stands where a layer has no feed-forward; the block arrangement skips the sublayer."""
