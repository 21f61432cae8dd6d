"""The dense gated feed-forward (SwiGLU, or with another activation of the gate)."""
from __future__ import annotations

from typing import Dict

import torch

from ..config.spec import PartSpec
from ..csrc import ops
from ..weights.loader import TensorDecl
from .base import FeedForward, NormedLazy, Runtime, StepContext, register_feed_forward
from .linear import Linear


@register_feed_forward("swiglu")
class SwiGLUFeedForward(FeedForward):
    """f = W_down (silu(W_gate n) * W_up n), silu(g) = g / (1 + exp(-g)), no bias
    (ExiledOfCode/KuiperLLama kuiper/source/model/llama3.cpp:692-718, swiglu_kernel.cu:18-21;
    gate = w1, up = w3, down = w2, tools/export_llama3.py:583-585).  Gate and up are stacked
    into one matrix at load (and the activation is applied in that product's epilogue where the
    tensor-core kernel runs).  ``activation`` "gelu_tanh" puts the tanh form of gelu in silu's place, "relu" a relu; "clamped" is
    min(g, limit) * sigmoid(alpha * min(g, limit)) * (clamp(u, -limit, limit) + shift) (no clamp when ``limit`` is None).  Spec:
    ``hidden_size``, ``intermediate_size``, ``activation`` ("silu"), for "clamped" ``limit``, ``alpha`` (1), ``shift`` (0), ``names``."""

    accepts_lazy_norm = True
    may_accumulate = True

    @classmethod
    def manifest(cls, spec: PartSpec, prefix: str) -> Dict[str, TensorDecl]:
        hid, inter, n = spec["hidden_size"], spec["intermediate_size"], spec["names"]
        return {prefix + n["gate"]: TensorDecl((inter, hid)), prefix + n["up"]: TensorDecl((inter, hid)),
                prefix + n["down"]: TensorDecl((hid, inter))}

    def __init__(self, spec, prefix, tensors, runtime: Runtime):
        super().__init__(spec, prefix, tensors, runtime)
        self.hidden, self.inter = int(spec["hidden_size"]), int(spec["intermediate_size"])
        self.activation = str(spec.get("activation") or "silu")
        if self.activation == "clamped":
            limit = spec.get("limit")
            self.activation = (0.0 if limit is None else float(limit), float(spec.get("alpha", 1.0)), float(spec.get("shift", 0.0)))
        elif self.activation not in ops.GATED_ACTIVATIONS:
            raise ValueError(f"unknown activation {self.activation!r} (known: {', '.join(sorted(ops.GATED_ACTIVATIONS))}, clamped)")
        n = spec["names"]
        dev, dt = runtime.device, runtime.dtype
        gate, up = (tensors[prefix + n[k]].to(device=dev, dtype=dt) for k in ("gate", "up"))
        # One product for gate and up.  Where the tensor-core kernel can apply the activation in
        # its epilogue, the rows are stored as alternating blocks of 64 gate and 64 up rows.
        self.fused = ops.swiglu_fusable(self.hidden, self.inter, dt)
        self.gate_up = Linear(ops.interleave_gate_up(gate, up) if self.fused else torch.cat([gate, up], dim=0), runtime)
        del gate, up
        self.down = Linear(tensors[prefix + n["down"]], runtime)

    def forward(self, x, step: StepContext):
        if isinstance(x, NormedLazy):
            if self.fused and self.activation == "silu" and ops.stream_fusable(x.shape[0], self.gate_up.weight):
                # gate, up and the activation in one kernel that also finishes the norm before them
                act = ops.gemm_skinny_stream(self.gate_up.weight, x.scaled, row_scale=(x.ss, x.eps), swiglu=True)
                return self.down.forward(act, allow_partials=True, sink=getattr(step, "residual_sink", None))
            x = x.dense()
        return self.down.forward(self._activated(x), allow_partials=True, sink=getattr(step, "residual_sink", None))

    def result(self, x: torch.Tensor) -> torch.Tensor:
        """The same for a caller that adds it itself: rows in the compute dtype, or float32 pieces."""
        return self.down.forward(self._activated(x), allow_partials=True)

    def _activated(self, x: torch.Tensor) -> torch.Tensor:
        act = torch.empty((x.shape[0], self.inter), dtype=self.runtime.dtype, device=x.device)
        if self.fused:
            ops.matmul_swiglu(x, self.gate_up.weight, act, activation=self.activation)
        else:
            ops.swiglu(self.gate_up.forward(x), act, activation=self.activation)
        return act
