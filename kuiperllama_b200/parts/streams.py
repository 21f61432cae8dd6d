"""Several residual streams: how a sublayer reads them and writes into them."""
from __future__ import annotations

from typing import Dict

import torch

from ..config.spec import PartSpec
from ..csrc import ops
from ..weights.loader import TensorDecl
from .base import Runtime, StreamLinks, register_streams


@register_streams("hyper_connection")
class HyperConnection(StreamLinks):
    """Learned weights between ``streams`` residual streams and one sublayer f (after Zhu et al., "Hyper-Connections", 2024, in its
    static form):

        u = sum_s a[s] x_s;   y = f(u);   x_t <- sum_s M[s, t] x_s + multiplier * b[t] * y

    Spec: ``streams``, ``multiplier`` (1) and the tensors' names ``in`` (a), ``out`` (b) and ``mix`` (M).  All of it is 32-bit; the
    norm kernels do it (``ops.stream_norm``).  KuiperLLama has one stream (kuiper/source/model/llama3.cpp:155-164)."""

    @classmethod
    def manifest(cls, spec: PartSpec, prefix: str) -> Dict[str, TensorDecl]:
        S, n = spec["streams"], spec["names"]
        return {prefix + n["in"]: TensorDecl((S,), role="vector", init="one_plus_normal"),
                prefix + n["out"]: TensorDecl((S,), role="vector", init="one_plus_normal"),
                prefix + n["mix"]: TensorDecl((S, S), role="vector")}

    def __init__(self, spec, prefix, tensors, runtime: Runtime):
        super().__init__(spec, prefix, tensors, runtime)
        self.streams = int(spec["streams"])
        if not 1 <= self.streams <= ops.MAX_STREAMS:
            raise ValueError(f"the kernels take 1 to {ops.MAX_STREAMS} residual streams, got {self.streams}")
        n = spec["names"]
        f32 = lambda key: tensors[prefix + n[key]].to(device=runtime.device, dtype=torch.float32).contiguous()
        self.in_weights, self.mix = f32("in"), f32("mix")
        self.out_weights = (f32("out") * float(spec.get("multiplier", 1.0))).contiguous()
