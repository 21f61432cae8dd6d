"""y = x W^T: the one place that picks a matrix-product kernel.

Weights are [out, in] row-major without bias, as in ExiledOfCode/KuiperLLama
(kuiper/source/op/kernels/cuda/matmul_kernel.cu:6-54, MatmulLayer has_bias=false,
kuiper/include/op/matmul.h:12-13).  In a float32 run every product uses the plain 32-bit
kernel.  In a bfloat16 run the kernel is picked by shape; each of them accumulates in
32 bits.
"""
from __future__ import annotations

from typing import Optional

import torch

from ..csrc import ops
from .base import Accumulated, NormedLazy, Runtime


class Linear:
    def __init__(self, weight: torch.Tensor, runtime: Runtime):
        assert weight.dim() == 2
        self.weight = weight.to(device=runtime.device, dtype=runtime.dtype).contiguous()
        self.out_features, self.in_features = self.weight.shape
        self.runtime = runtime

    def forward(self, x, out_dtype: Optional[torch.dtype] = None, out: Optional[torch.Tensor] = None,
                allow_partials: bool = False, sink=None):
        """[m, in] -> [m, out].  With ``allow_partials`` the result may instead be float32
        partial sums [S, m, out] (a product of few tokens whose K range was cut over CTAs);
        the norm and the rotary kernel add such pieces themselves, which saves a pass.

        ``x`` may be ``NormedLazy`` (rows of the residual stream times a norm's weight, 1 / rms
        still to be applied): a product of few tokens applies it in its epilogue, anything else
        asks for the dense rows.  With ``sink`` (the float32 residual stream and the norm that
        reads it next) such a product adds its result into the stream itself and returns
        ``Accumulated``."""
        m = x.shape[0]
        if sink is not None and m > ops.STREAM_SINK_MAX_ROWS:
            sink = None
        if allow_partials and out is None and ops.stream_fusable(m, self.weight) and (
                isinstance(x, NormedLazy) or sink is not None):
            lazy = isinstance(x, NormedLazy)
            got = ops.gemm_skinny_stream(self.weight, x.scaled if lazy else x, row_scale=(x.ss, x.eps) if lazy else None,
                                         sink=(sink.residual, sink.norm.weight) if sink is not None else None)
            return Accumulated(got[0], got[1], sink.norm) if sink is not None else got
        if isinstance(x, NormedLazy):
            x = x.dense()
        if allow_partials and out is None:
            parts = ops.gemm_skinny_partials(x, self.weight)
            if parts is not None:
                return parts
        if out is None:
            out = torch.empty((m, self.out_features), dtype=out_dtype or self.runtime.dtype, device=x.device)
        ops.matmul(x, self.weight, out)
        return out


class StackedInput:
    """Several projections of the same rows as one product: the weights are stacked along the
    output axis once (at the first ``forward``), and every projection is a column slice of the
    result.  A part that keeps its input projections here lets others (a residual gate that reads
    the same rows) ``add`` theirs, which saves a product each; kernels take the slices by column
    offset and the matrix's row stride.  Every projection starts at a multiple of ``ALIGN`` columns
    and so does every row (rows of zeros fill the gaps), so that slices of sizes like 2 or 3 heads
    leave the others on the 16-byte boundaries that vector loads and the tensor-core kernels want.  (KuiperLLama runs wq, wk, wv as three products,
    kuiper/source/model/llama3.cpp:610-639.)"""

    ALIGN = 8

    def __init__(self, runtime: Runtime):
        self.runtime = runtime
        self._pieces = []                  # (name, weight) until the first forward; name None: a gap of zeros
        self.columns = {}                  # name -> (first column, width)
        self.linear: Optional[Linear] = None
        self.total = 0
        self.last: Optional[torch.Tensor] = None     # the product of the latest forward, [m, total]
        self.rows: Optional[torch.Tensor] = None     # and the rows it read

    def add(self, name: str, weight: torch.Tensor) -> None:
        if self.linear is not None:
            raise RuntimeError("projections must be added before the first forward")
        if name in self.columns:
            raise ValueError(f"projection {name!r} is already stacked")
        w = weight.to(device=self.runtime.device, dtype=self.runtime.dtype)
        self._pad()
        self._pieces.append((name, w))
        self.columns[name] = (self.total, w.shape[0])
        self.total += w.shape[0]

    def _pad(self) -> None:
        gap = -self.total % self.ALIGN
        if gap and self._pieces:
            like = self._pieces[0][1]
            self._pieces.append((None, torch.zeros((gap, like.shape[1]), dtype=like.dtype, device=like.device)))
            self.total += gap

    def close(self) -> None:
        """No further projection may be added: ``total`` is the product's final width."""
        if self.linear is None:
            self._pad()
            self.linear = Linear(torch.cat([w for _, w in self._pieces], dim=0), self.runtime)
            self._pieces = []

    def column(self, name: str) -> int:
        return self.columns[name][0]

    def forward(self, x: torch.Tensor, allow_partials: bool = False) -> torch.Tensor:
        """[m, total].  With ``allow_partials`` the result may be float32 pieces [S, m, total] (see ``Linear.forward``), which the
        caller's kernel adds; ``view`` is then not to be used."""
        self.close()
        self.rows = x
        self.last = self.linear.forward(x, allow_partials=allow_partials)
        return self.last

    def view(self, name: str) -> torch.Tensor:
        """The named projection of the latest forward, [m, width] with the product's row stride."""
        c, w = self.columns[name]
        return self.last[:, c:c + w]
