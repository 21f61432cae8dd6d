"""Grouped-query attention over a window of recent keys, with the options that softmax attention in the plain
Llama form does not have: biased projections, a norm on q and k heads or over the whole projection, interleaved
rotary pairs, values of another size, a sink, sigmoid weights, pooled blocks before the window, chunks, a bias by
distance, short convolutions behind the projections, and values mixed with another layer's."""
from __future__ import annotations

import math
from typing import Dict, Optional

import torch

from ..cache import CacheView, KVRequest, StateRequest
from ..config.spec import PartSpec
from ..csrc import ops
from ..weights.loader import TensorDecl
from .base import Mixer, PositionEncoding, Runtime, StepContext, register_mixer
from .linear import Linear, StackedInput


def distance_buckets(distances: int, rows: int, largest: float) -> torch.Tensor:
    """int64 [distances]: the row of a bias table of ``rows`` rows that distance n reads.  The first rows // 2 distances have a
    row each; from there on the rows stand for distances that grow by a constant factor, the last row for ``largest`` and
    everything beyond: half + floor(ln(n / half) / ln(largest / half) * (rows - half)), at most rows - 1."""
    half = rows // 2
    out = []
    for n in range(distances):
        if n < half:
            out.append(n)
        elif largest <= half:
            out.append(rows - 1)
        else:
            out.append(min(rows - 1, half + int(math.floor(math.log(n / half) / math.log(largest / half) * (rows - half)))) if half else rows - 1)
    return torch.tensor(out, dtype=torch.int64)


@register_mixer("window_attention")
class WindowAttentionMixer(Mixer):
    """q = Wq n (+ bq), k = Wk n (+ bk), v = Wv n (+ bv) or, with ``values`` = "keys", v = k as projected; the first
    ``rotary_dim`` elements of every q and k head turn by the position (either pairing; no rotation without a
    position part); with ``head_norm`` every q and k head is then divided by its root mean square (eps inside the
    root) and multiplied by a weight per element shared by the heads where ``names`` gives ``q_norm`` / ``k_norm``;
    score = (q . k) * ``scale``; token i sees key j when 0 <= i - j < ``window`` (None: every earlier key) and, with
    ``pool`` = P, one mean key and mean value (of the keys and values as the cache holds them) for every block of P
    positions that lies wholly before the window; ``weights`` "softmax" over what is seen (with ``names['sink']`` a
    learned number per head joins the denominator as exp(sink)) or "sigmoid": sigmoid(score + b_h) with
    ``names['head_bias']``, not normalised; head h reads kv head h // (H / KV); out = Wo on the heads side by side.

    ``row_norm``: q and k are instead RMS-normed over their WHOLE projection before it is split into heads (``q_norm`` and
    ``k_norm`` then hold a weight per row of the projection; no biases, no rotation).  ``chunk`` = C: token i sees the keys
    j <= i of its own chunk of C positions, floor(i / C) = floor(j / C), counted from the sequence's first position.
    ``distance_bias`` {"rows", "largest"}: with ``names['distance_bias']`` [rows, heads] the score gets
    table[bucket(i - j), h] after the scaling (``distance_buckets``).  ``value_mix``: "keep" leaves the layer's values as
    projected for later layers of the step; "mix" caches (1 - lambda) v + lambda v_kept, lambda = ``names['value_mix']``, one number.

    ``conv`` = taps: every channel of q, k and v passes a causal filter of so many taps over time directly behind its projection
    (``names['q_conv']``, ``['k_conv']``, ``['v_conv']`` [channels, taps]; y_t = sum_j w[:, j] u_(t - taps + 1 + j), nothing before the
    sequence's start), before rotation and value mixing; the last taps - 1 projected rows are state of the sequence.  ``sink_score``: a
    number s, the same for every head and not learned: exp(s) joins the softmax's denominator.

    One product makes q | k | v; ``ops.qk_prepare`` does bias, rotation, norm and the cache write in one kernel;
    ``ops.qk_row_prepare`` does norm over rows, value mixing and cache write; ``ops.qkv_conv`` does convolutions, rotation, value mixing
    and cache write; ``ops.pool_blocks`` writes the means of the blocks
    that the step completes.  Chunks, a distance bias and values of another size run on the tensor cores for bfloat16 key and
    value sizes of 32, 64, 96 and 128 (``ops.attention_chunked_mma``), with a sink too.  Softmax without pooled blocks
    runs on the attention kernels of ``AttentionMixer`` where they take the sizes; a sink, sigmoid weights and pooled blocks
    are options of the windowed tensor-core kernel (bfloat16, equal key and value sizes of 64 or 128, groups of up to 16
    heads); everything else runs on the plain kernels.

    Spec: ``hidden_size``, ``num_heads``, ``num_kv_heads``, ``head_dim``, ``value_dim``, ``scale``, ``window``, ``values``
    ("own" | "keys"), ``weights`` ("softmax" | "sigmoid"), ``pool`` (None), ``head_norm`` (None | {"eps"}), ``row_norm``
    (None | {"eps"}), ``chunk``, ``distance_bias``, ``value_mix`` (None | "keep" | "mix"), ``conv``, ``sink_score``, ``names`` (q, k, o and
    optionally v, q_bias, k_bias, v_bias, q_norm, k_norm, sink, head_bias, distance_bias, value_mix, q_conv, k_conv, v_conv).  KuiperLLama's attention is
    the unbiased causal softmax over every earlier key (kuiper/source/model/llama3.cpp:610-639, mha_kernel.cu:61,74-106)."""

    KERNEL = "mma"                # "simt": the plain kernels also for bfloat16 (for comparisons)
    chunk = 0                     # positions per chunk; 0: no chunks

    @classmethod
    def manifest(cls, spec: PartSpec, prefix: str) -> Dict[str, TensorDecl]:
        hid, H, KV, hd = spec["hidden_size"], spec["num_heads"], spec["num_kv_heads"], spec["head_dim"]
        vd = spec.get("value_dim") or hd
        n = spec["names"]
        m = {prefix + n["q"]: TensorDecl((H * hd, hid)), prefix + n["k"]: TensorDecl((KV * hd, hid)),
             prefix + n["o"]: TensorDecl((hid, H * vd))}
        if spec.get("values", "own") != "keys":
            m[prefix + n["v"]] = TensorDecl((KV * vd, hid))
        for key, size in (("q_bias", H * hd), ("k_bias", KV * hd), ("v_bias", KV * vd), ("sink", H), ("head_bias", H)):
            if n.get(key):
                m[prefix + n[key]] = TensorDecl((size,), role="vector")
        for key, heads in (("q_norm", H), ("k_norm", KV)):
            if n.get(key):
                size = heads * hd if spec.get("row_norm") is not None else hd
                m[prefix + n[key]] = TensorDecl((size,), role="vector", init="one_plus_normal")
        if spec.get("distance_bias") is not None:
            m[prefix + n["distance_bias"]] = TensorDecl((spec["distance_bias"]["rows"], H), role="vector")
        if spec.get("value_mix") == "mix":
            m[prefix + n["value_mix"]] = TensorDecl((), role="vector")
        if spec.get("conv"):
            for key, size in (("q_conv", H * hd), ("k_conv", KV * hd), ("v_conv", KV * vd)):
                m[prefix + n[key]] = TensorDecl((size, spec["conv"]), role="vector")
        return m

    def __init__(self, spec, prefix, tensors, runtime: Runtime, position: Optional[PositionEncoding] = None):
        super().__init__(spec, prefix, tensors, runtime, position)
        self.hidden = int(spec["hidden_size"])
        self.H, self.KV, self.hd = int(spec["num_heads"]), int(spec["num_kv_heads"]), int(spec["head_dim"])
        self.vd = int(spec.get("value_dim") or self.hd)
        if self.H % self.KV:
            raise ValueError(f"{self.H} heads are not a multiple of {self.KV} kv heads")
        self.values_are_keys = spec.get("values", "own") == "keys"
        if self.values_are_keys and self.vd != self.hd:
            raise ValueError(f"values that are the keys have the keys' size {self.hd}, not {self.vd}")
        self.window = spec.get("window")
        self.pool = int(spec.get("pool") or 0)
        if self.pool and not self.window:
            raise ValueError("pooled blocks lie before a window: a window is needed")
        self.weights = str(spec.get("weights", "softmax"))
        if self.weights not in ops.ATTENTION_WEIGHTS:
            raise ValueError(f"unknown attention weights {self.weights!r} (softmax, sigmoid)")
        self.scale = float(spec["scale"])
        self.chunk = int(spec.get("chunk") or 0)
        self.value_mix = spec.get("value_mix")
        if self.value_mix not in (None, "keep", "mix"):
            raise ValueError(f"unknown value mixing {self.value_mix!r} (keep, mix)")
        row_norm = spec.get("row_norm")
        self.taps = int(spec.get("conv") or 0)
        if self.taps > ops.QKV_CONV_MAX_TAPS:
            raise ValueError(f"the convolution kernel takes up to {ops.QKV_CONV_MAX_TAPS} taps, got {self.taps}")
        rot = position.rotary() if position is not None else None
        # convolutions, and mixed values beside a rotation, are prepared by the kernel that does all three
        self.by_conv = self.taps > 0 or (self.value_mix is not None and rot is not None and row_norm is None)
        self.by_rows = not self.by_conv and (row_norm is not None or self.value_mix is not None)      # prepared a whole projection at a time
        norm = spec.get("head_norm") if not self.by_rows else row_norm
        self.head_norm, self.eps = norm is not None, float(norm["eps"]) if norm is not None else 0.0
        n = spec["names"]
        dev = runtime.device
        f32 = lambda key: tensors[prefix + n[key]].to(device=dev, dtype=torch.float32).contiguous() if n.get(key) else None
        self.q_bias, self.k_bias, self.v_bias = f32("q_bias"), f32("k_bias"), f32("v_bias")
        self.q_norm, self.k_norm = f32("q_norm"), f32("k_norm")
        self.sink, self.head_bias = f32("sink"), f32("head_bias")
        self.value_lambda = f32("value_mix").reshape(1) if self.value_mix == "mix" else None
        self.distance_bias = None
        if spec.get("distance_bias") is not None:
            # a column per distance up to the largest one (or as far as a chunk or window reaches): what a key at that distance gets
            rows, largest = int(spec["distance_bias"]["rows"]), float(spec["distance_bias"]["largest"])
            reach = [int(math.ceil(max(largest, rows // 2))) + 1] + [int(c) for c in (self.chunk, self.window) if c]
            table = f32("distance_bias")
            self.distance_bias = table[distance_buckets(min(reach), rows, largest).to(dev)].T.contiguous()
        if spec.get("sink_score") is not None:
            if self.sink is not None:
                raise ValueError("a learned sink and a fixed one exclude each other")
            self.sink = torch.full((self.H,), float(spec["sink_score"]), dtype=torch.float32, device=dev)
        # sizes and options for which the kernels with values of their own size are asked
        self.own_values = self.by_rows or self.by_conv or bool(self.chunk) or self.distance_bias is not None
        if self.own_values and (self.weights != "softmax" or self.pool):
            raise ValueError("chunks, a distance bias, convolutions and mixed values go with a softmax: no sigmoid weights, no pooled blocks")
        if self.by_conv and (self.values_are_keys or row_norm is not None or spec.get("head_norm") is not None
                             or any(t is not None for t in (self.q_bias, self.k_bias, self.v_bias))):
            raise ValueError("convolutions come without biases, norms on q and k, and values that are keys")
        if self.by_rows and (self.values_are_keys or spec.get("head_norm") is not None or position is not None and position.rotary() is not None
                             or any(t is not None for t in (self.q_bias, self.k_bias, self.v_bias))):
            raise ValueError("a norm over the whole projection and mixed values come without biases, head norm, rotation and values that are keys")
        if self.sink is not None and self.weights != "softmax":
            raise ValueError("a sink joins a softmax's denominator; sigmoid weights have none")
        self.inputs = StackedInput(runtime)                 # q | k | v from one product
        self.inputs.add("q", tensors[prefix + n["q"]])
        self.inputs.add("k", tensors[prefix + n["k"]])
        if not self.values_are_keys:
            self.inputs.add("v", tensors[prefix + n["v"]])
        self.o = Linear(tensors[prefix + n["o"]], runtime)
        self.inv_freq, self.rotary_dim = rot if rot is not None else (None, 0)
        self.magnitude = float(getattr(position, "magnitude", 1.0)) if rot is not None else 1.0
        if self.magnitude != 1.0 and not self.by_conv:
            raise ValueError("without convolutions this mixer's kernel rotates with unit magnitude")
        self.interleaved = getattr(position, "pairing", "half") == "interleaved"
        self.conv_weight = None
        if self.taps:
            self.inputs.close()                             # the filters lie by column of the product
            self.conv_weight = torch.zeros((self.taps, self.inputs.total), dtype=torch.float32, device=dev)
            for key in ("q", "k", "v"):
                c, w = self.inputs.columns[key]
                self.conv_weight[:, c:c + w] = f32(key + "_conv").T

    def kv_request(self) -> Optional[KVRequest]:
        value_dim = None if self.vd == self.hd else self.vd
        if self.pool:
            return KVRequest(kv_heads=self.KV, head_dim=self.hd, kind="pooled", window=self.window, value_dim=value_dim, pool=self.pool)
        return KVRequest(kv_heads=self.KV, head_dim=self.hd, kind="full", window=self.window, value_dim=value_dim, chunk=self.chunk or None)

    def state_request(self) -> Optional[StateRequest]:
        return StateRequest(((self.taps - 1) * self.inputs.total,), torch.float32) if self.taps > 1 else None

    def forward(self, x, step: StepContext, cache: CacheView) -> torch.Tensor:
        if hasattr(x, "dense"):
            x = x.dense()
        if self.own_values:
            return self._forward_own_values(x, step, cache)
        n, dt = step.n_tokens, self.runtime.dtype
        proj = self.inputs.forward(x)
        q_col = self.inputs.column("q")
        write = cache.writable
        ops.qk_prepare(proj, q_col, self.inputs.column("k"), None if self.values_are_keys else self.inputs.column("v"),
                       step.positions, step.token_slot, cache.block_table, cache.k if write else None, cache.v if write else None,
                       n, self.H, self.KV, self.hd, self.vd, q_bias=self.q_bias, k_bias=self.k_bias, v_bias=self.v_bias,
                       inv_freq=self.inv_freq, rotary_dim=self.rotary_dim, interleaved=self.interleaved, head_norm=self.head_norm,
                       eps=self.eps, q_norm_weight=self.q_norm, k_norm_weight=self.k_norm)
        if self.pool and write:
            ops.pool_blocks(cache.k, cache.v, cache.block_table, cache.pooled, step, self.KV, self.hd, self.vd)
        # rows that belong to no sequence (a small step's padding) are not written by the kernels: keep them defined
        make = torch.zeros if step.padded else torch.empty
        attn = make((n, self.H * self.vd), dtype=dt, device=proj.device)
        q = proj[:, q_col:q_col + self.H * self.hd]
        window = int(self.window or 0)
        if self.weights == "softmax" and not self.pool and self.sink is None and self.vd == self.hd:
            ops.attention(q, proj.stride(0), attn, cache.k, cache.v, cache.block_table, step, self.H, self.KV, self.hd, self.scale, window)
        elif (dt == torch.bfloat16 and self.KERNEL == "mma" and self.vd == self.hd and self.hd in ops.MMA_HEAD_DIMS and self.H // self.KV <= 16
              and proj.stride(0) % 2 == 0 and q.data_ptr() % 4 == 0):
            # the tensor cores: sink, sigmoid weights and pooled rows are options of the windowed kernel
            splits = 1
            if step.is_decode:
                splits = ops.decode_attention_splits(step.n_seqs, self.KV, self.hd, getattr(step, "context_class", 0))
            ops.attention_mma(q, proj.stride(0), attn, cache.k, cache.v, cache.block_table, step.cu_tokens, step.seq_slots, step.seq_starts,
                              step.seq_new, step.n_seqs, step.max_new, n, self.H, self.KV, self.hd, self.scale, window, splits,
                              few_rows=step.is_decode, sink=self.sink, weights=self.weights, head_bias=self.head_bias,
                              pooled=cache.pooled if self.pool else None)
        elif self.weights == "softmax" and not self.pool:
            ops.attention_simt(q, proj.stride(0), attn, cache.k, cache.v, cache.block_table, step.positions, step.token_slot, n,
                               self.H, self.KV, self.hd, self.scale, window, value_dim=self.vd, sink=self.sink)
        else:
            ops.attention_pooled(q, attn, cache.k, cache.v, cache.block_table, step.positions, step.token_slot, n, self.H, self.KV,
                                 self.hd, self.vd, self.scale, window, weights=self.weights, sink=self.sink, head_bias=self.head_bias,
                                 pooled=cache.pooled if self.pool else None)
        return self.o.forward(attn, allow_partials=True)

    def _prepare(self, x, step: StepContext, cache: CacheView) -> torch.Tensor:
        """The queries [n, H * head_dim], ready for the scores; keys and values are in the cache."""
        n, dt = step.n_tokens, self.runtime.dtype
        write = cache.writable
        k_cache, v_cache = (cache.k, cache.v) if write else (None, None)
        if self.by_conv:
            if self.taps > 1 and not write:
                raise ValueError("an execution with convolutions keeps a state of its own; it cannot read another one's cache")
            proj = self.inputs.forward(x, allow_partials=step.is_decode)      # single tokens: the product's pieces, which the kernel adds
            q, keep, first = self._mixed_values(x, step)
            ops.qkv_conv(proj, self.inputs.column("q"), self.inputs.column("k"), self.inputs.column("v"), q, step, cache.block_table,
                         k_cache, v_cache, self.H, self.KV, self.hd, self.vd, conv_weight=self.conv_weight, state=cache.state if self.taps > 1 else None,
                         inv_freq=self.inv_freq, rotary_dim=self.rotary_dim, magnitude=self.magnitude, interleaved=self.interleaved,
                         v_first=first, v_lambda=self.value_lambda, v_keep=keep)
            return q
        if not self.by_rows:
            proj = self.inputs.forward(x)
            q_col = self.inputs.column("q")
            ops.qk_prepare(proj, q_col, self.inputs.column("k"), None if self.values_are_keys else self.inputs.column("v"),
                           step.positions, step.token_slot, cache.block_table, k_cache, v_cache, n, self.H, self.KV, self.hd, self.vd,
                           q_bias=self.q_bias, k_bias=self.k_bias, v_bias=self.v_bias, inv_freq=self.inv_freq, rotary_dim=self.rotary_dim,
                           interleaved=self.interleaved, head_norm=self.head_norm, eps=self.eps, q_norm_weight=self.q_norm,
                           k_norm_weight=self.k_norm)
            return proj[:, q_col:q_col + self.H * self.hd]
        proj = self.inputs.forward(x, allow_partials=True)          # few tokens: the product's pieces, which the kernel adds
        q, keep, first = self._mixed_values(x, step)
        ops.qk_row_prepare(proj, self.inputs.column("q"), self.inputs.column("k"), self.inputs.column("v"), q, step, cache.block_table,
                           k_cache, v_cache, self.H, self.KV, self.hd, self.vd, norm=self.head_norm, eps=self.eps, q_norm_weight=self.q_norm,
                           k_norm_weight=self.k_norm, v_first=first, v_lambda=self.value_lambda, v_keep=keep)
        return q

    def _mixed_values(self, x, step: StepContext):
        """(rows for the queries; rows for the values this layer leaves for later ones, or None; those an earlier one left, or None)."""
        make = torch.zeros if step.padded else torch.empty
        rows = lambda width: make((step.n_tokens, width), dtype=self.runtime.dtype, device=x.device)
        keep = first = None
        if self.value_mix == "keep":
            keep = step.shared["values"] = rows(self.KV * self.vd)
        elif self.value_mix == "mix":
            first = step.shared["values"]
        return rows(self.H * self.hd), keep, first

    def _forward_own_values(self, x, step: StepContext, cache: CacheView) -> torch.Tensor:
        n, dt = step.n_tokens, self.runtime.dtype
        q = self._prepare(x, step, cache)
        # rows that belong to no sequence (a small step's padding) are not written by the kernels: keep them defined
        make = torch.zeros if step.padded else torch.empty
        attn = make((n, self.H * self.vd), dtype=dt, device=q.device)
        window = int(self.window or 0)
        if (dt == torch.bfloat16 and self.KERNEL == "mma" and self.hd in ops.CHUNKED_MMA_DIMS and self.vd in ops.CHUNKED_MMA_DIMS
                and self.H // self.KV <= 16 and q.stride(0) % 2 == 0 and q.data_ptr() % 4 == 0):
            splits = 1
            if step.is_decode:
                # never more pieces than the pages that a chunk or window spans
                reach = [-(-int(r) // ops.PAGE) + 1 for r in (self.chunk, window) if r]
                splits = min([ops.decode_attention_splits(step.n_seqs, self.KV, self.hd, getattr(step, "context_class", 0))] + reach)
            ops.attention_chunked_mma(q, q.stride(0), attn, cache.k, cache.v, cache.block_table, step, self.H, self.KV, self.hd, self.vd,
                                      self.scale, window=window, chunk=self.chunk, distance_bias=self.distance_bias, sink=self.sink,
                                      splits=splits, few_rows=step.is_decode)
        else:
            ops.attention_simt(q, q.stride(0), attn, cache.k, cache.v, cache.block_table, step.positions, step.token_slot, n, self.H, self.KV,
                               self.hd, self.scale, window, value_dim=self.vd, sink=self.sink, chunk=self.chunk, distance_bias=self.distance_bias)
        return self.o.forward(attn, allow_partials=True)
