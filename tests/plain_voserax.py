"""A plain, slow implementation of the Voserax decoder in float64 on the CPU: whole sequences, no cache,
one function per mechanism, written from the design's equations.  It shares no code with the package.

A model is an embedding table, a table of position vectors, a list of layers between several residual streams, a final norm and
the embedding table again as the classifier:

    e = embed[token] + pos[position];   x_1 = ... = x_S = e
    for every sublayer f of every layer:   u = sum_s a_s x_s;   y = f(N(u));   x_t <- sum_s M[s, t] x_s + m b_t y
    logits = embed N(sum_s x_s),   N(y) = y / sqrt(mean(y^2) + eps) * w

with vectors a, b and a matrix M of each sublayer's own and one constant m of the model.  A layer is an attention and, where it
has one, a feed-forward.

* attention: q, k, v projections, each followed by a short causal convolution per channel; part of every q and k head turns by
  the position (pairs of elements half the turned part apart, YaRN frequencies and magnitude); a window of recent keys; a
  softmax whose denominator has one added; in every layer that mixes values but the first of them
  v <- (1 - lambda) v + lambda v_first, v_first being that first layer's values behind their convolution.
* feed-forward: W_down (relu(W_gate h) * (W_up h)), or clamped experts chosen by softmax scores plus a correction and weighted
  by the scores, of which the last few are the identity, plus an expert for every token times one sigmoid per token.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional, Tuple

import torch

F = torch.float64
GATE_SLOPE = 1.702


def rms_norm(x: torch.Tensor, w: Optional[torch.Tensor], eps: float) -> torch.Tensor:
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def stream_input(x: torch.Tensor, a: torch.Tensor) -> torch.Tensor:
    """x [S, n, width] -> sum_s a[s] x[s]."""
    return torch.einsum("s,snw->nw", a, x)


def stream_update(x: torch.Tensor, mix: torch.Tensor, b: torch.Tensor, y: torch.Tensor, m: float) -> torch.Tensor:
    """Every stream from all old ones: x'[t] = sum_s mix[s, t] x[s] + m b[t] y."""
    return torch.einsum("st,snw->tnw", mix, x) + m * b[:, None, None] * y


def short_conv(u: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """u [n, channels], w [channels, taps]: y[t, c] = sum_j w[c, j] u[t - taps + 1 + j, c], zeros before the first row."""
    n, taps = u.shape[0], w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=u.dtype), u])
    return sum(w[:, j] * padded[j:j + n] for j in range(taps))


def frequencies(dims: int, base: float, scaling: Optional[dict]) -> Tuple[List[float], float]:
    """(the frequency of every pair, what cos and sin are multiplied by)."""
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return plain, 1.0
    factor, original = scaling["factor"], scaling["original"]
    index = lambda turns: dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(index(scaling["fast"])), 0), min(math.ceil(index(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * r + f * (1.0 - r))
    return out, 0.1 * math.log(factor) + 1.0


def rotate(x: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    """x [n, heads, d]: the first rot.dims elements of every head turn by the row's index."""
    if rot is None:
        return x
    half = rot["dims"] // 2
    freq, mag = frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    angle = torch.arange(x.shape[0], dtype=F)[:, None] * torch.tensor(freq, dtype=F)
    c, s = mag * torch.cos(angle)[:, None, :], mag * torch.sin(angle)[:, None, :]
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], dim=-1)


def window_mask(n: int, size: Optional[int]) -> torch.Tensor:
    i = torch.arange(n)[:, None]
    j = torch.arange(n)[None, :]
    seen = j <= i
    return seen if size is None else seen & (i - j < size)


def softmax_with_one(scores: torch.Tensor) -> torch.Tensor:
    """exp(s_j) / (1 + sum exp(s_j)) over the last dimension; masked scores are -inf."""
    top = scores.amax(-1, keepdim=True).clamp_min(0.0)
    e = torch.exp(scores - top)
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


def attention(h: torch.Tensor, m: dict, w: Dict[str, torch.Tensor], v_first: Optional[torch.Tensor]) -> Tuple[torch.Tensor, torch.Tensor]:
    """(the mixer's result, the layer's values before mixing).  ``v_first``: the values to mix in, or None."""
    n = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, own = (short_conv(h @ w[c].T, w[c + ".conv"]) for c in ("q", "k", "v"))
    q, k = rotate(q.view(n, H, d), m.get("rot")), rotate(k.view(n, G, d), m.get("rot"))
    v = own if v_first is None else (1.0 - w["vmix"]) * own + w["vmix"] * v_first
    rep = H // G
    k, v = k.repeat_interleave(rep, dim=1), v.view(n, G, dv).repeat_interleave(rep, dim=1)
    scores = torch.einsum("ihd,jhd->hij", q, k) * m["scale"]
    size = (m.get("mask") or {}).get("size")
    p = softmax_with_one(scores.masked_fill(~window_mask(n, size)[None], -math.inf))
    return torch.einsum("hij,jhd->ihd", p, v).reshape(n, H * dv) @ w["o"].T, own


def dense(h: torch.Tensor, w: Dict[str, torch.Tensor]) -> torch.Tensor:
    return (torch.relu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def expert(h: torch.Tensor, gate: torch.Tensor, up: torch.Tensor, down: torch.Tensor, limit: float) -> torch.Tensor:
    g = torch.clamp(h @ gate.T, max=limit)
    u = torch.clamp(h @ up.T, min=-limit, max=limit)
    return (g * torch.sigmoid(GATE_SLOPE * g) * (u + 1.0)) @ down.T


def route(h: torch.Tensor, router: torch.Tensor, correction: torch.Tensor, r: dict) -> Tuple[torch.Tensor, torch.Tensor, torch.Tensor]:
    """(choice [n, top], weight [n, top], margin [n]): softmax scores, the choice by score + correction; the margin is the gap
    between the last chosen and the first unchosen choice score."""
    s = torch.softmax(h @ router.T, dim=-1)
    best = torch.sort(s + correction, dim=-1, descending=True, stable=True)
    idx = best.indices[:, :r["top"]]
    margin = torch.full((h.shape[0],), math.inf, dtype=F)
    if r["top"] < s.shape[1]:
        margin = best.values[:, r["top"] - 1] - best.values[:, r["top"]]
    return idx, torch.gather(s, 1, idx), margin


def moe(h: torch.Tensor, mlp: dict, w: Dict[str, torch.Tensor], margins: Optional[list] = None) -> torch.Tensor:
    choice, weight, margin = route(h, w["router"], w["correction"], mlp["router"])
    if margins is not None:
        margins.append(margin)
    E = mlp["router"]["experts"]
    out = torch.zeros_like(h)
    for e in range(w["router"].shape[0]):
        t, c = (choice == e).nonzero(as_tuple=True)
        if t.numel():
            y = h[t] if e >= E else expert(h[t], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"], mlp["expert"]["limit"])
            out[t] += weight[t, c][:, None] * y
    if mlp.get("shared") is not None:
        y = expert(h, w["shared.gate"], w["shared.up"], w["shared.down"], mlp["shared"]["limit"])
        out = out + torch.sigmoid(h @ w["shared.sg"].T) * y
    return out


def sub(weights: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v.to(F) for k, v in weights.items() if k.startswith(prefix)}


def forward(config: dict, weights: Dict[str, torch.Tensor], tokens: List[int], margins: Optional[list] = None) -> Tuple[torch.Tensor, List[torch.Tensor]]:
    """(logits [n, vocab], the sum of the streams after every layer) of one whole sequence.  ``margins`` collects every router's margin."""
    eps, mult = float(config["norm"]["eps"]), float(config["residual_mult"])
    embed = weights["embed"].to(F)
    e = embed[torch.tensor(tokens, dtype=torch.long)] + weights["pos"].to(F)[:len(tokens)]
    x = e.unsqueeze(0).repeat(config["streams"], 1, 1)
    streams, v_first = [], None
    for i, layer in enumerate(config["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        hc = sub(weights, p + "hc1.")
        y, own = attention(rms_norm(stream_input(x, hc["in"]), weights[p + "norm1"].to(F), eps), m, sub(weights, p + "mix."),
                           v_first if m.get("v_mix") else None)
        if m.get("v_mix") and v_first is None:
            v_first = own
        x = stream_update(x, hc["mix"], hc["out"], y, mult)
        if mlp is not None:
            hc, w = sub(weights, p + "hc2."), sub(weights, p + "mlp.")
            h = rms_norm(stream_input(x, hc["in"]), weights[p + "norm2"].to(F), eps)
            x = stream_update(x, hc["mix"], hc["out"], dense(h, w) if mlp["kind"] == "dense" else moe(h, mlp, w, margins), mult)
        streams.append(x.sum(0))
    return rms_norm(x.sum(0), weights["final.norm"].to(F), eps) @ embed.T, streams
