"""A plain, slow implementation of the Vepolix decoder in float64 on the CPU: whole sequences, no cache,
one function per mechanism, written from the design's equations.  It shares no code with the package.

A model is an embedding table, a list of parallel layers, a final norm and a classifier:

    x = scale * embed[token] + sinusoid(position)
    h = N1(x);  x += mixer(h) + ff(h)             (both read the same normed rows; ff may be absent)
    logits = head N(x),   N(y) = y / sqrt(mean(y^2) + eps) * w

Mixers (positions count from 0):

* ``attention``: q, k, v projections without biases, H query heads on G key/value heads; q and k RMS-normed over the WHOLE
  projection with a weight per row; no rotation; score = scale (q . k) + table[bucket(i - j), h]; query i sees key
  j <= i of its own chunk of C positions; ordinary softmax; in every layer that mixes values but the first of them
  v <- (1 - lambda) v + lambda v_first, v_first being that first layer's projected values.
* ``mlstm``: a matrix memory with exponential gates and a running maximum (Beck et al., "xLSTM: Extended Long Short-Term
  Memory", 2024), see ``mlstm_recurrence``; each head's output over its root mean square, times a weight, times
  sigmoid(W_g h).

Feed-forward: W_down (gelu(W_gate h) * (W_up h)), or experts of the same form with silu, chosen by sigmoid scores plus a
correction among the best groups (a group's score: the sum of its two best), weighted by the scores without it, plus a
shared expert.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional, Tuple

import torch

F = torch.float64


def rms_norm(x: torch.Tensor, w: Optional[torch.Tensor], eps: float) -> torch.Tensor:
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def sinusoid(n: int, width: int) -> torch.Tensor:
    """[n, width]: entry 2i is sin(p / 10000^(2i / width)), entry 2i + 1 the cosine of the same angle."""
    out = torch.zeros(n, width, dtype=F)
    for c in range(width):
        angle = torch.arange(n, dtype=F) * 10000.0 ** (-2.0 * (c // 2) / width)
        out[:, c] = torch.sin(angle) if c % 2 == 0 else torch.cos(angle)
    return out


def bucket(n: int, rows: int, largest: float) -> int:
    """The table row of distance n: one row per distance below rows / 2, then logarithmic up to ``largest``."""
    half = rows // 2
    if n < half:
        return n
    if largest <= half:
        return rows - 1
    return min(rows - 1, half + int(math.floor(math.log(n / half) / math.log(largest / half) * (rows - half))))


def distance_bias(n: int, table: torch.Tensor, largest: float) -> torch.Tensor:
    """[H, n, n]: the bias of query i and key j <= i (zero where j > i)."""
    rows = table.shape[0]
    per_distance = torch.stack([table[bucket(d, rows, largest)] for d in range(n)])      # [n, H]
    i = torch.arange(n)[:, None]
    j = torch.arange(n)[None, :]
    return per_distance[(i - j).clamp_min(0)].permute(2, 0, 1)


def chunk_mask(n: int, size: Optional[int]) -> torch.Tensor:
    i = torch.arange(n)[:, None]
    j = torch.arange(n)[None, :]
    seen = j <= i
    return seen if size is None else seen & (i // size == j // size)


def attention(h: torch.Tensor, m: dict, w: Dict[str, torch.Tensor], eps: float, v_first: Optional[torch.Tensor]) -> Tuple[torch.Tensor, torch.Tensor]:
    """(the mixer's result, the layer's values as projected).  ``v_first``: the values to mix in, or None."""
    n = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(h @ w["q"].T, w["q.norm"], eps).view(n, H, d)
    k = rms_norm(h @ w["k"].T, w["k.norm"], eps).view(n, G, d)
    own = h @ w["v"].T
    v = own if v_first is None else (1.0 - w["vmix"]) * own + w["vmix"] * v_first
    v = v.view(n, G, dv)
    rep = H // G
    k, v = k.repeat_interleave(rep, dim=1), v.repeat_interleave(rep, dim=1)
    scores = torch.einsum("ihd,jhd->hij", q, k) * m["scale"] + distance_bias(n, w["rel"], m["bias_max"])
    size = (m.get("mask") or {}).get("size")
    p = torch.softmax(scores.masked_fill(~chunk_mask(n, size)[None], -math.inf), dim=-1)
    return torch.einsum("hij,jhd->ihd", p, v).reshape(n, H * dv) @ w["o"].T, own


def mlstm_sums(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, i: torch.Tensor, f: torch.Tensor) -> Tuple[torch.Tensor, torch.Tensor]:
    """q, k [n, d] and v [n, dv] of one head, log gates i, f [n] -> (S'^T q [n, dv], max(|n' . q|, exp(-m')) + 1e-6 [n]).
    S, n and m start at zero:  m' = max(f + m, i);  S' = exp(f + m - m') S + exp(i - m') k v^T;  n' likewise with k alone."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=F)
    z = torch.zeros(k.shape[1], dtype=F)
    m = torch.zeros((), dtype=F)
    num, den = [], []
    for t in range(q.shape[0]):
        m_new = torch.maximum(f[t] + m, i[t])
        keep, take = torch.exp(f[t] + m - m_new), torch.exp(i[t] - m_new)
        S = keep * S + take * torch.outer(k[t], v[t])
        z = keep * z + take * k[t]
        m = m_new
        num.append(S.T @ q[t])
        den.append(torch.maximum((z @ q[t]).abs(), torch.exp(-m)) + 1e-6)
    return torch.stack(num), torch.stack(den)


def mlstm_recurrence(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, i: torch.Tensor, f: torch.Tensor) -> torch.Tensor:
    """[n, dv]: one head's output, the sum over the denominator."""
    num, den = mlstm_sums(q, k, v, i, f)
    return num / den[:, None]


def log_gates(h: torch.Tensor, w: Dict[str, torch.Tensor], cap: float) -> Tuple[torch.Tensor, torch.Tensor]:
    """[n, H] each: the log input gate and the log forget gate."""
    soft = lambda z: cap * torch.tanh(z / cap)
    return soft(h @ w["i"].T + w["i.b"]), torch.nn.functional.logsigmoid(soft(h @ w["f"].T + w["f.b"]))


def mlstm(h: torch.Tensor, m: dict, w: Dict[str, torch.Tensor], eps: float) -> torch.Tensor:
    n = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T).view(n, H, d) * d ** -0.5
    k = (h @ w["k"].T).view(n, H, d)
    v = (h @ w["v"].T).view(n, H, dv)
    i, f = log_gates(h, w, m["gate_cap"])
    o = torch.stack([mlstm_recurrence(q[:, a], k[:, a], v[:, a], i[:, a], f[:, a]) for a in range(H)], dim=1)
    o = rms_norm(o, None, eps).reshape(n, H * dv) * w["norm"] * torch.sigmoid(h @ w["g"].T)
    return o @ w["o"].T


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def gated(h: torch.Tensor, gate: torch.Tensor, up: torch.Tensor, down: torch.Tensor, act) -> torch.Tensor:
    return (act(h @ gate.T) * (h @ up.T)) @ down.T


def route(h: torch.Tensor, router: torch.Tensor, correction: torch.Tensor, r: dict) -> Tuple[torch.Tensor, torch.Tensor]:
    """(choice [n, top], weight [n, top]): sigmoid scores, the choice by score + correction inside the best groups."""
    s = torch.sigmoid(h @ router.T)
    c = s + correction
    E = c.shape[1]
    grp = r.get("groups") or {"count": 1, "keep": 1}
    per = E // grp["count"]
    by_group = c.view(-1, grp["count"], per)
    group_score = torch.sort(by_group, dim=-1, descending=True).values[..., :2].sum(-1)
    best = torch.sort(group_score, dim=-1, descending=True, stable=True).indices[:, :grp["keep"]]
    allowed = torch.zeros(c.shape[0], grp["count"], dtype=torch.bool)
    allowed.scatter_(1, best, True)
    masked = c.masked_fill(~allowed.repeat_interleave(per, dim=1), -math.inf)
    idx = torch.sort(masked, dim=-1, descending=True, stable=True).indices[:, :r["top"]]
    return idx, torch.gather(s, 1, idx) * r.get("scale", 1.0)


def route_margin(h: torch.Tensor, router: torch.Tensor, correction: torch.Tensor, r: dict) -> torch.Tensor:
    """[n]: how close the choice is to another one: the smaller of the gap between the last chosen and the first unchosen
    allowed score and the gap between the last kept and the first dropped group (inf where there is no other choice)."""
    s = torch.sigmoid(h @ router.T)
    c = s + correction
    E = c.shape[1]
    grp = r.get("groups") or {"count": 1, "keep": 1}
    per = E // grp["count"]
    group_score = torch.sort(c.view(-1, grp["count"], per), dim=-1, descending=True).values[..., :2].sum(-1)
    gs = torch.sort(group_score, dim=-1, descending=True, stable=True)
    gap = torch.full((c.shape[0],), math.inf, dtype=F)
    if grp["keep"] < grp["count"]:
        gap = torch.minimum(gap, gs.values[:, grp["keep"] - 1] - gs.values[:, grp["keep"]])
    allowed = torch.zeros(c.shape[0], grp["count"], dtype=torch.bool)
    allowed.scatter_(1, gs.indices[:, :grp["keep"]], True)
    val = torch.sort(c.masked_fill(~allowed.repeat_interleave(per, dim=1), -math.inf), dim=-1, descending=True).values
    if r["top"] < E:
        gap = torch.minimum(gap, val[:, r["top"] - 1] - val[:, r["top"]])
    return gap


def moe(h: torch.Tensor, mlp: dict, w: Dict[str, torch.Tensor], margins: Optional[list] = None) -> torch.Tensor:
    choice, weight = route(h, w["router"], w["correction"], mlp["router"])
    if margins is not None:
        margins.append(route_margin(h, w["router"], w["correction"], mlp["router"]))
    out = torch.zeros_like(h)
    for e in range(w["router"].shape[0]):
        t, c = (choice == e).nonzero(as_tuple=True)
        if t.numel():
            out[t] += weight[t, c][:, None] * gated(h[t], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"], silu)
    if mlp.get("shared") is not None:
        out = out + gated(h, w["shared.gate"], w["shared.up"], w["shared.down"], silu)
    return out


def sub(weights: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v.to(F) for k, v in weights.items() if k.startswith(prefix)}


def forward(config: dict, weights: Dict[str, torch.Tensor], tokens: List[int], margins: Optional[list] = None) -> Tuple[torch.Tensor, List[torch.Tensor]]:
    """(logits [n, vocab], the stream after every layer) of one whole sequence.  ``margins`` collects every router's ``route_margin``."""
    eps = float(config["norm"]["eps"])
    x = weights["embed"].to(F)[torch.tensor(tokens, dtype=torch.long)] * config["embedding"]["scale"]
    x = x + sinusoid(x.shape[0], x.shape[1])
    streams, v_first = [], None
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = rms_norm(x, weights[p + "norm1"].to(F), eps)
        w = sub(weights, p + "mix.")
        if layer["type"] == "attention":
            y, own = attention(h, m, w, eps, v_first if m.get("v_mix") else None)
            if m.get("v_mix") and v_first is None:
                v_first = own
        else:
            y = mlstm(h, m, w, eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            w = sub(weights, p + "mlp.")
            y = y + (gated(h, w["gate"], w["up"], w["down"], gelu_tanh) if mlp["kind"] == "dense" else moe(h, mlp, w, margins))
        x = x + y
        streams.append(x)
    x = rms_norm(x, weights["final.norm"].to(F), eps)
    return x @ weights["head"].to(F).T, streams
