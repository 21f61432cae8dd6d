"""Small Vepolix configurations and random weights for the tests, written as model folders (config.json, model.safetensors in
bfloat16).  The sizes differ from layer to layer and avoid equalities that would hide a mix-up (key size = value size, heads = kv
heads, all groups kept, top = 1, a bias table that is longer than a chunk, equal scales)."""
from __future__ import annotations

import functools
import json
import os
from typing import Dict, Optional, Sequence

import torch

import plain_vepolix as P
from terolix_helpers import tokens, write_folder  # noqa: F401  (shared by the tests)


def _att(heads, kv_heads, dim, vdim, scale, bias_max, size, v_mix, rel_rows=32):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "bias_max": bias_max,
                                           "mask": None if size is None else {"size": size}, "v_mix": v_mix, "rel_rows": rel_rows}}


def _mem(heads, dim, vdim, cap):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff, groups=None, scale=1.0, shared=None):
    m = {"kind": "moe", "router": {"experts": experts, "top": top, "scale": scale}, "expert": {"ff": ff}}
    if groups is not None:
        m["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def _model(vocab, width, layers, eps=1e-5, scale=3.0):
    return {"architecture": "Vepolix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}


CONFIGS: Dict[str, dict] = {
    # both mixers with several sizes and in no regular order; the first attention mixes no values, two later ones share; a layer
    # without feed-forward; experts with and without groups and a shared one; groups of two and of one expert; top 1; bias tables
    # of several lengths, one that is longer than its chunk; a chunk shorter than a page, one that is no multiple of anything, none
    "mixed": _model(97, 64, [
        dict(_att(4, 2, 12, 20, 0.4, 50, 37, False, 16), mlp=_moe(6, 2, 24, (3, 2), 1.7, 40)),
        dict(_mem(3, 8, 12, 9.0), mlp=_dense(72)),
        dict(_att(6, 3, 16, 8, 0.25, 100, 70, True, 32), mlp=None),
        dict(_mem(2, 24, 10, 4.0), mlp=_moe(5, 1, 16)),
        dict(_att(2, 1, 8, 24, 0.5, 20, 150, True, 24), mlp=_dense(40)),
        dict(_mem(5, 4, 16, 15.0), mlp=_moe(8, 3, 8, (2, 1), 0.6)),
        dict(_att(3, 3, 20, 8, 0.3, 300, None, True, 20), mlp=_moe(4, 4, 12, (4, 4), 2.0, 8))]),
    # sizes that are multiples of nothing: rows on no 16-byte boundary, an odd width (the last entry of the sinusoid is a sine
    # alone), odd value sizes, a chunk of one and of two positions
    "odd": _model(131, 101, [
        dict(_mem(3, 7, 5, 11.0), mlp=_dense(50)),
        dict(_att(5, 5, 10, 6, 0.35, 31, 2, True, 12), mlp=_moe(7, 3, 18, None, 1.3, 13)),
        dict(_mem(1, 33, 9, 6.0), mlp=None),
        dict(_att(6, 2, 18, 15, 0.2, 64, 41, True, 32), mlp=_moe(9, 2, 9, (3, 2), 0.9)),
        dict(_att(2, 2, 6, 5, 0.5, 9, 1, False, 8), mlp=_dense(21))], eps=3e-6, scale=1.0),
    # sizes on which the bfloat16 tensor-core kernels run (16-byte rows everywhere; key and value sizes of 32, 64 and 128; memories of
    # 64, 128 and 256 rows and slices that do not come out even)
    "wide": _model(320, 256, [
        dict(_mem(4, 64, 96, 12.0), mlp=_dense(192)),
        dict(_att(8, 2, 64, 32, 0.125, 128, 96, True), mlp=_moe(8, 2, 64, (4, 3), 1.5, 128)),
        dict(_mem(2, 256, 40, 8.0), mlp=_moe(16, 4, 128, (4, 2), 2.5, 64)),
        dict(_att(4, 1, 128, 64, 0.09, 200, 150, True), mlp=_dense(256)),
        dict(_mem(3, 128, 64, 10.0), mlp=_moe(12, 4, 64)),
        dict(_att(6, 2, 32, 128, 0.2, 60, 70, False), mlp=_dense(128))], eps=1e-6, scale=2.0),
}
# one mechanism alone (a layer needs a mixer: the feed-forwards ride on a tiny memory)
CONFIGS["only_attention"] = _model(61, 64, [dict(CONFIGS["mixed"]["layers"][2], mlp=None)])
CONFIGS["only_mlstm"] = _model(61, 64, [dict(CONFIGS["mixed"]["layers"][1], mlp=None)])
CONFIGS["only_dense"] = _model(61, 64, [dict(_mem(1, 4, 4, 5.0), mlp=_dense(136))])
CONFIGS["only_moe"] = _model(61, 64, [dict(_mem(1, 4, 4, 5.0), mlp=_moe(12, 3, 24, (4, 2), 1.4, 16))])
CONFIGS["only_v_mix"] = _model(61, 64, [dict(_att(4, 2, 8, 16, 0.3, 40, 50, True, 16), mlp=None), dict(_att(2, 2, 12, 16, 0.3, 40, 64, True, 16), mlp=None),
                                        dict(_att(2, 1, 12, 32, 0.3, 30, 33, True, 10), mlp=None)])
# chunks that decoding passes over: a page, a page and a half, a prime
CONFIGS["chunks"] = _model(53, 48, [
    dict(_att(3, 3, 12, 8, 0.4, 100, 64, True, 16), mlp=None),
    dict(_mem(2, 8, 12, 9.0), mlp=None),
    dict(_att(4, 1, 12, 24, 0.3, 50, 96, True, 20), mlp=_moe(4, 2, 16, None, 1.0, 8)),
    dict(_att(2, 1, 8, 12, 0.3, 500, 127, False, 32), mlp=None)])


def tensor_shapes(c: dict) -> Dict[str, tuple]:
    W = c["width"]
    s = {"embed": (c["vocab"], W), "final.norm": (W,), "head": (c["vocab"], W)}
    for i, layer in enumerate(c["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        s[p + "norm1"] = (W,)
        if layer["type"] == "attention":
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            s.update({p + "mix.q": (H * d, W), p + "mix.k": (G * d, W), p + "mix.v": (G * dv, W), p + "mix.o": (W, H * dv),
                      p + "mix.q.norm": (H * d,), p + "mix.k.norm": (G * d,), p + "mix.rel": (m["rel_rows"], H)})
            if m["v_mix"]:
                s[p + "mix.vmix"] = ()
        else:
            H, d, dv = m["heads"], m["dim"], m["vdim"]
            s.update({p + "mix.q": (H * d, W), p + "mix.k": (H * d, W), p + "mix.v": (H * dv, W), p + "mix.g": (H * dv, W), p + "mix.o": (W, H * dv),
                      p + "mix.norm": (H * dv,), p + "mix.i": (H, W), p + "mix.i.b": (H,), p + "mix.f": (H, W), p + "mix.f.b": (H,)})
        mlp = layer["mlp"]
        if mlp is None:
            continue
        gated = lambda at, f: {at + "gate": (f, W), at + "up": (f, W), at + "down": (W, f)}
        if mlp["kind"] == "dense":
            s.update(gated(p + "mlp.", mlp["ff"]))
            continue
        E = mlp["router"]["experts"]
        s[p + "mlp.router"], s[p + "mlp.correction"] = (E, W), (E,)
        for e in range(E):
            s.update(gated(f"{p}mlp.e{e}.", mlp["expert"]["ff"]))
        if mlp.get("shared") is not None:
            s.update(gated(p + "mlp.shared.", mlp["shared"]["ff"]))
    return s


def random_weights(c: dict, seed: int, gain: float = 1.0) -> Dict[str, torch.Tensor]:
    """bfloat16 tensors.  Matrices N(0, gain / sqrt(fan-in)); norm weights around 1; biases of order 1/2, the forget gates' around 2
    (memories that last); bias tables of order 1; mixing factors around 0.4; corrections of order 0.3 and routers wide enough that
    the choices differ from token to token."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(c).items():
        r = torch.randn(shape, generator=g)
        if name == "embed":
            t = r
        elif name.endswith(("norm1", ".norm")):
            t = 1.0 + 0.2 * r
        elif name.endswith(".rel"):
            t = r
        elif name.endswith(".vmix"):
            t = 0.4 + 0.2 * r
        elif name.endswith(".f.b"):
            t = 2.0 + r
        elif name.endswith(".correction"):
            t = 0.3 * r
        elif name.endswith((".router", "mix.i", "mix.f")):
            t = 2.5 * r / shape[1] ** 0.5
        elif len(shape) == 2:
            t = r * gain / shape[1] ** 0.5
        else:
            t = 0.5 * r
        out[name] = t.to(torch.bfloat16)
    return out


def read_folder(folder: str):
    from safetensors.torch import load_file
    with open(os.path.join(folder, "config.json")) as f:
        c = json.load(f)
    return c, {k: v.double() for k, v in load_file(os.path.join(folder, "model.safetensors")).items()}


CLOSE_CALL = 0.02     # a router's choice counts as close where another one lies within so much of the scores (sigmoids)


@functools.lru_cache(maxsize=128)
def _oracle(folder: str, toks: tuple):
    c, W = read_folder(folder)
    margins = []
    logits = P.forward(c, W, list(toks), margins)[0].float()
    logits.close_from = len(toks)                    # the first row at which some router's choice is a close call
    if margins:
        close = (torch.stack(margins).min(dim=0).values < CLOSE_CALL).nonzero()
        if close.numel():
            logits.close_from = int(close[0])
    return logits


def oracle_logits(folder: str, toks: Sequence[int]) -> torch.Tensor:
    """float32 logits [T, vocab] of the whole sequence from the plain implementation (computed in float64).  Its attribute
    ``close_from`` is the first row at which a router's choice is a close call (the number of rows if there is none)."""
    return _oracle(folder, tuple(int(t) for t in toks))


def row_errors(got: torch.Tensor, ref: torch.Tensor) -> torch.Tensor:
    got, ref = got.detach().double().cpu(), ref.detach().double().cpu()
    d = got - ref
    d = d - d.mean(dim=-1, keepdim=True)
    return d.pow(2).mean(dim=-1).sqrt() / (ref - ref.mean(dim=-1, keepdim=True)).pow(2).mean(dim=-1).sqrt().clamp_min(1e-9)


def assert_logits(got: torch.Tensor, ref: torch.Tensor, dtype: str, what: str, rows: Optional[Sequence[int]] = None) -> None:
    """Per row, the difference with its mean taken off, root mean square over the vocabulary, relative to the reference row's
    spread.  float32 (the sharp test: only the order of sums differs): 1e-4 for every row.  bfloat16 is judged by shares (half
    of the rows within 5 %, nine in ten within 30 %), because a router with a close call picks another expert than float64 does,
    which moves that row by much of its spread, under every cut and batch alike; where the shares fail and ``ref`` comes from
    ``oracle_logits`` of a whole sequence, the rows before the plain implementation's first close call are judged instead (each
    within a tenth).  ``rows``: rows that must hold the float32 limit, or a tenth of their spread in bfloat16, each (the rows a test
    is about)."""
    assert got.shape == ref.shape, f"{what}: shape {tuple(got.shape)} vs {tuple(ref.shape)}"
    assert torch.isfinite(got).all(), f"{what}: non-finite logits"
    err = row_errors(got, ref)
    worst = int(err.argmax())
    if rows is not None:
        limit = 1e-4 if dtype == "float32" else 1e-1
        for r in rows:
            assert float(err[r]) <= limit, f"{what}: row {r} is off by {float(err[r]):.3e} of its spread (limit {limit:.0e})"
    if dtype == "float32":
        assert float(err.max()) <= 1e-4, f"{what}: row {worst} is off by {float(err.max()):.3e} of its spread (limit 1e-04)"
        return
    half, most = float(err.quantile(0.5)), float(err.quantile(0.9))
    sure = getattr(ref, "close_from", None)
    if (half > 5e-2 or most > 3e-1) and sure is not None and sure < err.numel() and (sure == 0 or float(err[:sure].max()) <= 1e-1):
        return
    assert half <= 5e-2, f"{what}: half of the rows are off by more than {half:.3e} of their spread (limit 5e-02)"
    if err.numel() >= 20:
        assert most <= 3e-1, f"{what}: a tenth of the rows is off by more than {most:.3e} of their spread (limit 3e-01)"
