"""Small Voserax configurations and random weights for the tests, written as model folders (config.json, model.safetensors in
bfloat16).  The sizes differ from layer to layer and avoid equalities that would hide a mix-up (key size = value size, heads = kv
heads, as many streams as taps, the same limits for experts and shared expert, top = 1, no identity expert)."""
from __future__ import annotations

import functools
import json
import os
from typing import Dict, Optional, Sequence

import torch

import plain_voserax as P
from terolix_helpers import tokens, write_folder  # noqa: F401  (shared by the tests)


def _rot(dims, base=10000.0, factor=None, original=256, fast=16.0, slow=1.0):
    return {"base": base, "dims": dims, "scaling": None if factor is None else {"factor": factor, "original": original, "fast": fast, "slow": slow}}


def _att(heads, kv_heads, dim, vdim, scale, conv, rot, size, v_mix, mlp=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "conv": conv, "rot": rot,
                                           "mask": None if size is None else {"size": size}, "v_mix": v_mix}, "mlp": mlp}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff, limit, identity=None, shared=None):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}
    if identity is not None:
        m["router"]["identity"] = identity
    if shared is not None:
        m["shared"] = {"ff": shared[0], "limit": shared[1]}
    return m


def _model(vocab, width, streams, mult, layers, eps=1e-5, positions=500):
    return {"architecture": "Voserax", "vocab": vocab, "width": width, "streams": streams, "residual_mult": mult, "norm": {"eps": eps},
            "max_positions": positions, "layers": layers}


CONFIGS: Dict[str, dict] = {
    # several sizes in no regular order: the first layer mixes no values, three later ones share; layers without feed-forward; experts
    # with and without identity and shared ones; taps 1 to 6; windows shorter than a page, off and on its border, none; no rotation
    "mixed": _model(97, 64, 3, 0.8, [
        _att(4, 2, 12, 20, 0.4, 3, _rot(8, 5000.0, 4.0), 37, False, _moe(6, 2, 24, 1.5, 2, (40, 0.9))),
        _att(6, 3, 16, 8, 0.3, 4, _rot(16, 10000.0), 70, True, _dense(72)),
        _att(2, 1, 8, 24, 0.5, 6, None, 150, True, None),
        _att(3, 3, 20, 8, 0.3, 1, _rot(4, 300.0, 2.5, 64, 8.0, 2.0), None, True, _moe(5, 4, 16, 0.7, None, (8, 2.0))),
        _att(8, 4, 10, 6, 0.35, 2, _rot(6, 700.0, 8.0), 64, True, _moe(4, 3, 12, 1.0, 3))]),
    # sizes that are multiples of nothing: rows on no 16-byte boundary, odd widths, key and value sizes, five streams, windows of one
    # and two keys
    "odd": _model(131, 101, 5, 1.3, [
        _att(5, 5, 10, 7, 0.35, 4, _rot(6, 900.0, 3.0), 2, True, _moe(7, 3, 18, 1.2, 1, (13, 0.6))),
        _att(6, 2, 18, 15, 0.2, 5, _rot(18, 2000.0), 41, False, _dense(50)),
        _att(5, 5, 7, 7, 0.4, 2, _rot(2, 50.0), 1, True, _moe(9, 2, 9, 0.8))], eps=3e-6),
    # sizes on which the bfloat16 tensor-core kernels run (16-byte rows everywhere; key and value sizes of 32, 64, 96 and 128)
    "wide": _model(320, 256, 2, 0.6, [
        _att(8, 2, 64, 32, 0.125, 4, _rot(32, 50000.0, 4.0, 128), 96, True, _moe(8, 2, 64, 1.1, 3, (128, 0.8))),
        _att(6, 1, 96, 64, 0.1, 3, _rot(48, 20000.0, 2.0, 200), 65, True, _dense(192)),
        _att(4, 2, 128, 96, 0.09, 2, _rot(64, 500000.0), 150, False, _moe(12, 4, 128, 0.9, 4, (64, 1.7))),
        _att(2, 2, 32, 32, 0.2, 4, _rot(32, 10000.0, 16.0, 512, 32.0, 1.0), None, True, _moe(16, 5, 64, 2.0)),
        _att(12, 4, 96, 128, 0.1, 8, None, 130, False, _dense(256))], eps=1e-6),
}
# one mechanism alone
CONFIGS["only_attention"] = _model(61, 64, 1, 1.0, [_att(4, 2, 16, 24, 0.3, 1, None, 33, False)])
CONFIGS["only_rotation"] = _model(61, 64, 1, 0.9, [_att(4, 2, 32, 24, 0.3, 1, _rot(24, 500.0, 4.0, 60, 8.0, 1.0), 80, False)])
CONFIGS["only_conv"] = _model(61, 64, 1, 1.1, [_att(4, 1, 12, 16, 0.3, 5, None, 40, False), _att(3, 3, 16, 8, 0.3, 2, None, None, False)])
CONFIGS["only_streams"] = _model(61, 48, 4, 0.7, [_att(2, 1, 8, 12, 0.4, 1, None, 20, False), _att(2, 2, 12, 8, 0.4, 2, None, 30, False)])
CONFIGS["only_dense"] = _model(61, 64, 1, 1.0, [_att(1, 1, 4, 4, 0.5, 1, None, 4, False, _dense(136))])
CONFIGS["only_moe"] = _model(61, 64, 1, 1.0, [_att(1, 1, 4, 4, 0.5, 1, None, 4, False, _moe(12, 4, 24, 0.8, 5, (16, 1.4)))])
CONFIGS["only_v_mix"] = _model(61, 64, 1, 1.0, [_att(4, 2, 8, 16, 0.3, 3, _rot(8), 50, True), _att(2, 2, 12, 16, 0.3, 1, None, 64, True),
                                                _att(2, 1, 12, 32, 0.3, 2, _rot(4, 99.0), 33, True)])
# windows that decoding passes over: a page, a page and a half, a prime
CONFIGS["windows"] = _model(53, 48, 2, 0.9, [
    _att(3, 3, 12, 8, 0.4, 4, _rot(8, 1000.0), 64, True),
    _att(4, 1, 12, 24, 0.3, 3, _rot(12, 1000.0, 4.0), 96, True, _moe(4, 2, 16, 1.0, 1, (8, 0.9))),
    _att(2, 1, 8, 12, 0.3, 2, None, 127, False)])


def tensor_shapes(c: dict) -> Dict[str, tuple]:
    W, S = c["width"], c["streams"]
    s = {"embed": (c["vocab"], W), "pos": (c["max_positions"], W), "final.norm": (W,)}
    for i, layer in enumerate(c["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer["mlp"]
        H, G, d, dv, K = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
        for q in (1, 2) if mlp is not None else (1,):
            s.update({f"{p}norm{q}": (W,), f"{p}hc{q}.in": (S,), f"{p}hc{q}.out": (S,), f"{p}hc{q}.mix": (S, S)})
        for n, size in (("q", H * d), ("k", G * d), ("v", G * dv)):
            s[f"{p}mix.{n}"], s[f"{p}mix.{n}.conv"] = (size, W), (size, K)
        s[p + "mix.o"] = (W, H * dv)
        if m["v_mix"]:
            s[p + "mix.vmix"] = ()
        if mlp is None:
            continue
        gated = lambda at, f: {at + "gate": (f, W), at + "up": (f, W), at + "down": (W, f)}
        if mlp["kind"] == "dense":
            s.update(gated(p + "mlp.", mlp["ff"]))
            continue
        E = mlp["router"]["experts"]
        scored = E + mlp["router"].get("identity", 0)
        s[p + "mlp.router"], s[p + "mlp.correction"] = (scored, W), (scored,)
        for e in range(E):
            s.update(gated(f"{p}mlp.e{e}.", mlp["expert"]["ff"]))
        if mlp.get("shared") is not None:
            s.update(gated(p + "mlp.shared.", mlp["shared"]["ff"]))
            s[p + "mlp.shared.sg"] = (1, W)
    return s


def random_weights(c: dict, seed: int, gain: float = 1.0) -> Dict[str, torch.Tensor]:
    """bfloat16 tensors.  Matrices N(0, gain / sqrt(fan-in)); norm weights around 1; filters whose last tap is the largest; stream
    weights that keep the streams apart and of a size; position vectors of half the embeddings' size; mixing factors around 0.4;
    corrections and routers wide enough that the choices differ from token to token and identity experts are among them."""
    g = torch.Generator().manual_seed(seed)
    S = c["streams"]
    out = {}
    for name, shape in tensor_shapes(c).items():
        r = torch.randn(shape, generator=g)
        if name == "embed":
            t = r
        elif name == "pos":
            t = 0.5 * r
        elif name.endswith(("norm1", "norm2", ".norm")):
            t = 1.0 + 0.2 * r
        elif name.endswith(".conv"):
            t = 0.4 * r
            t[:, -1] += 0.8
        elif ".hc" in name:
            t = 0.3 * r
            if name.endswith(".mix"):
                t = 0.3 * r / S ** 0.5 + 0.9 * torch.eye(S)
            elif name.endswith(".in"):
                t = 0.3 * r + 1.0 / S
            else:
                t = 0.3 * r + 0.8
        elif name.endswith(".vmix"):
            t = 0.4 + 0.2 * r
        elif name.endswith(".correction"):
            t = 0.1 * r
        elif name.endswith(".router"):
            t = 2.0 * r / shape[1] ** 0.5
        elif name.endswith(".sg"):
            t = 1.5 * r / shape[1] ** 0.5
        else:
            t = r * gain / shape[1] ** 0.5
        out[name] = t.to(torch.bfloat16)
    return out


def read_folder(folder: str):
    from safetensors.torch import load_file
    with open(os.path.join(folder, "config.json")) as f:
        c = json.load(f)
    return c, {k: v.double() for k, v in load_file(os.path.join(folder, "model.safetensors")).items()}


CLOSE_CALL = 0.01     # a router's choice counts as close where another one lies within so much of the choice scores


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
