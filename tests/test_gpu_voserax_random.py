"""Seeded random Voserax configurations (width, streams, multiplier, head counts, key and value sizes, taps, rotations, windows, experts,
identity and shared experts, limits, layer count: every size and constant config.json carries) through the framework against
the plain implementation: a whole prompt, a prompt followed by single tokens, and two unequal requests in one batch decoded
together, in float32 and bfloat16.  The prompts are longer than most of the drawn windows, so they act in the prompt and in decoding."""
from __future__ import annotations

import random

import pytest
import torch

from voserax_helpers import assert_logits, oracle_logits, random_weights, tokens, write_folder

pytestmark = pytest.mark.gpu
N_CONFIGS = 16


def random_config(seed: int) -> dict:
    r = random.Random(seed)
    width = r.choice([40, 64, 96, 101, 160, 256])
    shared_values = r.choice([(1, 48), (2, 24), (3, 16), (4, 12), (1, 64), (2, 32)])          # kv heads x value size of the layers that mix
    layers = []
    for _ in range(r.randint(1, 5)):
        kind = r.choice(["dense", "moe", "moe", None])
        mlp = None
        if kind == "dense":
            mlp = {"kind": "dense", "ff": r.choice([8, 33, 64, 128, 200])}
        elif kind == "moe":
            E, extra = r.randint(1, 14), r.choice([0, 0, 1, 2, 5])
            mlp = {"kind": "moe", "router": {"experts": E, "top": r.randint(1, min(E + extra, 5))},
                   "expert": {"ff": r.choice([8, 24, 32, 64, 96]), "limit": r.choice([0.5, 1.0, 3.0])}}
            if extra:
                mlp["router"]["identity"] = extra
            if r.random() < 0.6:
                mlp["shared"] = {"ff": r.choice([8, 20, 64, 128]), "limit": r.choice([0.4, 1.2, 7.0])}
        v_mix = r.random() < 0.6
        kv = shared_values[0] if v_mix else r.choice([1, 2, 3, 4])
        dim = r.choice([2, 7, 12, 16, 24, 32, 64, 96, 128])
        rot = None
        if r.random() < 0.8:
            rot = {"base": r.choice([50.0, 1000.0, 10000.0, 500000.0]), "dims": 2 * r.randint(1, dim // 2)}
            if r.random() < 0.8:
                fast = r.choice([2.0, 8.0, 32.0])
                rot["scaling"] = {"factor": r.choice([1.5, 4.0, 16.0]), "original": r.choice([16, 100, 1024]), "fast": fast, "slow": fast / r.choice([2.0, 8.0, 32.0])}
        m = {"heads": kv * r.randint(1, 4), "kv_heads": kv, "dim": dim, "vdim": shared_values[1] if v_mix else r.choice([dim, 4, 15, 32, 64, 96, 128]),
             "scale": round(r.uniform(0.3, 1.5) / dim ** 0.5, 4), "conv": r.choice([1, 2, 3, 4, 4, 5, 9]), "rot": rot, "v_mix": v_mix,
             "mask": r.choice([None] + [{"size": s} for s in (1, 2, 7, 31, 32, 33, 64, 65, 80, 200)])}
        layers.append({"type": "attention", "mixer": m, "mlp": mlp})
    return {"architecture": "Voserax", "vocab": r.randint(50, 700), "width": width, "streams": r.choice([1, 2, 3, 4, 6]),
            "residual_mult": r.choice([0.5, 1.0, 1.4]), "norm": {"eps": r.choice([1e-6, 1e-5, 1e-4])}, "max_positions": r.choice([90, 128, 1000]), "layers": layers}


@pytest.mark.parametrize("seed", range(N_CONFIGS))
def test_random_configuration(seed, tmp_path_factory):
    from kuiperllama_b200.engine import Engine, SequenceInput, load_model
    c = random_config(8000 + seed)
    folder = write_folder(str(tmp_path_factory.mktemp(f"voserax-random-{seed}")), c, random_weights(c, seed))
    V = c["vocab"]
    a, b = tokens(90, V, seed=seed), tokens(37, V, seed=seed + 500)
    ref_a, ref_b = oracle_logits(folder, a), oracle_logits(folder, b)
    what = f"random {seed}"
    for dtype in ("float32", "bfloat16"):
        with torch.inference_mode():
            model = load_model(folder, dtype=dtype, device="cuda:0")
            eng = Engine(model, model.new_cache(max_tokens=64 * 8))
            inp = lambda slot, toks: SequenceInput(slot, list(toks), list(range(len(toks))))
            s = eng.alloc_slot()
            assert_logits(eng.step([inp(s, a)]), ref_a, dtype, f"{what}: whole")
            eng.free_slot(s)
            s = eng.alloc_slot()
            rows = [eng.step([inp(s, a[:61])]).clone()] + [eng.step([inp(s, [t])]).clone() for t in a[61:]]
            assert_logits(torch.cat(rows), ref_a, dtype, f"{what}: prompt, then tokens")
            eng.free_slot(s)
            s, t = eng.alloc_slot(), eng.alloc_slot()
            first = eng.step([inp(s, a[:70]), inp(t, b[:3])])
            ra, rb = [first[:70].clone()], [first[70:].clone()]
            for k in range(20):
                out = eng.step([inp(s, [a[70 + k]]), inp(t, [b[3 + k]])])
                ra.append(out[:1].clone())
                rb.append(out[1:].clone())
            eng.free_slot(s)
            for k in range(23, 37):                                       # the longer-lived request goes on alone
                rb.append(eng.step([inp(t, [b[k]])]).clone())
            eng.free_slot(t)
            assert_logits(torch.cat(ra), ref_a, dtype, f"{what}: in a batch, first request")
            assert_logits(torch.cat(rb), ref_b, dtype, f"{what}: in a batch, second request")
        eng.check_device_errors()
