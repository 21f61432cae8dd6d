"""Seeded random Vepolix configurations (width, head counts, key and value sizes, chunks, bias tables and their reach, scales, gate
caps, experts and groups, shared experts, layer order: every size and constant config.json carries) through the framework against
the plain implementation: a whole prompt, a prompt followed by single tokens, and two unequal requests in one batch decoded
together, in float32 and bfloat16.  The prompts are longer than most of the drawn chunks, so chunks act in the prompt and in decoding."""
from __future__ import annotations

import random

import pytest
import torch

from vepolix_helpers import assert_logits, oracle_logits, random_weights, tokens, write_folder

pytestmark = pytest.mark.gpu
N_CONFIGS = 16


def random_config(seed: int) -> dict:
    r = random.Random(seed)
    width = r.choice([40, 64, 96, 101, 160, 256])
    shared_values = r.choice([(1, 48), (2, 24), (3, 16), (4, 12), (6, 8)])          # kv heads x value size of the layers that mix
    layers = []
    for _ in range(r.randint(2, 6)):
        kind = r.choice(["dense", "moe", "moe", None])
        mlp = None
        if kind == "dense":
            mlp = {"kind": "dense", "ff": r.choice([8, 33, 64, 128, 200])}
        elif kind == "moe":
            count = r.choice([1, 1, 2, 3, 4])
            per = r.randint(1, 5)
            keep = r.randint(1, count)
            mlp = {"kind": "moe", "router": {"experts": count * per, "top": r.randint(1, min(keep * per, 5)), "scale": r.choice([0.5, 1.0, 2.5])},
                   "expert": {"ff": r.choice([8, 24, 32, 64, 96])}}
            if count > 1 or r.random() < 0.3:
                mlp["router"]["groups"] = {"count": count, "keep": keep}
            if r.random() < 0.6:
                mlp["shared"] = {"ff": r.choice([8, 20, 64, 128])}
        if r.random() < 0.5:
            v_mix = r.random() < 0.6
            kv = shared_values[0] if v_mix else r.choice([1, 2, 3, 4])
            dim = r.choice([2, 7, 12, 16, 24, 32, 64, 128])
            m = {"heads": kv * r.randint(1, 4), "kv_heads": kv, "dim": dim, "vdim": shared_values[1] if v_mix else r.choice([dim, 4, 15, 32, 64, 128]),
                 "scale": round(r.uniform(0.3, 1.5) / dim ** 0.5, 4), "bias_max": r.choice([5, 20, 64, 100, 1000]), "v_mix": v_mix,
                 "mask": r.choice([None] + [{"size": s} for s in (1, 2, 7, 31, 32, 33, 64, 65, 80, 200)]), "rel_rows": r.choice([2, 6, 16, 21, 32])}
            layers.append({"type": "attention", "mixer": m, "mlp": mlp})
        else:
            layers.append({"type": "mlstm", "mixer": {"heads": r.randint(1, 6), "dim": r.choice([1, 4, 8, 16, 24, 64, 72, 128]),
                                                      "vdim": r.choice([1, 4, 8, 24, 40, 64, 80]), "gate_cap": r.choice([2.0, 6.5, 12.0, 20.0])}, "mlp": mlp})
    return {"architecture": "Vepolix", "vocab": r.randint(50, 700), "width": width, "norm": {"eps": r.choice([1e-6, 1e-5, 1e-4])},
            "embedding": {"scale": r.choice([1.0, 3.5, 10.0])}, "layers": layers}


@pytest.mark.parametrize("seed", range(N_CONFIGS))
def test_random_configuration(seed, tmp_path_factory):
    from kuiperllama_b200.engine import Engine, SequenceInput, load_model
    c = random_config(7000 + seed)
    folder = write_folder(str(tmp_path_factory.mktemp(f"vepolix-random-{seed}")), c, random_weights(c, seed))
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
