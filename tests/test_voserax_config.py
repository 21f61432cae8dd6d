"""The Voserax configuration on the CPU: reading config.json, its faults, the model it describes, the tensors that model reads,
what it asks of the cache, the YaRN frequencies, and the plain implementation's own mechanisms against values worked out by hand."""
from __future__ import annotations

import json
import math

import pytest
import torch

import plain_voserax as P
from voserax_helpers import CONFIGS, random_weights, tensor_shapes


def _cfg(name):
    from kuiperllama_b200.config import config_from_dict
    return config_from_dict(json.loads(json.dumps(CONFIGS[name])))


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_manifest_names_and_shapes(name):
    from kuiperllama_b200.engine.model import ignorable_tensor_suffixes, model_manifest
    cfg = _cfg(name)
    assert type(cfg).__name__ == "VoseraxConfig"
    spec = cfg.to_model_spec()
    got = {k: tuple(v.shape) for k, v in model_manifest(spec).items()}
    want = tensor_shapes(CONFIGS[name])
    # the factor of the first layer that mixes values is in the checkpoint and is not read
    mixing = [i for i, l in enumerate(CONFIGS[name]["layers"]) if l["mixer"]["v_mix"]]
    for i in mixing[:1]:
        assert want.pop(f"l{i}.mix.vmix") == () and f"l{i}.mix.vmix" in ignorable_tensor_suffixes(spec)
    assert got == want


def test_round_trip_and_spec():
    from kuiperllama_b200.config import config_from_dict
    cfg = _cfg("mixed")
    assert config_from_dict(cfg.to_dict()).to_dict() == cfg.to_dict() == CONFIGS["mixed"]
    spec = cfg.to_model_spec()
    assert spec.lm_head_name is None and spec.embedding_name == "embed" and spec.embedding_multiplier is None and spec.max_positions == 500
    assert spec.embedding_position.kind == "learned" and spec.embedding_position["positions"] == 500
    assert all(l.arrangement == "streams" and l.mixer.kind == "window_attention" for l in spec.layers)
    assert all(l.mixer_streams["streams"] == 3 and l.mixer_streams["multiplier"] == 0.8 for l in spec.layers)
    assert spec.layers[2].feed_forward is None and spec.layers[2].feed_forward_norm is None and spec.layers[2].feed_forward_streams is None
    assert {"l2.norm2", "l2.hc2.in", "l2.hc2.out", "l2.hc2.mix", "l0.mix.vmix", "l1.mix.vmix"} == set(spec.ignorable_suffixes)
    assert [l.mixer.get("value_mix") for l in spec.layers] == [None, "keep", "mix", "mix", "mix"]
    a = spec.layers[0].mixer
    assert (a["num_heads"], a["num_kv_heads"], a["head_dim"], a["value_dim"], a["scale"], a["window"], a["conv"], a["sink_score"]) == (4, 2, 12, 20, 0.4, 37, 3, 0.0)
    assert spec.layers[3].mixer["window"] is None and spec.layers[2].position is None
    r = spec.layers[0].position
    assert (r.kind, r["rotary_dim"], r["theta"], r["scaling"]["rope_type"], r["scaling"]["factor"]) == ("rope", 8, 5000.0, "yarn", 4.0)
    assert spec.layers[1].position["scaling"] is None
    moe, dense = spec.layers[0].feed_forward, spec.layers[1].feed_forward
    assert (dense.kind, dense["intermediate_size"], dense["activation"]) == ("swiglu", 72, "relu")
    assert (moe["experts"], moe["identity"], moe["top"], moe["expert_size"], moe["limit"], moe["alpha"], moe["shift"], moe["scores"], moe["renormalise"],
            moe["shared_size"], moe["shared_limit"]) == (6, 2, 2, 24, 1.5, 1.702, 1.0, "softmax", False, 40, 0.9)
    assert spec.layers[3].feed_forward["identity"] == 0 and spec.layers[4].feed_forward["shared_size"] is None


def test_the_longest_sequence_comes_from_the_position_table():
    from kuiperllama_b200.config import config_from_dict
    c = json.loads(json.dumps(CONFIGS["mixed"]))
    del c["max_positions"]
    cfg = config_from_dict(c)
    assert cfg.with_tensor_shapes({"pos": (321, 64)}).to_model_spec().max_positions == 321
    assert _cfg("mixed").with_tensor_shapes({"pos": (321, 64)}).to_model_spec().max_positions == 500


def test_faults_are_listed_together():
    from kuiperllama_b200.config import ConfigError, config_from_dict
    c = json.loads(json.dumps(CONFIGS["mixed"]))
    c["streams"] = 0
    c["norm"] = {}
    del c["residual_mult"]
    c["layers"][0]["mixer"]["kv_heads"] = 3                        # 4 heads
    c["layers"][0]["mixer"]["mask"] = {"size": 0}
    c["layers"][0]["mixer"]["rot"]["dims"] = 14                    # heads of 12
    del c["layers"][0]["mlp"]["shared"]["limit"]
    del c["layers"][1]["mixer"]["conv"]
    c["layers"][1]["mixer"]["rot"]["scaling"] = {"factor": 2.0}
    c["layers"][2]["type"] = "delta"
    c["layers"][3]["mlp"]["router"]["top"] = 9                     # 5 experts
    c["layers"][4]["mixer"]["v_mix"] = 1
    c["layers"][4]["mlp"]["router"]["identity"] = -1
    with pytest.raises(ConfigError) as e:
        config_from_dict(c)
    msg = str(e.value)
    for part in ('"streams"', '"eps"', '"residual_mult"', "layers[0]", '"kv_heads" 3', '"size"', '"dims" 14', '"shared": "limit"', "layers[1]", '"conv"',
                 '"original"', "layers[2]", '"type"', "layers[3]", '"top" 9', "layers[4]", '"v_mix"', '"identity"'):
        assert part in msg, (part, msg)
    c = json.loads(json.dumps(CONFIGS["mixed"]))
    c["layers"][2]["mixer"]["vdim"] = 16                           # other layers mix 24 values
    with pytest.raises(ConfigError, match="mix values"):
        config_from_dict(c)


def test_cache_requests_and_state():
    """Attention asks for paged keys and values of sizes of their own over its window, and for its last taps - 1 projected rows
    (every projection padded to eight columns)."""
    from kuiperllama_b200.cache import KVRequest
    from kuiperllama_b200.config.spec import PartSpec
    from kuiperllama_b200.parts import Runtime, part_class
    spec = _cfg("mixed").to_model_spec()
    W = random_weights(CONFIGS["mixed"], 0)
    rt = Runtime(torch.device("cpu"), torch.float32)
    kv, sizes = [], []
    for layer in spec.layers:
        pos = None if layer.position is None else part_class("position", "rope")(layer.position, layer.prefix, W, rt)
        m = part_class("mixer", layer.mixer.kind)(layer.mixer, layer.prefix, W, rt, pos)
        kv.append(m.kv_request())
        sizes.append(None if m.state_request() is None else m.state_request().shape)
    assert kv == [KVRequest(2, 12, "full", 37, 20), KVRequest(3, 16, "full", 70, 8), KVRequest(1, 8, "full", 150, 24), KVRequest(3, 20, "full", None, 8),
                  KVRequest(4, 10, "full", 64, 6)]
    up = lambda n: -(-n // 8) * 8
    assert sizes == [(2 * (48 + 24 + 40),), (3 * (96 + 48 + 24),), (5 * (16 + 8 + 24),), None, (up(80) + up(40) + up(24),)]
    with pytest.raises(ValueError, match="taps"):
        part_class("mixer", "window_attention")(PartSpec("window_attention", dict(spec.layers[0].mixer.params, conv=40)), "l0.", W, rt)


@pytest.mark.parametrize("rot", [{"dims": 8, "base": 5000.0, "scaling": {"factor": 4.0, "original": 256, "fast": 16.0, "slow": 1.0}},
                                 {"dims": 20, "base": 100.0, "scaling": {"factor": 2.0, "original": 4096, "fast": 32.0, "slow": 32.0}},
                                 {"dims": 6, "base": 10.0, "scaling": {"factor": 40.0, "original": 8, "fast": 9.0, "slow": 0.001}},
                                 {"dims": 12, "base": 777.0, "scaling": None}])
def test_frequencies_and_magnitude(rot):
    from kuiperllama_b200.config.spec import PartSpec
    from kuiperllama_b200.parts import Runtime
    from kuiperllama_b200.parts.position import RotaryPosition
    sc = None if rot["scaling"] is None else dict(rot["scaling"], rope_type="yarn")
    part = RotaryPosition(PartSpec("rope", {"head_dim": 32, "rotary_dim": rot["dims"], "theta": rot["base"], "scaling": sc}), "", {},
                          Runtime(torch.device("cpu"), torch.float32))
    want, mag = P.frequencies(rot["dims"], rot["base"], rot["scaling"])
    assert torch.allclose(part.inv_freq.double(), torch.tensor(want, dtype=torch.float64), rtol=1e-6) and abs(part.magnitude - mag) < 1e-12


# ----------------------------------------------------------------------------- the plain implementation against hand values

def test_plain_frequencies():
    # dims 4, base 100: f = 1, 0.1.  index(t) = 4 ln(100 / (2 pi t)) / (2 ln 100): of t = 100 / (2 pi) it is 0, of t = 1 / (2 pi) it is 2
    t0, t2 = 100 / (2 * math.pi), 1 / (2 * math.pi)
    f, mag = P.frequencies(4, 100.0, {"factor": 10.0, "original": 100.0, "fast": t0 * 1.0000001, "slow": t2 * 1.0000001})
    assert abs(f[0] - 1.0) < 1e-12 and abs(f[1] - (0.5 * 0.1 + 0.5 * 0.01)) < 1e-12          # ramp 0 and 1/2 of lo = 0, hi = 2
    assert abs(mag - (0.1 * math.log(10.0) + 1.0)) < 1e-12
    # hi is kept below dims, lo at zero or above
    f, _ = P.frequencies(4, 100.0, {"factor": 10.0, "original": 100.0, "fast": 1e9, "slow": 1e-9})
    assert abs(f[1] - (0.1 * (1 - 1 / 3) + 0.01 / 3)) < 1e-12
    # a ramp without length steps from one to the next
    f, _ = P.frequencies(8, 10.0, {"factor": 2.0, "original": 1.0, "fast": 10.0, "slow": 9.0})
    assert abs(f[0] - 1.0) < 1e-12 and abs(f[1] - 0.5 * 10 ** -0.25) < 1e-12


def test_plain_rotation():
    x = torch.zeros(3, 1, 6, dtype=torch.float64)
    x[2, 0] = torch.tensor([1.0, 2.0, 3.0, 4.0, 5.0, 6.0])
    y = P.rotate(x, {"dims": 4, "base": 100.0, "scaling": None})[2, 0]
    for i, (u, v, a) in enumerate([(1.0, 3.0, 2.0), (2.0, 4.0, 0.2)]):
        assert abs(float(y[i]) - (u * math.cos(a) - v * math.sin(a))) < 1e-12 and abs(float(y[i + 2]) - (v * math.cos(a) + u * math.sin(a))) < 1e-12
    assert y[4:].tolist() == [5.0, 6.0]


def test_plain_convolution_window_and_softmax():
    u = torch.tensor([[1.0, 10.0], [2.0, 20.0], [3.0, 30.0]], dtype=torch.float64)
    w = torch.tensor([[0.5, 1.0, 2.0], [0.0, 0.0, 1.0]], dtype=torch.float64)
    assert P.short_conv(u, w).tolist() == [[2.0, 10.0], [5.0, 20.0], [8.5, 30.0]]
    m = P.window_mask(6, 3)
    assert m[4].tolist() == [False, False, True, True, True, False] and m[1].tolist() == [True, True] + [False] * 4 and P.window_mask(4, None)[3].all()
    p = P.softmax_with_one(torch.tensor([[0.0, 0.0, -math.inf], [-900.0, -900.0, -900.0], [800.0, 0.0, 0.0]], dtype=torch.float64))
    assert torch.allclose(p, torch.tensor([[1 / 3, 1 / 3, 0.0], [0.0, 0.0, 0.0], [1.0, 0.0, 0.0]], dtype=torch.float64))


def test_plain_streams():
    x = torch.tensor([1.0, 2.0, 5.0], dtype=torch.float64).view(3, 1, 1)
    mix = torch.tensor([[1.0, 10.0, 0.0], [0.0, 1.0, 3.0], [2.0, 0.0, 1.0]], dtype=torch.float64)          # [from, to]
    y, b = torch.full((1, 1), 4.0, dtype=torch.float64), torch.tensor([1.0, 0.0, -1.0], dtype=torch.float64)
    assert P.stream_update(x, mix, b, y, 0.5).flatten().tolist() == [1 + 10 + 2, 10 + 2, 6 + 5 - 2]
    assert P.stream_input(x, torch.tensor([1.0, -1.0, 2.0], dtype=torch.float64)).item() == 9.0


def test_plain_experts_and_router():
    one = torch.ones(1, 1, dtype=torch.float64)
    sig = lambda z: 1 / (1 + math.exp(-z))
    assert abs(float(P.expert(one, 3 * one, 0.5 * one, one, 2.0)) - 2 * sig(1.702 * 2) * 1.5) < 1e-12
    assert abs(float(P.expert(one, -3 * one, -9 * one, one, 2.0)) - -3 * sig(1.702 * -3) * -1.0) < 1e-12     # no lower clamp of the gate
    assert abs(float(P.expert(one, one, 9 * one, one, 2.0)) - sig(1.702) * 3.0) < 1e-12
    h = torch.tensor([[1.0, 2.0]], dtype=torch.float64)
    w = {"gate": torch.tensor([[1.0, 0.0], [0.0, -1.0]], dtype=torch.float64), "up": torch.ones(2, 2, dtype=torch.float64), "down": torch.eye(2, dtype=torch.float64)}
    assert P.dense(h, w).tolist() == [[3.0, 0.0]]
    z = torch.log(torch.tensor([[0.5, 0.3, 0.15, 0.05]], dtype=torch.float64))
    eye = torch.eye(4, dtype=torch.float64)
    idx, wt, margin = P.route(z, eye, torch.tensor([0.0, 0.0, 0.0, 0.6], dtype=torch.float64), {"top": 2})
    assert idx.tolist() == [[3, 0]] and torch.allclose(wt, torch.tensor([[0.05, 0.5]], dtype=torch.float64)) and abs(float(margin) - 0.2) < 1e-12
    # an identity expert gives the input back; the shared expert is weighed by one number
    mlp = {"router": {"experts": 3, "identity": 1, "top": 1}, "shared": {"ff": 1, "limit": 1.0}, "expert": {"ff": 1, "limit": 1.0}}
    t = {"router": torch.tensor([[0.0, 0.0]] * 3 + [[9.0, 9.0]], dtype=torch.float64), "correction": torch.zeros(4, dtype=torch.float64),
         "shared.gate": torch.ones(1, 2, dtype=torch.float64), "shared.up": torch.zeros(1, 2, dtype=torch.float64),
         "shared.down": torch.tensor([[1.0], [0.0]], dtype=torch.float64), "shared.sg": torch.tensor([[2.0, -1.0]], dtype=torch.float64)}
    got = P.moe(h, mlp, t)
    s = 1 / (1 + 3 * math.exp(-27.0))
    assert torch.allclose(got, torch.tensor([[s * 1.0 + 0.5 * sig(1.702), s * 2.0]], dtype=torch.float64))
