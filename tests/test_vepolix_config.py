"""The Vepolix configuration on the CPU: reading config.json, its faults, the model it describes, the tensors that model reads,
what it asks of the cache (pages of chunks among them), the bias buckets and the sinusoid's frequencies, and the plain
implementation's own mechanisms against values worked out by hand."""
from __future__ import annotations

import json
import math

import pytest
import torch

import plain_vepolix as P
from vepolix_helpers import CONFIGS, tensor_shapes


def _cfg(name):
    from kuiperllama_b200.config import config_from_dict
    return config_from_dict(json.loads(json.dumps(CONFIGS[name])))


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_manifest_names_and_shapes(name):
    from kuiperllama_b200.engine.model import ignorable_tensor_suffixes, model_manifest
    cfg = _cfg(name)
    assert type(cfg).__name__ == "VepolixConfig"
    spec = cfg.to_model_spec()
    got = {k: tuple(v.shape) for k, v in model_manifest(spec).items()}
    want = tensor_shapes(CONFIGS[name])
    # the factor of the first layer that mixes values is in the checkpoint and is not read
    mixing = [i for i, l in enumerate(CONFIGS[name]["layers"]) if l["type"] == "attention" and l["mixer"]["v_mix"]]
    for i in mixing[:1]:
        assert want.pop(f"l{i}.mix.vmix") == () and f"l{i}.mix.vmix" in ignorable_tensor_suffixes(spec)
    assert got == want


def test_round_trip_and_spec():
    from kuiperllama_b200.config import config_from_dict
    cfg = _cfg("mixed")
    again = config_from_dict(cfg.to_dict())
    assert again.to_dict() == cfg.to_dict() and again.to_dict()["layers"] == CONFIGS["mixed"]["layers"]
    spec = cfg.to_model_spec()
    assert spec.lm_head_name == "head" and spec.embedding_name == "embed" and spec.embedding_multiplier == 3.0 and spec.hidden_size == 64
    assert all(l.arrangement == "parallel" and l.feed_forward_norm is None and l.mixer_norm["eps"] == 1e-5 for l in spec.layers)
    assert [l.mixer.kind for l in spec.layers] == ["window_attention", "mlstm", "window_attention", "mlstm", "window_attention", "mlstm",
                                                   "window_attention"]
    assert spec.layers[0].position.kind == "sinusoidal" and spec.layers[0].position["base"] == 10000.0
    assert all(l.position is None for l in spec.layers[1:])
    assert [l.mixer.get("value_mix") for l in spec.layers] == [None, None, "keep", None, "mix", None, "mix"]
    assert "value_mix" not in spec.layers[2].mixer["names"] and spec.layers[4].mixer["names"]["value_mix"] == "mix.vmix"
    a, m = spec.layers[2].mixer, spec.layers[1].mixer
    assert (a["num_heads"], a["num_kv_heads"], a["head_dim"], a["value_dim"], a["scale"], a["chunk"], a["distance_bias"]) \
        == (6, 3, 16, 8, 0.25, 70, {"rows": 32, "largest": 100.0})
    assert spec.layers[6].mixer["chunk"] is None
    assert (m["heads"], m["dim"], m["vdim"], m["cap"], m["den_eps"], m["norm_eps"]) == (3, 8, 12, 9.0, 1e-6, 1e-5)
    assert abs(m["q_scale"] - 8 ** -0.5) < 1e-15
    assert spec.layers[2].feed_forward is None
    dense, moe = spec.layers[1].feed_forward, spec.layers[0].feed_forward
    assert (dense.kind, dense["intermediate_size"], dense["activation"]) == ("swiglu", 72, "gelu_tanh")
    assert (moe["experts"], moe["top"], moe["expert_size"], moe["groups"], moe["keep_groups"], moe["group_top"], moe["scores"],
            moe["router_scale"], moe["renormalise"], moe["shared_size"]) == (6, 2, 24, 3, 2, 2, "sigmoid", 1.7, False, 40)
    plain = spec.layers[3].feed_forward
    assert (plain["groups"], plain["keep_groups"], plain["router_scale"], plain["shared_size"]) == (1, 1, 1.0, None)


def test_the_bias_tables_rows_come_from_the_tensors():
    from kuiperllama_b200.config import config_from_dict
    c = json.loads(json.dumps(CONFIGS["mixed"]))
    for l in c["layers"]:
        l["mixer"].pop("rel_rows", None)
    cfg = config_from_dict(c)
    assert cfg.to_model_spec().layers[0].mixer["distance_bias"]["rows"] == 32
    spec = cfg.with_tensor_shapes({"l0.mix.rel": (16, 4), "l2.mix.rel": (32, 6), "l4.mix.rel": (24, 2), "l6.mix.rel": (20, 3)}).to_model_spec()
    assert [spec.layers[i].mixer["distance_bias"]["rows"] for i in (0, 2, 4, 6)] == [16, 32, 24, 20]


def test_faults_are_listed_together():
    from kuiperllama_b200.config import ConfigError, config_from_dict
    c = json.loads(json.dumps(CONFIGS["mixed"]))
    c["vocab"] = 0
    c["norm"] = {}
    del c["embedding"]
    c["layers"][0]["mixer"]["kv_heads"] = 3                        # 4 heads
    c["layers"][0]["mixer"]["mask"] = {"size": 0}
    del c["layers"][1]["mixer"]["gate_cap"]
    c["layers"][2]["mixer"]["vdim"] = 16                           # other layers mix 24 values, this one has 48
    c["layers"][3]["mlp"]["router"]["top"] = 9                     # 5 experts
    c["layers"][4]["type"] = "slstm"
    c["layers"][5]["mlp"]["router"]["groups"]["count"] = 3         # 8 experts
    c["layers"][6]["mixer"]["v_mix"] = 1
    with pytest.raises(ConfigError) as e:
        config_from_dict(c)
    msg = str(e.value)
    for part in ('"vocab"', '"eps"', '"scale"', "layers[0]", '"kv_heads" 3', '"size"', "layers[1]", '"gate_cap"', "layers[3]", '"top" 9',
                 "layers[4]", '"type"', "layers[5]", "3 equal groups", "layers[6]", '"v_mix"'):
        assert part in msg, (part, msg)
    c = json.loads(json.dumps(CONFIGS["mixed"]))
    c["layers"][2]["mixer"]["vdim"] = 16
    with pytest.raises(ConfigError, match="mix values"):
        config_from_dict(c)


def test_cache_requests_and_state():
    """Attention asks for paged keys and values of sizes of their own over its chunk; a memory for its matrix, its vector and its
    maximum in a row that keeps 16-byte boundaries."""
    from kuiperllama_b200.cache import KVRequest
    from kuiperllama_b200.parts import part_class
    spec = _cfg("mixed").to_model_spec()
    got = []
    for layer in spec.layers:
        cls = part_class("mixer", layer.mixer.kind)
        m, p = cls.__new__(cls), layer.mixer
        if p.kind == "mlstm":
            m.H, m.d, m.dv = p["heads"], p["dim"], p["vdim"]
            m.z_off = m.H * m.d * m.dv
            m.m_off = m.z_off + m.H * m.d
            size = m.state_request().shape[0]
            assert m.kv_request() is None and size % 4 == 0 and 0 <= size - (m.m_off + m.H) < 4
        else:
            m.KV, m.hd, m.vd, m.window, m.pool, m.chunk = p["num_kv_heads"], p["head_dim"], p["value_dim"], None, 0, int(p["chunk"] or 0)
            got.append(m.kv_request())
    assert got == [KVRequest(2, 12, "full", None, 20, chunk=37), KVRequest(3, 16, "full", None, 8, chunk=70),
                   KVRequest(1, 8, "full", None, 24, chunk=150), KVRequest(3, 20, "full", None, 8)]


def test_pages_below_the_chunk_go_back():
    """On the host: before every step the pages wholly below the chunk of the step's first position are given back, none that the
    step or a later one reads; also where a chunk is shorter than a page, and with a promised step size."""
    from kuiperllama_b200.cache import KVRequest, SequenceCache
    for size in (1, 40, 64, 96, 200):
        cache = SequenceCache([KVRequest(1, 4, chunk=size)], [None], [None], 64 * 40, 64 * 40, torch.float32, "cpu", max_slots=1)
        g, s, length = cache.groups[0], cache.alloc_slot(), 0
        for new in (30, 60, 9, 1, 1, 150, 1, 333, 64, 64, 1):
            cache.reserve(s, length + new)
            first = next(b for b, p in enumerate(g.slot_pages[s]) if p >= 0)
            assert first * 64 <= length // size * size, (size, length, first)          # the chunk of the step's first token is whole
            assert first == length // size * size // 64, (size, length, first)         # and nothing below it is kept
            cache.lengths[s] = length = length + new
        assert g.pages.held() == len(g.pages_of(s))
        cache.free_slot(s)
        assert g.held() == 0 and cache.slots.held() == 0
    both = KVRequest(1, 4, window=30, chunk=100)
    cache = SequenceCache([both], [None], [None], 64 * 40, 64 * 40, torch.float32, "cpu", max_slots=2, window_step_tokens=70)
    g = cache.groups[0]
    assert g.first_needed(250) == 221 and g.first_needed(205) == 200 and g.window_tokens() == 30
    assert g.pool_size() <= 2 * (2 + 1)


def test_buckets_and_frequencies():
    from kuiperllama_b200.parts.position import SinusoidalPosition
    from kuiperllama_b200.parts.base import Runtime
    from kuiperllama_b200.config.spec import PartSpec
    from kuiperllama_b200.parts.window_attention import distance_buckets
    for rows, largest in ((32, 128), (16, 50), (7, 20), (8, 3), (32, 16), (2, 10), (20, 33.5)):
        got = distance_buckets(300, rows, largest).tolist()
        assert got == [P.bucket(n, rows, largest) if rows // 2 else rows - 1 for n in range(300)], (rows, largest)
        assert got[:rows // 2] == list(range(rows // 2)) and got[-1] == rows - 1 and got == sorted(got)
        assert all(b == rows - 1 for n, b in enumerate(got) if n >= max(largest, rows // 2))
    # 16 rows up to 50: half 8; distance 8 -> 8, 20 -> 8 + floor(ln 2.5 / ln 6.25 * 8) = 12, 49 -> 15
    assert [distance_buckets(60, 16, 50).tolist()[n] for n in (7, 8, 9, 20, 49, 50)] == [7, 8, 8, 12, 15, 15]
    for hidden in (8, 101):
        pos = SinusoidalPosition(PartSpec("sinusoidal", {"hidden_size": hidden, "base": 10000.0}), "", {}, Runtime(torch.device("cpu"), torch.float32))
        f = pos.embedding_frequencies().double().sum(0)
        want = torch.tensor([10000.0 ** (-2.0 * i / hidden) for i in range((hidden + 1) // 2)], dtype=torch.float64)
        assert float((f / want - 1).abs().max()) < 1e-13 and pos.rotary() is None


# ----------------------------------------------------------------------------- the plain implementation against hand values

def test_plain_sinusoid_chunks_and_bias():
    x = P.sinusoid(3, 5)
    assert torch.allclose(x[0], torch.tensor([0.0, 1.0, 0.0, 1.0, 0.0], dtype=torch.float64))
    f = [1.0, 10000.0 ** (-2 / 5), 10000.0 ** (-4 / 5)]
    assert torch.allclose(x[2], torch.tensor([math.sin(2 * f[0]), math.cos(2 * f[0]), math.sin(2 * f[1]), math.cos(2 * f[1]), math.sin(2 * f[2])],
                                             dtype=torch.float64))
    m = P.chunk_mask(7, 3)
    assert m[5].tolist() == [False, False, False, True, True, True, False] and m[6].tolist() == [False] * 6 + [True]
    assert m[2].tolist() == [True, True, True] + [False] * 4 and P.chunk_mask(4, None)[3].all()
    table = torch.arange(12, dtype=torch.float64).view(6, 2)
    b = P.distance_bias(9, table, 8)
    assert b.shape == (2, 9, 9) and b[1, 4, 4] == table[0, 1] and b[0, 4, 2] == table[2, 0] and b[0, 8, 0] == table[5, 0]


def test_plain_memory_and_norm_over_rows():
    # one head, d = dv = 1: gates that keep and take everything (f = 0, i = 0) give a plain running sum over a running count
    one = torch.ones(4, 1, dtype=torch.float64)
    v = torch.tensor([[1.0], [2.0], [3.0], [6.0]], dtype=torch.float64)
    zero = torch.zeros(4, dtype=torch.float64)
    o = P.mlstm_recurrence(one, one, v, zero, zero)
    n = torch.tensor([1.0, 2.0, 3.0, 4.0], dtype=torch.float64)
    assert torch.allclose(o[:, 0], v[:, 0].cumsum(0) / (n + 1e-6))
    # a small key: |n q| stays below exp(-m) = 1, so the sum is divided by one
    o = P.mlstm_recurrence(one, 0.1 * one, v, zero, zero)
    assert torch.allclose(o[:, 0], 0.1 * v[:, 0].cumsum(0) / (1 + 1e-6))
    # the maximum starts at 0: an input gate of -3 alone weighs e^-3 against a floor of e^0 (with f = 0)
    o = P.mlstm_recurrence(one[:1], one[:1], v[:1], torch.tensor([-3.0], dtype=torch.float64), zero[:1])
    assert abs(float(o) - math.exp(-3.0) / (1 + 1e-6)) < 1e-12
    # and one of +3 is the new maximum: weight 1, floor e^-3
    o = P.mlstm_recurrence(one[:1], one[:1], v[:1], torch.tensor([3.0], dtype=torch.float64), zero[:1])
    assert abs(float(o) - 1.0 / (1 + 1e-6)) < 1e-12
    x = torch.tensor([[3.0, 4.0, 0.0, 0.0]], dtype=torch.float64)
    assert torch.allclose(P.rms_norm(x, None, 0.0), x / 2.5)


def test_plain_router():
    # logits such that the scores are known; four experts in two groups, corrections that turn the choice but not the weights
    z = torch.tensor([[2.0, 1.0, 0.0, -1.0]], dtype=torch.float64)
    router = torch.eye(4, dtype=torch.float64)
    s = torch.sigmoid(z)[0]
    r = {"experts": 4, "top": 2, "scale": 1.5, "groups": {"count": 2, "keep": 1}}
    choice, weight = P.route(z, router, torch.zeros(4, dtype=torch.float64), r)
    assert choice.tolist() == [[0, 1]] and torch.allclose(weight[0], 1.5 * s[:2])
    corr = torch.tensor([0.0, 0.0, 0.9, 0.9], dtype=torch.float64)
    choice, weight = P.route(z, router, corr, r)
    assert choice.tolist() == [[2, 3]] and torch.allclose(weight[0], 1.5 * s[2:])
    # a group's score is the sum of its two best, not its best one: 0.95 + 0.1 loses against 0.6 + 0.6
    z = torch.logit(torch.tensor([[0.95, 0.1, 0.05, 0.6, 0.6, 0.05]], dtype=torch.float64))
    choice, _ = P.route(z, torch.eye(6, dtype=torch.float64), torch.zeros(6, dtype=torch.float64),
                        {"experts": 6, "top": 2, "groups": {"count": 2, "keep": 1}})
    assert choice.tolist() == [[3, 4]]
    # negative choice scores: experts of a dropped group stay out although their scores are larger than the kept ones'
    corr = torch.tensor([-3.0, -3.0, -4.0, -4.0], dtype=torch.float64)
    z = torch.logit(torch.tensor([[0.2, 0.3, 0.9, 0.9]], dtype=torch.float64))
    choice, weight = P.route(z, torch.eye(4, dtype=torch.float64), corr, {"experts": 4, "top": 2, "groups": {"count": 2, "keep": 1}})
    assert choice.tolist() == [[1, 0]] and torch.allclose(weight[0], torch.tensor([0.3, 0.2], dtype=torch.float64))
    # groups of one expert: its own score
    choice, _ = P.route(z, torch.eye(4, dtype=torch.float64), torch.zeros(4, dtype=torch.float64), {"experts": 4, "top": 1, "groups": {"count": 4, "keep": 2}})
    assert choice.tolist() == [[2]]
