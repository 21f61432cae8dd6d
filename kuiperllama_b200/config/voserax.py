"""Typed configuration of the Voserax decoder, read from its config.json.

Voserax is a small decoder-only design: embeddings plus a learned vector per position, layers between several residual streams
(hyper-connections: each sublayer reads a weighted sum of the streams and is written into all of them while they mix), a norm of
the streams' sum and the embedding table as the classifier.  A layer is an attention with short convolutions behind q, k
and v, YaRN rotation of part of each head, a window, a one in the softmax's denominator and values blended with the first such
layer's; and a feed-forward: dense with a relu gate, or clamped experts chosen by softmax scores plus a correction, of which the
last few are the identity, plus a shared expert times one sigmoid per token.  config.json::

    {"architecture": "Voserax", "vocab": V, "width": W, "streams": S, "residual_mult": m, "norm": {"eps": e}, "max_positions": P,
     "layers": [{"type": "attention",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "conv": taps, "v_mix": true or false,
                           "mask": {"size"} (null: every earlier key),
                           "rot": {"base", "dims", "scaling": {"factor", "original", "fast", "slow"} (optional)} (null: none)},
                 "mlp": {"kind": "dense", "ff": F} or null},
                {"type": "attention", "mixer": {...},
                 "mlp": {"kind": "moe", "router": {"experts", "top", "identity" (optional)}, "expert": {"ff", "limit"},
                         "shared": {"ff", "limit"} (optional)}}]}

Tensor names: ``embed``, ``pos``, ``final.norm`` and under ``l<i>.``: ``norm1``, ``norm2``, ``hc1.in|out|mix``, ``hc2.in|out|mix``,
``mix.q|k|v|o``, ``mix.q.conv`` and so on, ``mix.vmix``, ``mlp.gate|up|down`` or ``mlp.router``, ``mlp.correction``,
``mlp.e<k>.gate|up|down``, ``mlp.shared.gate|up|down|sg``.  ``max_positions`` may be left out where the tensors are at hand:
``with_tensor_shapes`` reads it from ``pos``.  ExiledOfCode/KuiperLLama has no such model; its model classes are picked in
``main`` (demo/main.cpp:58).
"""
from __future__ import annotations

import dataclasses
import json
from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from .registry import ConfigError, register_architecture
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

# Constants the design fixes (parameters of the parts, so another design may choose others).
SINK_SCORE = 0.0                 # exp(0) = 1 joins every softmax's denominator
MAGNITUDE_SLOPE = 0.1            # YaRN: cos and sin times 0.1 ln(factor) + 1
DENSE_ACTIVATION = "relu"        # dense: W_down (relu(W_gate h) * (W_up h))
GATE_SLOPE = 1.702               # experts: g sigmoid(1.702 g) (u + 1)
UP_SHIFT = 1.0
DEFAULT_MAX_POSITIONS = 4096     # where neither config.json nor the tensors say (random weights)


def _is_int(v: Any) -> bool:
    return isinstance(v, int) and not isinstance(v, bool)


def _is_num(v: Any) -> bool:
    return isinstance(v, (int, float)) and not isinstance(v, bool)


@register_architecture("Voserax")
@dataclass(frozen=True)
class VoseraxConfig:
    vocab: int
    width: int
    streams: int
    residual_mult: float
    norm_eps: float
    layers: Tuple[dict, ...]              # as in config.json, checked
    max_positions: Optional[int] = None

    architecture = "Voserax"

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "VoseraxConfig":
        problems: List[str] = []

        def integer(where: str, obj: Any, key: str, least: int = 1) -> int:
            v = obj.get(key) if isinstance(obj, dict) else None
            if not _is_int(v) or v < least:
                problems.append(f'{where}"{key}" must be {"a positive integer" if least == 1 else f"an integer of at least {least}"}, got {v!r}')
                return max(least, 1)
            return v

        def number(where: str, obj: Any, key: str, positive: bool = False) -> float:
            v = obj.get(key) if isinstance(obj, dict) else None
            if not _is_num(v) or (positive and v <= 0):
                problems.append(f'{where}"{key}" must be a {"positive " if positive else ""}number, got {v!r}')
                return 1.0
            return float(v)

        vocab, width, streams = (integer("", d, k) for k in ("vocab", "width", "streams"))
        mult = number("", d, "residual_mult")
        eps = number('"norm": ', d.get("norm"), "eps", positive=True)
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            problems.append('"layers" must be a list with at least one layer')
            layers = []
        mixed = []                        # value sizes of the layers that share values
        for i, layer in enumerate(layers):
            at = f"layers[{i}]: "
            if not isinstance(layer, dict) or layer.get("type") != "attention":
                problems.append(f'{at}"type" must be "attention", got {layer.get("type") if isinstance(layer, dict) else layer!r}')
                continue
            m = layer.get("mixer")
            if not isinstance(m, dict):
                problems.append(f'{at}"mixer" must be an object')
                continue
            H, G = integer(at, m, "heads"), integer(at, m, "kv_heads")
            dim, vdim = integer(at, m, "dim"), integer(at, m, "vdim")
            integer(at, m, "conv")
            number(at, m, "scale")
            if H % G:
                problems.append(f'{at}"heads" {H} is not a multiple of "kv_heads" {G}')
            if m.get("mask") is not None:
                integer(at + '"mask": ', m.get("mask"), "size")
            rot = m.get("rot")
            if rot is not None:
                dims = integer(at + '"rot": ', rot, "dims")
                base = number(at + '"rot": ', rot, "base", positive=True)
                if dims % 2 or dims > dim:
                    problems.append(f'{at}"rot": "dims" {dims} must be even and at most "dim" {dim}')
                if base == 1.0 and isinstance(rot, dict) and rot.get("base") == 1:
                    problems.append(f'{at}"rot": "base" must not be 1')
                if isinstance(rot, dict) and rot.get("scaling") is not None:
                    for k in ("factor", "original", "fast", "slow"):
                        number(at + '"rot": "scaling": ', rot["scaling"], k, positive=True)
            if not isinstance(m.get("v_mix", False), bool):
                problems.append(f'{at}"v_mix" must be true or false, got {m.get("v_mix")!r}')
            elif m.get("v_mix"):
                mixed.append((i, G * vdim))
            mlp = layer.get("mlp")
            if mlp is None:
                continue
            if not isinstance(mlp, dict) or mlp.get("kind") not in ("dense", "moe"):
                problems.append(f'{at}"mlp" must be null or have "kind": "dense" or "moe", got {mlp!r}')
            elif mlp["kind"] == "dense":
                integer(at + '"mlp": ', mlp, "ff")
            else:
                r = mlp.get("router")
                E, top = integer(at + '"mlp": "router": ', r, "experts"), integer(at + '"mlp": "router": ', r, "top")
                extra = 0
                if isinstance(r, dict) and r.get("identity") is not None:
                    extra = integer(at + '"mlp": "router": ', r, "identity", least=0)
                if top > E + extra:
                    problems.append(f'{at}"mlp": "top" {top} exceeds the {E + extra} experts')
                for part in ("expert", "shared"):
                    if part == "expert" or mlp.get("shared") is not None:
                        integer(f'{at}"mlp": "{part}": ', mlp.get(part), "ff")
                        number(f'{at}"mlp": "{part}": ', mlp.get(part), "limit", positive=True)
        if len({size for _, size in mixed}) > 1:
            problems.append("the layers that mix values must have equally many of them: " + ", ".join(f"layers[{i}] has {s}" for i, s in mixed))
        max_positions = d.get("max_positions")
        if max_positions is not None and (not _is_int(max_positions) or max_positions <= 0):
            problems.append(f'"max_positions" must be a positive integer, got {max_positions!r}')
        if problems:
            raise ConfigError("config.json (Voserax): " + "; ".join(problems))
        return cls(vocab=vocab, width=width, streams=streams, residual_mult=mult, norm_eps=eps,
                   layers=tuple(json.loads(json.dumps(l)) for l in layers), max_positions=max_positions)

    # ------------------------------------------------------------------ writing
    def to_dict(self) -> dict:
        d = {"architecture": self.architecture, "layers": json.loads(json.dumps(list(self.layers))), "norm": {"eps": self.norm_eps},
             "residual_mult": self.residual_mult, "streams": self.streams, "vocab": self.vocab, "width": self.width}
        if self.max_positions is not None:
            d["max_positions"] = self.max_positions
        return d

    # ------------------------------------------------------------------ sizes that only the tensors give
    def with_tensor_shapes(self, shapes: Dict[str, Tuple[int, ...]]) -> "VoseraxConfig":
        """The same configuration with ``max_positions`` from the tensor ``pos`` where config.json leaves it out."""
        shape = shapes.get("pos")
        if self.max_positions is not None or shape is None or len(shape) != 2 or shape[0] < 1:
            return self
        return dataclasses.replace(self, max_positions=int(shape[0]))

    # ------------------------------------------------------------------ the model it describes
    def _norm(self, name: str) -> PartSpec:
        return PartSpec("rmsnorm", {"size": self.width, "eps": self.norm_eps, "name": name})

    def _links(self, q: int) -> PartSpec:
        return PartSpec("hyper_connection", {"streams": self.streams, "multiplier": self.residual_mult,
                                             "names": {"in": f"hc{q}.in", "out": f"hc{q}.out", "mix": f"hc{q}.mix"}})

    def _mixer(self, m: dict, value_mix: Optional[str]) -> PartSpec:
        names = {k: f"mix.{k}" for k in ("q", "k", "v", "o")}
        names.update({f"{k}_conv": f"mix.{k}.conv" for k in ("q", "k", "v")})
        if value_mix == "mix":
            names["value_mix"] = "mix.vmix"
        return PartSpec("window_attention", {
            "hidden_size": self.width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"], "value_dim": m["vdim"],
            "scale": float(m["scale"]), "window": None if m.get("mask") is None else m["mask"]["size"], "conv": m["conv"],
            "sink_score": SINK_SCORE, "value_mix": value_mix, "names": names})

    def _position(self, m: dict) -> Optional[PartSpec]:
        rot = m.get("rot")
        if rot is None:
            return None
        scaling = None if rot.get("scaling") is None else dict(rot["scaling"], rope_type="yarn", magnitude_slope=MAGNITUDE_SLOPE)
        return PartSpec("rope", {"head_dim": m["dim"], "rotary_dim": rot["dims"], "theta": float(rot["base"]), "scaling": scaling})

    def _feed_forward(self, mlp: Optional[dict]) -> Optional[PartSpec]:
        if mlp is None:
            return None
        if mlp["kind"] == "dense":
            return PartSpec("swiglu", {"hidden_size": self.width, "intermediate_size": mlp["ff"], "activation": DENSE_ACTIVATION,
                                       "names": {"gate": "mlp.gate", "up": "mlp.up", "down": "mlp.down"}})
        r, shared = mlp["router"], mlp.get("shared")
        names = {"router": "mlp.router", "correction": "mlp.correction", "gate": "mlp.e{e}.gate", "up": "mlp.e{e}.up", "down": "mlp.e{e}.down"}
        params = {"hidden_size": self.width, "experts": r["experts"], "top": r["top"], "identity": r.get("identity") or 0,
                  "expert_size": mlp["expert"]["ff"], "limit": float(mlp["expert"]["limit"]), "alpha": GATE_SLOPE, "shift": UP_SHIFT,
                  "renormalise": False, "scores": "softmax", "shared_size": None, "names": names}
        if shared is not None:
            names.update({"shared_gate": "mlp.shared.gate", "shared_up": "mlp.shared.up", "shared_down": "mlp.shared.down",
                          "shared_scale": "mlp.shared.sg"})
            params.update(shared_size=shared["ff"], shared_limit=float(shared["limit"]))
        return PartSpec("moe", params)

    def to_model_spec(self) -> ModelSpec:
        layers, schedule = [], []
        first_mixed = next((i for i, l in enumerate(self.layers) if l["mixer"].get("v_mix")), None)
        unread = []                       # the first layer that mixes values has a factor nobody reads
        positions = self.max_positions or DEFAULT_MAX_POSITIONS
        for i, layer in enumerate(self.layers):
            m, mlp = layer["mixer"], layer.get("mlp")
            mix = None
            if m.get("v_mix"):
                mix = "keep" if i == first_mixed else "mix"
            if mix != "mix":
                unread.append(f"l{i}.mix.vmix")
            if mlp is None:
                unread += [f"l{i}.norm2"] + [f"l{i}.hc2.{k}" for k in ("in", "out", "mix")]
            layers.append(LayerSpec(
                prefix=f"l{i}.", arrangement="streams", mixer=self._mixer(m, mix), feed_forward=self._feed_forward(mlp),
                mixer_norm=self._norm("norm1"), feed_forward_norm=None if mlp is None else self._norm("norm2"), position=self._position(m),
                mixer_streams=self._links(1), feed_forward_streams=None if mlp is None else self._links(2)))
            schedule.append(ScheduleEntry(layer=i))
        spec = ModelSpec(
            architecture=self.architecture, hidden_size=self.width, vocab_size=self.vocab, max_positions=positions,
            layers=tuple(layers), schedule=tuple(schedule), embedding_name="embed", final_norm=self._norm("norm"),
            final_norm_prefix="final.", lm_head_name=None, ignorable_suffixes=tuple(unread),
            embedding_position=PartSpec("learned", {"hidden_size": self.width, "positions": positions, "name": "pos"}))
        spec.validate()
        return spec
