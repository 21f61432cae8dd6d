"""Typed configuration of the Vepolix decoder, read from its config.json.

Vepolix is a small decoder-only design: scaled embeddings with a sinusoid of the position added, layers of ONE RMS norm
whose rows both sublayers read, x += mixer(N(x)) + ff(N(x)), a final norm and a classifier of its own.  A layer's mixer is
``attention`` (no rotation; q and k normed over the whole projection; a learned bias by distance in logarithmic buckets; a
token sees its own chunk of positions; the values of every layer that mixes them are blended with the first such layer's)
or ``mlstm`` (a matrix memory with exponential gates).  The feed-forward is dense with a gelu gate, or a mixture of
silu-gated experts chosen by sigmoid scores plus a correction inside the best groups, plus a shared expert.  config.json::

    {"architecture": "Vepolix", "vocab": V, "width": W, "norm": {"eps": e}, "embedding": {"scale": s},
     "layers": [{"type": "attention",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "bias_max", "v_mix": true or false,
                           "mask": {"size"} (null: every earlier key)},
                 "mlp": {"kind": "dense", "ff": F} or null},
                {"type": "mlstm", "mixer": {"heads", "dim", "vdim", "gate_cap"},
                 "mlp": {"kind": "moe", "router": {"experts", "top", "scale", "groups": {"count", "keep"} (optional)},
                         "expert": {"ff"}, "shared": {"ff"} (optional)}}]}

Tensor names: ``embed``, ``head``, ``final.norm`` and under ``l<i>.``: ``norm1``, ``mix.*``, ``mlp.gate|up|down`` or ``mlp.router``,
``mlp.correction``, ``mlp.e<k>.gate|up|down``, ``mlp.shared.gate|up|down``.  The number of rows of a layer's bias table is not in
config.json; ``with_tensor_shapes`` reads it from the tensor ``l<i>.mix.rel``.  ExiledOfCode/KuiperLLama has no such model; its
model classes are picked in ``main`` (demo/main.cpp:58).
"""
from __future__ import annotations

import json
from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from .registry import ConfigError, register_architecture
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

MIXER_TYPES = ("attention", "mlstm")
# Constants the design fixes (parameters of the parts, so another design may choose others).
POSITION_BASE = 10000.0          # the sinusoid's frequencies are base^(-2i / width)
DENSE_ACTIVATION = "gelu_tanh"   # dense: W_down (gelu(W_gate h) * (W_up h)); experts have silu there
GROUP_TOP = 2                    # a group of experts is scored by the sum of its two best
DENOMINATOR_EPS = 1e-6           # the matrix memory's output is divided by max(|n . q|, exp(-m)) + 1e-6
DEFAULT_BIAS_ROWS = 32           # the bias table's rows where neither config.json nor the tensors say (random weights)
DEFAULT_MAX_POSITIONS = 1 << 17  # the design names no longest sequence; "max_positions" may raise it


def _is_int(v: Any) -> bool:
    return isinstance(v, int) and not isinstance(v, bool)


def _is_num(v: Any) -> bool:
    return isinstance(v, (int, float)) and not isinstance(v, bool)


@register_architecture("Vepolix")
@dataclass(frozen=True)
class VepolixConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    layers: Tuple[dict, ...]              # as in config.json, checked
    max_positions: int = DEFAULT_MAX_POSITIONS

    architecture = "Vepolix"

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "VepolixConfig":
        problems: List[str] = []

        def positive_int(where: str, obj: Any, key: str) -> int:
            v = obj.get(key) if isinstance(obj, dict) else None
            if not _is_int(v) or v <= 0:
                problems.append(f'{where}"{key}" must be a positive integer, got {v!r}')
                return 1
            return v

        def number(where: str, obj: Any, key: str, positive: bool = False) -> float:
            v = obj.get(key) if isinstance(obj, dict) else None
            if not _is_num(v) or (positive and v <= 0):
                problems.append(f'{where}"{key}" must be a {"positive " if positive else ""}number, got {v!r}')
                return 1.0
            return float(v)

        vocab = positive_int("", d, "vocab")
        width = positive_int("", d, "width")
        eps = number('"norm": ', d.get("norm"), "eps", positive=True)
        scale = number('"embedding": ', d.get("embedding"), "scale")
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            problems.append('"layers" must be a list with at least one layer')
            layers = []
        mixed = []                        # value sizes of the layers that share values
        for i, layer in enumerate(layers):
            at = f"layers[{i}]: "
            if not isinstance(layer, dict) or layer.get("type") not in MIXER_TYPES:
                problems.append(f'{at}"type" must be one of {list(MIXER_TYPES)}, got {layer.get("type") if isinstance(layer, dict) else layer!r}')
                continue
            m = layer.get("mixer")
            if not isinstance(m, dict):
                problems.append(f'{at}"mixer" must be an object')
                continue
            if layer["type"] == "attention":
                H, G = positive_int(at, m, "heads"), positive_int(at, m, "kv_heads")
                positive_int(at, m, "dim")
                vdim = positive_int(at, m, "vdim")
                number(at, m, "scale")
                number(at, m, "bias_max", positive=True)
                if m.get("mask") is not None:
                    positive_int(at + '"mask": ', m.get("mask"), "size")
                if m.get("rel_rows") is not None:
                    positive_int(at, m, "rel_rows")
                if H % G:
                    problems.append(f'{at}"heads" {H} is not a multiple of "kv_heads" {G}')
                if not isinstance(m.get("v_mix", False), bool):
                    problems.append(f'{at}"v_mix" must be true or false, got {m.get("v_mix")!r}')
                elif m.get("v_mix"):
                    mixed.append((i, G * vdim))
            else:
                for k in ("heads", "dim", "vdim"):
                    positive_int(at, m, k)
                number(at, m, "gate_cap", positive=True)
            mlp = layer.get("mlp")
            if mlp is None:
                continue
            if not isinstance(mlp, dict) or mlp.get("kind") not in ("dense", "moe"):
                problems.append(f'{at}"mlp" must be null or have "kind": "dense" or "moe", got {mlp!r}')
            elif mlp["kind"] == "dense":
                positive_int(at + '"mlp": ', mlp, "ff")
            else:
                r = mlp.get("router")
                E = positive_int(at + '"mlp": "router": ', r, "experts")
                top = positive_int(at + '"mlp": "router": ', r, "top")
                if isinstance(r, dict) and r.get("scale") is not None:
                    number(at + '"mlp": "router": ', r, "scale")
                positive_int(at + '"mlp": "expert": ', mlp.get("expert"), "ff")
                if mlp.get("shared") is not None:
                    positive_int(at + '"mlp": "shared": ', mlp.get("shared"), "ff")
                count = keep = 1
                grp = r.get("groups") if isinstance(r, dict) else None
                if grp is not None:
                    count = positive_int(at + '"mlp": "router": "groups": ', grp, "count")
                    keep = positive_int(at + '"mlp": "router": "groups": ', grp, "keep")
                if E % count or keep > count:
                    problems.append(f'{at}"mlp": {E} experts do not form {count} equal groups of which {keep} are kept')
                elif top > keep * (E // count):
                    problems.append(f'{at}"mlp": "top" {top} exceeds the {keep * (E // count)} experts of the kept groups')
        if len({size for _, size in mixed}) > 1:
            problems.append("the layers that mix values must have equally many of them: " + ", ".join(f"layers[{i}] has {s}" for i, s in mixed))
        max_positions = d.get("max_positions", DEFAULT_MAX_POSITIONS)
        if not _is_int(max_positions) or max_positions <= 0:
            problems.append(f'"max_positions" must be a positive integer, got {max_positions!r}')
        if problems:
            raise ConfigError("config.json (Vepolix): " + "; ".join(problems))
        return cls(vocab=vocab, width=width, norm_eps=eps, embedding_scale=scale, layers=tuple(json.loads(json.dumps(l)) for l in layers),
                   max_positions=max_positions)

    # ------------------------------------------------------------------ writing
    def to_dict(self) -> dict:
        d = {"architecture": self.architecture, "embedding": {"scale": self.embedding_scale},
             "layers": json.loads(json.dumps(list(self.layers))), "norm": {"eps": self.norm_eps}, "vocab": self.vocab, "width": self.width}
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            d["max_positions"] = self.max_positions
        return d

    # ------------------------------------------------------------------ sizes that only the tensors give
    def with_tensor_shapes(self, shapes: Dict[str, Tuple[int, ...]]) -> "VepolixConfig":
        """The same configuration with every size that config.json leaves to the tensors filled in from ``shapes`` (tensor
        name -> shape): the rows of a layer's bias table, ``rel_rows``, from ``l<i>.mix.rel``."""
        layers = json.loads(json.dumps(list(self.layers)))
        for i, layer in enumerate(layers):
            if layer["type"] == "attention" and layer["mixer"].get("rel_rows") is None:
                shape = shapes.get(f"l{i}.mix.rel")
                if shape is not None and len(shape) == 2 and shape[0] > 0:
                    layer["mixer"]["rel_rows"] = int(shape[0])
        return VepolixConfig(self.vocab, self.width, self.norm_eps, self.embedding_scale, tuple(layers), self.max_positions)

    # ------------------------------------------------------------------ the model it describes
    def _norm(self, name: str) -> PartSpec:
        return PartSpec("rmsnorm", {"size": self.width, "eps": self.norm_eps, "name": name})

    def _mixer(self, kind: str, m: dict, value_mix: Optional[str]) -> PartSpec:
        if kind == "mlstm":
            return PartSpec("mlstm", {
                "hidden_size": self.width, "heads": m["heads"], "dim": m["dim"], "vdim": m["vdim"], "cap": float(m["gate_cap"]),
                "q_scale": float(m["dim"]) ** -0.5, "den_eps": DENOMINATOR_EPS, "norm_eps": self.norm_eps,
                "names": {"q": "mix.q", "k": "mix.k", "v": "mix.v", "g": "mix.g", "o": "mix.o", "norm": "mix.norm", "i": "mix.i",
                          "i_bias": "mix.i.b", "f": "mix.f", "f_bias": "mix.f.b"}})
        names = {"q": "mix.q", "k": "mix.k", "v": "mix.v", "o": "mix.o", "q_norm": "mix.q.norm", "k_norm": "mix.k.norm",
                 "distance_bias": "mix.rel"}
        if value_mix == "mix":
            names["value_mix"] = "mix.vmix"
        return PartSpec("window_attention", {
            "hidden_size": self.width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"], "value_dim": m["vdim"],
            "scale": float(m["scale"]), "row_norm": {"eps": self.norm_eps}, "chunk": None if m.get("mask") is None else m["mask"]["size"],
            "distance_bias": {"rows": m.get("rel_rows") or DEFAULT_BIAS_ROWS, "largest": float(m["bias_max"])},
            "value_mix": value_mix, "names": names})

    def _feed_forward(self, mlp: Optional[dict]) -> Optional[PartSpec]:
        if mlp is None:
            return None
        if mlp["kind"] == "dense":
            return PartSpec("swiglu", {"hidden_size": self.width, "intermediate_size": mlp["ff"], "activation": DENSE_ACTIVATION,
                                       "names": {"gate": "mlp.gate", "up": "mlp.up", "down": "mlp.down"}})
        r, shared = mlp["router"], mlp.get("shared")
        grp = r.get("groups") or {"count": 1, "keep": 1}
        names = {"router": "mlp.router", "correction": "mlp.correction", "gate": "mlp.e{e}.gate", "up": "mlp.e{e}.up", "down": "mlp.e{e}.down"}
        if shared is not None:
            names.update({"shared_gate": "mlp.shared.gate", "shared_up": "mlp.shared.up", "shared_down": "mlp.shared.down"})
        return PartSpec("moe", {
            "hidden_size": self.width, "experts": r["experts"], "top": r["top"], "expert_size": mlp["expert"]["ff"],
            "limit": None, "alpha": 1.0, "shift": 0.0, "renormalise": False, "scores": "sigmoid",
            "router_scale": 1.0 if r.get("scale") is None else float(r["scale"]), "groups": grp["count"], "keep_groups": grp["keep"],
            "group_top": GROUP_TOP, "shared_size": None if shared is None else shared["ff"], "names": names})

    def to_model_spec(self) -> ModelSpec:
        layers, schedule = [], []
        first_mixed = next((i for i, l in enumerate(self.layers) if l["type"] == "attention" and l["mixer"].get("v_mix")), None)
        unread = []                       # the first layer that mixes values has a factor nobody reads
        for i, layer in enumerate(self.layers):
            mix = None
            if layer["type"] == "attention" and layer["mixer"].get("v_mix"):
                mix = "keep" if i == first_mixed else "mix"
            if layer["type"] == "attention" and mix != "mix":
                unread.append(f"l{i}.mix.vmix")
            # the sinusoid belongs to the model's first layer: the embedding kernel adds it
            position = PartSpec("sinusoidal", {"hidden_size": self.width, "base": POSITION_BASE}) if i == 0 else None
            layers.append(LayerSpec(
                prefix=f"l{i}.", arrangement="parallel", mixer=self._mixer(layer["type"], layer["mixer"], mix),
                feed_forward=self._feed_forward(layer.get("mlp")), mixer_norm=self._norm("norm1"), feed_forward_norm=None, position=position))
            schedule.append(ScheduleEntry(layer=i))
        spec = ModelSpec(
            architecture=self.architecture, hidden_size=self.width, vocab_size=self.vocab, max_positions=self.max_positions,
            layers=tuple(layers), schedule=tuple(schedule), embedding_name="embed", final_norm=self._norm("norm"),
            final_norm_prefix="final.", lm_head_name="head", ignorable_suffixes=tuple(unread), embedding_multiplier=self.embedding_scale)
        spec.validate()
        return spec
