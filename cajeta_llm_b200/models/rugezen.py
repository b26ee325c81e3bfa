"""Rugezen: configuration, layer plan and tensor names.

A decoder whose ``config.json`` lists its layers one by one (``layers``: ``type``, ``mixer`` sizes, ``mlp`` or null).
What it is put together from:

* a layer is a ``parallel`` block with two norms: ``x += residual_mult (mixer(norm1(x)) + ff(norm2(x)))``, both of the same
  ``x``; RMS norms with a plain weight;
* ``type`` ``attention``: grouped-query attention (part ``attention``) whose queries and keys are rotated over their first
  ``rot.dims`` entries in neighbouring pairs and divided by their root mean square per head, whose values are divided
  by theirs, whose scores are capped by ``softcap * tanh(s / softcap)``, and whose softmax has one more term ``e^0`` in the
  divisor (``sink_score`` 0); no window, no biases;
* ``type`` ``mingru``: a gated recurrence channel by channel (part ``mingru``) whose gates read the current token alone;
* ``mlp.kind`` ``dense``: ``W_down relu(W_up h + b)^2 + b`` (part ``dense_relu2`` with biases);
* ``loop``: layers ``start .. stop-1`` run ``times`` times with the same weights, each pass with a cache or state of its own
  (the plan's schedule names those layers once per pass); nothing happens between the passes.

Tensor names: ``embed``, ``l<i>.norm1|norm2``, ``l<i>.mix.q|k|v|o`` (``attention``), ``l<i>.mix.z|z.b|x|x.b|g|o``
(``mingru``), ``l<i>.mlp.up|up.b|down|down.b``, ``final.norm``, ``head``.  Every size and every constant that can differ
between models comes from ``config.json``.
"""
from __future__ import annotations

import json
from dataclasses import dataclass
from typing import Any, Dict, Tuple

from ..config.base import ConfigError, ConfigReader, ModelConfig, register_architecture
from ..parts.plan import LayerSpec, ModelPlan, PartSpec, ScheduleEntry

ARCHITECTURE = "Rugezen"
MIXER_TYPES = ("attention", "mingru")
SINK_SCORE = 0.0          # the softmax's divisor is one larger than the sum over the keys: a key of score 0 without a value


@dataclass(frozen=True)
class RugezenConfig(ModelConfig):
    width: int
    vocab: int
    norm_eps: float
    residual_mult: float
    layers_json: str              # ``layers`` as canonical JSON (a frozen dataclass holds no dicts)
    loop_json: str                # ``loop`` as canonical JSON, "null" for none
    eos_token_ids: Tuple[int, ...] = ()

    @property
    def layers(self):
        return json.loads(self.layers_json)

    @property
    def loop(self):
        return json.loads(self.loop_json)

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @classmethod
    def from_reader(cls, r: ConfigReader) -> "RugezenConfig":
        raw = r.raw
        arch = raw["architectures"][0] if "architectures" in raw else raw["architecture"]
        norm = raw.get("norm")
        if not isinstance(norm, dict) or "eps" not in norm:
            raise ConfigError(f"{r.source}: required key 'norm.eps' is missing")
        eps = _number(r.source, "norm.eps", norm["eps"])
        mult = _number(r.source, "residual_mult", raw.get("residual_mult", 1.0), positive=False)
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError(f"{r.source}: required key 'layers' is missing or is not a list of layers")
        for i, layer in enumerate(layers):
            _check_layer(r.source, i, layer)
        loop = raw.get("loop")
        if loop is not None:
            _need_ints(r.source, "loop", loop, ("times",))
            _need_ints(r.source, "loop", loop, ("start", "stop"), minimum=0)
            if not loop["start"] < loop["stop"] <= len(layers):
                raise ConfigError(f"{r.source}: loop must name layers start < stop <= {len(layers)}, found {loop['start']} .. {loop['stop']}")
        return cls(architecture=arch, width=r.integer("width", minimum=1), vocab=r.integer("vocab", minimum=1), norm_eps=eps,
                   residual_mult=mult, layers_json=json.dumps(layers, sort_keys=True), loop_json=json.dumps(loop, sort_keys=True),
                   eos_token_ids=tuple(r.integer_list("eos_token_id", ())))

    def to_json_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"architecture": self.architecture, "width": self.width, "vocab": self.vocab,
                             "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult, "layers": self.layers}
        if self.loop is not None:
            d["loop"] = self.loop
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d


def _need_ints(source: str, where: str, d: Any, keys, minimum: int = 1) -> None:
    if not isinstance(d, dict):
        raise ConfigError(f"{source}: {where} must be an object")
    for k in keys:
        v = d.get(k)
        if isinstance(v, bool) or not isinstance(v, int) or v < minimum:
            raise ConfigError(f"{source}: {where}.{k} must be an integer >= {minimum}, found {v!r}")


def _number(source: str, where: str, v: Any, positive: bool = True) -> float:
    if isinstance(v, bool) or not isinstance(v, (int, float)) or (positive and v <= 0):
        raise ConfigError(f"{source}: {where} must be a{' positive' if positive else ''} number, found {v!r}")
    return float(v)


def _check_layer(source: str, i: int, layer: Any) -> None:
    where = f"layers[{i}]"
    if not isinstance(layer, dict) or layer.get("type") not in MIXER_TYPES:
        raise ConfigError(f"{source}: {where}.type must be one of {', '.join(MIXER_TYPES)}, "
                          f"found {layer.get('type') if isinstance(layer, dict) else layer!r}")
    m = layer.get("mixer")
    if layer["type"] == "attention":
        _need_ints(source, f"{where}.mixer", m, ("heads", "kv_heads", "dim", "vdim"))
        if m["heads"] % m["kv_heads"] != 0:
            raise ConfigError(f"{source}: {where}.mixer: heads {m['heads']} is not a multiple of kv_heads {m['kv_heads']}")
        _number(source, f"{where}.mixer.scale", m.get("scale"))
        if m.get("softcap") is not None:
            _number(source, f"{where}.mixer.softcap", m["softcap"])
        rot = m.get("rot")
        if rot is not None:
            _need_ints(source, f"{where}.mixer.rot", rot, ("dims",))
            _number(source, f"{where}.mixer.rot.base", rot.get("base"))
            if rot["dims"] % 2 != 0 or rot["dims"] > m["dim"]:
                raise ConfigError(f"{source}: {where}.mixer.rot.dims must be even and at most dim")
    else:
        _need_ints(source, f"{where}.mixer", m, ("width",))
    ff = layer.get("mlp")
    if ff is None:
        return
    if not isinstance(ff, dict) or ff.get("kind") != "dense":
        raise ConfigError(f"{source}: {where}.mlp.kind must be 'dense' (or mlp null for no feed-forward)")
    _need_ints(source, f"{where}.mlp", ff, ("ff",))


def _mixer_spec(h: int, eps: float, kind: str, m: Dict[str, Any]) -> PartSpec:
    if kind == "mingru":
        return PartSpec("mingru", {"hidden_size": h, "width": m["width"]})
    rot = m.get("rot")
    position = PartSpec("none")
    if rot is not None:
        position = PartSpec("rope", {"head_dim": m["dim"], "rotary_dim": rot["dims"], "theta": float(rot["base"]), "pairs": True,
                                     "float64_table": True})
    return PartSpec("attention", {
        "hidden_size": h, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"], "value_dim": m["vdim"],
        "scale": float(m["scale"]), "softcap": float(m.get("softcap") or 0.0), "exact_cap": True, "qk_norm": {"eps": eps},
        "value_norm": {"eps": eps}, "sink_score": SINK_SCORE, "position": position, "names": {"q": "q", "k": "k", "v": "v", "o": "o"}})


def _feed_forward_spec(h: int, ff: Any):
    if ff is None:
        return None
    return PartSpec("dense_relu2", {"hidden_size": h, "intermediate_size": ff["ff"], "bias": True, "names": {"up": "up", "down": "down"}})


def build_plan(cfg: RugezenConfig) -> ModelPlan:
    h, eps, loop = cfg.width, cfg.norm_eps, cfg.loop
    norm = PartSpec("rmsnorm", {"dim": h, "eps": eps, "weight_name": ""})
    block = PartSpec("parallel", {"mixer_norm_name": "norm1", "feed_forward_norm_name": "norm2", "mixer_name": "mix",
                                  "feed_forward_name": "mlp", "residual_mult": cfg.residual_mult})
    layers = []
    for i, layer in enumerate(cfg.layers):
        ffn = _feed_forward_spec(h, layer.get("mlp"))
        layers.append(LayerSpec(prefix=f"l{i}", block=block, mixer=_mixer_spec(h, eps, layer["type"], layer["mixer"]),
                                feed_forward=ffn, mixer_norm=norm, feed_forward_norm=norm if ffn is not None else None))
    # the run order: a looped stretch of layers appears once per pass, each appearance with a cache plane or state of its own
    order = list(range(len(layers)))
    if loop is not None:
        order = order[:loop["start"]] + order[loop["start"]:loop["stop"]] * loop["times"] + order[loop["stop"]:]
    plan = ModelPlan(architecture=cfg.architecture, hidden_size=h, vocab_size=cfg.vocab, embedding_name="embed",
                     layers=tuple(layers), schedule=tuple(ScheduleEntry(layer=i) for i in order), final_norm=norm,
                     final_norm_prefix="final.norm", lm_head_name="head", eog_token_ids=cfg.eos_token_ids, max_position=None)
    plan.validate()
    return plan


register_architecture(ARCHITECTURE, RugezenConfig, build_plan, replace=True)
