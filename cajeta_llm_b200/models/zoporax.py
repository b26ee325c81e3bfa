"""Zoporax: configuration, layer plan and tensor names.

A decoder whose ``config.json`` lists its layers one by one (``layers``: ``type``, ``mixer`` sizes, ``mlp`` or null).
What it is put together from:

* a layer is a ``prenorm`` block with RMS norms (plain weight); a layer may have no feed-forward;
* ``type`` ``latent_attention``: attention over a compressed latent (part ``latent_attention``) whose queries pass a latent of
  their own (``q_rank``), with a rotation of the shared key part that pairs entry i with i + dims/2 and whose slow frequencies
  are stretched (``rot.scaling``, the YaRN form; cos and sin times its magnitude), a sliding window of ``mask.size`` and a
  sigmoid gate on every entry of the heads;
* ``type`` ``lightning``: linear attention with one constant decay per head (part ``lightning``), the heads normed together and
  gated;
* ``mlp.kind`` ``dense``: a gated feed-forward with gelu's tanh form and biases (part ``dense_gated``); ``moe``: experts without a
  gate and with gelu by the error function (part ``sparse_moe``) behind a router of sigmoid scores that picks the ``top`` largest
  among the ``groups.keep`` best of ``groups.count`` groups (a group's score: the sum of its two largest), weights = the picks'
  scores over their sum, times ``router.scale``; plus a shared expert of the same form behind a sigmoid gate;
* the head is the embedding table.

Tensor names: ``embed``, ``l<i>.norm1|norm2``, ``l<i>.mix.*`` (``latent_attention``: ``dq dq.norm uq dkv dkv.norm uk uv g o``;
``lightning``: ``q k v g norm o``), ``l<i>.mlp.gate|up|down`` each with ``.b``, or ``l<i>.mlp.router``, ``l<i>.mlp.e<k>.up|down``,
``l<i>.mlp.shared.up|down|sg``, ``final.norm``.  Every size and every constant that can differ between models comes from
``config.json``.
"""
from __future__ import annotations

import json
from dataclasses import dataclass
from typing import Any, Dict, Tuple

from ..config.base import ConfigError, ConfigReader, ModelConfig, register_architecture
from ..parts.plan import LayerSpec, ModelPlan, PartSpec, ScheduleEntry

ARCHITECTURE = "Zoporax"
MIXER_TYPES = ("latent_attention", "lightning")
NORM_FLOOR = 1e-20            # added to the sum of the picks' scores that their weights are divided by


@dataclass(frozen=True)
class ZoporaxConfig(ModelConfig):
    width: int
    vocab: int
    norm_eps: float
    layers_json: str              # ``layers`` as canonical JSON (a frozen dataclass holds no dicts)
    eos_token_ids: Tuple[int, ...] = ()

    @property
    def layers(self):
        return json.loads(self.layers_json)

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @classmethod
    def from_reader(cls, r: ConfigReader) -> "ZoporaxConfig":
        raw = r.raw
        arch = raw["architectures"][0] if "architectures" in raw else raw["architecture"]
        norm = raw.get("norm")
        if not isinstance(norm, dict) or "eps" not in norm:
            raise ConfigError(f"{r.source}: required key 'norm.eps' is missing")
        eps = _number(r.source, "norm.eps", norm["eps"])
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError(f"{r.source}: required key 'layers' is missing or is not a list of layers")
        for i, layer in enumerate(layers):
            _check_layer(r.source, i, layer)
        return cls(architecture=arch, width=r.integer("width", minimum=1), vocab=r.integer("vocab", minimum=1), norm_eps=eps,
                   layers_json=json.dumps(layers, sort_keys=True), eos_token_ids=tuple(r.integer_list("eos_token_id", ())))

    def to_json_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"architecture": self.architecture, "width": self.width, "vocab": self.vocab,
                             "norm": {"eps": self.norm_eps}, "layers": self.layers}
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


def _check_latent(source: str, where: str, m: Any) -> None:
    _need_ints(source, where, m, ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank"))
    _number(source, f"{where}.scale", m.get("scale"), positive=False)
    if m.get("mask") is not None:
        _need_ints(source, f"{where}.mask", m["mask"], ("size",))
    rot = m.get("rot")
    _need_ints(source, f"{where}.rot", rot, ("dims",))
    if rot["dims"] % 2 != 0 or rot["dims"] > m["rot_dim"] or _number(source, f"{where}.rot.base", rot.get("base")) <= 1.0:
        raise ConfigError(f"{source}: {where}.rot: dims must be even and at most rot_dim, base larger than 1")
    sc = rot.get("scaling")
    if sc is not None:
        if not isinstance(sc, dict):
            raise ConfigError(f"{source}: {where}.rot.scaling must be an object")
        for k in ("factor", "original", "fast", "slow"):
            _number(source, f"{where}.rot.scaling.{k}", sc.get(k))


def _check_lightning(source: str, where: str, m: Any) -> None:
    _need_ints(source, where, m, ("heads", "dim", "vdim"))
    decay = m.get("decay")
    if not isinstance(decay, list) or len(decay) != m["heads"]:
        raise ConfigError(f"{source}: {where}.decay must list a number for each of the {m['heads']} heads")
    for d in decay:
        if not 0.0 <= _number(source, f"{where}.decay", d, positive=False) <= 1.0:
            raise ConfigError(f"{source}: {where}.decay must be within [0, 1], found {d!r}")


def _check_layer(source: str, i: int, layer: Any) -> None:
    where = f"layers[{i}]"
    if not isinstance(layer, dict) or layer.get("type") not in MIXER_TYPES:
        raise ConfigError(f"{source}: {where}.type must be one of {', '.join(MIXER_TYPES)}, "
                          f"found {layer.get('type') if isinstance(layer, dict) else layer!r}")
    (_check_latent if layer["type"] == "latent_attention" else _check_lightning)(source, f"{where}.mixer", layer.get("mixer"))
    ff = layer.get("mlp")
    if ff is None:
        return
    if not isinstance(ff, dict) or ff.get("kind") not in ("dense", "moe"):
        raise ConfigError(f"{source}: {where}.mlp.kind must be 'dense' or 'moe' (or mlp null for no feed-forward)")
    if ff["kind"] == "dense":
        _need_ints(source, f"{where}.mlp", ff, ("ff",))
        return
    _need_ints(source, f"{where}.mlp.expert", ff.get("expert"), ("ff",))
    router = ff.get("router")
    _need_ints(source, f"{where}.mlp.router", router, ("experts", "top"))
    if router["top"] > router["experts"]:
        raise ConfigError(f"{source}: {where}.mlp.router.top is larger than .experts")
    if router.get("scale") is not None:
        _number(source, f"{where}.mlp.router.scale", router["scale"], positive=False)
    groups = router.get("groups")
    if groups is not None:
        _need_ints(source, f"{where}.mlp.router.groups", groups, ("count", "keep"))
        if router["experts"] % groups["count"] != 0 or groups["keep"] > groups["count"]:
            raise ConfigError(f"{source}: {where}.mlp.router.groups: experts must form 'count' equal groups and keep <= count")
        if groups["keep"] * (router["experts"] // groups["count"]) < router["top"]:
            raise ConfigError(f"{source}: {where}.mlp.router.groups: the kept groups hold fewer than 'top' experts")
    if ff.get("shared") is not None:
        _need_ints(source, f"{where}.mlp.shared", ff["shared"], ("ff",))


def _mixer_spec(h: int, eps: float, kind: str, m: Dict[str, Any]) -> PartSpec:
    if kind == "lightning":
        return PartSpec("lightning", {"hidden_size": h, "heads": m["heads"], "dim": m["dim"], "vdim": m["vdim"],
                                      "decay": tuple(float(d) for d in m["decay"]), "eps": eps})
    rot = m["rot"]
    position = PartSpec("rope", {"head_dim": m["rot_dim"], "rotary_dim": rot["dims"], "theta": float(rot["base"]), "float64_table": True,
                                 "scaling": rot.get("scaling")})
    return PartSpec("latent_attention", {
        "hidden_size": h, "heads": m["heads"], "dim": m["dim"], "rot_dim": m["rot_dim"], "vdim": m["vdim"], "kv_rank": m["kv_rank"],
        "q_rank": m["q_rank"], "scale": float(m["scale"]), "eps": eps, "position": position, "halves": True,
        "window": (m.get("mask") or {}).get("size", 0), "gate": "entries", "exact_weights": True})


def _feed_forward_spec(h: int, ff: Any):
    if ff is None:
        return None
    if ff["kind"] == "dense":
        return PartSpec("dense_gated", {"hidden_size": h, "intermediate_size": ff["ff"], "activation": "gelu_tanh", "bias": True,
                                        "names": {"gate": "gate", "up": "up", "down": "down"}})
    router, shared, groups = ff["router"], ff.get("shared"), ff["router"].get("groups")
    scale = router.get("scale")
    return PartSpec("sparse_moe", {
        "hidden_size": h, "num_experts": router["experts"], "top_k": router["top"], "expert_intermediate_size": ff["expert"]["ff"],
        "activation": "gelu", "score": "sigmoid", "weight_on": "output", "norm_topk_prob": True, "norm_floor": NORM_FLOOR,
        "route_scale": 1.0 if scale is None else float(scale),
        "route_groups": (groups["count"], groups["keep"]) if groups else None, "group_score": "top2",
        "shared_intermediate_size": shared["ff"] if shared else 0, "shared_gate": bool(shared),
        "names": {"router": "router", "up": "e{e}.up", "down": "e{e}.down", "shared_up": "shared.up", "shared_down": "shared.down",
                  "shared_sg": "shared.sg"}})


def build_plan(cfg: ZoporaxConfig) -> ModelPlan:
    h, eps = cfg.width, cfg.norm_eps
    norm = PartSpec("rmsnorm", {"dim": h, "eps": eps, "weight_name": ""})
    block = PartSpec("prenorm", {"mixer_norm_name": "norm1", "feed_forward_norm_name": "norm2", "mixer_name": "mix",
                                 "feed_forward_name": "mlp"})
    layers = []
    for i, layer in enumerate(cfg.layers):
        ffn = _feed_forward_spec(h, layer.get("mlp"))
        layers.append(LayerSpec(prefix=f"l{i}", block=block, mixer=_mixer_spec(h, eps, layer["type"], layer["mixer"]),
                                feed_forward=ffn, mixer_norm=norm, feed_forward_norm=norm if ffn is not None else None))
    plan = ModelPlan(architecture=cfg.architecture, hidden_size=h, vocab_size=cfg.vocab, embedding_name="embed",
                     layers=tuple(layers), schedule=tuple(ScheduleEntry(layer=i) for i in range(len(layers))), final_norm=norm,
                     final_norm_prefix="final.norm", lm_head_name=None, eog_token_ids=cfg.eos_token_ids, max_position=None)
    plan.validate()
    return plan


register_architecture(ARCHITECTURE, ZoporaxConfig, build_plan, replace=True)
