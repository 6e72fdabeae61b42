"""Typed configuration of the Zugutar decoder, read from the keys of its own config.json, and its
description in terms of parts.

The design: embedding rows as they are; layers with one RMS norm (the stored weight is the gain's distance
from one) whose output both sublayers read, ``x += mixer(N(x)) + ff(N(x))``; a range of layers may run several
times in a row with the same weights, each pass with a cache or state of its own, the embedding rows being
added to the stream in front of every pass but the first; a final norm; the embedding matrix again as the
output matrix, logits times a constant.  Two mixers.  ``attention``: softmax attention without positions,
queries multiplied by ``1 + coef ln(floor((p + 1) / every) + 1)``, a gate per output value.  ``parallel``: half
the sum of two mixers' outputs, each through an RMS norm over the stream's width: on the left softmax attention
with an RMS norm per head on q and k, rotation of a head's first values (halves pairing), a sink of score 0 and
a gate per head; on the right Mamba-2.  The feed-forward is a mixture of gated units with silu: sigmoid
scores, the largest chosen, an expert's score multiplying what it reads, beside a shared unit times the sigmoid
of one number per token.

config.json keys: ``architecture`` ("Zugutar"), ``vocab``, ``width``, ``norm.eps``, ``logit_scale``, ``layers``
(a list of ``{type, mixer, mlp}``) and, optionally, ``loop`` (``{start, stop, times}``).  Tensor names in the
weight file: ``embed``, ``l<i>.norm1``, ``l<i>.mix.<name>``, ``l<i>.mix.left.<name>``, ``l<i>.mix.right.<name>``,
``l<i>.mlp.<name>``, the convolution's bias ``.conv.b``, ``final.norm``.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Tuple

from ..errors import InvalidArgumentError, UnsupportedError
from .gusolix import _softmax_heads
from .nobupel import DEFAULT_MAX_POSITIONS, _integer, _need, _number, nobupel_stored_name, nobupel_tensor_alias
from .registry import register_architecture
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry


@dataclass(frozen=True)
class ZugutarLayer:
    kind: str                       # "attention" or "parallel"
    mixer: Dict[str, Any]           # the mixer's sizes and constants, checked
    mlp: Optional[Dict[str, Any]]   # the feed-forward's, None for a layer without one


@dataclass(frozen=True)
class ZugutarConfig:
    vocab: int
    width: int
    eps: float
    logit_scale: float
    layers: Tuple[ZugutarLayer, ...]
    loop: Optional[Tuple[int, int, int]]   # (start, stop, times)
    max_positions: int = DEFAULT_MAX_POSITIONS
    eos_token_ids: Tuple[int, ...] = ()
    architecture: str = "Zugutar"
    raw: Dict[str, Any] = field(default_factory=dict, compare=False, hash=False)

    # ---- reading -----------------------------------------------------------------
    @classmethod
    def from_dict(cls, data: Dict[str, Any]) -> "ZugutarConfig":
        _need("the configuration", data, ("vocab", "width", "layers", "norm"))
        _need("norm", data["norm"], ("eps",))
        if not isinstance(data["layers"], list) or not data["layers"]:
            raise InvalidArgumentError("layers must be a list with at least one layer")
        layers: List[ZugutarLayer] = []
        for index, entry in enumerate(data["layers"]):
            where = f"layers[{index}]"
            _need(where, entry, ("type", "mixer"))
            if entry["type"] == "attention":
                mixer = cls._attention(f"{where}.mixer", entry["mixer"])
            elif entry["type"] == "parallel":
                mixer = cls._parallel(f"{where}.mixer", entry["mixer"])
            else:
                raise UnsupportedError(f"{where}: unknown mixer type {entry['type']!r}; known: attention, parallel")
            mlp = None if entry.get("mlp") is None else cls._mlp(f"{where}.mlp", entry["mlp"])
            layers.append(ZugutarLayer(entry["type"], mixer, mlp))
        loop = None
        if data.get("loop") is not None:
            _need("loop", data["loop"], ("start", "stop", "times"))
            start, stop = (_integer(f"loop.{key}", data["loop"][key], 0) for key in ("start", "stop"))
            times = _integer("loop.times", data["loop"]["times"])
            if not start <= stop <= len(layers):
                raise InvalidArgumentError(f"loop {start}..{stop} does not lie within the {len(layers)} layers")
            loop = (start, stop, times)
        eos = data.get("eos_token_id")
        eos_ids = () if eos is None else ((int(eos),) if isinstance(eos, int) else tuple(int(x) for x in eos))
        return cls(vocab=_integer("vocab", data["vocab"]), width=_integer("width", data["width"]),
                   eps=_number("norm.eps", data["norm"]["eps"]),
                   logit_scale=_number("logit_scale", data.get("logit_scale", 1.0), positive=False), layers=tuple(layers), loop=loop,
                   max_positions=_integer("max_positions", data.get("max_positions", DEFAULT_MAX_POSITIONS)),
                   eos_token_ids=eos_ids, raw=dict(data))

    @staticmethod
    def _attention(where: str, mixer: Dict[str, Any]) -> Dict[str, Any]:
        out = _softmax_heads(where, mixer)
        out["q_temp"] = None
        temp = mixer.get("q_temp")
        if temp is not None:
            _need(f"{where}.q_temp", temp, ("coef", "every"))
            out["q_temp"] = {"coef": _number(f"{where}.q_temp.coef", temp["coef"], positive=False),
                             "every": _number(f"{where}.q_temp.every", temp["every"])}
        return out

    @staticmethod
    def _parallel(where: str, mixer: Dict[str, Any]) -> Dict[str, Any]:
        _need(where, mixer, ("left", "right"))
        left = _softmax_heads(f"{where}.left", mixer["left"])
        left["rot"] = None
        rot = mixer["left"].get("rot")
        if rot is not None:
            _need(f"{where}.left.rot", rot, ("dims", "base"))
            dims = _integer(f"{where}.left.rot.dims", rot["dims"], 0)
            if dims % 2 or dims > left["dim"]:
                raise InvalidArgumentError(f"{where}.left: rot.dims {dims} must be even and at most dim {left['dim']}")
            if dims:
                left["rot"] = {"dims": dims, "base": _number(f"{where}.left.rot.base", rot["base"])}
        keys = ("heads", "vdim", "state", "groups", "conv", "norm_groups")
        _need(f"{where}.right", mixer["right"], keys)
        right = {key: _integer(f"{where}.right.{key}", mixer["right"][key]) for key in keys}
        if right["heads"] % right["groups"]:
            raise InvalidArgumentError(f"{where}.right: heads {right['heads']} is not a multiple of groups {right['groups']}")
        if right["heads"] * right["vdim"] % right["norm_groups"]:
            raise InvalidArgumentError(f"{where}.right: norm_groups {right['norm_groups']} does not divide the "
                                       f"{right['heads']} heads of {right['vdim']}")
        return {"left": left, "right": right}

    @staticmethod
    def _mlp(where: str, mlp: Dict[str, Any]) -> Dict[str, Any]:
        _need(where, mlp, ("kind", "expert", "router"))
        if mlp["kind"] != "moe":
            raise UnsupportedError(f"{where}: unknown kind {mlp['kind']!r}; known: moe")
        _need(f"{where}.expert", mlp["expert"], ("ff",))
        _need(f"{where}.router", mlp["router"], ("experts", "top"))
        experts, top = (_integer(f"{where}.router.{key}", mlp["router"][key]) for key in ("experts", "top"))
        if top > experts:
            raise InvalidArgumentError(f"{where}.router: {top} of {experts} experts cannot be chosen")
        shared = None
        if mlp.get("shared") is not None:
            _need(f"{where}.shared", mlp["shared"], ("ff",))
            shared = _integer(f"{where}.shared.ff", mlp["shared"]["ff"])
        return {"ff": _integer(f"{where}.expert.ff", mlp["expert"]["ff"]), "experts": experts, "top": top, "shared": shared}

    def to_dict(self) -> Dict[str, Any]:
        """The config.json that reads back as this configuration."""
        layers = []
        for layer in self.layers:
            if layer.kind == "attention":
                mixer = {k: v for k, v in layer.mixer.items() if v is not None}
            else:
                mixer = {"left": {k: v for k, v in layer.mixer["left"].items() if v is not None}, "right": dict(layer.mixer["right"])}
            mlp = None
            if layer.mlp is not None:
                mlp = {"kind": "moe", "expert": {"ff": layer.mlp["ff"]},
                       "router": {"experts": layer.mlp["experts"], "top": layer.mlp["top"]}}
                if layer.mlp["shared"] is not None:
                    mlp["shared"] = {"ff": layer.mlp["shared"]}
            layers.append({"type": layer.kind, "mixer": mixer, "mlp": mlp})
        out: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                               "norm": {"eps": self.eps}, "logit_scale": self.logit_scale, "layers": layers,
                               "loop": None if self.loop is None else
                               {"start": self.loop[0], "stop": self.loop[1], "times": self.loop[2]}}
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            out["max_positions"] = self.max_positions
        if self.eos_token_ids:
            out["eos_token_id"] = list(self.eos_token_ids)
        return out

    # ---- derived -----------------------------------------------------------------
    def layer_runs(self) -> List[Tuple[int, bool]]:
        """(layer, whether the embedding rows are added first) in the order the layers run."""
        count = len(self.layers)
        if self.loop is None:
            return [(index, False) for index in range(count)]
        start, stop, times = self.loop
        runs = [(index, False) for index in range(start)]
        for turn in range(times):
            runs += [(index, turn > 0 and index == start) for index in range(start, stop)]
        return runs + [(index, False) for index in range(stop, count)]


_NAMES = ("q", "k", "v", "o")


def _attention_part(config: ZugutarConfig, m: Dict[str, Any]) -> PartSpec:
    return PartSpec("gqa_attention", {
        "hidden_size": config.width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"],
        "value_dim": m["vdim"], "qkv_bias": False, "window": None, "output_gate": True, "tile_heads": True,
        "query_temperature": m["q_temp"], "max_positions": config.max_positions, "softmax_scale": m["scale"],
        "position": PartSpec("none", {}), "projection_names": _NAMES})


def _parallel_part(config: ZugutarConfig, m: Dict[str, Any]) -> PartSpec:
    left, right = m["left"], m["right"]
    position = PartSpec("none", {})
    if left["rot"] is not None:
        position = PartSpec("rope_neox", {"head_dim": left["dim"], "rotary_dims": left["rot"]["dims"], "theta": left["rot"]["base"],
                                          "scaling": None, "exact_angles": True, "max_positions": config.max_positions})
    softmax = PartSpec("gqa_attention", {
        "hidden_size": config.width, "num_heads": left["heads"], "num_kv_heads": left["kv_heads"], "head_dim": left["dim"],
        "value_dim": left["vdim"], "qkv_bias": False, "window": None, "head_norm": True, "norm_eps": config.eps, "sink": True,
        "output_gate": "heads", "tile_heads": True, "softmax_scale": left["scale"], "position": position, "projection_names": _NAMES})
    recurrence = PartSpec("mamba2", {
        "hidden_size": config.width, "num_heads": right["heads"], "value_dim": right["vdim"], "state": right["state"],
        "groups": right["groups"], "taps": right["conv"], "norm_groups": right["norm_groups"], "norm_eps": config.eps})
    return PartSpec("parallel", {"branches": (("left", softmax, 0.5), ("right", recurrence, 0.5)),
                                 "hidden_size": config.width, "out_norm_eps": config.eps})


def zugutar_model_spec(config: ZugutarConfig) -> ModelSpec:
    """Zugutar in parts.  Every run of a layer is a schedule entry with a cache slot of its own."""
    norm = PartSpec("rmsnorm", {"size": config.width, "eps": config.eps, "weight_offset": 1.0})
    layers: List[LayerSpec] = []
    for index, layer in enumerate(config.layers):
        build = _attention_part if layer.kind == "attention" else _parallel_part
        parts = {"mixer_norm": norm, "mixer": build(config, layer.mixer)}
        f = layer.mlp
        if f is not None:
            params = {"hidden_size": config.width, "intermediate_size": f["ff"], "experts": f["experts"], "top": f["top"],
                      "score": "sigmoid", "activation": "silu", "weight_on": "input", "projection_names": ("gate", "up", "down")}
            if f["shared"] is not None:
                params.update(shared_size=f["shared"], shared_gate=True, shared_gate_name="sg")
            parts["ffn"] = PartSpec("moe_mlp", params)
        layers.append(LayerSpec(block="parallel", prefix=f"l{index}", parts=parts,
                                names={"mixer_norm": "norm1", "mixer": "mix", "ffn": "mlp"},
                                params={"hidden_size": config.width, "shared_norm": True}))
    spec = ModelSpec(
        architecture=config.architecture,
        vocab_size=config.vocab,
        hidden_size=config.width,
        max_position_embeddings=config.max_positions,
        embedding_name="embed.weight",
        layers=layers,
        schedule=[ScheduleEntry(layer=layer, cache=run, adds_embedding=again)
                  for run, (layer, again) in enumerate(config.layer_runs())],
        final_norm=norm,
        final_norm_name="final.norm",
        head_name=None,
        logit_scale=config.logit_scale,
    )
    spec.validate()
    return spec


register_architecture("Zugutar", ZugutarConfig.from_dict, zugutar_model_spec,
                      tensor_alias=nobupel_tensor_alias, stored_name=nobupel_stored_name)
