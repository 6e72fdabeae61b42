"""Typed configuration of the Nuvezen decoder, read from the keys of its own config.json, and its
description in terms of parts.

The design: embedding rows as they are; layers whose mixer and feed-forward both read the same stream,
each through an RMS norm of its own (the stored weight is the gain's distance from one), and join it
together, each scaled per channel, ``x += s1 mixer(N1(x)) + s2 ff(N2(x))``; a final norm; the embedding
matrix again as the output matrix.  A layer may run another layer's tensors with a cache of its own.
One mixer, ``latent_attention``: queries through a normed latent, keys and values as products of a cached
normed latent with one rotated key part (interleaved pairs) shared by the heads, a sliding window, a
softmax whose denominator also holds ``exp(sink_h)``.  Two feed-forwards.  ``dense``: a gated unit with
silu.  ``moe``: gated units with bounds on both halves, chosen by the router's logits and weighted by
the softmax over the chosen logits, beside a shared unit (bounds of its own) times the sigmoid of one
number per token.

config.json keys: ``architecture`` ("Nuvezen"), ``vocab``, ``width``, ``norm.eps`` and ``layers`` (a list
of ``{type, mixer, mlp}`` with, optionally, ``weights_of``).  Tensor names in the weight file: ``embed``,
``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.ls1``, ``l<i>.ls2``, ``l<i>.mix.<name>``, ``l<i>.mlp.<name>``,
``l<i>.mlp.e<k>.gate|up|down``, ``l<i>.mlp.shared.gate|up|down|sg``, ``final.norm``.
"""
from __future__ import annotations

import re
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Tuple

from ..errors import InvalidArgumentError, UnsupportedError
from .fasolorn import _mask, _rot
from .nobupel import DEFAULT_MAX_POSITIONS, _integer, _need, _number, nobupel_stored_name, nobupel_tensor_alias
from .registry import register_architecture
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry


@dataclass(frozen=True)
class NuvezenLayer:
    mixer: Dict[str, Any]           # the mixer's sizes and constants, checked
    mlp: Optional[Dict[str, Any]]   # the feed-forward's, None for a layer without one
    source: int                     # the layer whose tensors it runs (itself where it has its own)


@dataclass(frozen=True)
class NuvezenConfig:
    vocab: int
    width: int
    eps: float
    layers: Tuple[NuvezenLayer, ...]
    max_positions: int = DEFAULT_MAX_POSITIONS
    eos_token_ids: Tuple[int, ...] = ()
    architecture: str = "Nuvezen"
    raw: Dict[str, Any] = field(default_factory=dict, compare=False, hash=False)

    @classmethod
    def from_dict(cls, data: Dict[str, Any]) -> "NuvezenConfig":
        _need("the configuration", data, ("vocab", "width", "layers", "norm"))
        _need("norm", data["norm"], ("eps",))
        if not isinstance(data["layers"], list) or not data["layers"]:
            raise InvalidArgumentError("layers must be a list with at least one layer")
        layers: List[NuvezenLayer] = []
        for index, entry in enumerate(data["layers"]):
            where = f"layers[{index}]"
            _need(where, entry, ("type", "mixer"))
            if entry["type"] != "latent_attention":
                raise UnsupportedError(f"{where}: unknown mixer type {entry['type']!r}; known: latent_attention")
            mixer = cls._latent(f"{where}.mixer", entry["mixer"])
            mlp = None if entry.get("mlp") is None else cls._mlp(f"{where}.mlp", entry["mlp"])
            source = cls._source(where, entry, data["layers"], index)
            layers.append(NuvezenLayer(mixer, mlp, source))
        for index, layer in enumerate(layers):
            own = layers[layer.source]
            if layer.mixer != own.mixer or layer.mlp != own.mlp:
                raise InvalidArgumentError(f"layers[{index}] runs the tensors of layers[{layer.source}] and must have its sizes")
        eos = data.get("eos_token_id")
        eos_ids = () if eos is None else ((int(eos),) if isinstance(eos, int) else tuple(int(x) for x in eos))
        return cls(vocab=_integer("vocab", data["vocab"]), width=_integer("width", data["width"]),
                   eps=_number("norm.eps", data["norm"]["eps"]), layers=tuple(layers),
                   max_positions=_integer("max_positions", data.get("max_positions", DEFAULT_MAX_POSITIONS)),
                   eos_token_ids=eos_ids, raw=dict(data))

    @staticmethod
    def _source(where: str, entry: Dict[str, Any], entries: List[Dict[str, Any]], index: int) -> int:
        """The layer that owns the tensors layer `index` runs: ``weights_of``, followed to its end."""
        seen = {index}
        while entry.get("weights_of") is not None:
            index = _integer(f"{where}.weights_of", entry["weights_of"], 0)
            if index >= len(entries) or index in seen or not isinstance(entries[index], dict):
                raise InvalidArgumentError(f"{where}.weights_of does not lead to a layer with tensors of its own")
            seen.add(index)
            entry = entries[index]
        return index

    @staticmethod
    def _latent(where: str, mixer: Dict[str, Any]) -> Dict[str, Any]:
        _need(where, mixer, ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank", "scale", "rot"))
        out = {key: _integer(f"{where}.{key}", mixer[key])
               for key in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank")}
        out["scale"] = _number(f"{where}.scale", mixer["scale"])
        out["mask"] = _mask(where, mixer)
        out["rot"] = _rot(where, mixer, out["rot_dim"])
        if out["rot"] is None or out["rot"]["dims"] != out["rot_dim"]:
            raise InvalidArgumentError(f"{where}: rot.dims must equal rot_dim {out['rot_dim']}")
        return out

    @staticmethod
    def _mlp(where: str, mlp: Dict[str, Any]) -> Dict[str, Any]:
        _need(where, mlp, ("kind",))
        if mlp["kind"] == "dense":
            _need(where, mlp, ("ff",))
            return {"kind": "dense", "ff": _integer(f"{where}.ff", mlp["ff"])}
        if mlp["kind"] != "moe":
            raise UnsupportedError(f"{where}: unknown kind {mlp['kind']!r}; known: dense, moe")
        _need(where, mlp, ("expert", "router"))

        def unit(name):
            _need(f"{where}.{name}", mlp[name], ("ff", "limit"))
            return {"ff": _integer(f"{where}.{name}.ff", mlp[name]["ff"]),
                    "limit": _number(f"{where}.{name}.limit", mlp[name]["limit"])}

        router = mlp["router"]
        _need(f"{where}.router", router, ("experts", "top"))
        experts, top = (_integer(f"{where}.router.{key}", router[key]) for key in ("experts", "top"))
        if top > experts:
            raise InvalidArgumentError(f"{where}.router: {top} of {experts} experts cannot be chosen")
        return {"kind": "moe", "expert": unit("expert"), "experts": experts, "top": top,
                "shared": None if mlp.get("shared") is None else unit("shared")}

    def to_dict(self) -> Dict[str, Any]:
        """The config.json that reads back as this configuration."""
        layers = []
        for index, layer in enumerate(self.layers):
            mixer = {k: v for k, v in layer.mixer.items() if k not in ("mask", "rot")}
            if layer.mixer["mask"] is not None:
                mixer["mask"] = {"size": layer.mixer["mask"]}
            mixer["rot"] = dict(layer.mixer["rot"])
            mlp = layer.mlp
            if mlp is not None and mlp["kind"] == "moe":
                mlp = {"kind": "moe", "expert": dict(mlp["expert"]), "router": {"experts": mlp["experts"], "top": mlp["top"]}}
                if layer.mlp["shared"] is not None:
                    mlp["shared"] = dict(layer.mlp["shared"])
            entry = {"type": "latent_attention", "mixer": mixer, "mlp": mlp}
            if layer.source != index:
                entry["weights_of"] = layer.source
            layers.append(entry)
        out: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                               "norm": {"eps": self.eps}, "layers": layers}
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            out["max_positions"] = self.max_positions
        if self.eos_token_ids:
            out["eos_token_id"] = list(self.eos_token_ids)
        return out


# What the design fixes: the slope inside the sigmoid of the mixture's units.
UNIT_SLOPE = 1.702


def nuvezen_model_spec(config: NuvezenConfig) -> ModelSpec:
    """Nuvezen in parts.  A layer with tensors of its own becomes a layer of the description; every
    layer of config.json is an entry of the schedule, with a cache slot of its own."""
    norm = PartSpec("rmsnorm", {"size": config.width, "eps": config.eps, "weight_offset": 1.0})
    layers: List[LayerSpec] = []
    place: Dict[int, int] = {}      # index in config.json -> index among the described layers
    for index, layer in enumerate(config.layers):
        if layer.source != index:
            continue
        m = layer.mixer
        position = PartSpec("rope_interleaved", {
            "head_dim": m["rot_dim"], "rotary_dims": m["rot"]["dims"], "theta": m["rot"]["base"], "scaling": None,
            "exact_angles": True, "max_positions": config.max_positions})
        parts = {"mixer_norm": norm, "mixer": PartSpec("latent_attention", {
            "hidden_size": config.width, "num_heads": m["heads"], "head_dim": m["dim"], "rot_dim": m["rot_dim"],
            "value_dim": m["vdim"], "kv_rank": m["kv_rank"], "q_rank": m["q_rank"], "softmax_scale": m["scale"],
            "norm_eps": config.eps, "own_cache": True, "output_gate": False, "window": m["mask"], "sink": "learned",
            "position": position})}
        f = layer.mlp
        if f is not None:
            parts["ffn_norm"] = norm
            if f["kind"] == "dense":
                parts["ffn"] = PartSpec("gated_mlp", {"hidden_size": config.width, "intermediate_size": f["ff"],
                                                      "activation": "silu", "bias": False,
                                                      "projection_names": ("gate", "up", "down")})
            else:
                shared = f["shared"]
                params = {"hidden_size": config.width, "intermediate_size": f["expert"]["ff"], "experts": f["experts"],
                          "top": f["top"], "score": "logit", "activation": "clamped", "limit": f["expert"]["limit"],
                          "slope": UNIT_SLOPE, "projection_names": ("gate", "up", "down")}
                if shared is not None:
                    params.update(shared_size=shared["ff"], shared_limit=shared["limit"], shared_gate=True,
                                  shared_gate_name="sg")
                parts["ffn"] = PartSpec("moe_mlp", params)
        place[index] = len(layers)
        layers.append(LayerSpec(block="parallel", prefix=f"l{index}", parts=parts,
                                names={"mixer_norm": "norm1", "mixer": "mix", "mixer_scale": "ls1",
                                       "ffn_norm": "norm2", "ffn": "mlp", "ffn_scale": "ls2"},
                                params={"hidden_size": config.width, "layer_scale": True}))
    spec = ModelSpec(
        architecture=config.architecture,
        vocab_size=config.vocab,
        hidden_size=config.width,
        max_position_embeddings=config.max_positions,
        embedding_name="embed.weight",
        layers=layers,
        schedule=[ScheduleEntry(layer=place[layer.source], cache=index) for index, layer in enumerate(config.layers)],
        final_norm=norm,
        final_norm_name="final.norm",
        head_name=None,
    )
    spec.validate()
    return spec


_SECOND_BRANCH = re.compile(r"^l(\d+)\.(norm2|ls2)\.weight$")


def nuvezen_ignorable(config: NuvezenConfig, name: str) -> bool:
    """A file may hold the second branch's norm and scale for a layer without a feed-forward; nothing
    reads them."""
    match = _SECOND_BRANCH.match(name)
    if not match or int(match.group(1)) >= len(config.layers):
        return False
    layer = config.layers[int(match.group(1))]
    return layer.mlp is None and layer.source == int(match.group(1))


register_architecture("Nuvezen", NuvezenConfig.from_dict, nuvezen_model_spec,
                      tensor_alias=nobupel_tensor_alias, stored_name=nobupel_stored_name, ignorable=nuvezen_ignorable)
