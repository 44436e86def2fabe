"""Typed configuration of the Deginex decoder, read from its own config.json keys.

A Deginex model is a list of pre-norm layers on a residual of several streams (hyper-connections):
a sublayer reads a weighted sum of the streams through a layer norm with gain and bias, and its output
changes every stream through a small matrix.  A stretch of the layers may run several times in a row
with the same weights, each pass with its own cache; the output head is the embedding table:

    {"architecture": "Deginex", "vocab": V, "width": W, "norm": {"eps": e}, "streams": s,
     "loop": {"start": i, "stop": j, "times": n} | null,
     "layers": [{"type": "attention", "mixer": {...}, "mlp": {...} | null}, ...]}

    attention  heads, kv_heads, dim, vdim, scale, softcap, mask {size}
               (grouped-query attention without positions and biases; q and k divided by their root
               mean square per head; capped scores; keys visible inside the query's chunk of
               `mask.size` positions only; a sigmoid gate per column on the concatenated heads)
    mlp        kind "dense", ff;  or kind "moe", expert {ff}, router {experts, top}
               (a router with a bias, weights by a softmax over the chosen experts)

Nothing here is fixed to one model: every size, the order of the layers and every constant come
from the file; the tensor names ('embed', 'final.norm', 'final.norm.b', 'l<i>.norm1', 'l<i>.norm1.b',
'l<i>.hc1.in', 'l<i>.hc1.out', 'l<i>.hc1.mix', 'l<i>.mix.q', 'l<i>.mix.g', 'l<i>.mlp.gate',
'l<i>.mlp.e<j>.up', 'l<i>.mlp.router', 'l<i>.mlp.router.b', ...) are the design's.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, List, Mapping, Optional

from .metulix import _integer
from .qwen2 import ConfigError
from .spec import LayerCall, LayerSpec, ModelSpec, PartSpec
from .zadepel import _number

MIXERS = ("attention",)


def _check_attention(where: str, mixer: Mapping[str, Any]) -> None:
    heads = _integer(where, mixer, "heads")
    kv_heads = _integer(where, mixer, "kv_heads") if "kv_heads" in mixer else heads
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where}.heads must be a multiple of kv_heads")
    _integer(where, mixer, "dim")
    if "vdim" in mixer:
        _integer(where, mixer, "vdim")
    _number(where, mixer, "scale")
    if mixer.get("softcap") is not None and _number(where, mixer, "softcap") < 0:   # absent, null or 0: no cap
        raise ConfigError(f"config.json: {where}.softcap must not be negative")
    mask = mixer.get("mask")
    if mask is not None:            # absent or null: every earlier position is seen
        if not isinstance(mask, Mapping):
            raise ConfigError(f"config.json: {where}.mask must be an object with 'size', or null")
        _integer(where + ".mask", mask, "size")


def _check_mlp(where: str, mlp: Any) -> None:
    if not isinstance(mlp, Mapping) or mlp.get("kind") not in ("dense", "moe"):
        raise ConfigError(f"config.json: {where}.kind must be 'dense' or 'moe'")
    if mlp["kind"] == "dense":
        _integer(where, mlp, "ff")
        return
    expert, router = mlp.get("expert"), mlp.get("router")
    if not isinstance(expert, Mapping) or not isinstance(router, Mapping):
        raise ConfigError(f"config.json: {where} needs 'expert' and 'router' objects")
    _integer(where + ".expert", expert, "ff")
    if _integer(where + ".router", router, "top") > _integer(where + ".router", router, "experts"):
        raise ConfigError(f"config.json: {where}.router.top exceeds the number of experts")


@dataclass(frozen=True)
class DeginexConfig:
    vocab: int
    width: int
    eps: float
    streams: int
    layers: tuple                      # the layer entries as read (dicts), checked
    loop: Optional[tuple] = None       # (start, stop, times)
    eos_token_id: Optional[int] = None

    architecture = "Deginex"

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, data: Mapping[str, Any]) -> "DeginexConfig":
        vocab = _integer("the model", data, "vocab")
        width = _integer("the model", data, "width")
        streams = _integer("the model", data, "streams")
        norm = data.get("norm")
        if not isinstance(norm, Mapping) or "eps" not in norm:
            raise ConfigError("config.json: 'norm' must be an object with 'eps'")
        layers = data.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        loop = data.get("loop")
        if loop is not None:
            if not isinstance(loop, Mapping):
                raise ConfigError("config.json: 'loop' must be an object or null")
            loop = (_integer("loop", loop, "start", least=0), _integer("loop", loop, "stop", least=0),
                    _integer("loop", loop, "times"))
        eos = data.get("eos_token_id")
        if isinstance(eos, list):
            eos = eos[0] if eos else None
        config = cls(vocab, width, _number("norm", norm, "eps"), streams, tuple(copy.deepcopy(list(layers))),
                     loop, None if eos is None else int(eos))
        config.validate()
        return config

    def to_dict(self) -> Dict[str, Any]:
        data: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab,
                                "width": self.width, "norm": {"eps": self.eps}, "streams": self.streams,
                                "loop": None if self.loop is None else
                                {"start": self.loop[0], "stop": self.loop[1], "times": self.loop[2]},
                                "layers": copy.deepcopy(list(self.layers))}
        if self.eos_token_id is not None:
            data["eos_token_id"] = self.eos_token_id
        return data

    # --------------------------------------------------------------- validation
    def validate(self) -> None:
        if self.eps < 0:
            raise ConfigError("config.json: norm.eps must not be negative")
        if self.loop is not None:
            start, stop, _ = self.loop
            if not start < stop <= len(self.layers):
                raise ConfigError(f"config.json: loop must name layers start < stop <= {len(self.layers)}, "
                                  f"got start {start}, stop {stop}")
        for index, layer in enumerate(self.layers):
            where = f"layers[{index}]"
            if not isinstance(layer, Mapping) or not isinstance(layer.get("mixer"), Mapping):
                raise ConfigError(f"config.json: {where} must be an object with a 'mixer'")
            if layer.get("type") not in MIXERS:
                raise ConfigError(f"config.json: {where}.type '{layer.get('type')}' is not a mixer of this design "
                                  f"({', '.join(MIXERS)})")
            _check_attention(where + ".mixer", layer["mixer"])
            if layer.get("mlp") is not None:
                _check_mlp(where + ".mlp", layer["mlp"])

    # --------------------------------------------------------------------- spec
    def _attention(self, mixer: Mapping[str, Any]) -> PartSpec:
        return PartSpec("scaled_gqa_attention", {
            "hidden_size": self.width, "heads": int(mixer["heads"]),
            "kv_heads": int(mixer.get("kv_heads", mixer["heads"])),
            "dim": int(mixer["dim"]), "vdim": int(mixer.get("vdim", mixer["dim"])), "scale": float(mixer["scale"]),
            "position": PartSpec("none", {}), "temperature": False, "value_mix": "none", "bias": False,
            "chunk": int(mixer["mask"]["size"]) if mixer.get("mask") else 0,
            "softcap": float(mixer.get("softcap") or 0.0),
            "qk_norm": True, "qk_gain": False, "eps": self.eps, "column_gate": True})

    def _feed_forward(self, mlp: Optional[Mapping[str, Any]]) -> Optional[PartSpec]:
        if mlp is None:
            return None
        if mlp["kind"] == "dense":
            return PartSpec("gated_mlp", {
                "hidden_size": self.width, "intermediate_size": int(mlp["ff"]), "activation": "silu",
                "names": {"gate": "gate", "up": "up", "down": "down", "weight": "", "bias": ".b"}})
        router = mlp["router"]
        return PartSpec("routed_experts", {
            "hidden_size": self.width, "intermediate_size": int(mlp["expert"]["ff"]),
            "experts": int(router["experts"]), "top": int(router["top"]), "scores": "chosen_softmax",
            "correction": False, "router_bias": True, "activation": "silu", "shared": None})

    def build_spec(self) -> ModelSpec:
        """Lay the configuration out as parts: every layer is a `streams` arrangement of layer norms
        with gain and bias, its mixer `scaled_gqa_attention` (no positions, unit q and k, capped
        scores, chunks, a gate per column), its feed-forward a `gated_mlp`, `routed_experts`, or
        none.  The looped stretch appears in the run order once per pass, every call with a cache
        entry of its own."""
        norm = PartSpec("layernorm", {"width": self.width, "eps": self.eps, "weight_name": "",
                                      "bias_name": ".b"})
        layers: List[LayerSpec] = [
            LayerSpec(prefix=f"l{index}.", arrangement="streams", mixer=self._attention(layer["mixer"]),
                      feed_forward=self._feed_forward(layer.get("mlp")), mixer_norm=norm, feed_forward_norm=norm,
                      mixer_name="mix.", feed_forward_name="mlp.", mixer_norm_name="norm1",
                      feed_forward_norm_name="norm2")
            for index, layer in enumerate(self.layers)]
        order = list(range(len(layers)))
        if self.loop is not None:
            start, stop, times = self.loop
            order = order[:start] + order[start:stop] * times + order[stop:]
        return ModelSpec(
            architecture=self.architecture, hidden_size=self.width, vocab_size=self.vocab,
            max_position=0, embedding_name="embed", head_name=None, final_norm=norm,
            final_norm_prefix="final.norm", layers=tuple(layers),
            schedule=tuple(LayerCall(layer=i) for i in order), streams=self.streams)
