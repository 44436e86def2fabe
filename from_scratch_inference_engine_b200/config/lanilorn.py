"""Typed configuration of the Lanilorn decoder, read from its own config.json keys.

A Lanilorn model is a list of pre-norm layers (RMS norms) on a residual of several streams
(hyper-connections): a sublayer reads a weighted sum of the streams, its output is scaled column by
column and changes every stream through a small matrix.  The embedding rows are scaled, the output head is
the embedding table, its logits are scaled:

    {"architecture": "Lanilorn", "vocab": V, "width": W, "norm": {"eps": e}, "streams": s,
     "embedding": {"scale": c}, "logit_scale": l,
     "layers": [{"type": "attention" | "attention_2" | "gla", "mixer": {...}, "mlp": {...} | null}, ...]}

    attention    heads, kv_heads, dim, vdim (= dim), scale, mask {size}, rot {base, dims, scaling {factor, original,
                 fast, slow}}
                 (grouped-query attention whose values are its keys as projected; q and k RMS-normed over the whole
                 projection; YaRN rotation of the leading columns; a sliding window; a sink per head; a sigmoid
                 gate per head)
    attention_2  heads, kv_heads, dim, vdim, scale, diff, q_temp {coef, every}
                 (differential attention without positions: two softmax maps over the same values and their
                 normed difference; a query temperature by position; a sigmoid gate per head)
    gla          heads, dim, vdim, tau, and rank where weights are drawn at random (else the tensors say)
                 (gated linear attention: a recurrence with a decay per key column and token)
    mlp          kind "dense", ff (W_down relu(W_up h)^2)

Nothing here is fixed to one model: every size, the order of the layers and every constant come from the
file; the tensor names ('embed', 'final.norm', 'l<i>.norm1', 'l<i>.ls1', 'l<i>.hc1.in', 'l<i>.hc1.out',
'l<i>.hc1.mix', 'l<i>.mix.q', 'l<i>.mix.q.norm', 'l<i>.mix.sink', 'l<i>.mix.lq1', 'l<i>.mix.a2.b', 'l<i>.mlp.up', ...)
are the design's.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, List, Mapping, Optional

from .metulix import _integer
from .qwen2 import ConfigError
from .spec import LayerCall, LayerSpec, ModelSpec, PartSpec
from .zadepel import _number

MIXERS = ("attention", "attention_2", "gla")


def _object(where: str, data: Mapping[str, Any], key: str) -> Optional[Mapping[str, Any]]:
    """data[key] where it is an object, None where it is absent or null."""
    value = data.get(key)
    if value is not None and not isinstance(value, Mapping):
        raise ConfigError(f"config.json: {where}.{key} must be an object or null")
    return value


def _positive(where: str, data: Mapping[str, Any], key: str) -> float:
    value = _number(where, data, key)
    if value <= 0:
        raise ConfigError(f"config.json: {where}.{key} must be positive, got {value}")
    return value


def _check_heads(where: str, mixer: Mapping[str, Any]) -> None:
    heads = _integer(where, mixer, "heads")
    kv_heads = _integer(where, mixer, "kv_heads") if "kv_heads" in mixer else heads
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where}.heads must be a multiple of kv_heads")
    _integer(where, mixer, "dim")
    if "vdim" in mixer:
        _integer(where, mixer, "vdim")
    _number(where, mixer, "scale")


def _check_attention(where: str, mixer: Mapping[str, Any]) -> None:
    _check_heads(where, mixer)
    if mixer.get("vdim", mixer["dim"]) != mixer["dim"]:
        raise ConfigError(f"config.json: {where}.vdim must equal dim (the values are the keys)")
    mask = _object(where, mixer, "mask")
    if mask is not None:                # absent or null: every earlier position is seen
        _integer(where + ".mask", mask, "size")
    rot = _object(where, mixer, "rot")
    if rot is not None:                 # absent or null: no rotation
        _positive(where + ".rot", rot, "base")
        dims = _integer(where + ".rot", rot, "dims", least=0)
        if dims % 2 or dims > mixer["dim"]:
            raise ConfigError(f"config.json: {where}.rot.dims must be even and at most {mixer['dim']}")
        scaling = _object(where + ".rot", rot, "scaling")
        if scaling is not None:
            for key in ("factor", "original", "fast", "slow"):
                _positive(where + ".rot.scaling", scaling, key)
            if float(rot["base"]) <= 1:
                raise ConfigError(f"config.json: {where}.rot.base must exceed 1 where the rotation is scaled")


def _check_attention_2(where: str, mixer: Mapping[str, Any]) -> None:
    _check_heads(where, mixer)
    _number(where, mixer, "diff")
    temperature = _object(where, mixer, "q_temp")
    if temperature is not None:
        _number(where + ".q_temp", temperature, "coef")
        _positive(where + ".q_temp", temperature, "every")


def _check_gla(where: str, mixer: Mapping[str, Any]) -> None:
    for key in ("heads", "dim", "vdim"):
        _integer(where, mixer, key)
    _positive(where, mixer, "tau")
    if "rank" in mixer:
        _integer(where, mixer, "rank")


_CHECKS = {"attention": _check_attention, "attention_2": _check_attention_2, "gla": _check_gla}


def _check_mlp(where: str, mlp: Any) -> None:
    if not isinstance(mlp, Mapping) or mlp.get("kind") != "dense":
        raise ConfigError(f"config.json: {where}.kind must be 'dense'")
    _integer(where, mlp, "ff")


@dataclass(frozen=True)
class LanilornConfig:
    vocab: int
    width: int
    eps: float
    streams: int
    layers: tuple                      # the layer entries as read (dicts), checked
    embedding_scale: float = 1.0
    logit_scale: float = 1.0
    eos_token_id: Optional[int] = None

    architecture = "Lanilorn"

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, data: Mapping[str, Any]) -> "LanilornConfig":
        vocab = _integer("the model", data, "vocab")
        width = _integer("the model", data, "width")
        streams = _integer("the model", data, "streams")
        norm = data.get("norm")
        if not isinstance(norm, Mapping) or "eps" not in norm:
            raise ConfigError("config.json: 'norm' must be an object with 'eps'")
        layers = data.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        embedding = _object("the model", data, "embedding") or {}
        eos = data.get("eos_token_id")
        if isinstance(eos, list):
            eos = eos[0] if eos else None
        config = cls(vocab, width, _number("norm", norm, "eps"), streams, tuple(copy.deepcopy(list(layers))),
                     _number("embedding", embedding, "scale") if "scale" in embedding else 1.0,
                     _number("the model", data, "logit_scale") if data.get("logit_scale") is not None else 1.0,
                     None if eos is None else int(eos))
        config.validate()
        return config

    def to_dict(self) -> Dict[str, Any]:
        data: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab,
                                "width": self.width, "norm": {"eps": self.eps}, "streams": self.streams,
                                "embedding": {"scale": self.embedding_scale}, "logit_scale": self.logit_scale,
                                "layers": copy.deepcopy(list(self.layers))}
        if self.eos_token_id is not None:
            data["eos_token_id"] = self.eos_token_id
        return data

    # --------------------------------------------------------------- validation
    def validate(self) -> None:
        if self.eps < 0:
            raise ConfigError("config.json: norm.eps must not be negative")
        for index, layer in enumerate(self.layers):
            where = f"layers[{index}]"
            if not isinstance(layer, Mapping) or not isinstance(layer.get("mixer"), Mapping):
                raise ConfigError(f"config.json: {where} must be an object with a 'mixer'")
            if layer.get("type") not in MIXERS:
                raise ConfigError(f"config.json: {where}.type '{layer.get('type')}' is not a mixer of this design "
                                  f"({', '.join(MIXERS)})")
            _CHECKS[layer["type"]](where + ".mixer", layer["mixer"])
            if layer.get("mlp") is not None:
                _check_mlp(where + ".mlp", layer["mlp"])

    # --------------------------------------------------------------------- spec
    @staticmethod
    def _position(rot: Optional[Mapping[str, Any]]) -> PartSpec:
        if not rot:
            return PartSpec("none", {})
        params = {"theta": float(rot["base"]), "rotary_dim": int(rot["dims"])}
        scaling = rot.get("scaling")
        if not scaling:
            return PartSpec("rotary", params)
        return PartSpec("yarn_rotary", dict(params, **{k: float(scaling[k]) for k in ("factor", "original", "fast",
                                                                                      "slow")}))

    def _mixer(self, kind: str, mixer: Mapping[str, Any]) -> PartSpec:
        heads = int(mixer["heads"])
        params = {"hidden_size": self.width, "heads": heads, "dim": int(mixer["dim"]),
                  "vdim": int(mixer.get("vdim", mixer["dim"])), "eps": self.eps}
        if kind == "gla":
            if "rank" in mixer:
                params["rank"] = int(mixer["rank"])
            return PartSpec("gated_linear_attention", dict(params, tau=float(mixer["tau"])))
        params.update(kv_heads=int(mixer.get("kv_heads", heads)), scale=float(mixer["scale"]))
        if kind == "attention_2":
            temperature = mixer.get("q_temp")
            return PartSpec("difference_attention", dict(
                params, diff=float(mixer["diff"]),
                temperature=None if not temperature else (float(temperature["coef"]), float(temperature["every"]))))
        return PartSpec("scaled_gqa_attention", dict(
            params, position=self._position(mixer.get("rot")), temperature=False, value_mix="none", bias=False,
            window=int(mixer["mask"]["size"]) if mixer.get("mask") else 0, qk_norm=True, norm_span="projection",
            keys_as_values=True, sink=True, head_gate=True))

    def _feed_forward(self, mlp: Optional[Mapping[str, Any]]) -> Optional[PartSpec]:
        if mlp is None:
            return None
        return PartSpec("plain_mlp", {"hidden_size": self.width, "intermediate_size": int(mlp["ff"]),
                                      "activation": "relu2"})

    def build_spec(self) -> ModelSpec:
        """Lay the configuration out as parts: every layer is a `streams` arrangement of RMS norms whose
        sublayers' outputs are scaled column by column; its mixer `scaled_gqa_attention` (window, whole-projection
        norm, keys as values, sinks), `difference_attention` or `gated_linear_attention`; its
        feed-forward a `plain_mlp`, or none."""
        norm = PartSpec("rmsnorm", {"width": self.width, "eps": self.eps, "weight_name": ""})
        layers: List[LayerSpec] = [
            LayerSpec(prefix=f"l{index}.", arrangement="streams", mixer=self._mixer(layer["type"], layer["mixer"]),
                      feed_forward=self._feed_forward(layer.get("mlp")), mixer_norm=norm, feed_forward_norm=norm,
                      mixer_name="mix.", feed_forward_name="mlp.", mixer_norm_name="norm1",
                      feed_forward_norm_name="norm2", output_scale_names=("ls1", "ls2"))
            for index, layer in enumerate(self.layers)]
        return ModelSpec(
            architecture=self.architecture, hidden_size=self.width, vocab_size=self.vocab,
            max_position=0, embedding_name="embed", head_name=None, final_norm=norm,
            final_norm_prefix="final.norm", layers=tuple(layers),
            schedule=tuple(LayerCall(layer=i) for i in range(len(layers))), streams=self.streams,
            embedding_scale=self.embedding_scale, logit_scale=self.logit_scale)
