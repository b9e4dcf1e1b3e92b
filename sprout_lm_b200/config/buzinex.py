"""Typed configuration of the Buzinex decoder, read from its config.json.

config.json: ``architecture`` ("Buzinex"), ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``, ``logit_scale`` and
``logit_softcap`` (the logits are multiplied by the one, then capped by the other), and ``layers``, a list whose entries give
``type``, the sizes of that mixer (``mixer``) and the feed-forward (``mlp``: {``kind``: "dense", ``ff``}, silu-gated, or null
for none).  Mixers:

* ``latent_attention``: ``heads``, ``dim`` unrotated and ``rot_dim`` rotated query/key elements per head, ``vdim``, ``kv_rank``,
  ``scale``, ``mask.size`` (a sliding window), ``rot`` = {``base``, ``dims``} (interleaved pairs; the whole rotated part turns),
  a sink per head;
* ``attention``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``softcap`` on the scores, ``q_temp`` = {``coef``, ``every``}
  (queries grow with their position), query and key norms per head, no rotation, every earlier position;
* ``wkv``: ``heads``, ``dim``: RWKV time mixing (its decay's inner size is that of the checkpoint's tensors; ``rank`` names it for
  the random-weights mode).

Every size and constant comes from the file; only ``max_positions`` (the rotary tables' length) has a default.  Every sublayer
has a norm before and after it.  Tensor names: ``embed`` (also the head), ``l<i>.norm1|norm1b|norm2|norm2b``, ``l<i>.mix.*``,
``l<i>.mlp.gate|up|down``, ``final.norm``.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, replace
from typing import Any, Mapping

from .specs import ConfigError, LayerCall, LayerSpec, ModelSpec, PartSpec

DEFAULT_MAX_POSITIONS = 65536
MIXER_TYPES = ("latent_attention", "attention", "wkv")
MAX_DIM = {"dim": 512, "vdim": 512}          # what the attention's kernels hold per head
MAX_RANK = 1024                              # and of a latent
MAX_STATE_DIM = 1024                         # and of a recurrence's key vectors


def _is_int(value) -> bool:
    return isinstance(value, int) and not isinstance(value, bool)


def _number(value) -> bool:
    return isinstance(value, (int, float)) and not isinstance(value, bool) and math.isfinite(value)


def _positive_int(raw: Mapping, key: str, where: str, most: int | None = None) -> int:
    value = raw.get(key)
    if not _is_int(value) or value <= 0:
        raise ConfigError(f"Invalid Buzinex config: {where}.{key} must be a positive integer.")
    if most is not None and value > most:
        raise ConfigError(f"Invalid Buzinex config: {where}.{key} must be at most {most}.")
    return value


def _positive(raw: Mapping, key: str, where: str) -> float:
    value = raw.get(key)
    if not _number(value) or value <= 0:
        raise ConfigError(f"Invalid Buzinex config: {where}.{key} must be a positive number.")
    return float(value)


def _any_number(raw: Mapping, key: str, where: str) -> float:
    value = raw.get(key)
    if not _number(value):
        raise ConfigError(f"Invalid Buzinex config: {where}.{key} must be a number.")
    return float(value)


def _object(raw: Mapping, key: str, where: str) -> Mapping:
    value = raw.get(key)
    if not isinstance(value, Mapping):
        raise ConfigError(f"Invalid Buzinex config: {where}.{key} must be an object.")
    return value


def _parse_latent(m: Mapping, where: str) -> dict:
    out = {key: _positive_int(m, key, where) for key in ("heads", "dim", "rot_dim", "vdim")}
    out["kv_rank"] = _positive_int(m, "kv_rank", where, MAX_RANK)
    out["scale"] = _positive(m, "scale", where)
    out["mask"] = {"size": _positive_int(_object(m, "mask", where), "size", where + ".mask")}
    rot = _object(m, "rot", where)
    if rot.get("dims") != out["rot_dim"] or out["rot_dim"] % 2:
        raise ConfigError(f"Invalid Buzinex config: {where}.rot.dims must be rot_dim, an even number: the whole rotated part turns.")
    base = _positive(rot, "base", where + ".rot")
    if base <= 1:
        raise ConfigError(f"Invalid Buzinex config: {where}.rot.base must be above 1.")
    out["rot"] = {"base": base, "dims": out["rot_dim"]}
    return out


def _parse_attention(m: Mapping, where: str) -> dict:
    out = {key: _positive_int(m, key, where, MAX_DIM.get(key)) for key in ("heads", "kv_heads", "dim", "vdim")}
    if out["heads"] % out["kv_heads"]:
        raise ConfigError(f"Invalid Buzinex config: {where}.heads must be a multiple of kv_heads.")
    out["scale"], out["softcap"] = _positive(m, "scale", where), _positive(m, "softcap", where)
    temp = _object(m, "q_temp", where)
    out["q_temp"] = {"coef": _any_number(temp, "coef", where + ".q_temp"), "every": _positive_int(temp, "every", where + ".q_temp")}
    return out


def _parse_wkv(m: Mapping, where: str) -> dict:
    out = {"heads": _positive_int(m, "heads", where), "dim": _positive_int(m, "dim", where, MAX_STATE_DIM)}
    if m.get("rank") is not None:
        out["rank"] = _positive_int(m, "rank", where)
    return out


_PARSERS = {"latent_attention": _parse_latent, "attention": _parse_attention, "wkv": _parse_wkv}


def _parse_mlp(index: int, mlp) -> dict | None:
    where = f"layers[{index}].mlp"
    if mlp is None:
        return None
    if not isinstance(mlp, Mapping) or mlp.get("kind") != "dense":
        raise ConfigError(f"Invalid Buzinex config: {where} must be null or of kind 'dense'.")
    return {"kind": "dense", "ff": _positive_int(mlp, "ff", where)}


@dataclass(frozen=True)
class BuzinexLayer:
    type: str
    mixer: dict
    mlp: dict | None

    def to_dict(self) -> dict:
        return {"type": self.type, "mixer": self.mixer, "mlp": self.mlp}


@dataclass(frozen=True)
class BuzinexConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    logit_scale: float
    logit_softcap: float
    layers: tuple
    max_positions: int = DEFAULT_MAX_POSITIONS
    eos_token_ids: tuple = ()

    architecture = "Buzinex"

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "BuzinexConfig":
        if not isinstance(raw, Mapping) or raw.get("architecture") != cls.architecture:
            raise ConfigError("Invalid Buzinex config.")
        vocab, width = _positive_int(raw, "vocab", "config"), _positive_int(raw, "width", "config")
        eps = _positive(_object(raw, "norm", "config"), "eps", "config.norm")
        scale = _any_number(_object(raw, "embedding", "config"), "scale", "config.embedding")
        logit_scale, logit_cap = _any_number(raw, "logit_scale", "config"), _positive(raw, "logit_softcap", "config")
        if not isinstance(raw.get("layers"), list) or not raw["layers"]:
            raise ConfigError("Invalid Buzinex config: layers must be a non-empty list.")
        layers = []
        for index, layer in enumerate(raw["layers"]):
            if not isinstance(layer, Mapping) or layer.get("type") not in MIXER_TYPES or not isinstance(layer.get("mixer"), Mapping):
                raise ConfigError(f"Invalid Buzinex config: layers[{index}] needs a type of {', '.join(MIXER_TYPES)} and a mixer.")
            mixer = _PARSERS[layer["type"]](layer["mixer"], f"layers[{index}].mixer")
            layers.append(BuzinexLayer(layer["type"], mixer, _parse_mlp(index, layer.get("mlp"))))
        max_positions = raw.get("max_positions", DEFAULT_MAX_POSITIONS)
        if not _is_int(max_positions) or max_positions <= 0:
            raise ConfigError("Invalid Buzinex config: max_positions must be a positive integer.")
        eos_ids = ()
        if raw.get("eos_token_id") is not None:
            from .qwen2 import parse_eos_ids
            eos_ids = parse_eos_ids(raw["eos_token_id"], vocab)
        return cls(vocab=vocab, width=width, norm_eps=eps, embedding_scale=scale, logit_scale=logit_scale, logit_softcap=logit_cap,
                   layers=tuple(layers), max_positions=max_positions, eos_token_ids=eos_ids)

    def to_dict(self) -> dict:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
               "embedding": {"scale": self.embedding_scale}, "logit_scale": self.logit_scale, "logit_softcap": self.logit_softcap,
               "layers": [layer.to_dict() for layer in self.layers]}
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            out["max_positions"] = self.max_positions
        if self.eos_token_ids:
            out["eos_token_id"] = list(self.eos_token_ids)
        return out

    def with_eos(self, eos_token_id) -> "BuzinexConfig":
        from .qwen2 import parse_eos_ids
        return replace(self, eos_token_ids=parse_eos_ids(eos_token_id, self.vocab))

    # ------------------------------------------------------------------ parts
    def _mixer_spec(self, layer: BuzinexLayer) -> PartSpec:
        m, eps = layer.mixer, self.norm_eps
        if layer.type == "wkv":
            return PartSpec("rwkv_time_mixing", {"hidden_size": self.width, "heads": m["heads"], "dim": m["dim"], "eps": eps,
                                                 "decay_rank": m.get("rank"), "stem": "mix."})
        if layer.type == "latent_attention":
            position = PartSpec("rope_interleaved", {"dims": m["rot"]["dims"], "theta": m["rot"]["base"],
                                                     "max_positions": self.max_positions, "scaling": None})
            return PartSpec("latent_attention", {
                "hidden_size": self.width, "heads": m["heads"], "dim": m["dim"], "rot_dim": m["rot_dim"], "value_dim": m["vdim"],
                "kv_rank": m["kv_rank"], "scale": m["scale"], "eps": eps, "position": position, "window": m["mask"]["size"],
                "names": {key: "mix." + name for key, name in (("q", "q"), ("dkv", "dkv"), ("dkv_norm", "dkv.norm"), ("uk", "uk"),
                                                               ("uv", "uv"), ("sink", "sink"), ("o", "o"))}})
        return PartSpec("multimap_attention", {
            "hidden_size": self.width, "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"], "value_dim": m["vdim"],
            "scale": m["scale"], "position": PartSpec("none", {}), "maps": 1, "softcap": m["softcap"], "qk_norm_eps": eps,
            "query_growth": (m["q_temp"]["coef"], m["q_temp"]["every"]),
            "names": {key: "mix." + name for key, name in (("q", "q"), ("k", "k"), ("v", "v"), ("o", "o"), ("q_norm", "q.norm"),
                                                           ("k_norm", "k.norm"))}})

    def _mlp_spec(self, mlp: dict | None) -> PartSpec:
        if mlp is None:
            return PartSpec("none", {})
        return PartSpec("gated_mlp", {"hidden_size": self.width, "intermediate_size": mlp["ff"], "activation": "silu",
                                      "names": {key: "mlp." + key for key in ("gate", "up", "down")}})

    def model_spec(self) -> ModelSpec:
        norm = {"size": self.width, "eps": self.norm_eps, "suffix": ""}
        layers = []
        for index, layer in enumerate(self.layers):
            names = ("norm1", "norm1b") + (("norm2", "norm2b") if layer.mlp is not None else ())
            layers.append(LayerSpec("sandwich_norm", f"l{index}.", self._mixer_spec(layer), self._mlp_spec(layer.mlp),
                                    tuple(PartSpec("rmsnorm", {**norm, "name": name}) for name in names)))
        return ModelSpec(
            architecture=self.architecture, hidden_size=self.width, vocab_size=self.vocab, max_positions=self.max_positions,
            embedding=PartSpec("token_embedding", {"vocab_size": self.vocab, "hidden_size": self.width, "name": "embed", "suffix": "",
                                                   "scale": self.embedding_scale}),
            layers=tuple(layers), order=tuple(LayerCall(layer=i, cache=i) for i in range(len(layers))),
            final_norm=PartSpec("rmsnorm", {**norm, "name": "final.norm"}),
            head=PartSpec("lm_head", {"vocab_size": self.vocab, "hidden_size": self.width, "tied_to": "embed", "suffix": "",
                                      "scale": self.logit_scale, "softcap": self.logit_softcap, "any_inner_size": True}),
            eos_token_ids=self.eos_token_ids)
