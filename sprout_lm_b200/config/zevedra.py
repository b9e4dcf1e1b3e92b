"""Typed configuration of the Zevedra decoder, read from its config.json.

config.json: ``architecture`` ("Zevedra"), ``vocab``, ``width``, ``norm.eps``, ``residual_mult`` (what both sublayers of a layer
add is multiplied by it), ``embedding`` = {``scale``[, ``bigram``: {``buckets``, ``mul_prev``, ``mul_cur``}]} (a second table
whose row the last two tokens choose), optionally ``loop`` = {``start``, ``stop``, ``times``} (layers start .. stop - 1 run
``times`` times in a row with the same weights), and ``layers``, a list whose entries give ``type``, the sizes of that mixer
(``mixer``) and the feed-forward (``mlp``, or null for none).  Both mixers are two mixers side by side:

* ``parallel``: ``left`` (softmax attention over a sliding window of ``mask.size`` positions: ``heads``, ``kv_heads``, ``dim``,
  ``vdim``, ``conv`` taps on queries, keys and values, ``rot`` = {``base``, ``dims``} in interleaved pairs, unit-length queries
  and keys, values turned by their position and outputs turned back, ``scale``, a sigmoid gate per head) beside ``right`` (the
  gated delta rule: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``conv`` taps), summed with ``left_scale`` and ``right_scale``;
* ``parallel_2``: ``left`` (causal softmax attention with one added to its denominator: ``heads``, ``kv_heads``, ``dim``, ``vdim``,
  query and key norms over the whole projections, ``rot`` in half-split pairs, ``scale``, a sigmoid gate per element) beside
  ``right`` (a recurrence whose forget gate also decides what is written: ``heads``, ``dim``, ``vdim``), each normed over the
  width, half their sum.

``mlp``: {``kind``: "moe", ``expert``: {``ff``}, ``router``: {``experts``, ``top``}}: silu-gated experts chosen by sigmoid scores
that multiply an expert's input.  Every size and constant comes from the file; only ``max_positions`` (the rotary tables'
length) has a default.  Norms have one number for all elements.  Tensor names: ``embed``, ``bigram``, ``loop.step``,
``l<i>.norm1|norm2``, ``l<i>.mix.left.*``, ``l<i>.mix.right.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, replace
from typing import Any, Mapping

from .specs import ConfigError, LayerCall, LayerSpec, ModelSpec, PartSpec

DEFAULT_MAX_POSITIONS = 65536
MIXER_TYPES = ("parallel", "parallel_2")
MAX_TAPS = 8                    # what the convolution's kernel holds


def _is_int(value) -> bool:
    return isinstance(value, int) and not isinstance(value, bool)


def _number(value) -> bool:
    return isinstance(value, (int, float)) and not isinstance(value, bool) and math.isfinite(value)


def _positive_int(raw: Mapping, key: str, where: str) -> int:
    value = raw.get(key)
    if not _is_int(value) or value <= 0:
        raise ConfigError(f"Invalid Zevedra config: {where}.{key} must be a positive integer.")
    return value


def _positive(raw: Mapping, key: str, where: str) -> float:
    value = raw.get(key)
    if not _number(value) or value <= 0:
        raise ConfigError(f"Invalid Zevedra config: {where}.{key} must be a positive number.")
    return float(value)


def _any_number(raw: Mapping, key: str, where: str) -> float:
    value = raw.get(key)
    if not _number(value):
        raise ConfigError(f"Invalid Zevedra config: {where}.{key} must be a number.")
    return float(value)


def _object(raw: Mapping, key: str, where: str) -> Mapping:
    value = raw.get(key)
    if not isinstance(value, Mapping):
        raise ConfigError(f"Invalid Zevedra config: {where}.{key} must be an object.")
    return value


def _taps(raw: Mapping, where: str) -> int:
    taps = _positive_int(raw, "conv", where)
    if taps > MAX_TAPS:
        raise ConfigError(f"Invalid Zevedra config: {where}.conv must be at most {MAX_TAPS} taps.")
    return taps


def _heads(m: Mapping, where: str, grouped: bool) -> dict:
    out = {"heads": _positive_int(m, "heads", where), "dim": _positive_int(m, "dim", where), "vdim": _positive_int(m, "vdim", where)}
    if grouped:
        out["kv_heads"] = _positive_int(m, "kv_heads", where)
        if out["heads"] % out["kv_heads"]:
            raise ConfigError(f"Invalid Zevedra config: {where}.heads must be a multiple of kv_heads.")
    return out


def _softmax(m: Mapping, where: str, windowed: bool) -> dict:
    out = _heads(m, where, grouped=True)
    out["scale"] = _positive(m, "scale", where)
    rot = _object(m, "rot", where)
    dims = rot.get("dims")
    if not _is_int(dims) or dims < 0 or dims % 2 or dims > out["dim"]:
        raise ConfigError(f"Invalid Zevedra config: {where}.rot.dims must be even and at most dim.")
    base = _positive(rot, "base", where + ".rot")
    if base <= 1:
        raise ConfigError(f"Invalid Zevedra config: {where}.rot.base must be above 1.")
    out["rot"] = {"base": base, "dims": dims}
    if windowed:
        if out["vdim"] % 2:
            raise ConfigError(f"Invalid Zevedra config: {where}.vdim must be even: its elements turn in pairs.")
        out["conv"] = _taps(m, where)
        out["mask"] = {"size": _positive_int(_object(m, "mask", where), "size", where + ".mask")}
    return out


def _parse_mixer(index: int, kind: str, m: Mapping) -> dict:
    where = f"layers[{index}].mixer"
    left, right = _object(m, "left", where), _object(m, "right", where)
    out = {"left": _softmax(left, where + ".left", windowed=kind == "parallel"),
           "right": _heads(right, where + ".right", grouped=kind == "parallel")}
    if kind == "parallel":
        out["right"]["conv"] = _taps(right, where + ".right")
        if out["right"]["dim"] > 256:
            raise ConfigError(f"Invalid Zevedra config: {where}.right.dim must be at most 256.")
        for key in ("left_scale", "right_scale"):
            out[key] = _any_number(m, key, where)
    return out


def _parse_mlp(index: int, mlp) -> dict | None:
    where = f"layers[{index}].mlp"
    if mlp is None:
        return None
    if not isinstance(mlp, Mapping) or mlp.get("kind") != "moe":
        raise ConfigError(f"Invalid Zevedra config: {where} must be null or of kind 'moe'.")
    expert, router = _object(mlp, "expert", where), _object(mlp, "router", where)
    out = {"kind": "moe", "expert": {"ff": _positive_int(expert, "ff", where + ".expert")},
           "router": {"experts": _positive_int(router, "experts", where + ".router"), "top": _positive_int(router, "top", where + ".router")}}
    if out["router"]["top"] > out["router"]["experts"]:
        raise ConfigError(f"Invalid Zevedra config: {where}.router.top must be at most experts.")
    return out


@dataclass(frozen=True)
class ZevedraLayer:
    type: str
    mixer: dict
    mlp: dict | None

    def to_dict(self) -> dict:
        return {"type": self.type, "mixer": self.mixer, "mlp": self.mlp}


@dataclass(frozen=True)
class ZevedraConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    embedding_scale: float
    layers: tuple
    bigram: tuple | None = None                # (buckets, mul_prev, mul_cur)
    loop: tuple | None = None                  # (start, stop, times)
    max_positions: int = DEFAULT_MAX_POSITIONS
    eos_token_ids: tuple = ()

    architecture = "Zevedra"

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "ZevedraConfig":
        if not isinstance(raw, Mapping) or raw.get("architecture") != cls.architecture:
            raise ConfigError("Invalid Zevedra config.")
        vocab, width = _positive_int(raw, "vocab", "config"), _positive_int(raw, "width", "config")
        eps = _positive(_object(raw, "norm", "config"), "eps", "config.norm")
        mult = _any_number(raw, "residual_mult", "config")
        embedding = _object(raw, "embedding", "config")
        scale = _any_number(embedding, "scale", "config.embedding")
        bigram = None
        if embedding.get("bigram") is not None:
            spec = _object(embedding, "bigram", "config.embedding")
            for key in ("mul_prev", "mul_cur"):
                if not _is_int(spec.get(key)) or abs(spec[key]) >= 1 << 31:
                    raise ConfigError(f"Invalid Zevedra config: config.embedding.bigram.{key} must be an integer of at most 31 bits.")
            bigram = (_positive_int(spec, "buckets", "config.embedding.bigram"), spec["mul_prev"], spec["mul_cur"])
        if not isinstance(raw.get("layers"), list) or not raw["layers"]:
            raise ConfigError("Invalid Zevedra config: layers must be a non-empty list.")
        layers = []
        for index, layer in enumerate(raw["layers"]):
            if not isinstance(layer, Mapping) or layer.get("type") not in MIXER_TYPES or not isinstance(layer.get("mixer"), Mapping):
                raise ConfigError(f"Invalid Zevedra config: layers[{index}] needs a type of {', '.join(MIXER_TYPES)} and a mixer.")
            layers.append(ZevedraLayer(layer["type"], _parse_mixer(index, layer["type"], layer["mixer"]),
                                       _parse_mlp(index, layer.get("mlp"))))
        loop = None
        if raw.get("loop") is not None:
            spec = _object(raw, "loop", "config")
            start, stop, times = spec.get("start"), spec.get("stop"), spec.get("times")
            if not _is_int(start) or not _is_int(stop) or not _is_int(times) or not 0 <= start < stop <= len(layers) or times < 1:
                raise ConfigError("Invalid Zevedra config: loop needs 0 <= start < stop <= layers and times >= 1.")
            loop = (start, stop, times)
        max_positions = raw.get("max_positions", DEFAULT_MAX_POSITIONS)
        if not _is_int(max_positions) or max_positions <= 0:
            raise ConfigError("Invalid Zevedra config: max_positions must be a positive integer.")
        eos_ids = ()
        if raw.get("eos_token_id") is not None:
            from .qwen2 import parse_eos_ids
            eos_ids = parse_eos_ids(raw["eos_token_id"], vocab)
        return cls(vocab=vocab, width=width, norm_eps=eps, residual_mult=mult, embedding_scale=scale, layers=tuple(layers),
                   bigram=bigram, loop=loop, max_positions=max_positions, eos_token_ids=eos_ids)

    def to_dict(self) -> dict:
        embedding: dict = {"scale": self.embedding_scale}
        if self.bigram is not None:
            embedding["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), self.bigram))
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
               "residual_mult": self.residual_mult, "embedding": embedding, "layers": [layer.to_dict() for layer in self.layers]}
        if self.loop is not None:
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            out["max_positions"] = self.max_positions
        if self.eos_token_ids:
            out["eos_token_id"] = list(self.eos_token_ids)
        return out

    def with_eos(self, eos_token_id) -> "ZevedraConfig":
        from .qwen2 import parse_eos_ids
        return replace(self, eos_token_ids=parse_eos_ids(eos_token_id, self.vocab))

    # ------------------------------------------------------------------ parts
    def _rotary(self, kind: str, dims: int, base: float) -> PartSpec:
        return PartSpec(kind, {"dims": dims, "theta": base, "max_positions": self.max_positions, "scaling": None}) if dims else PartSpec("none", {})

    def _mixer_spec(self, layer: ZevedraLayer) -> PartSpec:
        m, eps = layer.mixer, self.norm_eps
        left, right = m["left"], m["right"]
        softmax = {"hidden_size": self.width, "heads": left["heads"], "kv_heads": left["kv_heads"], "dim": left["dim"],
                   "value_dim": left["vdim"], "scale": left["scale"], "maps": 1}
        sizes = {"hidden_size": self.width, "heads": right["heads"], "dim": right["dim"], "value_dim": right["vdim"], "eps": eps}
        names = ("mix.left.", "mix.right.")
        base = left["rot"]["base"]
        if layer.type == "parallel":
            attention = PartSpec("multimap_attention", {
                **softmax, "position": self._rotary("rope_interleaved", left["rot"]["dims"], base),
                "value_position": self._rotary("rope_interleaved", left["vdim"], base), "conv": left["conv"],
                "unit_norm_eps": eps, "mask": ("window", left["mask"]["size"]), "gate": "head"})
            delta = PartSpec("gated_delta_rule", {**sizes, "kv_heads": right["kv_heads"], "taps": right["conv"]})
            return PartSpec("parallel_mixers", {"mixers": (attention, delta), "scales": (m["left_scale"], m["right_scale"]),
                                                "names": names})
        attention = PartSpec("multimap_attention", {
            **softmax, "position": self._rotary("rope_yarn", left["rot"]["dims"], base), "qk_norm_eps": eps,
            "qk_norm_span": "projection", "unit_sink": True, "gate": "element"})
        return PartSpec("parallel_mixers", {
            "mixers": (attention, PartSpec("forget_write_attention", sizes)), "scales": (0.5, 0.5), "names": names,
            "norms": ("mix.left.out", "mix.right.out"), "norm_eps": eps, "hidden_size": self.width})

    def _mlp_spec(self, mlp: dict | None) -> PartSpec:
        if mlp is None:
            return PartSpec("none", {})
        return PartSpec("routed_experts", {
            "hidden_size": self.width, "experts": mlp["router"]["experts"], "identity": 0, "top": mlp["router"]["top"], "scale": 1.0,
            "expert_ff": mlp["expert"]["ff"], "expert_kind": "silu_glu", "correction": False, "renormalize": False,
            "scores": "sigmoid", "weight_on": "input", "names": {"router": "mlp.router", "expert": "mlp.e{}."}})

    def run_order(self) -> tuple[tuple, tuple]:
        """(layer calls, the index in them of every pass's first call): a looped layer is called once per pass, each call
        with a cache slot and a state entry of its own."""
        n = len(self.layers)
        if self.loop is None:
            return tuple(LayerCall(layer=i, cache=i) for i in range(n)), ()
        start, stop, times = self.loop
        calls, starts = [LayerCall(layer=i, cache=i) for i in range(start)], []
        for t in range(times):
            starts.append(len(calls))
            for i in range(start, stop):
                slot = i if t == 0 else n + (t - 1) * (stop - start) + (i - start)
                calls.append(LayerCall(layer=i, cache=slot, state=slot))
        calls += [LayerCall(layer=i, cache=i) for i in range(stop, n)]
        return tuple(calls), tuple(starts)

    def model_spec(self) -> ModelSpec:
        norm = {"size": self.width, "eps": self.norm_eps, "suffix": "", "one_number": True}
        layers = []
        for index, layer in enumerate(self.layers):
            names = ("norm1",) + (("norm2",) if layer.mlp is not None else ())
            layers.append(LayerSpec("pre_norm", f"l{index}.", self._mixer_spec(layer), self._mlp_spec(layer.mlp),
                                    tuple(PartSpec("rmsnorm", {**norm, "name": name}) for name in names),
                                    {"branch_scale": self.residual_mult}))
        order, starts = self.run_order()
        stream = PartSpec("loop_restart", {"hidden_size": self.width, "starts": starts, "name": "loop.step"}) if starts else None
        table = {"vocab_size": self.vocab, "hidden_size": self.width, "name": "embed", "suffix": "", "scale": self.embedding_scale}
        embedding = PartSpec("token_embedding", table)
        if self.bigram is not None:
            embedding = PartSpec("token_pair_embedding", {**table, **dict(zip(("buckets", "mul_prev", "mul_cur"), self.bigram))})
        return ModelSpec(
            architecture=self.architecture, hidden_size=self.width, vocab_size=self.vocab, max_positions=self.max_positions,
            embedding=embedding, layers=tuple(layers), order=order, stream=stream,
            final_norm=PartSpec("rmsnorm", {**norm, "name": "final.norm"}),
            head=PartSpec("lm_head", {"vocab_size": self.vocab, "hidden_size": self.width, "name": "head", "suffix": "",
                                      "any_inner_size": True}),
            eos_token_ids=self.eos_token_ids)
