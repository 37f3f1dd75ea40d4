"""Typed configuration of the Daburax design, read from its own ``config.json`` keys.

A Daburax folder names its design under ``architecture`` and describes every layer on its own:
``layers[i] = {"type": "retention" | "parallel", "mixer": its sizes and constants, "mlp": {"kind":
"moe", "expert", "router", "shared"} or null}``.  Beside the layers: ``width``, ``vocab``,
``streams``, ``residual_mult``, ``norm.eps``, ``embedding.scale`` and ``embedding.bigram``.  Every
size and constant of a model comes from this object.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping

from .model_config import ConfigError
from .vilepel_config import _eos, _need, _plain, _positive_int

MIXER_KEYS = {
    "retention": ("heads", "dim", "vdim", "decay"),
    "parallel": ("left", "right", "left_scale", "right_scale"),
}
LEFT_KEYS = ("heads", "kv_heads", "dim", "vdim", "scale")
RIGHT_KEYS = ("heads", "dim", "vdim", "gate_cap")


def _check_rot(m, where: str) -> None:
    rot = m.get("rot")
    if not rot:
        return
    dims = _need(rot, "dims", f"{where}.rot")
    if isinstance(dims, bool) or not isinstance(dims, int) or dims < 0 or dims % 2 or dims > m["dim"]:
        raise ConfigError(f"config.json: {where}.rot.dims must be an even number up to dim "
                          f"{m['dim']}, got {dims!r}")
    if not (float(_need(rot, "base", f"{where}.rot")) > 0):
        raise ConfigError(f"config.json: {where}.rot.base must be > 0")
    sc = rot.get("scaling")
    if sc is not None and not (float(_need(sc, "factor", f"{where}.rot.scaling")) > 0):
        raise ConfigError(f"config.json: {where}.rot.scaling.factor must be > 0")


@dataclass(frozen=True)
class DaburaxLayer:
    type: str
    mixer: Mapping[str, Any]
    mlp: Mapping[str, Any] | None

    def to_dict(self) -> dict:
        return {"type": self.type, "mixer": _plain(self.mixer), "mlp": _plain(self.mlp)}


@dataclass(frozen=True)
class DaburaxConfig:
    width: int
    vocab: int
    streams: int
    residual_mult: float
    norm_eps: float
    embedding_scale: float
    bigram: Mapping[str, int] | None
    layers: tuple[DaburaxLayer, ...]
    eos_token_ids: tuple[int, ...] = ()
    torch_dtype: str = "bfloat16"
    extra: Mapping[str, Any] = field(default_factory=dict, compare=False, repr=False)

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "DaburaxConfig":
        width = _positive_int(_need(d, "width", "the model"), "width")
        vocab = _positive_int(_need(d, "vocab", "the model"), "vocab")
        emb = _need(d, "embedding", "the model")
        raw_layers = _need(d, "layers", "the model")
        if not isinstance(raw_layers, (list, tuple)) or not raw_layers:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        layers = []
        for i, L in enumerate(raw_layers):
            where = f"layers[{i}]"
            kind = _need(L, "type", where)
            if kind not in MIXER_KEYS:
                raise ConfigError(f"config.json: {where} has type {kind!r}; known mixers are "
                                  f"{sorted(MIXER_KEYS)}")
            mixer = _need(L, "mixer", where)
            for k in MIXER_KEYS[kind]:
                _need(mixer, k, f"{where}.mixer")
            layers.append(DaburaxLayer(kind, mixer, L.get("mlp")))
        cfg = cls(width=width, vocab=vocab,
                  streams=_positive_int(_need(d, "streams", "the model"), "streams"),
                  residual_mult=float(_need(d, "residual_mult", "the model")),
                  norm_eps=float(_need(_need(d, "norm", "the model"), "eps", "norm")),
                  embedding_scale=float(_need(emb, "scale", "embedding")),
                  bigram=emb.get("bigram"), layers=tuple(layers),
                  eos_token_ids=_eos(d.get("eos_token_id"), vocab),
                  torch_dtype=str(d.get("torch_dtype", "bfloat16")),
                  extra={k: v for k, v in d.items()
                         if k not in ("architecture", "width", "vocab", "streams", "residual_mult",
                                      "norm", "embedding", "layers", "eos_token_id",
                                      "torch_dtype")})
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if not (self.norm_eps > 0):
            raise ConfigError(f"config.json: norm.eps must be > 0, got {self.norm_eps}")
        if self.bigram is not None:
            _positive_int(_need(self.bigram, "buckets", "embedding.bigram"), "bigram.buckets")
            for k in ("mul_prev", "mul_cur"):
                v = _need(self.bigram, k, "embedding.bigram")
                if isinstance(v, bool) or not isinstance(v, int) or v < 0:
                    raise ConfigError(f"config.json: embedding.bigram.{k} must be an integer >= 0")
        for i, L in enumerate(self.layers):
            where = f"layers[{i}].mixer"
            if L.type == "retention":
                self._check_heads(L.mixer, where)
                dec = L.mixer["decay"]
                if not isinstance(dec, (list, tuple)) or len(dec) != L.mixer["heads"]:
                    raise ConfigError(f"config.json: {where}.decay must list one decay for each of the "
                                      f"{L.mixer['heads']} heads")
                _check_rot(L.mixer, where)
            else:
                left, right = L.mixer["left"], L.mixer["right"]
                for side, keys in (("left", LEFT_KEYS), ("right", RIGHT_KEYS)):
                    for k in keys:
                        _need(L.mixer[side], k, f"{where}.{side}")
                    self._check_heads(L.mixer[side], f"{where}.{side}")
                _positive_int(left["kv_heads"], f"{where}.left.kv_heads")
                if left["heads"] % left["kv_heads"]:
                    raise ConfigError(f"config.json: layers[{i}] has {left['heads']} heads for "
                                      f"{left['kv_heads']} kv heads")
                _check_rot(left, f"{where}.left")
                if not (float(right["gate_cap"]) > 0):
                    raise ConfigError(f"config.json: {where}.right.gate_cap must be > 0")
            if L.mlp is not None:
                self._check_mlp(L.mlp, f"layers[{i}].mlp")

    @staticmethod
    def _check_heads(m, where: str) -> None:
        for k in ("heads", "dim", "vdim"):
            _positive_int(m[k], f"{where}.{k}")

    @staticmethod
    def _check_mlp(mlp, where: str) -> None:
        kind = _need(mlp, "kind", where)
        if kind != "moe":
            raise ConfigError(f"config.json: {where}.kind {kind!r} is not 'moe'")
        _positive_int(_need(_need(mlp, "expert", where), "ff", f"{where}.expert"), f"{where}.expert.ff")
        r = _need(mlp, "router", where)
        experts = _positive_int(_need(r, "experts", f"{where}.router"), "router.experts")
        top = _positive_int(_need(r, "top", f"{where}.router"), "router.top")
        identity = r.get("identity", 0)
        if isinstance(identity, bool) or not isinstance(identity, int) or identity < 0:
            raise ConfigError(f"config.json: {where}.router.identity must be an integer >= 0")
        outputs, g = experts + identity, r.get("groups")
        count = keep = 1
        if g is not None:
            count = _positive_int(_need(g, "count", f"{where}.router.groups"), "groups.count")
            keep = _positive_int(_need(g, "keep", f"{where}.router.groups"), "groups.keep")
            if outputs % count or keep > count:
                raise ConfigError(f"config.json: {where}: {outputs} router outputs do not form {count} "
                                  f"equal groups of which {keep} stay")
        if top > outputs // count * keep:
            raise ConfigError(f"config.json: {where}: {top} of {outputs // count * keep} outputs cannot "
                              "be chosen")
        if mlp.get("shared") is not None:
            _positive_int(_need(mlp["shared"], "ff", f"{where}.shared"), f"{where}.shared.ff")

    def to_dict(self) -> dict[str, Any]:
        d: dict[str, Any] = dict(self.extra)
        emb: dict[str, Any] = {"scale": self.embedding_scale}
        if self.bigram is not None:
            emb["bigram"] = _plain(self.bigram)
        d.update(architecture="Daburax", width=self.width, vocab=self.vocab, streams=self.streams,
                 residual_mult=self.residual_mult, norm={"eps": self.norm_eps}, embedding=emb,
                 layers=[L.to_dict() for L in self.layers], torch_dtype=self.torch_dtype)
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d
