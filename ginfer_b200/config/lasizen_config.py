"""Typed configuration of the Lasizen design, read from its own ``config.json`` keys.

A Lasizen folder names its design under ``architecture`` and describes every layer on its own:
``layers[i] = {"type": "delta" | "attention", "mixer": its sizes and constants, "mlp": {"kind":
"dense", "ff": n} or null}``.  Beside the layers: ``width``, ``vocab``, ``norm.eps``,
``embedding.scale``, ``logit_scale`` and ``loop = {start, stop, times}`` (layers ``start .. stop-1``
run ``times`` times in a row, each pass with caches and states of its own; absent or null: every
layer once).  Every size and constant of a model comes from this object.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping

from .model_config import ConfigError
from .vilepel_config import _eos, _need, _plain, _positive_int

MIXER_KEYS = {
    "delta": ("heads", "kv_heads", "dim", "vdim", "conv"),
    "attention": ("heads", "kv_heads", "dim", "vdim", "scale"),
}
_TOP_KEYS = ("architecture", "width", "vocab", "norm", "embedding", "logit_scale", "loop", "layers",
             "eos_token_id", "torch_dtype")


@dataclass(frozen=True)
class LasizenLayer:
    type: str
    mixer: Mapping[str, Any]
    mlp: Mapping[str, Any] | None

    def to_dict(self) -> dict:
        return {"type": self.type, "mixer": _plain(self.mixer), "mlp": _plain(self.mlp)}


@dataclass(frozen=True)
class LasizenConfig:
    width: int
    vocab: int
    norm_eps: float
    embedding_scale: float
    logit_scale: float
    layers: tuple[LasizenLayer, ...]
    loop: tuple[int, int, int] | None = None           # (start, stop, times)
    eos_token_ids: tuple[int, ...] = ()
    torch_dtype: str = "bfloat16"
    extra: Mapping[str, Any] = field(default_factory=dict, compare=False, repr=False)

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "LasizenConfig":
        width = _positive_int(_need(d, "width", "the model"), "width")
        vocab = _positive_int(_need(d, "vocab", "the model"), "vocab")
        eps = float(_need(_need(d, "norm", "the model"), "eps", "norm"))
        emb = d.get("embedding") or {}
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
            mlp = L.get("mlp")
            if mlp is not None:
                mk = _need(mlp, "kind", f"{where}.mlp")
                if mk != "dense":
                    raise ConfigError(f"config.json: {where}.mlp.kind {mk!r} is not 'dense'")
                _positive_int(_need(mlp, "ff", f"{where}.mlp"), f"{where}.mlp.ff")
            layers.append(LasizenLayer(kind, mixer, mlp))
        loop = d.get("loop")
        if loop is not None:
            loop = tuple(int(_need(loop, k, "loop")) for k in ("start", "stop", "times"))
        cfg = cls(width=width, vocab=vocab, norm_eps=eps,
                  embedding_scale=float(emb.get("scale", 1.0)),
                  logit_scale=float(d.get("logit_scale", 1.0)),
                  layers=tuple(layers), loop=loop,
                  eos_token_ids=_eos(d.get("eos_token_id"), vocab),
                  torch_dtype=str(d.get("torch_dtype", "bfloat16")),
                  extra={k: v for k, v in d.items() if k not in _TOP_KEYS})
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if not (self.norm_eps > 0):
            raise ConfigError(f"config.json: norm.eps must be > 0, got {self.norm_eps}")
        if self.loop is not None:
            a, b, times = self.loop
            if not (0 <= a < b <= len(self.layers)) or times < 1:
                raise ConfigError(f"config.json: loop {self.loop} does not fit "
                                  f"{len(self.layers)} layers (0 <= start < stop <= layers, "
                                  "times >= 1)")
        for i, L in enumerate(self.layers):
            m, where = L.mixer, f"layers[{i}].mixer"
            for k in ("heads", "kv_heads", "dim", "vdim"):
                _positive_int(m[k], f"{where}.{k}")
            if m["heads"] % m["kv_heads"]:
                raise ConfigError(f"config.json: layers[{i}] has {m['heads']} heads for "
                                  f"{m['kv_heads']} kv heads")
            if L.type == "delta":
                _positive_int(m["conv"], f"{where}.conv")
                continue
            if m.get("mask") is not None:            # no mask: every earlier token is seen
                _positive_int(_need(m["mask"], "size", f"{where}.mask"), "mask.size")
            rot = m.get("rot")
            if rot is None:                          # no rot: no rotation
                continue
            dims = _need(rot, "dims", f"{where}.rot")
            if isinstance(dims, bool) or not isinstance(dims, int) or dims < 0 or dims % 2 \
                    or dims > m["dim"]:
                raise ConfigError(f"config.json: layers[{i}] rotates {dims!r} of {m['dim']} "
                                  "channels; it must be an even number of them")
            base = float(_need(rot, "base", f"{where}.rot"))
            if not (base > 0):
                raise ConfigError(f"config.json: {where}.rot.base must be > 0")
            sc = rot.get("scaling")
            if sc is not None:
                for k in ("factor", "original", "fast", "slow"):
                    if not (float(_need(sc, k, f"{where}.rot.scaling")) > 0):
                        raise ConfigError(f"config.json: {where}.rot.scaling.{k} must be > 0")
                if base == 1.0:
                    raise ConfigError(f"config.json: {where}.rot.scaling needs a base other than 1")

    def run_order(self) -> list[int]:
        """The layers in the order in which a step runs them."""
        n = len(self.layers)
        if self.loop is None:
            return list(range(n))
        a, b, times = self.loop
        return list(range(a)) + list(range(a, b)) * times + list(range(b, n))

    def to_dict(self) -> dict[str, Any]:
        d: dict[str, Any] = dict(self.extra)
        d.update(architecture="Lasizen", width=self.width, vocab=self.vocab,
                 norm={"eps": self.norm_eps}, embedding={"scale": self.embedding_scale},
                 logit_scale=self.logit_scale, layers=[L.to_dict() for L in self.layers],
                 torch_dtype=self.torch_dtype)
        if self.loop is not None:
            d["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d
