"""Typed configuration of the Tubazen decoder.

``config.json`` of this design is nested; every size and every constant that may differ between models is
read from it (or, for the ranks of the decays and the rows of the distance bias, from the shapes of the model's
tensors):

    architecture: "Tubazen"     vocab, width, max_positions     norm: {eps}     logit_scale
    layers: [ {type: "gla" | "parallel", mixer: {...}, mlp: {kind: "dense", ff} | null}, ... ]
      gla      {heads, dim, vdim, tau}                       (+ decay_rank when no weight file gives it)
      parallel {left_scale, right_scale,
                left:  {heads, kv_heads, dim, vdim, scale, bias_max, q_temp: {coef, every}}
                       (q_temp absent: queries as they are)  (+ bias_rows when no weight file gives it)
                right: {heads, dim}                          (+ decay_rank when no weight file gives it)}
    max_positions: rows of the position table, and so the longest sequence.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, replace
from typing import Any, Mapping, Optional, Tuple

from .registry import ConfigError
from .salepel import _num, _sub


def _rank(m, name, where):
    return None if m.get(name) is None else _num(m, name, where)


def _with(out, **optional):
    out.update({k: v for k, v in optional.items() if v is not None})
    return out


@dataclass(frozen=True)
class GlaMeta:
    """Linear attention whose memory fades per key channel."""
    heads: int
    dim: int
    vdim: int
    tau: float
    decay_rank: Optional[int] = None     # rows of the decay's first projection; from the tensors when a file is read

    @classmethod
    def from_dict(cls, m, where):
        dim = _num(m, "dim", where)
        m = dict(m, vdim=m.get("vdim", dim))
        return cls(_num(m, "heads", where), dim, _num(m, "vdim", where), _num(m, "tau", where, float),
                   _rank(m, "decay_rank", where))

    def to_dict(self):
        return _with({"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "tau": self.tau}, decay_rank=self.decay_rank)


@dataclass(frozen=True)
class LeftMeta:
    """Attention with a learned bias per (distance bucket, head)."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    bias_max: int                        # from this distance on every key has the last bucket
    temp_coef: float                     # queries times 1 + coef ln(floor((p + 1) / every) + 1)
    temp_every: int                      # 0: queries as they are
    bias_rows: Optional[int] = None      # buckets; from the tensors when a file is read

    @classmethod
    def from_dict(cls, m, where):
        heads, dim = _num(m, "heads", where), _num(m, "dim", where)
        m = dict(m, kv_heads=m.get("kv_heads", heads), vdim=m.get("vdim", dim), scale=m.get("scale", dim ** -0.5))
        coef, every = 0.0, 0
        if m.get("q_temp") is not None:
            t = _sub(m, "q_temp", where)
            coef, every = _num(t, "coef", where + ".q_temp", float), _num(t, "every", where + ".q_temp")
            if every <= 0:
                raise ConfigError(f"{where}.q_temp.every must be positive, got {every}")
        return cls(heads, _num(m, "kv_heads", where), dim, _num(m, "vdim", where), _num(m, "scale", where, float),
                   _num(m, "bias_max", where), coef, every, _rank(m, "bias_rows", where))

    def to_dict(self):
        out = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale,
               "bias_max": self.bias_max}
        if self.temp_every:
            out["q_temp"] = {"coef": self.temp_coef, "every": self.temp_every}
        return _with(out, bias_rows=self.bias_rows)


@dataclass(frozen=True)
class RightMeta:
    """The delta rule with a decay, a removal rate and a key of its own."""
    heads: int
    dim: int
    decay_rank: Optional[int] = None

    @classmethod
    def from_dict(cls, m, where):
        return cls(_num(m, "heads", where), _num(m, "dim", where), _rank(m, "decay_rank", where))

    def to_dict(self):
        return _with({"heads": self.heads, "dim": self.dim}, decay_rank=self.decay_rank)


@dataclass(frozen=True)
class ParallelMeta:
    left: LeftMeta
    right: RightMeta
    left_scale: float
    right_scale: float

    @classmethod
    def from_dict(cls, m, where):
        m = dict(m, left_scale=m.get("left_scale", 1.0), right_scale=m.get("right_scale", 1.0))
        return cls(LeftMeta.from_dict(_sub(m, "left", where), where + ".left"),
                   RightMeta.from_dict(_sub(m, "right", where), where + ".right"),
                   _num(m, "left_scale", where, float), _num(m, "right_scale", where, float))

    def to_dict(self):
        return {"left": self.left.to_dict(), "right": self.right.to_dict(), "left_scale": self.left_scale,
                "right_scale": self.right_scale}


MIXERS = {"gla": GlaMeta, "parallel": ParallelMeta}


@dataclass(frozen=True)
class TubazenLayer:
    mixer: Any                    # GlaMeta | ParallelMeta
    ff: Optional[int]             # width of the dense feed-forward; None: a layer without one

    def to_dict(self):
        kind = "gla" if isinstance(self.mixer, GlaMeta) else "parallel"
        return {"type": kind, "mixer": self.mixer.to_dict(), "mlp": None if self.ff is None else {"kind": "dense", "ff": self.ff}}


@dataclass(frozen=True)
class TubazenMeta:
    vocab: int
    width: int
    max_positions: int
    eps: float
    logit_scale: float
    layers: Tuple[TubazenLayer, ...]
    eos: tuple = ()

    @classmethod
    def from_dict(cls, cfg: Mapping[str, Any]) -> "TubazenMeta":
        layers_in = cfg.get("layers")
        if not isinstance(layers_in, (list, tuple)) or not layers_in:
            raise ConfigError("config.json lacks the list 'layers'")
        layers = []
        for i, entry in enumerate(layers_in):
            where = f"layers[{i}]"
            if not isinstance(entry, Mapping):
                raise ConfigError(f"{where} must be an object")
            if entry.get("type") not in MIXERS:
                raise ConfigError(f"{where}.type must be one of {sorted(MIXERS)}, got {entry.get('type')!r}")
            mixer = MIXERS[entry["type"]].from_dict(_sub(entry, "mixer", where), where + ".mixer")
            mlp, ff = entry.get("mlp"), None
            if mlp is not None:
                if not isinstance(mlp, Mapping) or mlp.get("kind") != "dense":
                    raise ConfigError(f"{where}.mlp must be null or an object of kind 'dense'")
                ff = _num(mlp, "ff", where + ".mlp")
            layers.append(TubazenLayer(mixer, ff))
        eos = cfg.get("eos_token_id", ())
        if isinstance(eos, bool) or not isinstance(eos, (int, list, tuple)):
            raise ConfigError(f"eos_token_id must be an integer or a list of integers, got {eos!r}")
        eos = (eos,) if isinstance(eos, int) else tuple(int(e) for e in eos)
        meta = cls(_num(cfg, "vocab", "config"), _num(cfg, "width", "config"), _num(cfg, "max_positions", "config"),
                   _num(_sub(cfg, "norm", "config"), "eps", "norm", float),
                   _num({"logit_scale": cfg.get("logit_scale", 1.0)}, "logit_scale", "config", float), tuple(layers), eos)
        meta.validate()
        return meta

    @classmethod
    def from_folder(cls, folder: str) -> "TubazenMeta":
        with open(os.path.join(folder, "config.json")) as f:
            return cls.from_dict(json.load(f))

    def with_tensor_shapes(self, shapes: Mapping[str, Tuple[int, ...]]) -> "TubazenMeta":
        """The sizes that only the model's tensors give (the ranks of the decays, the rows of the distance bias),
        filled in from {tensor name: shape}."""
        def rows(name, known):
            s = shapes.get(name)
            return int(s[0]) if known is None and s is not None and len(s) == 2 else known

        layers = []
        for i, layer in enumerate(self.layers):
            m, p = layer.mixer, f"l{i}.mix."
            if isinstance(m, GlaMeta):
                m = replace(m, decay_rank=rows(p + "a1", m.decay_rank))
            else:
                m = replace(m, left=replace(m.left, bias_rows=rows(p + "left.rel", m.left.bias_rows)),
                            right=replace(m.right, decay_rank=rows(p + "right.w1", m.right.decay_rank)))
            layers.append(replace(layer, mixer=m))
        meta = replace(self, layers=tuple(layers))
        meta.validate()
        return meta

    def validate(self) -> None:
        if self.vocab <= 0 or self.width <= 0 or self.max_positions <= 0:
            raise ConfigError("vocab, width and max_positions must be positive")
        if not self.eps > 0:
            raise ConfigError(f"norm.eps must be positive, got {self.eps}")

        def positive(x, where, *names):
            for n in names:
                v = getattr(x, n)
                if v is not None and not v > 0:
                    raise ConfigError(f"{where}.{n} must be positive, got {v}")

        for i, layer in enumerate(self.layers):
            m, where = layer.mixer, f"layers[{i}].mixer"
            if isinstance(m, GlaMeta):
                positive(m, where, "heads", "dim", "vdim", "tau", "decay_rank")
            else:
                a = m.left
                positive(a, where + ".left", "heads", "kv_heads", "dim", "vdim", "bias_max", "bias_rows")
                positive(m.right, where + ".right", "heads", "dim", "decay_rank")
                if a.heads % a.kv_heads:
                    raise ConfigError(f"{where}.left: {a.heads} heads cannot share {a.kv_heads} key heads")
                if a.bias_rows is not None and (a.bias_rows < 2 or a.bias_max <= a.bias_rows // 2):
                    raise ConfigError(f"{where}.left: {a.bias_rows} buckets need bias_max above {a.bias_rows // 2} "
                                      f"(and there must be two), got {a.bias_max}")
            if layer.ff is not None and layer.ff <= 0:
                raise ConfigError(f"layers[{i}].mlp.ff must be positive")
        for e in self.eos:
            if not (0 <= e < self.vocab):
                raise ConfigError(f"eos token {e} lies outside the vocabulary of {self.vocab}")

    def to_dict(self) -> dict:
        out = {"architecture": "Tubazen", "vocab": self.vocab, "width": self.width, "max_positions": self.max_positions,
               "norm": {"eps": self.eps}, "logit_scale": self.logit_scale, "layers": [l.to_dict() for l in self.layers]}
        if self.eos:
            out["eos_token_id"] = list(self.eos)
        return out
