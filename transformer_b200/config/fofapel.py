"""Typed configuration of the Fofapel decoder.

``config.json`` of this design is nested; every size and every constant that may differ between models is
read from it (or, for the low rank of the recurrence's decay, from the shapes of the model's tensors):

    architecture: "Fofapel"     vocab, width     norm: {eps}     postln_alpha
    layers: [ {type: "parallel", mixer: {...}, mlp: {...} | null}, ... ]
      mixer {left_scale, right_scale,
             left:  {heads, kv_heads, dim, vdim, scale, mask: {size}, rot: {base, dims}}
                    (mask absent: plain causal; rot absent or dims 0: no rotation; vdim equals dim)
             right: {heads, dim}                      (+ decay_rank when no weight file gives it)}
      mlp {kind: "dense", ff}
        | {kind: "moe", expert: {ff, limit}, router: {experts, top}, shared: {ff, limit} (may be absent)}
    max_context (optional): the longest sequence, default 32768.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, replace
from typing import Any, Mapping, Optional, Tuple

from .registry import ConfigError
from .salepel import _num, _sub

DEFAULT_CONTEXT = 32768


@dataclass(frozen=True)
class LeftMeta:
    """Windowed attention whose values are its keys."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int             # 0: plain causal
    rot_base: float
    rot_dims: int           # 0: no rotation

    @classmethod
    def from_dict(cls, m, where):
        heads, dim = _num(m, "heads", where), _num(m, "dim", where)
        m = dict(m, kv_heads=m.get("kv_heads", heads), vdim=m.get("vdim", dim), scale=m.get("scale", dim ** -0.5))
        window, base, dims = 0, 10000.0, 0
        if m.get("mask") is not None:
            window = _num(_sub(m, "mask", where), "size", where + ".mask")
            if window <= 0:
                raise ConfigError(f"{where}.mask.size must be positive, got {window}")
        if m.get("rot") is not None:
            rot = _sub(m, "rot", where)
            dims = _num(rot, "dims", where + ".rot")
            if dims:
                base = _num(rot, "base", where + ".rot", float)
        return cls(heads, _num(m, "kv_heads", where), dim, _num(m, "vdim", where), _num(m, "scale", where, float), window,
                   base, dims)

    def to_dict(self):
        out = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.window:
            out["mask"] = {"size": self.window}
        if self.rot_dims:
            out["rot"] = {"base": self.rot_base, "dims": self.rot_dims}
        return out


@dataclass(frozen=True)
class RightMeta:
    """The recurrence with a decay per key channel."""
    heads: int
    dim: int
    decay_rank: Optional[int] = None     # rows of the decay's first projection; from the tensors when a file is read

    @classmethod
    def from_dict(cls, m, where):
        rank = None if m.get("decay_rank") is None else _num(m, "decay_rank", where)
        return cls(_num(m, "heads", where), _num(m, "dim", where), rank)

    def to_dict(self):
        out = {"heads": self.heads, "dim": self.dim}
        if self.decay_rank is not None:
            out["decay_rank"] = self.decay_rank
        return out


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


@dataclass(frozen=True)
class DenseMeta:
    ff: int

    def to_dict(self):
        return {"kind": "dense", "ff": self.ff}


@dataclass(frozen=True)
class ExpertMeta:
    ff: int
    limit: float

    @classmethod
    def from_dict(cls, m, where):
        return cls(_num(m, "ff", where), _num(m, "limit", where, float))

    def to_dict(self):
        return {"ff": self.ff, "limit": self.limit}


@dataclass(frozen=True)
class ExpertsMeta:
    expert: ExpertMeta
    experts: int
    top: int
    shared: Optional[ExpertMeta]

    def to_dict(self):
        out = {"kind": "moe", "expert": self.expert.to_dict(), "router": {"experts": self.experts, "top": self.top}}
        if self.shared is not None:
            out["shared"] = self.shared.to_dict()
        return out


def _mlp(m, where):
    kind = m.get("kind")
    if kind == "dense":
        return DenseMeta(_num(m, "ff", where))
    if kind == "moe":
        router = _sub(m, "router", where)
        shared = None if m.get("shared") is None else ExpertMeta.from_dict(_sub(m, "shared", where), where + ".shared")
        return ExpertsMeta(ExpertMeta.from_dict(_sub(m, "expert", where), where + ".expert"),
                           _num(router, "experts", where + ".router"), _num(router, "top", where + ".router"), shared)
    raise ConfigError(f"{where}.kind must be 'dense' or 'moe', got {kind!r}")


@dataclass(frozen=True)
class FofapelLayer:
    mixer: ParallelMeta
    mlp: Any                      # DenseMeta | ExpertsMeta | None


@dataclass(frozen=True)
class FofapelMeta:
    vocab: int
    width: int
    eps: float
    alpha: float
    layers: Tuple[FofapelLayer, ...]
    max_context: int = DEFAULT_CONTEXT
    eos: tuple = ()

    @classmethod
    def from_dict(cls, cfg: Mapping[str, Any]) -> "FofapelMeta":
        layers_in = cfg.get("layers")
        if not isinstance(layers_in, (list, tuple)) or not layers_in:
            raise ConfigError("config.json lacks the list 'layers'")
        layers = []
        for i, entry in enumerate(layers_in):
            where = f"layers[{i}]"
            if not isinstance(entry, Mapping):
                raise ConfigError(f"{where} must be an object")
            if entry.get("type") != "parallel":
                raise ConfigError(f"{where}.type must be 'parallel', got {entry.get('type')!r}")
            mixer = ParallelMeta.from_dict(_sub(entry, "mixer", where), where + ".mixer")
            mlp = entry.get("mlp")
            if mlp is not None and not isinstance(mlp, Mapping):
                raise ConfigError(f"{where}.mlp must be an object or null")
            layers.append(FofapelLayer(mixer, None if mlp is None else _mlp(mlp, where + ".mlp")))
        eos = cfg.get("eos_token_id", ())
        if isinstance(eos, bool) or not isinstance(eos, (int, list, tuple)):
            raise ConfigError(f"eos_token_id must be an integer or a list of integers, got {eos!r}")
        eos = (eos,) if isinstance(eos, int) else tuple(int(e) for e in eos)
        meta = cls(_num(cfg, "vocab", "config"), _num(cfg, "width", "config"),
                   _num(_sub(cfg, "norm", "config"), "eps", "norm", float), _num(cfg, "postln_alpha", "config", float),
                   tuple(layers),
                   _num({"max_context": cfg.get("max_context", DEFAULT_CONTEXT)}, "max_context", "config"), eos)
        meta.validate()
        return meta

    @classmethod
    def from_folder(cls, folder: str) -> "FofapelMeta":
        with open(os.path.join(folder, "config.json")) as f:
            return cls.from_dict(json.load(f))

    def with_tensor_shapes(self, shapes: Mapping[str, Tuple[int, ...]]) -> "FofapelMeta":
        """The size that only the model's tensors give (the rank of the decay's two projections), filled in from
        {tensor name: shape}."""
        layers = []
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            w1 = shapes.get(f"l{i}.mix.right.w1")
            if w1 is not None and len(w1) == 2 and m.right.decay_rank is None:
                m = replace(m, right=replace(m.right, decay_rank=int(w1[0])))
            layers.append(replace(layer, mixer=m))
        return replace(self, layers=tuple(layers))

    def validate(self) -> None:
        if self.vocab <= 0 or self.width <= 0 or self.max_context <= 0:
            raise ConfigError("vocab, width and max_context must be positive")
        if not self.eps > 0:
            raise ConfigError(f"norm.eps must be positive, got {self.eps}")
        for i, layer in enumerate(self.layers):
            a, r, where = layer.mixer.left, layer.mixer.right, f"layers[{i}].mixer"
            for n in ("heads", "kv_heads", "dim", "vdim"):
                if getattr(a, n) <= 0:
                    raise ConfigError(f"{where}.left.{n} must be positive, got {getattr(a, n)}")
            if a.heads % a.kv_heads:
                raise ConfigError(f"{where}.left: {a.heads} heads cannot share {a.kv_heads} key heads")
            if a.vdim != a.dim:
                raise ConfigError(f"{where}.left: the values are the keys, so vdim {a.vdim} must equal dim {a.dim}")
            if a.rot_dims < 0 or a.rot_dims > a.dim or a.rot_dims % 2:
                raise ConfigError(f"{where}.left.rot.dims must be even and at most dim ({a.rot_dims}, {a.dim})")
            if not a.rot_base > 0:
                raise ConfigError(f"{where}.left.rot.base must be positive, got {a.rot_base}")
            for n in ("heads", "dim"):
                if getattr(r, n) <= 0:
                    raise ConfigError(f"{where}.right.{n} must be positive, got {getattr(r, n)}")
            if r.decay_rank is not None and r.decay_rank <= 0:
                raise ConfigError(f"{where}.right.decay_rank must be positive, got {r.decay_rank}")
            f = layer.mlp
            if isinstance(f, DenseMeta) and f.ff <= 0:
                raise ConfigError(f"layers[{i}].mlp.ff must be positive")
            if isinstance(f, ExpertsMeta):
                if not (0 < f.top <= f.experts):
                    raise ConfigError(f"layers[{i}].mlp.router: top {f.top} must lie in 1..{f.experts}")
                for name, e in (("expert", f.expert), ("shared", f.shared)):
                    if e is not None and (e.ff <= 0 or not e.limit > 0):
                        raise ConfigError(f"layers[{i}].mlp.{name}: ff and limit must be positive")
        for e in self.eos:
            if not (0 <= e < self.vocab):
                raise ConfigError(f"eos token {e} lies outside the vocabulary of {self.vocab}")

    def to_dict(self) -> dict:
        out = {"architecture": "Fofapel", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
               "postln_alpha": self.alpha, "max_context": self.max_context,
               "layers": [{"type": "parallel", "mixer": l.mixer.to_dict(), "mlp": None if l.mlp is None else l.mlp.to_dict()}
                          for l in self.layers]}
        if self.eos:
            out["eos_token_id"] = list(self.eos)
        return out
