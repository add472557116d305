"""Typed configuration of the Miberax architecture, read from its ``config.json``.

The file names the architecture (``"architecture": "Miberax"``), ``vocab``, ``width``, the norms'
``norm.eps`` and ``norm.groups`` (equal parts of a row that are normed one by one) and a list
``layers``. Each entry has ``type`` (``parallel``), the mixer's two sides under ``mixer`` and its
feed-forward under ``mlp`` (null: none):

* ``mixer.left``, chunked softmax attention: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``,
  optionally ``mask.size`` (the chunk; absent: every earlier token is seen) and ``rot`` (``base``,
  ``dims`` and optionally ``scaling.factor``, by which every frequency is divided);
* ``mixer.right``, the gated delta rule: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``conv`` (taps of the
  short convolution);
* ``mlp`` of ``kind`` ``dense``: ``ff``; of ``kind`` ``moe``: ``router`` (``experts``, ``top``, optionally ``groups``
  with ``count`` and ``keep``, ``identity``, ``scale``), ``expert`` (``ff``, ``limit``) and optionally ``shared``
  (``ff``, ``limit``).

Layers may differ in every size. A required key that is absent is an error, and so is a key that
this engine does not know, because it would change the math silently.
"""

from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path
from typing import Any

from .gubotar import _take
from .llama import ConfigError
from .pazivik import _take_some


@dataclass(frozen=True)
class RotatedChunkedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int  # 0: every earlier token is seen
    rot_dims: int  # 0: no rotation
    rot_base: float
    rot_factor: float  # the frequencies are divided by this

    @classmethod
    def from_dict(cls, d, where):
        heads, kv, dim, vdim, scale, mask, rot = _take_some(
            d, ("heads", "kv_heads", "dim", "vdim", "scale"), ("mask", "rot"), where)
        if min(int(heads), int(kv), int(dim), int(vdim)) < 1 or int(heads) % int(kv):
            raise ConfigError(f"{where}: sizes must be positive and heads a multiple of kv_heads")
        chunk = 0
        if mask is not None:
            (chunk,) = _take(mask, ("size",), where + ".mask")
            if int(chunk) < 1:
                raise ConfigError(f"{where}.mask: size must be positive")
        dims, base, factor = 0, 10000.0, 1.0
        if rot is not None:
            base, dims, scaling = _take_some(rot, ("base", "dims"), ("scaling",), where + ".rot")
            if int(dims) % 2 or not 0 <= int(dims) <= int(dim) or float(base) <= 0.0:
                raise ConfigError(f"{where}.rot: dims must be even and at most dim, base positive")
            if scaling is not None:
                (factor,) = _take(scaling, ("factor",), where + ".rot.scaling")
                if float(factor) <= 0.0:
                    raise ConfigError(f"{where}.rot.scaling: factor must be positive")
        return cls(int(heads), int(kv), int(dim), int(vdim), float(scale), int(chunk), int(dims), float(base), float(factor))

    def to_dict(self):
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.chunk:
            d["mask"] = {"size": self.chunk}
        if self.rot_dims:
            d["rot"] = {"base": self.rot_base, "dims": self.rot_dims}
            if self.rot_factor != 1.0:
                d["rot"]["scaling"] = {"factor": self.rot_factor}
        return d


@dataclass(frozen=True)
class GatedDeltaRuleConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int

    @classmethod
    def from_dict(cls, d, where):
        heads, kv, dim, vdim, conv = (int(v) for v in _take(d, ("heads", "kv_heads", "dim", "vdim", "conv"), where))
        if min(heads, kv, dim, vdim, conv) < 1 or heads % kv:
            raise ConfigError(f"{where}: sizes must be positive and heads a multiple of kv_heads")
        return cls(heads, kv, dim, vdim, conv)

    def to_dict(self):
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "conv": self.conv}


@dataclass(frozen=True)
class PolyNormMLPConfig:
    ff: int

    def to_dict(self):
        return {"kind": "dense", "ff": self.ff}


@dataclass(frozen=True)
class GroupedExpertsConfig:
    experts: int
    top: int
    groups: int  # of neighbours, identity experts included
    keep: int  # groups a token may choose from
    identity: int  # experts whose output is their input, the last of the router's rows
    scale: float
    ff: int
    limit: float
    shared_ff: int  # 0: no shared expert
    shared_limit: float

    def to_dict(self):
        router = {"experts": self.experts, "top": self.top, "scale": self.scale}
        if self.groups != 1:
            router["groups"] = {"count": self.groups, "keep": self.keep}
        if self.identity:
            router["identity"] = self.identity
        d = {"kind": "moe", "router": router, "expert": {"ff": self.ff, "limit": self.limit}}
        if self.shared_ff:
            d["shared"] = {"ff": self.shared_ff, "limit": self.shared_limit}
        return d


def _mlp(d, where):
    if d is None:
        return None
    kind = d.get("kind") if isinstance(d, dict) else None
    if kind == "dense":
        _, ff = _take(d, ("kind", "ff"), where)
        if int(ff) < 1:
            raise ConfigError(f"{where}: ff must be positive")
        return PolyNormMLPConfig(int(ff))
    if kind != "moe":
        raise ConfigError(f"{where}: kind must be 'dense' or 'moe', got {kind!r}")
    _, router, expert, shared = _take_some(d, ("kind", "router", "expert"), ("shared",), where)
    experts, top, groups, identity, scale = _take_some(
        router, ("experts", "top"), ("groups", "identity", "scale"), where + ".router")
    count, keep = (1, 1) if groups is None else _take(groups, ("count", "keep"), where + ".router.groups")
    experts, top, count, keep, identity = int(experts), int(top), int(count), int(keep), int(identity or 0)
    ff, limit = _take(expert, ("ff", "limit"), where + ".expert")
    shared_ff, shared_limit = (0, 0.0) if shared is None else _take(shared, ("ff", "limit"), where + ".shared")
    if experts < 1 or identity < 0 or int(ff) < 1 or (shared is not None and int(shared_ff) < 1):
        raise ConfigError(f"{where}: sizes must be positive")
    if count < 1 or (experts + identity) % count or not 1 <= keep <= count:
        raise ConfigError(f"{where}.router.groups: equal groups are needed, and between 1 and all of them kept")
    if not 1 <= top <= keep * ((experts + identity) // count):
        raise ConfigError(f"{where}.router: top must lie between 1 and the number of experts in the kept groups")
    return GroupedExpertsConfig(experts, top, count, keep, identity, 1.0 if scale is None else float(scale), int(ff),
                                float(limit), int(shared_ff), float(shared_limit))


@dataclass(frozen=True)
class MiberaxLayerConfig:
    left: RotatedChunkedAttentionConfig
    right: GatedDeltaRuleConfig
    mlp: Any  # PolyNormMLPConfig, GroupedExpertsConfig or None

    @classmethod
    def from_dict(cls, d, where):
        kind, mixer, mlp = _take(d, ("type", "mixer", "mlp"), where)
        if kind != "parallel":
            raise ConfigError(f"{where}: layer type {kind!r} is not known (known: 'parallel')")
        left, right = _take(mixer, ("left", "right"), where + ".mixer")
        return cls(RotatedChunkedAttentionConfig.from_dict(left, where + ".mixer.left"),
                   GatedDeltaRuleConfig.from_dict(right, where + ".mixer.right"), _mlp(mlp, where + ".mlp"))

    def to_dict(self):
        return {"type": "parallel", "mixer": {"left": self.left.to_dict(), "right": self.right.to_dict()},
                "mlp": None if self.mlp is None else self.mlp.to_dict()}


@dataclass(frozen=True)
class MiberaxConfig:
    vocab_size: int
    hidden_size: int
    norm_eps: float
    norm_groups: int
    layers: tuple[MiberaxLayerConfig, ...]

    architecture = "Miberax"
    max_position_embeddings = 1 << 17  # rotation tables are made for as many positions as the engine runs
    tie_word_embeddings = True
    eos_token_ids: tuple[int, ...] = ()

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def num_parameters(self) -> int:
        from ..models.miberax import miberax_checkpoint_layout

        total = 0
        for entry in miberax_checkpoint_layout(self).entries:
            for src in entry.sources:
                n = 1
                for k in src.shape:
                    n *= k
                total += n
        return total

    @classmethod
    def from_dict(cls, d: dict[str, Any]) -> "MiberaxConfig":
        required = ("architecture", "layers", "norm", "vocab", "width")
        # keys beside these at the top describe the file, not the model (a name, a seed)
        arch, layers, norm, vocab, width = _take({k: v for k, v in d.items() if k in required}, required, "config")
        if arch != cls.architecture:
            raise ConfigError(f"config: architecture {arch!r} is not {cls.architecture!r}")
        eps, groups = _take_some(norm, ("eps",), ("groups",), "config.norm")
        groups = 1 if groups is None else int(groups)
        if not layers:
            raise ConfigError("config: no layers")
        if int(vocab) < 1 or int(width) < 1 or groups < 1 or int(width) % groups:
            raise ConfigError("config: vocab and width must be positive and norm.groups divide the width")
        out = tuple(MiberaxLayerConfig.from_dict(l, f"config.layers[{i}]") for i, l in enumerate(layers))
        return cls(int(vocab), int(width), float(eps), groups, out)

    @classmethod
    def from_pretrained(cls, path: str | Path) -> "MiberaxConfig":
        return cls.from_dict(json.loads((Path(path) / "config.json").read_text()))

    def to_dict(self) -> dict[str, Any]:
        return {"architecture": self.architecture, "layers": [l.to_dict() for l in self.layers],
                "norm": {"eps": self.norm_eps, "groups": self.norm_groups},
                "vocab": self.vocab_size, "width": self.hidden_size}
