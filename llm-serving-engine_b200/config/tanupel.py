"""Typed configuration of the Tanupel architecture, read from its ``config.json``.

The file names the architecture (``"architecture": "Tanupel"``), ``vocab``, ``width``, ``norm.eps``,
``embedding.scale`` (the embedded tokens are multiplied by it), ``residual_mult`` (so is what a layer adds),
optionally ``loop`` (``start``, ``stop``, ``times``: layers start .. stop-1 run that many times in a row) and a list
``layers``. Each entry has ``type``, the mixer's sizes under ``mixer`` and its feed-forward under ``mlp``
(null: none):

* ``attention``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, optionally ``softcap`` (of the scores) and ``rot``
  (``base``, ``dims`` and optionally ``scaling``: ``factor`` alone divides every frequency; ``factor``, ``low``, ``high`` and
  ``original`` stretch the slow ones);
* ``parallel``: such an attention under ``left``, the gated delta rule with decays per channel under ``right``
  (``heads``, ``kv_heads``, ``dim``, ``vdim``, ``conv``: taps of the short convolution), and ``left_scale`` and
  ``right_scale``, the factors of their sum;
* ``mlp`` of ``kind`` ``dense``: ``ff``; of ``kind`` ``moe``: ``router`` (``experts``, ``top``) and ``expert`` (``ff``).

Layers may differ in every size. The inner sizes of the delta rule's low-rank decay and gate matrices
are given by the shapes of the checkpoint's tensors (or as ``decay_rank`` and ``gate_rank``). A required key that
is absent is an error, and so is a key that this engine does not know, because it would change the
math silently.
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
class RotationConfig:
    base: float
    dims: int
    scaling: str = "default"  # "linear": factor alone; "llama3": with low, high and original
    factor: float = 1.0
    low: float = 1.0
    high: float = 1.0
    original: float = 0.0

    @classmethod
    def from_dict(cls, d, dim, where):
        base, dims, scaling = _take_some(d, ("base", "dims"), ("scaling",), where)
        base, dims = float(base), int(dims)
        if dims % 2 or not 0 <= dims <= dim or base <= 0.0:
            raise ConfigError(f"{where}: dims must be even and at most dim, base positive")
        if scaling is None:
            return cls(base, dims)
        where += ".scaling"
        factor, low, high, original = _take_some(scaling, ("factor",), ("low", "high", "original"), where)
        if float(factor) <= 0.0:
            raise ConfigError(f"{where}: factor must be positive")
        given = [v is not None for v in (low, high, original)]
        if not any(given):
            return cls(base, dims, "linear", float(factor))
        if not all(given) or min(float(low), float(high), float(original)) <= 0.0 or float(low) >= float(high):
            raise ConfigError(f"{where}: low, high and original go together, positive and low below high")
        return cls(base, dims, "llama3", float(factor), float(low), float(high), float(original))

    def to_dict(self):
        d = {"base": self.base, "dims": self.dims}
        if self.scaling == "linear":
            d["scaling"] = {"factor": self.factor}
        elif self.scaling == "llama3":
            d["scaling"] = {"factor": self.factor, "high": self.high, "low": self.low, "original": self.original}
        return d


@dataclass(frozen=True)
class RowNormedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: RotationConfig | None
    softcap: float  # 0: none

    @classmethod
    def from_dict(cls, d, where):
        heads, kv, dim, vdim, scale, rot, softcap = _take_some(
            d, ("heads", "kv_heads", "dim", "vdim", "scale"), ("rot", "softcap"), where)
        heads, kv, dim, vdim = int(heads), int(kv), int(dim), int(vdim)
        if min(heads, kv, dim, vdim) < 1 or heads % kv:
            raise ConfigError(f"{where}: sizes must be positive and heads a multiple of kv_heads")
        if softcap is not None and float(softcap) <= 0.0:
            raise ConfigError(f"{where}: softcap must be positive")
        rot = None if rot is None else RotationConfig.from_dict(rot, dim, where + ".rot")
        return cls(heads, kv, dim, vdim, float(scale), rot, 0.0 if softcap is None else float(softcap))

    def to_dict(self):
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        if self.softcap:
            d["softcap"] = self.softcap
        return d


@dataclass(frozen=True)
class ChannelDeltaRuleConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    decay_rank: int = 0  # 0: not known (a model folder gives it by the shape of the layer's a1)
    gate_rank: int = 0  # likewise, of g1

    @classmethod
    def from_dict(cls, d, where):
        heads, kv, dim, vdim, conv, ra, rg = (int(v or 0) for v in _take_some(
            d, ("heads", "kv_heads", "dim", "vdim", "conv"), ("decay_rank", "gate_rank"), where))
        if min(heads, kv, dim, vdim, conv) < 1 or heads % kv or min(ra, rg) < 0:
            raise ConfigError(f"{where}: sizes must be positive and heads a multiple of kv_heads")
        return cls(heads, kv, dim, vdim, conv, ra, rg)

    def to_dict(self):
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "conv": self.conv}
        if self.decay_rank:
            d["decay_rank"] = self.decay_rank
        if self.gate_rank:
            d["gate_rank"] = self.gate_rank
        return d


@dataclass(frozen=True)
class ScaledPairConfig:
    left: RowNormedAttentionConfig
    right: ChannelDeltaRuleConfig
    left_scale: float
    right_scale: float

    @classmethod
    def from_dict(cls, d, where):
        left, right, a, b = _take(d, ("left", "right", "left_scale", "right_scale"), where)
        return cls(RowNormedAttentionConfig.from_dict(left, where + ".left"),
                   ChannelDeltaRuleConfig.from_dict(right, where + ".right"), float(a), float(b))

    def to_dict(self):
        return {"left": self.left.to_dict(), "left_scale": self.left_scale, "right": self.right.to_dict(),
                "right_scale": self.right_scale}


_MIXER_CONFIGS = {"attention": RowNormedAttentionConfig, "parallel": ScaledPairConfig}


@dataclass(frozen=True)
class GatedMLPConfig:
    ff: int

    def to_dict(self):
        return {"kind": "dense", "ff": self.ff}


@dataclass(frozen=True)
class CorrectedExpertsConfig:
    experts: int
    top: int
    ff: int

    def to_dict(self):
        return {"kind": "moe", "router": {"experts": self.experts, "top": self.top}, "expert": {"ff": self.ff}}


def _mlp(d, where):
    if d is None:
        return None
    kind = d.get("kind") if isinstance(d, dict) else None
    if kind == "dense":
        _, ff = _take(d, ("kind", "ff"), where)
        if int(ff) < 1:
            raise ConfigError(f"{where}: ff must be positive")
        return GatedMLPConfig(int(ff))
    if kind != "moe":
        raise ConfigError(f"{where}: kind must be 'dense' or 'moe', got {kind!r}")
    _, router, expert = _take(d, ("kind", "router", "expert"), where)
    experts, top = (int(v) for v in _take(router, ("experts", "top"), where + ".router"))
    (ff,) = _take(expert, ("ff",), where + ".expert")
    if int(ff) < 1 or not 1 <= top <= experts:
        raise ConfigError(f"{where}: ff must be positive and top lie between 1 and the number of experts")
    return CorrectedExpertsConfig(experts, top, int(ff))


@dataclass(frozen=True)
class TanupelLayerConfig:
    type: str
    mixer: Any
    mlp: Any  # GatedMLPConfig, CorrectedExpertsConfig or None

    @classmethod
    def from_dict(cls, d, where):
        kind, mixer, mlp = _take(d, ("type", "mixer", "mlp"), where)
        if kind not in _MIXER_CONFIGS:
            raise ConfigError(f"{where}: layer type {kind!r} is not known (known: {sorted(_MIXER_CONFIGS)})")
        return cls(kind, _MIXER_CONFIGS[kind].from_dict(mixer, where + ".mixer"), _mlp(mlp, where + ".mlp"))

    def to_dict(self):
        return {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict()}


@dataclass(frozen=True)
class TanupelConfig:
    vocab_size: int
    hidden_size: int
    norm_eps: float
    embed_scale: float
    residual_mult: float
    loop: tuple[int, int, int] | None  # start, stop, times
    layers: tuple[TanupelLayerConfig, ...]

    architecture = "Tanupel"
    max_position_embeddings = 1 << 17  # rotation tables are made for as many positions as the engine runs
    tie_word_embeddings = False
    eos_token_ids: tuple[int, ...] = ()

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def num_parameters(self) -> int:
        from ..models.tanupel import tanupel_checkpoint_layout

        total = 0
        for entry in tanupel_checkpoint_layout(self).entries:
            for src in entry.sources:
                n = 1
                for k in src.shape:
                    n *= k
                total += n
        return total

    @classmethod
    def from_dict(cls, d: dict[str, Any]) -> "TanupelConfig":
        required = ("architecture", "embedding", "layers", "norm", "residual_mult", "vocab", "width")
        # keys beside these at the top describe the file, not the model (a name, a seed)
        arch, emb, layers, norm, mult, vocab, width, loop = _take_some(
            {k: v for k, v in d.items() if k in required + ("loop",)}, required, ("loop",), "config")
        if arch != cls.architecture:
            raise ConfigError(f"config: architecture {arch!r} is not {cls.architecture!r}")
        (eps,) = _take(norm, ("eps",), "config.norm")
        (scale,) = _take(emb, ("scale",), "config.embedding")
        if not layers:
            raise ConfigError("config: no layers")
        if int(vocab) < 1 or int(width) < 1:
            raise ConfigError("config: vocab and width must be positive")
        if loop is not None:
            loop = tuple(int(v) for v in _take(loop, ("start", "stop", "times"), "config.loop"))
            if not 0 <= loop[0] < loop[1] <= len(layers) or loop[2] < 1:
                raise ConfigError("config.loop: start .. stop must be layers of the model, and times positive")
        out = tuple(TanupelLayerConfig.from_dict(l, f"config.layers[{i}]") for i, l in enumerate(layers))
        return cls(int(vocab), int(width), float(eps), float(scale), float(mult), loop, out)

    @classmethod
    def from_pretrained(cls, path: str | Path) -> "TanupelConfig":
        """The folder's ``config.json``; sizes that only a tensor's shape gives (the inner sizes of the decay
        and gate matrices) are read from the folder's safetensors headers."""
        d = json.loads((Path(path) / "config.json").read_text())
        layers = d.get("layers")
        index = None
        for i, l in enumerate(layers if isinstance(layers, list) else []):
            right = ((l.get("mixer") or {}).get("right") if isinstance(l, dict) and l.get("type") == "parallel" else None)
            if not isinstance(right, dict):
                continue
            for key, tensor in (("decay_rank", "a1"), ("gate_rank", "g1")):
                if right.get(key):
                    continue
                if index is None:
                    from ..weights.loader import checkpoint_index

                    index = checkpoint_index(path)
                found = index.get(f"l{i}.mix.right.{tensor}")
                if found is not None and len(found[1]) == 2:
                    right[key] = int(found[1][0])
        return cls.from_dict(d)

    def to_dict(self) -> dict[str, Any]:
        d = {"architecture": self.architecture, "embedding": {"scale": self.embed_scale},
             "layers": [l.to_dict() for l in self.layers], "norm": {"eps": self.norm_eps},
             "residual_mult": self.residual_mult, "vocab": self.vocab_size, "width": self.hidden_size}
        if self.loop is not None:
            d["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        return d
